from . import bebulorn, fedutar, fuvozen, fuvuvik, qwen2, ribozen, rikolix  # noqa: F401  (register Bebulorn, Fedutar, Fuvozen, Fuvuvik, Ribozen, Rikolix and Qwen2ForCausalLM)
