from . import bebulorn, fedutar, fuvozen, fuvuvik, qwen2, rikolix  # noqa: F401  (register Bebulorn, Fedutar, Fuvozen, Fuvuvik, Rikolix and Qwen2ForCausalLM)
