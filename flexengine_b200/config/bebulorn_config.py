"""Typed configuration of the Bebulorn decoder, read from its ``config.json``.

The file is nested: ``vocab``, ``width``, ``norm`` {eps}, ``residual_mult``, ``loop`` {start, stop, times} (layers
start .. stop - 1 run ``times`` times in a row; absent: every layer once) and ``layers``, a list whose entries give ``type``
(which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (a dense or a routed feed-forward, or null).  Mixers:
``attention`` (softmax attention without positions, scores squashed by tanh, a sliding window), ``lightning`` (linear
attention with a fixed decay per head) and ``delta`` (the gated delta rule).  Every size and constant comes from this file.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .fuvozen_config import _get
from .model_config import ConfigError

MIXERS = ("attention", "lightning", "delta")


@dataclass(frozen=True)
class SoftcapAttentionConfig:
    heads: int
    kv_heads: int
    dim: int             # query/key size of a head
    vdim: int            # value size of a head
    scale: float         # what the scores are multiplied by (and by a learned number per head)
    softcap: float       # scores become softcap * tanh(score / softcap); 0: as they are
    window: int          # how many keys a query sees, itself among them; 0: every earlier one


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple         # one number per head


@dataclass(frozen=True)
class DeltaConfig:
    heads: int           # value heads; head h uses query/key head h // (heads / kv_heads)
    kv_heads: int
    dim: int
    vdim: int
    conv: int            # taps of the short convolutions over time


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int


@dataclass(frozen=True)
class MoeMlpConfig:
    experts: int
    top: int
    expert_ff: int
    shared_ff: int       # size of the expert every token runs; 0: none


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class BebulornLayer:
    type: str
    mixer: Any
    mlp: Any             # DenseMlpConfig, MoeMlpConfig or None


@dataclass(frozen=True)
class BebulornConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float     # what a sublayer's normed output is multiplied by on its way into the stream
    loop: LoopConfig | None
    layers: tuple
    eos_token_ids: tuple = ()
    bos_token_id: int | None = None

    ARCHITECTURE = "Bebulorn"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "BebulornConfig":
        layers = _get(data, "layers", list)
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one entry")
        parsed = []
        for i, entry in enumerate(layers):
            kind = _get(entry, "type", str)
            parsed.append(BebulornLayer(kind, cls._mixer(i, kind, entry), cls._mlp(i, entry.get("mlp"))))
        loop = None
        if data.get("loop") is not None:
            loop = LoopConfig(start=_get(data, "loop.start", int), stop=_get(data, "loop.stop", int), times=_get(data, "loop.times", int))
            if not (0 <= loop.start < loop.stop <= len(parsed)) or loop.times < 1:
                raise ConfigError("config.json: 'loop' must name a span of layers, start < stop, and run it at least once")
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else (tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (int(eos),))
        cfg = cls(vocab=_get(data, "vocab", int), width=_get(data, "width", int), norm_eps=_get(data, "norm.eps", float),
                  residual_mult=_get(data, "residual_mult", float, default=1.0, required=False),
                  loop=loop, layers=tuple(parsed), eos_token_ids=eos_ids,
                  bos_token_id=None if data.get("bos_token_id") is None else int(data["bos_token_id"]))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        if not cfg.norm_eps > 0.0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cfg

    @staticmethod
    def _mixer(i: int, kind: str, entry: Mapping[str, Any]):
        if kind == "attention":
            heads = _get(entry, "mixer.heads", int)
            mixer = SoftcapAttentionConfig(
                heads=heads, kv_heads=_get(entry, "mixer.kv_heads", int, default=heads, required=False),
                dim=_get(entry, "mixer.dim", int), vdim=_get(entry, "mixer.vdim", int), scale=_get(entry, "mixer.scale", float),
                softcap=_get(entry, "mixer.softcap", float, default=0.0, required=False),
                window=_get(entry, "mixer.mask.size", int, default=0, required=False))
            if mixer.window < 0 or (mixer.window == 0 and entry["mixer"].get("mask") is not None):
                raise ConfigError(f"layer {i}: mask.size must be positive")
            if mixer.softcap < 0.0:
                raise ConfigError(f"layer {i}: softcap must not be negative")
        elif kind == "lightning":
            decay = _get(entry, "mixer.decay", list)
            mixer = LightningConfig(heads=_get(entry, "mixer.heads", int), dim=_get(entry, "mixer.dim", int),
                                    vdim=_get(entry, "mixer.vdim", int), decay=tuple(float(x) for x in decay))
            if len(mixer.decay) != mixer.heads:
                raise ConfigError(f"layer {i}: 'decay' must list one number per head")
        elif kind == "delta":
            heads = _get(entry, "mixer.heads", int)
            mixer = DeltaConfig(heads=heads, kv_heads=_get(entry, "mixer.kv_heads", int, default=heads, required=False),
                                dim=_get(entry, "mixer.dim", int), vdim=_get(entry, "mixer.vdim", int), conv=_get(entry, "mixer.conv", int))
            if mixer.conv < 1:
                raise ConfigError(f"layer {i}: conv must be at least one tap")
        else:
            raise ConfigError(f"layer {i}: unknown mixer type {kind!r}; known: {', '.join(MIXERS)}")
        if min(mixer.heads, mixer.dim, mixer.vdim) <= 0:
            raise ConfigError(f"layer {i}: head counts and sizes must be positive")
        kv_heads = getattr(mixer, "kv_heads", 1)
        if kv_heads <= 0 or mixer.heads % kv_heads:
            raise ConfigError(f"layer {i}: heads must be a multiple of kv_heads")
        return mixer

    @staticmethod
    def _mlp(i: int, data):
        if data is None:
            return None
        kind = _get(data, "kind", str)
        if kind == "dense":
            mlp = DenseMlpConfig(ff=_get(data, "ff", int))
            if mlp.ff <= 0:
                raise ConfigError(f"layer {i}: mlp.ff must be positive")
            return mlp
        if kind == "moe":
            mlp = MoeMlpConfig(experts=_get(data, "router.experts", int), top=_get(data, "router.top", int),
                               expert_ff=_get(data, "expert.ff", int),
                               shared_ff=_get(data, "shared.ff", int, default=0, required=data.get("shared") is not None))
            if not (1 <= mlp.top <= mlp.experts) or mlp.expert_ff <= 0:
                raise ConfigError(f"layer {i}: a token uses between 1 and 'experts' experts of a positive size")
            if mlp.shared_ff < 0 or (mlp.shared_ff == 0 and data.get("shared") is not None):
                raise ConfigError(f"layer {i}: shared.ff must be positive")
            return mlp
        raise ConfigError(f"layer {i}: unknown mlp kind {kind!r}; known: dense, moe")
