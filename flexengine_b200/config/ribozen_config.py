"""Typed configuration of the Ribozen decoder, read from its ``config.json``.

The file is nested: ``vocab``, ``width``, ``norm`` {eps}, ``embedding`` {scale} and ``layers``, a list whose entries give
``type`` (which mixer), ``mixer`` (its sizes and constants) and ``mlp`` (a routed feed-forward, or null).  Mixers: ``mlstm``
(a matrix memory with exponential gates), ``mamba2`` (a state-space layer with one decay per head) and ``parallel`` (softmax
attention under a window that keeps the first tokens, beside a selective scan with a decay per channel and state entry).
Every size and constant comes from this file.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .fuvozen_config import _get
from .model_config import ConfigError

MIXERS = ("mlstm", "parallel", "mamba2")


@dataclass(frozen=True)
class MlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float      # both gates' pre-activations become gate_cap * tanh(. / gate_cap)


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int          # of the keys and queries (B and C); head h uses group h // (heads / groups)
    norm_groups: int
    conv: int            # taps of the short convolution over time


@dataclass(frozen=True)
class RotaryScalingConfig:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float       # scores become softcap * tanh(score / softcap); 0: as they are
    window: int          # how many keys a query sees, itself among them; 0: every earlier one
    keep_first: int      # the first so many tokens of the sequence are seen as well
    rot_base: float
    rot_dims: int        # entries of a head that turn; 0: none
    rot_scaling: RotaryScalingConfig | None


@dataclass(frozen=True)
class SelectiveScanConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowAttentionConfig
    right: SelectiveScanConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MoeMlpConfig:
    experts: int
    top: int
    expert_ff: int
    shared_ff: int       # size of the expert every token runs; 0: none


@dataclass(frozen=True)
class RibozenLayer:
    type: str
    mixer: Any
    mlp: MoeMlpConfig | None


@dataclass(frozen=True)
class RibozenConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: tuple
    eos_token_ids: tuple = ()
    bos_token_id: int | None = None

    ARCHITECTURE = "Ribozen"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "RibozenConfig":
        layers = _get(data, "layers", list)
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one entry")
        parsed = []
        for i, entry in enumerate(layers):
            kind = _get(entry, "type", str)
            parsed.append(RibozenLayer(kind, cls._mixer(i, kind, entry), cls._mlp(i, entry.get("mlp"))))
        eos = data.get("eos_token_id")
        eos_ids = () if eos is None else (tuple(int(e) for e in eos) if isinstance(eos, (list, tuple)) else (int(eos),))
        cfg = cls(vocab=_get(data, "vocab", int), width=_get(data, "width", int), norm_eps=_get(data, "norm.eps", float),
                  embedding_scale=_get(data, "embedding.scale", float, default=1.0, required=False), layers=tuple(parsed),
                  eos_token_ids=eos_ids, bos_token_id=None if data.get("bos_token_id") is None else int(data["bos_token_id"]))
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        if not cfg.norm_eps > 0.0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cfg

    @classmethod
    def _mixer(cls, i: int, kind: str, entry: Mapping[str, Any]):
        if kind == "mlstm":
            m = MlstmConfig(heads=_get(entry, "mixer.heads", int), dim=_get(entry, "mixer.dim", int), vdim=_get(entry, "mixer.vdim", int),
                            gate_cap=_get(entry, "mixer.gate_cap", float))
            if min(m.heads, m.dim, m.vdim) <= 0:
                raise ConfigError(f"layer {i}: head counts and sizes must be positive")
            if not m.gate_cap > 0.0:
                raise ConfigError(f"layer {i}: gate_cap must be positive")
            return m
        if kind == "mamba2":
            m = Mamba2Config(heads=_get(entry, "mixer.heads", int), vdim=_get(entry, "mixer.vdim", int), state=_get(entry, "mixer.state", int),
                             groups=_get(entry, "mixer.groups", int, default=1, required=False),
                             norm_groups=_get(entry, "mixer.norm_groups", int, default=1, required=False), conv=_get(entry, "mixer.conv", int))
            if min(m.heads, m.vdim, m.state) <= 0:
                raise ConfigError(f"layer {i}: head counts and sizes must be positive")
            if m.groups <= 0 or m.heads % m.groups:
                raise ConfigError(f"layer {i}: heads must be a multiple of groups")
            if m.norm_groups <= 0 or (m.heads * m.vdim) % m.norm_groups:
                raise ConfigError(f"layer {i}: norm_groups must cut heads * vdim into equal parts")
            if m.conv < 1:
                raise ConfigError(f"layer {i}: conv must be at least one tap")
            return m
        if kind == "parallel":
            return ParallelConfig(left=cls._attention(i, _get(entry, "mixer.left", dict)), right=cls._scan(i, _get(entry, "mixer.right", dict)),
                                  left_scale=_get(entry, "mixer.left_scale", float, default=1.0, required=False),
                                  right_scale=_get(entry, "mixer.right_scale", float, default=1.0, required=False))
        raise ConfigError(f"layer {i}: unknown mixer type {kind!r}; known: {', '.join(MIXERS)}")

    @staticmethod
    def _attention(i: int, data: Mapping[str, Any]) -> WindowAttentionConfig:
        heads, dim = _get(data, "heads", int), _get(data, "dim", int)
        scaling = None
        if isinstance(data.get("rot"), Mapping) and data["rot"].get("scaling") is not None:
            scaling = RotaryScalingConfig(*(_get(data, f"rot.scaling.{key}", float) for key in ("factor", "original", "fast", "slow")))
            if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0.0:
                raise ConfigError(f"layer {i}: the numbers of rot.scaling must be positive")
        rotated = data.get("rot") is not None
        m = WindowAttentionConfig(
            heads=heads, kv_heads=_get(data, "kv_heads", int, default=heads, required=False), dim=dim, vdim=_get(data, "vdim", int),
            scale=_get(data, "scale", float), softcap=_get(data, "softcap", float, default=0.0, required=False),
            window=_get(data, "mask.size", int, default=0, required=data.get("mask") is not None),
            keep_first=_get(data, "mask.keep_first", int, default=0, required=False),
            rot_base=_get(data, "rot.base", float, default=10000.0, required=rotated),
            rot_dims=_get(data, "rot.dims", int, default=0, required=rotated), rot_scaling=scaling)
        if min(m.heads, m.dim, m.vdim) <= 0:
            raise ConfigError(f"layer {i}: head counts and sizes must be positive")
        if m.kv_heads <= 0 or m.heads % m.kv_heads:
            raise ConfigError(f"layer {i}: heads must be a multiple of kv_heads")
        if m.window < 0 or (m.window == 0 and data.get("mask") is not None):
            raise ConfigError(f"layer {i}: mask.size must be positive")
        if m.keep_first < 0:
            raise ConfigError(f"layer {i}: mask.keep_first must not be negative")
        if m.softcap < 0.0:
            raise ConfigError(f"layer {i}: softcap must not be negative")
        if m.rot_dims < 0 or m.rot_dims % 2 or m.rot_dims > m.dim:
            raise ConfigError(f"layer {i}: rot.dims must be even and at most dim")
        if m.rot_dims and not m.rot_base > 1.0:
            raise ConfigError(f"layer {i}: rot.base must be above 1")
        return m

    @staticmethod
    def _scan(i: int, data: Mapping[str, Any]) -> SelectiveScanConfig:
        m = SelectiveScanConfig(inner=_get(data, "inner", int), state=_get(data, "state", int), dt_rank=_get(data, "dt_rank", int),
                                conv=_get(data, "conv", int))
        if min(m.inner, m.state, m.dt_rank) <= 0:
            raise ConfigError(f"layer {i}: inner, state and dt_rank must be positive")
        if m.conv < 1:
            raise ConfigError(f"layer {i}: conv must be at least one tap")
        return m

    @staticmethod
    def _mlp(i: int, data):
        if data is None:
            return None
        kind = _get(data, "kind", str)
        if kind != "moe":
            raise ConfigError(f"layer {i}: unknown mlp kind {kind!r}; known: moe")
        mlp = MoeMlpConfig(experts=_get(data, "router.experts", int), top=_get(data, "router.top", int),
                           expert_ff=_get(data, "expert.ff", int),
                           shared_ff=_get(data, "shared.ff", int, default=0, required=data.get("shared") is not None))
        if not (1 <= mlp.top <= mlp.experts) or mlp.expert_ff <= 0:
            raise ConfigError(f"layer {i}: a token uses between 1 and 'experts' experts of a positive size")
        if mlp.shared_ff < 0 or (mlp.shared_ff == 0 and data.get("shared") is not None):
            raise ConfigError(f"layer {i}: shared.ff must be positive")
        return mlp
