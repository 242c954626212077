"""Bebulorn as a plan of parts: a decoder whose sublayers have a layer norm (weight and bias) on both sides and enter the
stream times one constant.  Mixers: softmax attention without positions (unit-norm values, a learned number per head on the
scores, scores squashed by tanh, a sliding window), lightning attention (linear attention with one fixed decay per head,
silu on queries, keys and values, one norm over all heads, a sigmoid gate) and the gated delta rule (short convolutions,
unit vectors, a decay and a step size per token and head).  Feed-forwards: dense with a relu gate, or routed over experts
without a gate (exact GELU) beside a shared one.  A span of the layers may run several times in a row with the same
weights; every pass has cache and state of its own, and before every pass but the first the embedding's output is added to
the stream.

Checkpoint names: ``embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1|norm1b|norm2|norm2b`` (each norm with a
``.b``), ``l<i>.mix.q|k|v|o`` and, by mixer, ``.temp``; ``.g|norm``; ``.q.conv|k.conv|v.conv|b|a|A_log|dt_bias|norm|g``;
``l<i>.mlp.gate|up|down`` or ``l<i>.mlp.router``, ``.e<k>.up|down``, ``.shared.up|down``.  Matrices are [out, in]; the
projections of one input are bound as one matrix, all experts of a layer as one.

Cache groups: a paged group per distinct (key/value heads, head size, window); a float32 state group per distinct state
size of the lightning layers, and one per distinct (state, convolution history) of the delta layers; each with a slot per
run of a layer (a layer of the repeated span has one per pass).
"""
from __future__ import annotations

import math
from dataclasses import replace

from ..config.bebulorn_config import BebulornConfig, DeltaConfig, DenseMlpConfig, LightningConfig, MoeMlpConfig, SoftcapAttentionConfig
from ..config.registry import register_architecture
from ..parts.delta import GatedDeltaMixer
from ..parts.spec import (CacheGroupSpec, LayerSpec, ModelPlan, PartSpec, RunEntry, WeightBinding, WeightSource)


def run_order(cfg: BebulornConfig):
    """[(layer, the embedding's output is added before it)] in the order the layers run."""
    count = len(cfg.layers)
    if cfg.loop is None:
        return [(i, False) for i in range(count)]
    start, stop, times = cfg.loop.start, cfg.loop.stop, cfg.loop.times
    order = [(i, False) for i in range(start)]
    for turn in range(times):
        order += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return order + [(i, False) for i in range(stop, count)]


def build_bebulorn_plan(cfg: BebulornConfig, present=None) -> ModelPlan:
    """``present``: the tensor names of a checkpoint; the second pair of norms of a layer without a feed-forward is then
    named as ignored instead of unexpected."""
    D, V = cfg.width, cfg.vocab
    norm = PartSpec("layernorm", {"hidden_size": D, "eps": cfg.norm_eps})
    groups: list = []
    group_of: dict = {}            # key -> [group index, slots so far]
    layers, bindings, ignored, places = [], [], [], []
    init = {}

    def src(name, *shape, rule=None):
        fan_in = shape[-1] if len(shape) > 1 else 1
        init[name] = rule or ("normal", 0.0, 1.0 / math.sqrt(max(fan_in, 1)))
        return WeightSource(name, tuple(shape))

    def slot_in(key, need):
        if key not in group_of:
            group_of[key] = [len(groups), 0]
            groups.append(need)
        gi, slot = group_of[key]
        group_of[key][1] += 1
        return gi, slot

    near_one = ("normal", 1.0, 0.1)

    def norm_bindings(target, name):
        return [WeightBinding(target("weight"), (src(name, D, rule=near_one),), kind="vector"),
                WeightBinding(target("bias"), (src(name + ".b", D, rule=("normal", 0.0, 0.1)),), kind="vector")]

    bindings += [WeightBinding(("embedding", "weight"), (src("embed", V, D, rule=("normal", 0.0, 1.0)),)),
                 WeightBinding(("lm_head", "weight"), (src("head", V, D),))]
    bindings += norm_bindings(lambda local: ("final_norm", local), "final.norm")
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        mp = p + "mix."
        m = layer.mixer

        def target(part, local):
            return ("layer", i, part, local)

        if isinstance(m, SoftcapAttentionConfig):
            head = -(-max(m.dim, m.vdim) // 16) * 16
            kind = "window" if m.window else "full"
            mixer = PartSpec("gated_attention", {
                "hidden_size": D, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                "eps": cfg.norm_eps, "mask": kind, "mask_size": m.window, "value_norm": True, "head_scales": True,
                "softcap": m.softcap, "gate": "none"})
            places.append((("paged", m.kv_heads, head, m.window),
                           CacheGroupSpec(name=f"attention_{m.kv_heads}x{head}_{m.window or 'all'}", kind=kind, slots=0,
                                          kv_heads=m.kv_heads, head_dim=head, window=m.window)))
            bindings += [
                WeightBinding(target("mixer", "qkvg.weight"), (src(mp + "q", m.heads * m.dim, D), src(mp + "k", m.kv_heads * m.dim, D),
                                                               src(mp + "v", m.kv_heads * m.vdim, D))),
                WeightBinding(target("mixer", "head_scales"), (src(mp + "temp", m.heads, rule=near_one),), kind="vector"),
                WeightBinding(target("mixer", "o.weight"), (src(mp + "o", D, m.heads * m.vdim),)),
            ]
        elif isinstance(m, LightningConfig):
            n = m.heads * m.dim * m.vdim
            mixer = PartSpec("retention", {
                "hidden_size": D, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": m.decay, "eps": cfg.norm_eps,
                "activation": "silu", "key_scale": 1.0, "norm": "all_heads", "gate": "sigmoid"})
            places.append((("lightning", n), CacheGroupSpec(name=f"lightning_state_{n}", kind="state", slots=0, state_shape=(n,),
                                                            state_dtype="float32")))
            inner = m.heads * m.vdim
            bindings += [
                WeightBinding(target("mixer", "qkvg.weight"), (src(mp + "q", m.heads * m.dim, D), src(mp + "k", m.heads * m.dim, D),
                                                               src(mp + "v", inner, D), src(mp + "g", inner, D))),
                WeightBinding(target("mixer", "norm.weight"), (src(mp + "norm", inner, rule=near_one),), kind="vector"),
                WeightBinding(target("mixer", "o.weight"), (src(mp + "o", D, inner),)),
            ]
        else:
            assert isinstance(m, DeltaConfig)
            params = {"hidden_size": D, "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv,
                      "eps": cfg.norm_eps}
            mixer = PartSpec("gated_delta", params)
            n = GatedDeltaMixer(**params).state_elements
            places.append((("delta", n), CacheGroupSpec(name=f"delta_state_{n}", kind="state", slots=0, state_shape=(n,),
                                                        state_dtype="float32")))
            qk, inner = m.kv_heads * m.dim, m.heads * m.vdim
            taps = ("normal", 0.0, 1.0 / math.sqrt(m.conv))
            bindings += [
                WeightBinding(target("mixer", "qkvgba.weight"), (src(mp + "q", qk, D), src(mp + "k", qk, D), src(mp + "v", inner, D),
                                                                 src(mp + "g", inner, D), src(mp + "b", m.heads, D), src(mp + "a", m.heads, D))),
                WeightBinding(target("mixer", "conv.weight"), (src(mp + "q.conv", qk, m.conv, rule=taps), src(mp + "k.conv", qk, m.conv, rule=taps),
                                                               src(mp + "v.conv", inner, m.conv, rule=taps)), kind="vector"),
                WeightBinding(target("mixer", "A_log"), (src(mp + "A_log", m.heads, rule=("normal", -1.0, 1.0)),), kind="vector"),
                WeightBinding(target("mixer", "dt_bias"), (src(mp + "dt_bias", m.heads, rule=("normal", -2.0, 1.0)),), kind="vector"),
                WeightBinding(target("mixer", "norm.weight"), (src(mp + "norm", m.vdim, rule=near_one),), kind="vector"),
                WeightBinding(target("mixer", "o.weight"), (src(mp + "o", D, inner),)),
            ]
        mlp = layer.mlp
        fp = p + "mlp."
        if mlp is None:
            feed_forward = None
            ignored += [p + name + tail for name in ("norm2", "norm2b") for tail in ("", ".b")]
        elif isinstance(mlp, DenseMlpConfig):
            f = mlp.ff
            feed_forward = PartSpec("gated_mlp", {"hidden_size": D, "intermediate_size": f, "activation": "relu"})
            bindings += [WeightBinding(target("feed_forward", "gate_up.weight"), (src(fp + "gate", f, D), src(fp + "up", f, D))),
                         WeightBinding(target("feed_forward", "down.weight"), (src(fp + "down", D, f),))]
        else:
            assert isinstance(mlp, MoeMlpConfig)
            f, s = mlp.expert_ff, mlp.shared_ff
            # the softmax over all experts, divided by the sum of the chosen ones' shares, is the softmax over the chosen alone
            feed_forward = PartSpec("routed_experts", {
                "hidden_size": D, "experts": mlp.experts, "top": mlp.top, "expert_size": f, "shared_size": s,
                "router": "softmax_chosen", "activation": "gelu"})
            bindings += [
                WeightBinding(target("feed_forward", "router.weight"), (src(fp + "router", mlp.experts, D),), kind="float32"),
                WeightBinding(target("feed_forward", "experts.up.weight"), tuple(src(f"{fp}e{e}.up", f, D) for e in range(mlp.experts))),
                WeightBinding(target("feed_forward", "experts.down.weight"), tuple(src(f"{fp}e{e}.down", D, f) for e in range(mlp.experts))),
            ]
            if s:
                bindings += [WeightBinding(target("feed_forward", "shared.up.weight"), (src(fp + "shared.up", s, D),)),
                             WeightBinding(target("feed_forward", "shared.down.weight"), (src(fp + "shared.down", D, s),))]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if feed_forward is not None else ()):
            bindings += norm_bindings(lambda local, name=name: target(name, local), p + name)
        layers.append(LayerSpec(mixer=mixer, feed_forward=feed_forward, norm=norm, block="sandwich",
                                block_params={"residual_scale": cfg.residual_mult}))

    run = []
    for i, again in run_order(cfg):
        gi, slot = slot_in(*places[i])
        run.append(RunEntry(layer=i, cache_group=gi, cache_slot=slot, write_cache=True, before=0 if again else -1))
    counts = {gi: n for gi, n in group_of.values()}
    groups = [replace(g, slots=counts[gi]) for gi, g in enumerate(groups)]
    junctions = (PartSpec("readd"),) if any(again for _, again in run_order(cfg)) else ()
    if present is not None:
        ignored = [name for name in ignored if name in present]
    return ModelPlan(architecture=BebulornConfig.ARCHITECTURE, vocab_size=V, hidden_size=D, layers=layers, run=run,
                     cache_groups=groups, final_norm=norm, bindings=bindings, eos_token_ids=cfg.eos_token_ids,
                     bos_token_id=cfg.bos_token_id, init={"default": ("normal", 0.0, 0.02), "suffix": init},
                     junctions=junctions, ignored=tuple(ignored) if present is not None else ())


def plan_for_checkpoint(cfg: BebulornConfig, shapes) -> ModelPlan:
    return build_bebulorn_plan(cfg, present=set(shapes))


register_architecture(BebulornConfig.ARCHITECTURE, BebulornConfig, build_bebulorn_plan, refine=plan_for_checkpoint)
