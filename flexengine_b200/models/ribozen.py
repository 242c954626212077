"""Ribozen as a plan of parts: a pre-norm decoder whose branches enter the stream times a learned number per channel.
Mixers: a matrix memory with exponential gates and a running maximum (``mlstm``); a state-space layer with one decay per head
and token (``mamba2``); and two mixers side by side (``parallel``): softmax attention under a window that keeps the first
tokens (biases, norms over whole projections, a rotation with blended frequencies, squashed scores, a gate per entry) and a
selective scan with a decay per channel, state entry and token.  Feed-forwards are routed: sigmoid scores as weights of the
experts' inputs, and a shared expert.

Checkpoint names: ``embed``, ``head``, ``final.norm``, and per layer i ``l<i>.norm1|norm2|ls1|ls2``; ``l<i>.mix.q|k|v|g|i|f|o|norm``
(and ``.i.b``, ``.f.b``); ``l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o``; ``l<i>.mix.left.q|k|v|g|o`` (biases ``.q.b|k.b|v.b``,
norms ``.q.norm|k.norm``) and ``l<i>.mix.right.in|conv|conv.b|x|dt|dt.b|A_log|D|o``; ``l<i>.mlp.router``, ``.e<k>.gate|up|down``,
``.shared.gate|up|down``.  Matrices are [out, in]; the projections of one input are bound as one matrix, all experts of a layer
as one.

Cache groups: a paged group per distinct (key/value heads, head size, window, kept tokens) and a float32 state group per
distinct seat size of each kind of recurrence, with a slot per layer.
"""
from __future__ import annotations

import math
from dataclasses import replace

from ..config.registry import register_architecture
from ..config.ribozen_config import Mamba2Config, MlstmConfig, ParallelConfig, RibozenConfig
from ..parts.matrix_memory import MatrixMemoryMixer
from ..parts.spec import (CacheGroupSpec, LayerSpec, ModelPlan, PartSpec, RunEntry, WeightBinding, WeightSource)
from ..parts.state_space import HeadStateSpaceMixer, SelectiveScanMixer


def build_ribozen_plan(cfg: RibozenConfig, present=None) -> ModelPlan:
    """``present``: the tensor names of a checkpoint; the second norm and scale of a layer without a feed-forward are then
    named as ignored where the checkpoint has them."""
    D, V = cfg.width, cfg.vocab
    norm = PartSpec("rmsnorm", {"hidden_size": D, "eps": cfg.norm_eps})
    groups: list = []
    group_of: dict = {}            # key -> [group index, slots so far]
    layers, bindings, ignored, run = [], [], [], []
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

    def state_slot(kind, elements):
        return slot_in((kind, elements), CacheGroupSpec(name=f"{kind}_state_{elements}", kind="state", slots=0, state_shape=(elements,),
                                                        state_dtype="float32"))

    near_one, near_zero = ("normal", 1.0, 0.1), ("normal", 0.0, 0.1)
    bindings += [WeightBinding(("embedding", "weight"), (src("embed", V, D, rule=("normal", 0.0, 1.0 / math.sqrt(D))),)),
                 WeightBinding(("final_norm", "weight"), (src("final.norm", D, rule=near_one),), kind="vector"),
                 WeightBinding(("lm_head", "weight"), (src("head", V, D),))]
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        mp = p + "mix."
        m = layer.mixer

        def target(part, local):
            return ("layer", i, part, local)

        def vector(local, name, *shape, rule=near_one):
            bindings.append(WeightBinding(target("mixer", local), (src(name, *shape, rule=rule),), kind="vector"))

        if isinstance(m, MlstmConfig):
            params = {"hidden_size": D, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap, "eps": cfg.norm_eps}
            mixer = PartSpec("matrix_memory", params)
            place = state_slot("memory", MatrixMemoryMixer(**params).state_elements)
            qk, inner = m.heads * m.dim, m.heads * m.vdim
            bindings += [
                WeightBinding(target("mixer", "qkvgif.weight"), (src(mp + "q", qk, D), src(mp + "k", qk, D), src(mp + "v", inner, D),
                                                                 src(mp + "g", inner, D), src(mp + "i", m.heads, D), src(mp + "f", m.heads, D))),
                WeightBinding(target("mixer", "gates.bias"), (src(mp + "i.b", m.heads, rule=("normal", -1.0, 1.0)),
                                                              src(mp + "f.b", m.heads, rule=("normal", 3.0, 1.0))), kind="vector"),
                WeightBinding(target("mixer", "o.weight"), (src(mp + "o", D, inner),)),
            ]
            vector("norm.weight", mp + "norm", inner)
            entry = RunEntry(layer=i, cache_group=place[0], cache_slot=place[1])
        elif isinstance(m, Mamba2Config):
            params = {"hidden_size": D, "heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "norm_groups": m.norm_groups,
                      "conv": m.conv, "eps": cfg.norm_eps}
            part = HeadStateSpaceMixer(**params)
            mixer = PartSpec("head_state_space", params)
            place = state_slot("head_space", part.state_elements)
            bindings += [WeightBinding(target("mixer", "in.weight"), (src(mp + "in", part.input_width, D),)),
                         WeightBinding(target("mixer", "o.weight"), (src(mp + "o", D, part.inner_width),))]
            vector("conv.weight", mp + "conv", part.channels, m.conv, rule=("normal", 0.0, 1.0 / math.sqrt(m.conv)))
            vector("conv.bias", mp + "conv.b", part.channels, rule=near_zero)
            vector("dt_bias", mp + "dt_bias", m.heads, rule=("normal", -2.0, 1.0))
            vector("A_log", mp + "A_log", m.heads, rule=("normal", -1.0, 1.0))
            vector("D", mp + "D", m.heads)
            vector("norm.weight", mp + "norm", part.inner_width)
            entry = RunEntry(layer=i, cache_group=place[0], cache_slot=place[1])
        else:
            assert isinstance(m, ParallelConfig)
            L, R = m.left, m.right
            head = -(-max(L.dim, L.vdim) // 16) * 16
            kind = "window" if L.window else "full"
            scaling = L.rot_scaling
            left = PartSpec("gated_attention", {
                "hidden_size": D, "heads": L.heads, "kv_heads": L.kv_heads, "dim": L.dim, "vdim": L.vdim, "scale": L.scale,
                "rot_base": L.rot_base, "rot_dims": L.rot_dims,
                "rot_scaling": None if scaling is None else (scaling.factor, scaling.original, scaling.fast, scaling.slow),
                "qk_norm": True, "norm_weights": True, "norm_scope": "all", "eps": cfg.norm_eps, "bias": True, "mask": kind,
                "mask_size": L.window, "keep_first": L.keep_first if L.window else 0, "softcap": L.softcap, "gate": "element"})
            right_params = {"hidden_size": D, "inner": R.inner, "state": R.state, "dt_rank": R.dt_rank, "conv": R.conv}
            right_part = SelectiveScanMixer(**right_params)
            mixer = PartSpec("parallel", {"hidden_size": D, "sides": (("left", left, m.left_scale),
                                                                      ("right", PartSpec("selective_scan", right_params), m.right_scale))})
            keep = L.keep_first if L.window else 0
            place = slot_in(("paged", L.kv_heads, head, L.window, keep),
                            CacheGroupSpec(name=f"attention_{L.kv_heads}x{head}_{L.window or 'all'}_{keep}", kind=kind, slots=0,
                                           kv_heads=L.kv_heads, head_dim=head, window=L.window, keep=keep))
            beside = state_slot("selective", right_part.state_elements)
            lp, rp = mp + "left.", mp + "right."
            qw, kw, vw = L.heads * L.dim, L.kv_heads * L.dim, L.kv_heads * L.vdim
            bindings += [
                WeightBinding(target("mixer", "left.qkvg.weight"), (src(lp + "q", qw, D), src(lp + "k", kw, D), src(lp + "v", vw, D),
                                                                    src(lp + "g", L.heads * L.vdim, D))),
                WeightBinding(target("mixer", "left.qkv.bias"), tuple(src(lp + name, n, rule=near_zero)
                                                                      for name, n in (("q.b", qw), ("k.b", kw), ("v.b", vw))), kind="vector"),
                WeightBinding(target("mixer", "left.o.weight"), (src(lp + "o", D, L.heads * L.vdim),)),
                WeightBinding(target("mixer", "right.in.weight"), (src(rp + "in", right_part.input_width, D),)),
                WeightBinding(target("mixer", "right.x.weight"), (src(rp + "x", R.dt_rank + 2 * R.state, R.inner),)),
                WeightBinding(target("mixer", "right.dt.weight"), (src(rp + "dt", R.inner, R.dt_rank),)),
                WeightBinding(target("mixer", "right.o.weight"), (src(rp + "o", D, R.inner),)),
            ]
            vector("left.q_norm.weight", lp + "q.norm", qw)
            vector("left.k_norm.weight", lp + "k.norm", kw)
            vector("right.conv.weight", rp + "conv", R.inner, R.conv, rule=("normal", 0.0, 1.0 / math.sqrt(R.conv)))
            vector("right.conv.bias", rp + "conv.b", R.inner, rule=near_zero)
            vector("right.dt.bias", rp + "dt.b", R.inner, rule=("normal", -2.0, 1.0))
            vector("right.A_log", rp + "A_log", R.inner, R.state, rule=("normal", 0.5, 0.7))
            vector("right.D", rp + "D", R.inner)
            entry = RunEntry(layer=i, cache_group=place[0], cache_slot=place[1], more=(beside,))
        run.append(entry)
        mlp = layer.mlp
        fp = p + "mlp."
        if mlp is None:
            feed_forward = None
            ignored += [p + "norm2", p + "ls2"]
        else:
            f, s = mlp.expert_ff, mlp.shared_ff
            feed_forward = PartSpec("routed_experts", {"hidden_size": D, "experts": mlp.experts, "top": mlp.top, "expert_size": f,
                                                       "shared_size": s, "router": "sigmoid", "weigh": "input"})
            bindings += [
                WeightBinding(target("feed_forward", "router.weight"), (src(fp + "router", mlp.experts, D),), kind="float32"),
                WeightBinding(target("feed_forward", "experts.gate_up.weight"),
                              tuple(src(f"{fp}e{e}.{name}", f, D) for e in range(mlp.experts) for name in ("gate", "up"))),
                WeightBinding(target("feed_forward", "experts.down.weight"), tuple(src(f"{fp}e{e}.down", D, f) for e in range(mlp.experts))),
            ]
            if s:
                bindings += [WeightBinding(target("feed_forward", "shared.gate_up.weight"), (src(fp + "shared.gate", s, D), src(fp + "shared.up", s, D))),
                             WeightBinding(target("feed_forward", "shared.down.weight"), (src(fp + "shared.down", D, s),))]
        branches = (("input_norm", "norm1", "mixer_scale", "ls1"), ("post_mixer_norm", "norm2", "feed_forward_scale", "ls2"))
        for norm_part, norm_name, scale_part, scale_name in branches[:1 if feed_forward is None else 2]:
            bindings += [WeightBinding(target(norm_part, "weight"), (src(p + norm_name, D, rule=near_one),), kind="vector"),
                         WeightBinding(target(scale_part, "weight"), (src(p + scale_name, D, rule=("normal", 0.5, 0.2)),), kind="vector")]
        layers.append(LayerSpec(mixer=mixer, feed_forward=feed_forward, norm=norm, block="scaled_prenorm", block_params={"hidden_size": D}))

    counts = {gi: n for gi, n in group_of.values()}
    groups = [replace(g, slots=counts[gi]) for gi, g in enumerate(groups)]
    if present is not None:
        ignored = [name for name in ignored if name in present]
    embedding = PartSpec("token_table", {"vocab_size": V, "hidden_size": D, "scale": cfg.embedding_scale})
    return ModelPlan(architecture=RibozenConfig.ARCHITECTURE, vocab_size=V, hidden_size=D, layers=layers, run=run,
                     cache_groups=groups, final_norm=norm, bindings=bindings, embedding=embedding,
                     eos_token_ids=cfg.eos_token_ids, bos_token_id=cfg.bos_token_id,
                     init={"default": ("normal", 0.0, 0.02), "suffix": init},
                     ignored=tuple(ignored) if present is not None else ())


def plan_for_checkpoint(cfg: RibozenConfig, shapes) -> ModelPlan:
    return build_ribozen_plan(cfg, present=set(shapes))


register_architecture(RibozenConfig.ARCHITECTURE, RibozenConfig, build_ribozen_plan, refine=plan_for_checkpoint)
