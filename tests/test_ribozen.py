"""The Ribozen decoder in the engine against the plain implementation (``plain_ribozen``): each mechanism alone (branches times a
number per channel, softmax attention with biases, norms over whole projections, a blended rotation, squashed scores, a gate per
entry and a window that keeps the first tokens, the matrix memory with exponential gates, the state-space layer with one decay per
head, the selective scan, two mixers side by side, experts that read their input times a sigmoid score), whole prompts against
token-by-token decoding, portions down to two tokens, mixed batches with pages and seats used again, keys just inside and just
outside a window and among and after the kept ones, states that must remember, the first tokens, long decoding, other sizes, and
greedy generation through the engine's entry point.

Everything runs on the CPU with the reference kernels handed to the engine (host logic: plan, cache groups, run order,
metadata) and, marked ``gpu``, with the CUDA kernels in float32 and bfloat16.  float32 is compared row by row with the
float64 oracle; bfloat16 through a whole model is measured against what rounding alone does.
"""
import json
import os
import random
import subprocess
import sys
import types

import numpy as np
import pytest
import torch

import helpers
import kernel_refs
import plain_ribozen as plain
from flexengine_b200.cache import CacheManager
from flexengine_b200.config import ConfigError, EngineConfig, resolve
from flexengine_b200.engine import ModelRunner, StepEntry
from flexengine_b200.engine.runtime import Engine
from flexengine_b200.parts import CacheGroupSpec, PartSpec, RunEntry, build_part
from flexengine_b200.parts.norm import ScaledBranch
from flexengine_b200.weights import load_model, write_random_model
from test_fedutar import (CASES, DEVICES, F64, as64, bf16_exact, bind_by_checkpoint_names, close, drive, ops_for, randn, row_errors,
                          simple_ctx)

EPS = 1e-5


# ---- configurations ---------------------------------------------------------------------------------------------------
def rotation(dims, base=10000.0, factor=None, original=64, fast=8.0, slow=1.0):
    rot = {"base": base, "dims": dims}
    if factor is not None:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return rot


def left_side(heads, kv_heads, dim, vdim, window, keep, rot=None, softcap=20.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep},
            "rot": rot or rotation(dim // 2 * 2, factor=3.0), "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap}


def right_side(inner, state, rank, conv):
    return {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def mamba2(heads, vdim, state, groups, norm_groups, conv):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def moe(experts, top, ff, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(vocab, width, eps, scale, layers):
    return {"architecture": "Ribozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


# X: every mixer once; a window shorter than a page; part of a head rotated; values wider than keys; a layer without a feed-forward
# Y: two parallel layers of different windows and kept counts (more than a page, one token), one and three taps, as many
#    groups as heads and one, one expert chosen, no shared expert, odd sizes, an embedding scale of one
# Z: heads of 64 and 128 (the tensor-core kernels in bfloat16), sizes in multiples of the kernels' tiles and beyond them
CONFIGS = {
    "X": config(211, 64, 1e-5, 5.0, [
        (mamba2(4, 12, 10, 2, 4, 4), moe(5, 2, 24, shared=40)),
        (parallel(left_side(4, 2, 16, 24, 9, 3, rotation(12, factor=2.0, original=40)), right_side(40, 6, 5, 3), 0.7, 1.3), None),
        (mlstm(3, 8, 12, 9.0), moe(4, 3, 16, shared=24))]),
    "Y": config(301, 96, 3e-6, 1.0, [
        (parallel(left_side(3, 1, 24, 8, 33, 19, rotation(24, 500.0), softcap=4.0), right_side(30, 9, 3, 1), 1.2, 0.5), moe(6, 1, 40)),
        (mlstm(2, 20, 6, 15.0), moe(3, 2, 24, shared=16)),
        (mamba2(6, 5, 7, 6, 3, 2), moe(8, 4, 16)),
        (parallel(left_side(6, 6, 10, 10, 20, 1, rotation(6, 100.0, factor=8.0, original=30, fast=4.0)), right_side(52, 20, 7, 4)), moe(3, 2, 24, shared=16)),
        (mamba2(3, 8, 16, 1, 1, 3), None)]),
    "Z": config(400, 128, 1e-6, 11.0, [
        (parallel(left_side(8, 2, 64, 64, 40, 5), right_side(256, 16, 8, 4), 0.9, 1.1), moe(4, 2, 64, shared=64)),
        (mamba2(4, 64, 72, 2, 2, 4), moe(8, 3, 32, shared=128)),
        (mlstm(2, 64, 128, 10.0), moe(4, 4, 64, shared=64)),
        (parallel(left_side(4, 4, 128, 96, 70, 33, rotation(64, 1000.0, factor=4.0, original=128)), right_side(128, 40, 16, 2)), moe(6, 1, 64, shared=32))]),
}
PAGE = {"X": 16, "Y": 8, "Z": 16}
LENGTHS = {"X": [5, 33, 70, 1, 47], "Y": [2, 40, 77, 23], "Z": [150, 64, 90]}


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp(f"ribozen_{name}")
        write_random_model(cfg, str(d), seed=171 + i)
        out[name] = str(d)
    return out


def make_runner(model_dir, dtype, device, pages, page, seats=4):
    _cfg, plan, model = load_model(model_dir, dtype, device)
    cache = CacheManager(plan.cache_groups, pages, page, seats, {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype], device)
    return ModelRunner(model, cache, ops=ops_for(device))


_PLAIN = {}


def plain_logits(model_dir, ids):
    key = (model_dir, tuple(ids))
    if key not in _PLAIN:
        _PLAIN[key] = plain.forward_logits(*plain.read_model_folder(model_dir), ids)
    return _PLAIN[key]


def as_rounding_allows(model_dir, pairs, what):
    """bfloat16 through a whole model.  A router's close call changes a token's experts and, through the states, the tokens after
    it, so the measure is what rounding alone does: the same sequences through the reference kernels in bfloat16 (whole prompts, on
    the CPU), both against the float64 oracle.  The device's median and ninth-decile row errors may be twice the reference
    kernels' and 0.03 / 0.06 more."""
    device_errors, reference_errors = [], []
    reference = make_runner(model_dir, "bfloat16", "cpu", 64, 16, seats=1)
    for ids, positions, rows in pairs:
        want = plain_logits(model_dir, ids)[positions]
        device_errors.append(row_errors(rows, want))
        rounded = reference.step([StepEntry("ref", ids, list(positions))])
        reference.finish("ref")
        reference_errors.append(row_errors(rounded, want))
    device_errors, reference_errors = torch.cat(device_errors), torch.cat(reference_errors)
    for q, slack in ((0.5, 0.03), (0.9, 0.06)):
        mine, allowed = float(device_errors.quantile(q)), 2.0 * float(reference_errors.quantile(q)) + slack
        assert mine <= allowed, f"{what}: quantile {q} of the row errors is {mine:.3f}, rounding alone allows {allowed:.3f}"


def compare(model_dir, results, requests, dtype, what):
    pairs = []
    for rid, ids in requests.items():
        rows = sorted(p for (r, p) in results if r == rid)
        assert rows == list(range(len(ids))), f"{what}: request {rid} misses rows"
        got = torch.stack([results[(rid, p)] for p in rows])
        if dtype == "float32":
            close(got, plain_logits(model_dir, ids), dtype, f"{what} request {rid}", bars=(3e-4, 0.0))
        pairs.append((ids, rows, got))
    if dtype != "float32":
        as_rounding_allows(model_dir, pairs, what)


def requests_for(name, seed=3):
    rng = random.Random(seed)
    return {f"r{i}": helpers.random_prompt(rng, n, CONFIGS[name]["vocab"]) for i, n in enumerate(LENGTHS[name])}


# ---- configuration, plan, cache ----------------------------------------------------------------------------------------
def test_plan_of_parts_and_cache_groups():
    _typed, plan = resolve(CONFIGS["Y"])
    assert plan.architecture == "Ribozen" and [layer.block for layer in plan.layers] == ["scaled_prenorm"] * 5
    assert [layer.mixer.kind for layer in plan.layers] == ["parallel", "matrix_memory", "head_state_space", "parallel", "head_state_space"]
    assert plan.layers[-1].feed_forward is None and plan.layers[0].feed_forward.params["router"] == "sigmoid"
    groups = {g.name: g for g in plan.cache_groups}
    wide, narrow = groups["attention_1x32_33_19"], groups["attention_6x16_20_1"]
    assert (wide.kind, wide.window, wide.keep, wide.slots) == ("window", 33, 19, 1) and (narrow.window, narrow.keep) == (20, 1)
    # 2 heads of 20 x 6, their memories of the keys, their maxima; 6 heads of 7 x 5 behind which one row of 30 + 2 x 6 x 7 channels lies
    assert groups["memory_state_284"].state_shape == (284,) and groups["head_space_state_328"].state_shape == (328,)
    assert groups["selective_state_272"].slots == 1              # 30 x 9 and no history: one tap
    assert plan.embedding.params["scale"] == 1.0
    parallel_runs = [e for e in plan.run if e.more]
    assert [e.layer for e in parallel_runs] == [0, 3] and all(plan.cache_groups[e.more[0][0]].kind == "state" for e in parallel_runs)
    names = {s.name for b in plan.bindings for s in b.sources}
    assert {"final.norm", "l0.mix.left.q.b", "l0.mix.left.k.norm", "l0.mix.right.dt.b", "l1.mix.f.b", "l1.mix.norm", "l2.mix.dt_bias",
            "l2.mix.conv.b", "l3.mlp.shared.up", "l2.mlp.e7.down", "head", "l4.ls1"} <= names
    assert not {"l4.norm2", "l4.ls2", "l0.mlp.shared.up"} & names


def test_configuration_errors_are_named():
    def broken(change):
        cfg = json.loads(json.dumps(CONFIGS["X"]))
        change(cfg)
        return cfg

    left = lambda c: c["layers"][1]["mixer"]["left"]
    right = lambda c: c["layers"][1]["mixer"]["right"]
    cases = [
        (lambda c: left(c).update(kv_heads=3), "kv_heads"), (lambda c: left(c)["mask"].update(size=0), "mask.size"),
        (lambda c: left(c)["mask"].update(keep_first=-1), "keep_first"), (lambda c: left(c).update(softcap=-1.0), "softcap"),
        (lambda c: left(c).pop("scale"), "scale"), (lambda c: left(c)["rot"].update(dims=7), "rot.dims"),
        (lambda c: left(c)["rot"].update(dims=18), "rot.dims"), (lambda c: left(c)["rot"].update(base=1.0), "rot.base"),
        (lambda c: left(c)["rot"]["scaling"].pop("slow"), "slow"), (lambda c: left(c)["rot"]["scaling"].update(factor=0.0), "scaling"),
        (lambda c: right(c).update(conv=0), "conv"), (lambda c: right(c).update(dt_rank=0), "dt_rank"), (lambda c: right(c).pop("inner"), "inner"),
        (lambda c: c["layers"][1]["mixer"].pop("right"), "right"), (lambda c: c["layers"][0]["mixer"].update(groups=3), "groups"),
        (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "norm_groups"), (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
        (lambda c: c["layers"][2]["mixer"].update(gate_cap=0.0), "gate_cap"), (lambda c: c["layers"][2]["mixer"].pop("vdim"), "vdim"),
        (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "experts"), (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared.ff"),
        (lambda c: c["layers"][0]["mlp"].update(shared={}), "shared.ff"), (lambda c: c["layers"][0].update(type="mystery"), "mystery"),
        (lambda c: c["layers"][0]["mlp"].update(kind="mystery"), "mystery"), (lambda c: c["norm"].update(eps=0.0), "eps"),
    ]
    for change, word in cases:
        with pytest.raises(ConfigError, match=word):
            resolve(broken(change))


def test_tensors_of_absent_parts(tmp_path):
    """The norm and the scale of a feed-forward that a layer does not have may be there and are ignored; any other stranger is
    refused by name, as is a missing bias."""
    from flexengine_b200.weights.safetensors_io import write_safetensors
    write_random_model(CONFIGS["X"], str(tmp_path), seed=1)
    _c, weights = plain.read_model_folder(str(tmp_path))
    tensors = {k: v.to(torch.bfloat16) for k, v in weights.items()}

    def write():
        write_safetensors(str(tmp_path / "model.safetensors"), [(n, tuple(t.shape), t.dtype) for n, t in tensors.items()],
                          lambda n: tensors[n])
    for name in ("l1.norm2", "l1.ls2"):
        tensors[name] = torch.ones(64, dtype=torch.bfloat16)
    write()
    load_model(str(tmp_path), "float32", "cpu")
    tensors["l1.mlp.router"] = torch.ones(8, 64, dtype=torch.bfloat16)
    write()
    with pytest.raises(Exception, match="l1.mlp.router"):
        load_model(str(tmp_path), "float32", "cpu")
    del tensors["l1.mlp.router"], tensors["l1.mix.left.v.b"]
    write()
    with pytest.raises(Exception, match="l1.mix.left.v.b"):
        load_model(str(tmp_path), "float32", "cpu")


@pytest.mark.parametrize("keep,page,held", [(0, 4, [5, 6]), (1, 4, [0, 5, 6]), (4, 4, [0, 5, 6]), (5, 4, [0, 1, 5, 6]), (3, 8, [0, 2, 3])])
def test_a_window_gives_pages_back_but_not_those_of_the_kept_tokens(keep, page, held):
    """27 tokens under a window of 5: the next query sees positions 23 .. 26 and the first ``keep``."""
    spec = CacheGroupSpec("w", "window", slots=1, kv_heads=1, head_dim=16, window=5, keep=keep)
    cache = CacheManager([spec], 16, page, 2, torch.float32, "cpu")
    for n in (9, 2, 16):
        cache.reserve("a", cache.tokens_of("a") + n)
        cache.commit("a", n)
        cache.assert_invariants()
    assert [j for j, p in enumerate(cache.table("a", 0)) if p >= 0] == held
    cache.free("a")
    cache.assert_invariants()
    assert cache.used_pages == 0
    with pytest.raises(ValueError, match="keep"):
        CacheGroupSpec("w", "full", slots=1, kv_heads=1, head_dim=16, keep=2)


# ---- each mechanism alone -----------------------------------------------------------------------------------------
def run_mixer(mixer, more=()):
    entry = RunEntry(layer=0, cache_group=0, cache_slot=0, write_cache=True, more=more)
    return lambda ctx, rows: mixer.forward(ctx, rows, entry)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("width", [40, 97, 192, 2052, 1030])
def test_branches_enter_the_stream_times_a_number_per_channel(device, dtype, width):
    """x <- x + s y, then the norm of the sum, in one kernel: all rows in place, chosen rows without writing, the branch in float32 and
    in the compute dtype."""
    dt = getattr(torch, dtype)
    T, D = 11, width
    x = torch.randn(T, D, generator=torch.Generator().manual_seed(1)) * 3.0
    y = bf16_exact(randn(T, D, seed=2, scale=2.0))
    scale, weight = randn(D, seed=3), randn(D, seed=4) + 1.0
    norm = build_part("norm", PartSpec("rmsnorm", {"hidden_size": D, "eps": EPS}))
    norm.bind({"weight": weight.to(device)})
    ctx = simple_ctx(device, dt)
    new = x.to(F64) + scale.to(F64) * y.to(F64)
    want = plain.rms_norm(new, weight.to(F64), EPS)
    rows = torch.tensor([7, 0, 10], dtype=torch.int32)
    for branch in (y.to(device=device, dtype=dt), y.to(device)):
        residual = x.to(device).clone()
        chosen = norm.forward(ctx, residual, ScaledBranch(branch, scale.to(device)), rows=rows.to(device))
        assert torch.equal(residual.cpu(), x)
        close(chosen.float().cpu(), want[rows.long()], dtype, "chosen rows", bars=(1e-5, 3e-2))
        got = norm.forward(ctx, residual, ScaledBranch(branch, scale.to(device)))
        close(got.float().cpu(), want, dtype, "all rows", bars=(1e-5, 3e-2))
        assert (residual.cpu().double() - new).abs().max() < 1e-5


def attention_weights(D, m, seed):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {"o": randn(D, H * dv, seed=seed + 4, scale=(H * dv) ** -0.5), "g": randn(H * dv, D, seed=seed + 5, scale=D ** -0.5),
         "q.norm": 1.0 + randn(H * d, seed=seed + 6, scale=0.3), "k.norm": 1.0 + randn(G * d, seed=seed + 7, scale=0.3)}
    for i, (name, rows) in enumerate((("q", H * d), ("k", G * d), ("v", G * dv))):
        w[name] = randn(rows, D, seed=seed + i, scale=D ** -0.5)
        w[name + ".b"] = randn(rows, seed=seed + 10 + i, scale=0.5)
    return w


ATTENTION_NAMES = {"qkvg.weight": ["q", "k", "v", "g"], "qkv.bias": ["q.b", "k.b", "v.b"], "o.weight": ["o"], "q_norm.weight": ["q.norm"],
                   "k_norm.weight": ["k.norm"]}


def attention_spec(D, m):
    scaling = (m["rot"] or {}).get("scaling")
    return PartSpec("gated_attention", {
        "hidden_size": D, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"],
        "rot_base": m["rot"]["base"], "rot_dims": m["rot"]["dims"],
        "rot_scaling": None if scaling is None else tuple(scaling[k] for k in ("factor", "original", "fast", "slow")), "qk_norm": True,
        "norm_weights": True, "norm_scope": "all", "eps": EPS, "bias": True, "mask": "window", "mask_size": m["mask"]["size"],
        "keep_first": m["mask"]["keep_first"], "softcap": m["softcap"], "gate": "element"})


def attention_part(D, m, weights, device, dt):
    mixer = build_part("mixer", attention_spec(D, m))
    bind_by_checkpoint_names(mixer, weights, ATTENTION_NAMES, device, dt)
    head = -(-max(m["dim"], m["vdim"]) // 16) * 16
    return mixer, [CacheGroupSpec("keys", "window", slots=1, kv_heads=m["kv_heads"], head_dim=head, window=m["mask"]["size"],
                                  keep=m["mask"]["keep_first"])]


# heads, kv_heads, dim, vdim, window, kept: values wider and narrower than keys, one head, groups of one, three and four, windows of
# one key and beyond the sequence, none, one, a page's and more kept than a window holds; 64 and 128 for the tensor-core kernels
ATTENTION_SHAPES = [(4, 2, 16, 24, 9, 3), (2, 1, 32, 16, 4, 9), (3, 3, 16, 16, 1, 1), (8, 2, 64, 64, 20, 5), (1, 1, 40, 8, 100, 2), (6, 3, 64, 128, 13, 16),
                    (6, 2, 128, 128, 17, 0), (12, 4, 24, 64, 3, 4), (5, 5, 48, 48, 12, 32)]


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_alone(device, dtype, shape):
    """Scores spread wider than the cap: a cap that is left out or a bias, weight or gain in the wrong place shows."""
    dt = getattr(torch, dtype)
    D, T = 48, 41
    m = left_side(*shape, rot=rotation(shape[2] // 4 * 2, 300.0, factor=2.5, original=24, fast=3.0), softcap=1.5, scale=2.0 * shape[2] ** -0.5)
    weights = attention_weights(D, m, seed=10)
    mixer, specs = attention_part(D, m, weights, device, dt)
    h = randn(T, D, seed=11)
    want = plain.windowed_attention(h.to(F64), as64(weights), "", m, EPS)
    for cuts in ([T], [1] * T, [7, 2, 19, 2, 1, 10], [2, 37, 2], [1, 1, 2, 1, 36]):
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"attention {shape} cut {cuts[:5]}")


@pytest.mark.parametrize("rot", [rotation(16), rotation(64, 50000.0, 4.0, 512, 32.0, 1.0), rotation(32, 100.0, 8.0, 100, 2.0, 2.0), rotation(8, 10.0, 1.0, 7, 50.0, 0.01),
                                 rotation(2, 5.0, 2.0, 64, 4.0, 1.0), rotation(48, 1e6, 40.0, 4096, 32.0, 1.0)])
def test_blended_rotation_frequencies(rot):
    freq, gain = plain.rotation_frequencies(rot)
    m = left_side(2, 1, 64, 64, 8, 1, rot=rot)
    mixer = build_part("mixer", attention_spec(32, m))
    assert torch.allclose(mixer.inverse_frequencies("cpu").double(), freq, rtol=1e-6, atol=0.0) and abs(mixer.rot_gain - gain) < 1e-12


def peaked(D, m, seed, gain):
    """Weights under which queries and keys are channels 0..15 of the input, times ``gain`` over their root mean square, the same
    for every head; no biases."""
    weights = attention_weights(D, m, seed)
    for name in ("q", "k"):
        weights[name][:] = 0.0
        weights[name + ".b"][:] = 0.0
        weights[name + ".norm"][:] = gain
        for head in range(weights[name].shape[0] // m["dim"]):
            weights[name][head * m["dim"]:head * m["dim"] + 16, :16] = torch.eye(16)
    return weights


def one_key_stands_out(T, at, D, seed):
    """Every row points anywhere but one direction, row ``at`` and the last one along it: if the last query sees row ``at``, half of its
    output comes from there, else all of it from itself."""
    h = randn(T, D, seed=seed)
    direction = randn(16, seed=seed + 1)
    direction[:2] = 0.0                                            # the two entries that turn
    direction = direction / direction.norm()
    h[:, :16] -= (h[:, :16] @ direction)[:, None] * direction
    h[at, :16] = 4.0 * direction
    h[-1, :16] = 4.0 * direction
    return bf16_exact(h)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("back", [15, 16, 31, 32, 129, 130, 639])
@pytest.mark.parametrize("dim", [16, 64])
def test_a_key_just_inside_and_just_outside_the_window(device, dtype, decoded, back, dim):
    """The window is ``back`` (just outside) or ``back`` + 1 (just inside): on both sides of a page border, far back, in prompts and
    decoded."""
    dt = getattr(torch, dtype)
    D, T = 32, 655
    h = one_key_stands_out(T, T - 1 - back, D, seed=31)
    last = {}
    for window in (back, back + 1):
        m = left_side(4, 2, dim, 16, window, 2, rot=rotation(2), softcap=60.0, scale=1.0)
        weights = peaked(D, m, 30, 3.0)
        mixer, specs = attention_part(D, m, weights, device, dt)
        want = plain.windowed_attention(h.to(F64), as64(weights), "", m, EPS)
        last[window] = want[-1]
        cuts = [300, 354, 1] if decoded else [2, 330, 321, 2]
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, f"window {window}")
    assert (last[back] - last[back + 1]).abs().max() > 0.12 * last[back + 1].abs().max()


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("at", [0, 5, 15, 16, 31, 32, 70])
@pytest.mark.parametrize("dim", [16, 128])
def test_the_last_kept_token_and_the_next(device, dtype, decoded, at, dim):
    """The key at position ``at``, hundreds of positions back, with ``at`` tokens kept (just not seen) and ``at`` + 1 (just seen): kept
    tokens that end inside, at the end and after a page and a tile of keys."""
    dt = getattr(torch, dtype)
    D, T = 32, 500
    h = one_key_stands_out(T, at, D, seed=41)
    last = {}
    for keep in (at, at + 1):
        m = left_side(4, 1, dim, 32, 37, keep, rot=rotation(2), softcap=60.0, scale=1.0)
        weights = peaked(D, m, 40, 3.0)
        mixer, specs = attention_part(D, m, weights, device, dt)
        want = plain.windowed_attention(h.to(F64), as64(weights), "", m, EPS)
        last[keep] = want[-1]
        cuts = [301, 198, 1] if decoded else [2, 130, 2, 364, 2]
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, f"kept {keep}")
    assert (last[at] - last[at + 1]).abs().max() > 0.12 * last[at + 1].abs().max()


def state_spec(mixer):
    need = mixer.cache_need()
    return [CacheGroupSpec("state", "state", slots=1, state_shape=need["state_shape"], state_dtype=need["state_dtype"])]


def mlstm_weights(D, m, seed):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    return {"q": randn(H * d, D, seed=seed, scale=D ** -0.5), "k": randn(H * d, D, seed=seed + 1, scale=D ** -0.5),
            "v": randn(H * dv, D, seed=seed + 2, scale=D ** -0.5), "g": randn(H * dv, D, seed=seed + 3, scale=D ** -0.5),
            "i": randn(H, D, seed=seed + 4, scale=3.0 * D ** -0.5), "f": randn(H, D, seed=seed + 5, scale=3.0 * D ** -0.5),
            "i.b": randn(H, seed=seed + 6), "f.b": randn(H, seed=seed + 7) + 2.0, "norm": 1.0 + randn(H * dv, seed=seed + 8, scale=0.3),
            "o": randn(D, H * dv, seed=seed + 9, scale=(H * dv) ** -0.5)}


def mlstm_part(D, m, weights, device, dt):
    mixer = build_part("mixer", PartSpec("matrix_memory", {"hidden_size": D, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
                                                           "gate_cap": m["gate_cap"], "eps": EPS}))
    bind_by_checkpoint_names(mixer, weights, {"qkvgif.weight": ["q", "k", "v", "g", "i", "f"], "gates.bias": ["i.b", "f.b"], "norm.weight": ["norm"],
                                              "o.weight": ["o"]}, device, dt)
    return mixer, state_spec(mixer)


WAYS_TO_CUT = ([45], [1] * 45, [7, 2, 19, 2, 1, 14], [2, 41, 2], [1, 1, 2, 1, 40], [9, 3, 8, 4, 5, 16])


# heads, dim, vdim, cap: values narrower and wider than keys, one head, sizes that are no multiples of four or a tile, tiles of 64
# filled and overfilled
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(3, 8, 12, 9.0), (2, 24, 40, 1.5), (1, 12, 12, 20.0), (5, 6, 9, 4.0), (2, 64, 64, 12.0), (1, 128, 72, 15.0), (6, 65, 100, 5.0),
                                   (3, 36, 130, 2.0), (2, 7, 300, 8.0)])
def test_matrix_memory_alone(device, dtype, shape):
    dt = getattr(torch, dtype)
    D = 48
    m = mlstm(*shape)["mixer"]
    weights = mlstm_weights(D, m, seed=50)
    mixer, specs = mlstm_part(D, m, weights, device, dt)
    h = randn(45, D, seed=51)
    want = plain.mlstm(h.to(F64), as64(weights), "", m, EPS)
    for cuts in WAYS_TO_CUT:
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"mlstm {shape} cut {cuts[:5]}", bars=(2e-4, 0.15))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("input_bias", [-12.0, 0.0, 12.0])
def test_the_running_maximum_and_the_floor_of_the_divisor(device, dtype, input_bias):
    """Input gates far below one (the divisor is exp(-m) = 1 and the maximum stays at its start), near it and far above it (the
    maximum grows at once); the first tokens tell a maximum that starts at zero from one that starts at minus infinity."""
    dt = getattr(torch, dtype)
    D = 32
    m = mlstm(3, 16, 8, 30.0)["mixer"]
    weights = mlstm_weights(D, m, seed=55)
    weights["i.b"][:] = input_bias
    weights["v"][:] *= 50.0 if input_bias < 0 else 1.0
    mixer, specs = mlstm_part(D, m, weights, device, dt)
    h = randn(90, D, seed=56)
    want = plain.mlstm(h.to(F64), as64(weights), "", m, EPS)
    for cuts in ([90], [1] * 90, [3, 2, 64, 2, 19]):
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"input bias {input_bias} cut {cuts[:5]}", bars=(3e-4, 0.15))


def far_memory(D, T):
    h = randn(T, D, seed=61, scale=0.2)
    h[:, 0] = 0.0
    h[3, 0] = 8.0
    silent = h.clone()
    silent[3, 0] = 0.0
    return h, silent


FAR_CUTS = [[700], [2, 330, 366, 2], [300, 380] + [1] * 20]


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("cuts", FAR_CUTS)
def test_the_matrix_memory_remembers_over_hundreds_of_tokens(device, dtype, cuts):
    """Forget gates next to one; one token writes far more than the others and is known hundreds of tokens later."""
    dt = getattr(torch, dtype)
    D, T = 32, 700
    m = mlstm(2, 16, 16, 12.0)["mixer"]
    weights = mlstm_weights(D, m, seed=60)
    weights["f"][:] = 0.0
    weights["f.b"][:] = torch.tensor([9.0, 30.0])
    weights["i"][:] = 0.0
    weights["i"][:, 0] = 1.0
    weights["i.b"][:] = -1.0
    weights["k"][:, 0] = 1.0
    mixer, specs = mlstm_part(D, m, weights, device, dt)
    h, silent = far_memory(D, T)
    want = plain.mlstm(h.to(F64), as64(weights), "", m, EPS)           # a query across the memory's one direction leaves a small sum
    other = plain.mlstm(silent.to(F64), as64(weights), "", m, EPS)
    assert (other[-1] - want[-1]).abs().max() > 0.3 * want[-1].abs().max()
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, "far memory", bars=(5e-3, 0.2))


def mamba2_weights(D, m, seed):
    H, dv, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner, C = H * dv, H * dv + 2 * G * N
    return {"in": randn(inner + C + H, D, seed=seed, scale=D ** -0.5), "conv": randn(C, taps, seed=seed + 1, scale=taps ** -0.5),
            "conv.b": randn(C, seed=seed + 2, scale=0.5), "dt_bias": randn(H, seed=seed + 3) - 1.0, "A_log": randn(H, seed=seed + 4),
            "D": randn(H, seed=seed + 5) + 1.0, "norm": 1.0 + randn(inner, seed=seed + 6, scale=0.3), "o": randn(D, inner, seed=seed + 7, scale=inner ** -0.5)}


def mamba2_part(D, m, weights, device, dt):
    mixer = build_part("mixer", PartSpec("head_state_space", dict(m, hidden_size=D, eps=EPS)))
    names = {"in.weight": ["in"], "conv.weight": ["conv"], "conv.bias": ["conv.b"], "dt_bias": ["dt_bias"], "A_log": ["A_log"], "D": ["D"],
             "norm.weight": ["norm"], "o.weight": ["o"]}
    bind_by_checkpoint_names(mixer, weights, names, device, dt)
    return mixer, state_spec(mixer)


# heads, vdim, state, groups, norm_groups, taps: one group and a group per head, parts of a norm across and inside heads, one to six
# taps, sizes that are no multiples of four or a tile, tiles of 64 filled and overfilled
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(4, 12, 10, 2, 4, 4), (6, 5, 7, 6, 3, 2), (3, 8, 16, 1, 1, 3), (1, 7, 5, 1, 7, 1), (4, 64, 64, 2, 2, 4), (2, 72, 130, 2, 1, 6),
                                   (8, 16, 128, 4, 8, 4), (2, 200, 33, 1, 5, 3)])
def test_head_state_space_alone(device, dtype, shape):
    dt = getattr(torch, dtype)
    D = 48
    m = mamba2(*shape)["mixer"]
    weights = mamba2_weights(D, m, seed=70)
    mixer, specs = mamba2_part(D, m, weights, device, dt)
    h = randn(45, D, seed=71)
    want = plain.mamba2(h.to(F64), as64(weights), "", m, EPS)
    for cuts in WAYS_TO_CUT:
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"mamba2 {shape} cut {cuts[:5]}", bars=(2e-4, 8e-2))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("cuts", FAR_CUTS)
def test_head_state_space_remembers_over_hundreds_of_tokens(device, dtype, cuts):
    dt = getattr(torch, dtype)
    D, T = 32, 700
    m = mamba2(2, 16, 12, 1, 2, 2)["mixer"]
    weights = mamba2_weights(D, m, seed=80)
    weights["A_log"][:] = -9.0
    weights["in"][-2:] *= 0.1                                      # step sizes that hardly move
    weights["in"][:, 0] = 1.0
    weights["conv.b"][:] = 0.0
    mixer, specs = mamba2_part(D, m, weights, device, dt)
    h, silent = far_memory(D, T)
    want = plain.mamba2(h.to(F64), as64(weights), "", m, EPS)
    other = plain.mamba2(silent.to(F64), as64(weights), "", m, EPS)
    assert (other[-1] - want[-1]).abs().max() > 0.3 * want[-1].abs().max()
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, "far memory", bars=(3e-4, 0.2))


def scan_weights(D, m, seed):
    I, N, R, taps = m["inner"], m["state"], m["dt_rank"], m["conv"]
    return {"in": randn(2 * I, D, seed=seed, scale=D ** -0.5), "conv": randn(I, taps, seed=seed + 1, scale=taps ** -0.5),
            "conv.b": randn(I, seed=seed + 2, scale=0.5), "x": randn(R + 2 * N, I, seed=seed + 3, scale=2.0 * I ** -0.5),
            "dt": randn(I, R, seed=seed + 4, scale=R ** -0.5), "dt.b": randn(I, seed=seed + 5) - 1.0,
            "A_log": randn(I, N, seed=seed + 6), "D": randn(I, seed=seed + 7) + 1.0, "o": randn(D, I, seed=seed + 8, scale=I ** -0.5)}


SCAN_NAMES = {"in.weight": ["in"], "conv.weight": ["conv"], "conv.bias": ["conv.b"], "x.weight": ["x"], "dt.weight": ["dt"], "dt.bias": ["dt.b"],
              "A_log": ["A_log"], "D": ["D"], "o.weight": ["o"]}


def scan_part(D, m, weights, device, dt):
    mixer = build_part("mixer", PartSpec("selective_scan", dict(m, hidden_size=D)))
    bind_by_checkpoint_names(mixer, weights, SCAN_NAMES, device, dt)
    return mixer, state_spec(mixer)


# inner, state, rank, taps: every width of the kernel's groups of lanes, states that do not fill them, ranks in and out of step with eight
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(40, 6, 5, 3), (30, 9, 3, 1), (256, 16, 8, 4), (52, 20, 7, 4), (128, 40, 16, 2), (33, 1, 1, 2), (72, 64, 24, 5), (24, 100, 4, 4), (12, 300, 2, 3)])
def test_selective_scan_alone(device, dtype, shape):
    dt = getattr(torch, dtype)
    D = 48
    m = right_side(*shape)
    weights = scan_weights(D, m, seed=90)
    mixer, specs = scan_part(D, m, weights, device, dt)
    h = randn(45, D, seed=91)
    want = plain.mamba(h.to(F64), as64(weights), "", m)
    for cuts in WAYS_TO_CUT:
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"scan {shape} cut {cuts[:5]}", bars=(2e-4, 0.12))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("cuts", FAR_CUTS)
def test_the_selective_scan_remembers_over_hundreds_of_tokens(device, dtype, cuts):
    dt = getattr(torch, dtype)
    D, T = 32, 700
    m = right_side(48, 16, 4, 3)
    weights = scan_weights(D, m, seed=95)
    weights["A_log"][:] = -9.0
    weights["dt"][:] *= 0.1
    weights["in"][:, 0] = 1.0
    weights["conv.b"][:] = 0.1
    mixer, specs = scan_part(D, m, weights, device, dt)
    h, silent = far_memory(D, T)
    want = plain.mamba(h.to(F64), as64(weights), "", m)
    other = plain.mamba(silent.to(F64), as64(weights), "", m)
    assert (other[-1] - want[-1]).abs().max() > 0.3 * want[-1].abs().max()
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, "far memory", bars=(3e-4, 0.2))


@pytest.mark.parametrize("device,dtype", CASES)
def test_recurrences_over_a_portion_of_thousands_of_tokens(device, dtype):
    dt = getattr(torch, dtype)
    D, T = 16, 2300
    cuts = [2200, 98, 1, 1]
    h = randn(T, D, seed=101)
    for m, make, weigh, oracle in ((mlstm(2, 16, 24, 10.0)["mixer"], mlstm_part, mlstm_weights, lambda w, m: plain.mlstm(h.to(F64), w, "", m, EPS)),
                                   (mamba2(3, 20, 16, 1, 3, 4)["mixer"], mamba2_part, mamba2_weights, lambda w, m: plain.mamba2(h.to(F64), w, "", m, EPS)),
                                   (right_side(40, 16, 4, 4), scan_part, scan_weights, lambda w, m: plain.mamba(h.to(F64), w, "", m))):
        weights = weigh(D, m, seed=100)
        mixer, specs = make(D, m, weights, device, dt)
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=160), oracle(as64(weights), m), dtype, f"a long portion {m}", bars=(5e-4, 0.2))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [((4, 2, 16, 24, 9, 3), (40, 6, 5, 3), 0.7, 1.3), ((8, 2, 64, 64, 20, 5), (256, 16, 8, 4), 1.5, 0.25), ((3, 1, 24, 8, 33, 0), (30, 9, 3, 1), 1.0, -1.0)])
def test_two_mixers_side_by_side(device, dtype, shape):
    dt = getattr(torch, dtype)
    D, T = 64, 45
    m = parallel(left_side(*shape[0]), right_side(*shape[1]), *shape[2:])["mixer"]
    weights = {f"left.{k}": v for k, v in attention_weights(D, m["left"], seed=110).items()}
    weights.update({f"right.{k}": v for k, v in scan_weights(D, m["right"], seed=130).items()})
    mixer = build_part("mixer", PartSpec("parallel", {"hidden_size": D, "sides": (
        ("left", attention_spec(D, m["left"]), m["left_scale"]), ("right", PartSpec("selective_scan", dict(m["right"], hidden_size=D)), m["right_scale"]))}))
    names = {f"{side}.{local}": [f"{side}.{n}" for n in sources] for side, table in (("left", ATTENTION_NAMES), ("right", SCAN_NAMES))
             for local, sources in table.items()}
    bind_by_checkpoint_names(mixer, weights, names, device, dt)
    keys, state = mixer.cache_need()
    specs = [CacheGroupSpec("keys", keys["kind"], slots=1, kv_heads=keys["kv_heads"], head_dim=keys["head_dim"], window=keys["window"], keep=keys["keep"]),
             CacheGroupSpec("state", "state", slots=1, state_shape=state["state_shape"], state_dtype="float32")]
    h = randn(T, D, seed=111)
    want = plain.parallel(h.to(F64), as64(weights), "", m, EPS)
    for cuts in WAYS_TO_CUT:
        close(drive(run_mixer(mixer, more=((1, 0),)), specs, h, cuts, device, dt), want, dtype, f"side by side {shape} cut {cuts[:5]}", bars=(2e-4, 8e-2))


def routed_weights(D, mlp, seed):
    E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
    w = {"router": randn(E, D, seed=seed, scale=2.0 * D ** -0.5)}
    sizes = {f"e{e}": F for e in range(E)}
    if mlp.get("shared"):
        sizes["shared"] = mlp["shared"]["ff"]
    for i, (name, size) in enumerate(sizes.items()):
        w[name + ".gate"] = randn(size, D, seed=seed + 10 + 3 * i, scale=2.0 * D ** -0.5)
        w[name + ".up"] = randn(size, D, seed=seed + 11 + 3 * i, scale=2.0 * D ** -0.5)
        w[name + ".down"] = randn(D, size, seed=seed + 12 + 3 * i, scale=size ** -0.5)
    return w


def routed_part(D, mlp, weights, device, dt):
    E, shared = mlp["router"]["experts"], (mlp.get("shared") or {"ff": 0})["ff"]
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": D, "experts": E, "top": mlp["router"]["top"], "expert_size": mlp["expert"]["ff"], "shared_size": shared,
        "router": "sigmoid", "weigh": "input"}))
    names = {"router.weight": ["router"], "experts.gate_up.weight": [f"e{e}.{n}" for e in range(E) for n in ("gate", "up")],
             "experts.down.weight": [f"e{e}.down" for e in range(E)]}
    if shared:
        names.update({"shared.gate_up.weight": ["shared.gate", "shared.up"], "shared.down.weight": ["shared.down"]})
    bind_by_checkpoint_names(part, weights, names, device, dt)
    return part


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(5, 2, 24, 40), (6, 1, 40, 0), (4, 4, 64, 8), (8, 3, 32, 128), (1, 1, 16, 16), (12, 2, 64, 64), (40, 6, 9, 24)])
def test_routed_feed_forward_alone(device, dtype, shape):
    """The chosen experts and their scores are compared as well as the sum.  Rows whose choice is a close call are left out in
    bfloat16."""
    dt = getattr(torch, dtype)
    D = 64
    mlp = moe(*shape)
    weights = routed_weights(D, mlp, seed=20)
    part = routed_part(D, mlp, weights, device, dt)
    for T in (1, 7, 90, 300):
        h = randn(T, D, seed=5 + T)
        gaps = []
        want = plain.routed_feed_forward(h.to(F64), as64(weights), "", mlp, gaps)
        chosen, share = plain.route(h.to(F64) @ weights["router"].to(F64).T, mlp["router"]["top"])
        ctx = simple_ctx(device, dt)
        logits = ctx.ops.linear(h.to(device=device, dtype=dt), part.router_weight, None, out_float32=True)
        got_chosen, got_share = ctx.ops.route_top(logits, part.top, 1.0, sigmoid=True)
        sure = gaps[0] > (1e-5 if dtype == "float32" else 2e-2) if gaps else torch.ones(T, dtype=torch.bool)
        for row in sure.nonzero().flatten().tolist():
            mine = dict(zip(got_chosen[row].tolist(), got_share[row].tolist()))
            theirs = dict(zip(chosen[row].tolist(), share[row].tolist()))
            assert mine.keys() == theirs.keys() and all(abs(mine[e] - theirs[e]) < 1e-5 for e in mine)
        if bool(sure.any()):
            got = part.forward(ctx, h.to(device=device, dtype=dt))
            close(got.float().cpu()[sure], want[sure], dtype, f"routed {shape} rows {T}")


def test_parts_refuse_options_that_do_not_go_together():
    base = {"hidden_size": 32, "heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 1.0}
    for more, word in (({"bias": True}, "norm over the whole"), ({"keep_first": 2}, "window"), ({"mask": "chunk", "mask_size": 4, "keep_first": 2}, "window"),
                       ({"rot_scaling": (2.0, 8, 4, 1)}, "norm over the whole")):
        with pytest.raises(ValueError, match=word):
            build_part("mixer", PartSpec("gated_attention", dict(base, **more)))
    experts = {"hidden_size": 32, "experts": 4, "top": 2, "expert_size": 8}
    for more in ({"weigh": "sideways"}, {"weigh": "input", "identity": 1}, {"router": "sigmoid", "correction": True}):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_experts", dict(experts, **more)))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("head_state_space", {"hidden_size": 8, "heads": 3, "vdim": 4, "state": 4, "groups": 2, "norm_groups": 1, "conv": 2, "eps": EPS}))


# ---- kernels alone (GPU) ---------------------------------------------------------------------------------------------------
PORTIONS, SEATS = [1, 2, 3, 63, 64, 65, 127, 130, 5], [2, 0, -1, 5, 1, 4, 8, 3, 6]


def one_step(lengths, seats):
    return (torch.tensor([0] + list(np.cumsum(lengths)), dtype=torch.int32), torch.tensor(seats, dtype=torch.int32), sum(lengths))


def near(got, want, bar, what):
    want = want.cpu()
    err = float((got.float().cpu() - want.float()).abs().max())
    assert err <= bar * max(1e-3, float(want.float().abs().max())), f"{what}: error {err:.3e} of {float(want.abs().max()):.3e}"


@pytest.mark.gpu
@pytest.mark.parametrize("divided", [False, True])
@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 2, 64, 128), (3, 3, 24, 40), (6, 1, 130, 72), (2, 2, 17, 9), (8, 4, 128, 64)])
def test_head_scan_kernels_against_the_references(heads, groups, dim, vdim, divided):
    """One step of portions around the length of a block, over seats that hold a state, fresh ones and a request without a seat:
    outputs and states afterwards, decays from one to nothing; then one token a request over the same seats."""
    from flexengine_b200 import ops
    dev = "cuda:0"
    gen = torch.Generator().manual_seed(7)
    per = heads * (dim * vdim + dim)
    for lengths in (PORTIONS, [1] * 9):
        cu, slots, T = one_step(lengths, SEATS)
        rows = torch.randn(T, 2 * groups * dim + heads * vdim + 3, generator=gen)
        gates = torch.stack([-torch.rand(T, heads, generator=gen) ** 4 * 30.0, torch.rand(T, heads, generator=gen), torch.rand(T, heads, generator=gen)])
        state = torch.randn(9, per + 5, generator=gen) * 0.5
        skip = None if divided else torch.randn(heads, generator=gen)
        extra = {"divided": 1e-6} if divided else {"skip": skip}

        def parts(x):
            return x[:, :groups * dim], x[:, groups * dim:2 * groups * dim], x[:, 2 * groups * dim:2 * groups * dim + heads * vdim]
        want_state = state.clone()
        want = kernel_refs.head_scan(*parts(rows), gates, want_state, slots, cu, heads, groups, dim, vdim, query_scale=0.3, **extra)
        moved = state.to(dev)
        on_device = {k: (v.to(dev) if torch.is_tensor(v) else v) for k, v in extra.items()}
        got = ops.head_scan(*parts(rows.to(dev)), gates.to(dev), moved, slots.to(dev), cu.to(dev), heads, groups, dim, vdim, query_scale=0.3,
                            max_q_len=max(lengths), **on_device)
        if divided:                       # a divisor near its floor magnifies rounding: such entries are compared by what they were divided
            assert torch.isfinite(got).all()
            near(torch.tanh(got.cpu() / 50.0), torch.tanh(want / 50.0), 2e-3, "outputs")
        else:
            near(got, want, 3e-5, "outputs")
        near(moved, want_state, 3e-5, "states")


@pytest.mark.gpu
@pytest.mark.parametrize("heads", [1, 3, 8])
def test_memory_gates_against_the_reference(heads):
    from flexengine_b200 import ops
    dev = "cuda:0"
    cu, slots, T = one_step(PORTIONS, SEATS)
    gen = torch.Generator().manual_seed(8)
    rows, bias = torch.randn(T, 2 * heads + 3, generator=gen) * 6.0, torch.randn(2 * heads, generator=gen)
    state = torch.randn(9, heads + 7, generator=gen).abs()
    want_state = state.clone()
    want = kernel_refs.memory_gates(rows, bias, 9.0, want_state, 5, slots, cu, heads)
    moved = state.to(dev)
    got = ops.memory_gates(rows.to(dev), bias.to(dev), 9.0, moved, 5, slots.to(dev), cu.to(dev), heads)
    got = got.cpu()
    assert (got[0] - want[0]).abs().max() < 5e-5 and ((got[1:] - want[1:]).abs() <= 1e-4 * want[1:] + 1e-7).all()
    assert (moved.cpu() - want_state).abs().max() < 2e-5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("channels,taps", [(40, 4), (37, 3), (516, 2), (1030, 1), (24, 7)])
def test_convolution_kernel_against_the_reference(channels, taps, dtype):
    from flexengine_b200 import ops
    dev, dt = "cuda:0", getattr(torch, dtype)
    gen = torch.Generator().manual_seed(9)
    for lengths in (PORTIONS, [1] * 9, [2, 1, 3, 1, 1, 2, 8, 9, 1]):
        cu, slots, T = one_step(lengths, SEATS)
        u = torch.randn(T, channels + 5, generator=gen).to(dt)
        conv, bias = torch.randn(taps, channels, generator=gen), torch.randn(channels, generator=gen)
        at = 8
        state = torch.randn(9, at + (taps - 1) * channels + 3, generator=gen)
        rows, dt_bias, minus_a = torch.randn(T, 6, generator=gen), torch.randn(5, generator=gen), -torch.rand(5, generator=gen)
        want_state = state.clone()
        want, want_gates = kernel_refs.conv_silu(u[:, 2:2 + channels], conv, bias, want_state, at, slots, cu, steps=(rows[:, :5], dt_bias, minus_a))
        moved = state.to(dev)
        got, gates = ops.conv_silu(u.to(dev)[:, 2:2 + channels], conv.to(dev), bias.to(dev), moved, at, slots.to(dev), cu.to(dev),
                                   steps=(rows.to(dev)[:, :5], dt_bias.to(dev), minus_a.to(dev)), max_q_len=max(lengths))
        near(got, want, 1e-5 if dtype == "float32" else 8e-3, "rows")
        near(gates, want_gates, 1e-5, "steps")
        assert torch.equal(moved.cpu(), want_state)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inner,N,rank", [(256, 16, 16), (100, 5, 3), (70, 24, 8), (64, 64, 5), (40, 128, 8), (9, 200, 2)])
def test_selective_scan_kernels_against_the_references(inner, N, rank, dtype):
    """Portions around the length of a tile over kept, fresh and absent seats, rows with strides of their own; then one token a
    request with the step sizes' projection inside."""
    from flexengine_b200 import ops
    dev, dt = "cuda:0", getattr(torch, dtype)
    bar = 3e-5 if dtype == "float32" else 8e-3
    gen = torch.Generator().manual_seed(10)
    cu, slots, T = one_step(PORTIONS, SEATS)
    x, z, low = torch.randn(T, inner, generator=gen).to(dt), torch.randn(T, inner + 3, generator=gen).to(dt), torch.randn(T, rank + 2 * N, generator=gen).to(dt)
    steps, dt_bias, skip = torch.randn(T, inner, generator=gen), torch.randn(inner, generator=gen), torch.randn(inner, generator=gen)
    minus_a = -torch.exp(torch.randn(inner, N, generator=gen))
    weight = (torch.randn(inner, rank, generator=gen) * rank ** -0.5).to(dt)
    state = torch.randn(9, -(-inner * N // 4) * 4 + 4, generator=gen)
    want_state = state.clone()
    want = kernel_refs.selective_scan(x, steps, dt_bias, minus_a, low[:, rank:], skip, z[:, 1:1 + inner], want_state, slots, cu, scale=0.6)
    d = {k: v.to(dev) for k, v in dict(x=x, z=z, low=low, steps=steps, dt_bias=dt_bias, skip=skip, minus_a=minus_a, weight=weight, state=state, slots=slots,
                                       cu=cu).items()}
    wide = torch.zeros(T, inner + 5, dtype=dt, device=dev)
    ops.selective_scan(d["x"], d["steps"], d["dt_bias"], d["minus_a"], d["low"][:, rank:], d["skip"], d["z"][:, 1:1 + inner], d["state"], d["slots"], d["cu"],
                       scale=0.6, into=wide[:, 2:2 + inner])
    near(wide[:, 2:2 + inner], want, bar, "outputs")
    assert not wide[:, :2].any() and not wide[:, 2 + inner:].any()
    near(d["state"], want_state, 3e-5, "states")
    R = len(SEATS)
    want = kernel_refs.selective_decode(x[:R], low[:R], weight, dt_bias, minus_a, skip, z[:R, :inner], want_state, slots)
    got = ops.selective_decode(d["x"][:R], d["low"][:R], d["weight"], d["dt_bias"], d["minus_a"], d["skip"], d["z"][:R, :inner], d["state"], d["slots"])
    near(got, want, bar, "one token a request")
    near(d["state"], want_state, 5e-5, "states after one token")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inner,groups", [(64, 2), (96, 1), (90, 6), (4096, 8), (5000, 1), (14000, 1)])
def test_gated_group_norm_kernel_against_the_reference(inner, groups, dtype):
    from flexengine_b200 import ops
    gen = torch.Generator().manual_seed(11)
    y, z, w = torch.randn(7, inner, generator=gen), torch.randn(7, inner + 4, generator=gen), torch.randn(inner, generator=gen)
    want = kernel_refs.gated_group_rmsnorm(y, z[:, :inner], w, EPS, groups, torch.float32)
    got = ops.gated_group_rmsnorm(y.cuda(), z.cuda()[:, :inner], w.cuda(), EPS, groups, getattr(torch, dtype))
    near(got, want, 1e-5 if dtype == "float32" else 8e-3, "rows")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(4, 2, 32, 8), (8, 2, 64, 16), (6, 6, 16, 16), (16, 1, 128, 16), (3, 1, 48, 4), (12, 3, 64, 16), (2, 1, 256, 16)])
@pytest.mark.parametrize("lengths", [[(0, 70)], [(299, 1), (37, 1), (1, 1)], [(40, 33), (130, 1), (0, 2), (15, 300)], [(1000, 1)] * 3, [(0, 1100)], [(700, 130)]])
def test_kept_first_tokens_in_every_attention_kernel(dtype, shape, lengths):
    """Windows and kept counts that end inside and at the ends of tiles and pages, with and without squashed scores, in every
    attention kernel by name.  The pages that neither holds are not in the table."""
    from flexengine_b200 import ops
    nq, nkv, d, page = shape
    dt, dev = getattr(torch, dtype), "cuda:0"
    gen = torch.Generator().manual_seed(5)
    R = len(lengths)
    starts, counts = [s for s, _ in lengths], [n for _, n in lengths]
    T, most = sum(counts), max(s + n for s, n in lengths)
    per = -(-most // page)
    pages = R * per + 3
    full = torch.randperm(pages, generator=gen)[:R * per].view(R, per).to(torch.int32)
    kc = (torch.randn(pages, nkv, page, d, generator=gen) * 0.7).to(device=dev, dtype=dt)
    vc = torch.randn(pages, nkv, page, d, generator=gen).to(device=dev, dtype=dt)
    q = torch.randn(T, nq * d + 8, generator=gen).to(device=dev, dtype=dt)
    cu = torch.tensor([0] + list(np.cumsum(counts)), dtype=torch.int32, device=dev)
    ctx = types.SimpleNamespace(cu_q=cu, q_start=torch.tensor(starts, dtype=torch.int32, device=dev),
                                token_request=torch.repeat_interleave(torch.arange(R, dtype=torch.int32), torch.tensor(counts)).to(dev),
                                max_q_len=max(counts), max_ctx_len=most, host_lengths=counts, host_starts=starts)
    scale = 1.5 * d ** -0.5
    for window, keep, cap in ((50, 6, 3.0), (20, 64, 0.0), (64, 33, 20.0), (1, 1, 0.0), (128, 200, 5.0)):
        table = full.clone()
        for r, s in enumerate(starts):                    # what a window's cache has given back
            first_needed = max(0, s - window + 1) // page
            table[r, -(-keep // page):first_needed] = -1
        table = table.to(dev)
        score = {"softcap": cap} if cap else {}
        want = kernel_refs.paged_attention(q, kc, vc, table, ctx, nq, nkv, d, page, scale, window, keep_first=keep, **score)
        runs = {"as the step would choose": lambda: ops.paged_attention(q, kc, vc, table, ctx, nq, nkv, d, page, scale, window, keep_first=keep, **score)}
        if dtype == "bfloat16":
            common = (q, q.stride(0), kc, vc, table, ctx.cu_q, ctx.q_start)
            more = dict(score, keep=keep)
            if max(counts) == 1 and nq // nkv <= 16:
                for splits in (1, 3, 8):
                    runs[f"cluster of {splits}"] = lambda splits=splits: ops.paged_decode_cluster(*common, R, nq, nkv, d, page, scale, window, splits, **more)
                for splits in (1, 5, 40):
                    runs[f"{splits} splits and a merge"] = lambda splits=splits: ops.paged_decode_mma(*common, R, nq, nkv, d, page, scale, window, splits, **more)
            runs["mma.sync portions"] = lambda: ops.paged_prefill_mma(*common, T, R, max(counts), nq, nkv, d, page, scale, window, **more)
            if d in (64, 128):
                for splits in (1, 4):
                    runs[f"tcgen05 portions, keys split {splits} ways"] = lambda splits=splits: ops.paged_prefill_tcgen05(
                        *common, T, R, max(counts), nq, nkv, d, page, scale, window, splits=splits, **more)
        for what, run in runs.items():
            near(run(), want, 2e-4 if dtype == "float32" else 3e-2, f"{what}, window {window}, kept {keep}")
    ops.check_status(dev)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,width,experts", [(1, 64, 5), (8, 2048, 8), (301, 132, 16), (37, 4, 1), (50, 1028, 64), (9, 66, 7), (20, 128, 65)])
def test_router_logits_kernel_against_the_reference(T, width, experts, dtype):
    """Also what goes to the float32 product instead: widths that do not come in fours, more than 64 experts.  A token's logits do
    not depend on what else is in the batch."""
    from flexengine_b200 import ops
    h = randn(T, width, seed=12).to(device="cuda:0", dtype=getattr(torch, dtype))
    w = randn(experts, width, seed=13, scale=width ** -0.5).cuda()
    got = ops.router_logits(h, w)
    near(got, (h.double() @ w.double().T).float(), 1e-5, "logits")
    for row in (0, T // 2, T - 1):
        assert torch.equal(ops.router_logits(h[row:row + 1].contiguous(), w), got[row:row + 1])


@pytest.mark.gpu
@pytest.mark.parametrize("T,D,F,experts,top", [(700, 1024, 1024, 4, 2), (1500, 1024, 1536, 3, 1), (300, 256, 128, 6, 3), (6, 128, 64, 8, 2), (3, 72, 36, 5, 2), (200, 68, 36, 5, 2)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("activation", ["silu", "clamped", "relu2", "gelu"])
def test_weights_on_the_experts_inputs_in_every_grouped_product(T, D, F, experts, top, dtype, activation):
    from flexengine_b200 import ops
    dt = getattr(torch, dtype)
    gen = torch.Generator().manual_seed(3)
    single = activation in ("relu2", "gelu")
    h = randn(T, D, seed=4).to(device="cuda:0", dtype=dt)
    first = randn(experts, F if single else 2 * F, D, seed=5, scale=2.0 * D ** -0.5).to(device="cuda:0", dtype=dt)
    down = randn(experts, D, F, seed=6, scale=F ** -0.5).to(device="cuda:0", dtype=dt)
    chosen = torch.stack([torch.randperm(experts, generator=gen)[:top] for _ in range(T)]).to(torch.int32).cuda()
    weights = torch.rand(T, top, generator=gen).cuda()
    options = dict(activation=activation, limit=2.0 if activation == "clamped" else 0.0, weigh_input=True)
    got = ops.routed_experts(h, chosen, weights, first, down, **options)
    want = kernel_refs.routed_experts(h, chosen, weights, first, down, **options)
    near(got, want.cpu(), 1e-4 if dtype == "float32" else 3e-2, "rows")
    ops.check_status("cuda:0")


# ---- whole models -------------------------------------------------------------------------------------------------------
def scenario(kind, requests, rng):
    if kind == "whole":
        return helpers.steps_whole(requests)
    if kind == "last_decoded":
        return helpers.steps_last_decoded(requests, tail=12)
    if kind == "portions":
        return helpers.steps_portions(requests, rng)
    doubled = dict(requests)
    doubled.update({rid + "x": ids[::-1] for rid, ids in requests.items()})     # more requests than seats: seats are used again
    return helpers.steps_mixed(doubled, rng, live=4)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("kind", ["whole", "last_decoded", "portions", "mixed"])
@pytest.mark.parametrize("name", ["X", "Y", "Z"])
def test_model_against_plain(model_dirs, name, kind, device, dtype):
    rng = random.Random(5)
    steps = scenario(kind, requests_for(name), rng)
    page = PAGE[name]
    pages = helpers.peak_pages(steps, page) + (0 if kind == "mixed" else 1)         # just enough: pages are used again
    runner = make_runner(model_dirs[name], dtype, device, pages, page, seats=4)
    results = helpers.run_steps(runner, steps)
    assert runner.cache.used_pages == 0 and len(runner.cache.free_state_slots) == 4
    fed = {}
    for entries, _ in steps:
        for rid, toks, _w in entries:
            fed.setdefault(rid, []).extend(toks)
    compare(model_dirs[name], results, fed, dtype, f"{name}/{kind}/{dtype}")
    if device != "cpu":
        ops_for(device).check_status(device)


def test_the_stream_after_every_layer_against_plain(model_dirs):
    """The residual stream after every layer, with what is pending put in: the plain implementation's."""
    for name in ("X", "Y", "Z"):
        ids = requests_for(name)["r1"]
        cfg, weights = plain.read_model_folder(model_dirs[name])
        after = []
        plain.forward_logits(cfg, weights, ids, after)
        _cfg, plan, model = load_model(model_dirs[name], "float32", "cpu")
        cache = CacheManager(plan.cache_groups, 16, 16, 1, torch.float32, "cpu")
        runner = ModelRunner(model, cache, ops=kernel_refs)
        cache.reserve("a", len(ids))
        ctx = runner.build_context([StepEntry("a", ids, [])])
        residual, pending = model.embedding.forward(ctx), None
        for at, entry in enumerate(plan.run):
            pending = model.blocks[entry.layer].forward(ctx, residual, pending, entry)
            settled = residual.double() + pending.weight.double() * pending.y.double()
            assert (settled - after[at]).abs().max() < 2e-5 * float(after[at].abs().max()), f"{name}: layer {at}"


STACKS = {
    "one parallel layer without a feed-forward": config(50, 32, 1e-5, 3.0, [(parallel(left_side(2, 1, 16, 16, 5, 2), right_side(24, 4, 3, 2)), None)]),
    "matrix memories only": config(97, 48, 1e-5, 7.0, [(mlstm(2, 8, 8, 6.0), moe(2, 1, 8)), (mlstm(1, 24, 16, 3.0), None), (mlstm(4, 4, 12, 12.0), moe(3, 3, 8, shared=8))]),
    "one head state space": config(64, 40, 1e-6, 1.0, [(mamba2(2, 10, 6, 2, 4, 5), moe(3, 2, 16, shared=8))]),
    "kept tokens beyond a window, no cap": config(61, 32, 1e-5, 2.0, [
        (parallel(dict(left_side(4, 2, 8, 8, 3, 11), softcap=0.0), right_side(16, 3, 2, 3), 0.4, 2.0), moe(2, 2, 24))]),
    "every earlier key": config(83, 56, 1e-6, 4.0, [
        (parallel({k: v for k, v in left_side(7, 7, 8, 8, 1, 0).items() if k != "mask"}, right_side(20, 5, 9, 4)), moe(4, 2, 12, shared=20)),
        (mamba2(4, 6, 12, 1, 2, 1), None)]),
}


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("stack", list(STACKS))
def test_stacks_of_other_shapes(tmp_path, stack, device, dtype):
    cfg = STACKS[stack]
    write_random_model(cfg, str(tmp_path), seed=3)
    ids = helpers.random_prompt(random.Random(1), 45, cfg["vocab"])
    runner = make_runner(str(tmp_path), dtype, device, 8, 8)
    got = [runner.step([StepEntry("a", ids[:20], list(range(20)))]), runner.step([StepEntry("a", ids[20:44], list(range(24)))]),
           runner.step([StepEntry("a", ids[44:], [0])])]
    rows = torch.cat([g.float().cpu() for g in got])
    want = plain.forward_logits(cfg, plain.read_model_folder(str(tmp_path))[1], ids)
    if dtype == "float32":
        close(rows, want, dtype, stack, bars=(3e-4, 0.0))
    else:
        _PLAIN[(str(tmp_path), tuple(ids))] = want
        as_rounding_allows(str(tmp_path), [(ids, list(range(len(ids))), rows)], stack)
    runner.finish("a")
    runner.cache.assert_invariants()


@pytest.mark.parametrize("device,dtype", CASES)
def test_together_and_alone(model_dirs, device, dtype):
    """Unequal requests in one batch against each alone: the same logits (to rounding in bfloat16)."""
    name = "Z"
    requests = requests_for(name, seed=9)
    together = make_runner(model_dirs[name], dtype, device, 32, PAGE[name])
    logits = together.step([StepEntry(rid, ids, [len(ids) - 1]) for rid, ids in requests.items()])
    for row, (rid, ids) in enumerate(requests.items()):
        alone = make_runner(model_dirs[name], dtype, device, 16, PAGE[name])
        close(logits[row:row + 1], alone.step([StepEntry(rid, ids, [len(ids) - 1])]), dtype, rid, bars=(1e-4, 8e-2))


@pytest.mark.parametrize("device,dtype", CASES)
def test_first_tokens_and_long_decoding(model_dirs, device, dtype):
    """A prompt of one token, then 150 tokens decoded one by one beside a neighbour that arrives later and leaves: every row
    against the whole sequence.  The window passes over decoded tokens, pages fill and are given back, the kept ones stay."""
    name = "Y"
    rng = random.Random(12)
    ids = helpers.random_prompt(rng, 151, CONFIGS[name]["vocab"])
    other = helpers.random_prompt(rng, 60, CONFIGS[name]["vocab"])
    runner = make_runner(model_dirs[name], dtype, device, 30, PAGE[name], seats=2)
    rows, other_rows = [], []
    for p in range(len(ids)):
        entries = [StepEntry("long", ids[p:p + 1], [0])]
        q = p - 40
        if 0 <= q < len(other):
            entries.append(StepEntry("other", other[q:q + 1], [0]))
        logits = runner.step(entries)
        rows.append(logits[0].float().cpu())
        if len(entries) == 2:
            other_rows.append(logits[1].float().cpu())
        if q == len(other) - 1:
            runner.finish("other")
        runner.cache.assert_invariants()
    for got, seq, what in ((rows, ids, "long decoding"), (other_rows, other, "the neighbour")):
        if dtype == "float32":
            close(torch.stack(got), plain_logits(model_dirs[name], seq), dtype, what, bars=(3e-4, 0.0))
        else:
            as_rounding_allows(model_dirs[name], [(seq, list(range(len(seq))), torch.stack(got))], what)


# ---- generation through the engine ----------------------------------------------------------------------------------
def greedy(model_dir, prompt, count):
    cfg, weights = plain.read_model_folder(model_dir)
    ids = list(prompt)
    for _ in range(count):
        ids.append(int(plain.forward_logits(cfg, weights, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["X", "Y"])
def test_greedy_generation_through_the_engine(model_dirs, name, device, graphs):
    if graphs and device == "cpu":
        pytest.skip("CUDA graphs need a CUDA device")
    rng = random.Random(1)
    prompts = [helpers.random_prompt(rng, n, CONFIGS[name]["vocab"]) for n in (5, 17, 33, 1, 40, 9)]
    cfg = EngineConfig(model=model_dirs[name], device=device, dtype="float32", max_model_len=128, max_num_seqs=3,
                       max_num_batched_tokens=24, prefill_chunk_size=8, kv_block_size=PAGE[name], kv_num_blocks=48,
                       max_output_tokens=16, scheduler_policy="decode_first", cuda_graph=graphs, overlap_steps=device != "cpu")
    engine = Engine.from_model_dir(model_dirs[name], cfg, ops=ops_for(device))
    outputs = engine.generate(prompts, max_tokens=6)
    for prompt, out in zip(prompts, outputs):
        assert out.token_ids == greedy(model_dirs[name], prompt, 6)
    assert engine.cache.used_pages == 0


@pytest.mark.gpu
def test_trace_replay_program(model_dirs, tmp_path):
    """``bin/trace_run`` as a user starts it: steps on standard input, logits in files."""
    name = "X"
    ids = requests_for(name)["r1"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[20:], "want": [len(ids) - 21]}, {"id": "b", "tokens": ids[:3], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": ids[3:5], "want": [1]}], "end": ["b"]}]
    program = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    want = plain_logits(model_dirs[name], ids)
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        done = subprocess.run([sys.executable, program, "--model", model_dirs[name], "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert done.returncode == 0, done.stderr[-2000:]
        assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
        vocab = CONFIGS[name]["vocab"]
        rows = [np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, vocab) for n in range(3)]
        got = torch.from_numpy(np.concatenate(rows))
        if dtype == "float32":
            close(got, want[[0, 19, len(ids) - 1, 4]], dtype, "trace_run float32", bars=(3e-4, 0.0))
        else:
            as_rounding_allows(model_dirs[name], [(ids, [0, 19, len(ids) - 1, 4], got)], "trace_run bfloat16")
