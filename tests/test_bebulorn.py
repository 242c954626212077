"""The Bebulorn decoder in the engine against the plain implementation (``plain_bebulorn``): each mechanism alone (layer norms
on both sides of a branch with a residual factor and rows a junction adds, softmax attention with squashed scores, a factor per
head, unit-norm values and a window, lightning attention, the gated delta rule, both feed-forwards), whole prompts against
token-by-token decoding, portions down to two tokens, mixed batches with pages and seats used again, keys just inside and
just outside a window and on page borders, states that must remember and forget, the first tokens, long decoding, other
sizes, and greedy generation through the engine's entry point.

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
import plain_bebulorn as plain
from flexengine_b200.cache import CacheManager
from flexengine_b200.config import ConfigError, EngineConfig, resolve
from flexengine_b200.engine import ModelRunner, StepEntry
from flexengine_b200.engine.runtime import Engine
from flexengine_b200.parts import CacheGroupSpec, PartSpec, RunEntry, build_part
from flexengine_b200.parts.norm import PostNormed
from flexengine_b200.weights import load_model, write_random_model
from test_fedutar import (CASES, DEVICES, F64, as64, bf16_exact, bind_by_checkpoint_names, close, drive, ops_for, randn, row_errors,
                          simple_ctx)


# ---- configurations ---------------------------------------------------------------------------------------------------
def attention(heads, kv_heads, dim, vdim, window, softcap=20.0, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                           "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap}}


def lightning(heads, dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(vocab, width, eps, mult, layers, loop=None):
    cfg = {"architecture": "Bebulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# U: a repeated span in the middle; value heads wider than key heads; a window shorter than a page; a layer without a feed-forward
# V: the repeated span is the whole stack, three passes; as many key/value heads as heads, and one; convolutions of one and two
#    taps; one expert chosen, no shared expert; a residual factor of one; odd sizes
# W: no repeated span; heads of 64 and 128 (the tensor-core kernels in bfloat16), two windows; all experts chosen in one layer
CONFIGS = {
    "U": config(211, 64, 1e-5, 0.7, [
        (lightning(3, 8, 12, [0.9, 0.99, 1.0]), dense(72)),
        (attention(4, 2, 16, 24, 9, softcap=5.0), moe(5, 2, 24, shared=40)),
        (delta(4, 2, 8, 12, 4), None),
        (lightning(2, 12, 8, [0.5, 0.97]), moe(4, 3, 16, shared=24))], loop=(1, 3, 2)),
    "V": config(301, 96, 3e-6, 1.0, [
        (delta(3, 3, 16, 8, 2), moe(6, 1, 40)),
        (attention(3, 1, 24, 8, 33), dense(112)),
        (delta(6, 2, 10, 14, 1), dense(56)),
        (lightning(2, 20, 6, [0.8, 0.995]), moe(3, 2, 24, shared=16))], loop=(0, 4, 3)),
    "W": config(400, 128, 1e-6, 0.3, [
        (attention(8, 2, 64, 64, 40, softcap=8.0), dense(192)),
        (lightning(2, 64, 128, [0.98, 0.999]), moe(4, 4, 64, shared=64)),
        (delta(4, 2, 64, 64, 3), dense(128)),
        (attention(4, 4, 128, 128, 70, softcap=50.0), moe(8, 3, 32, shared=128)),
        (delta(2, 2, 128, 128, 4), None)]),
}
PAGE = {"U": 16, "V": 8, "W": 16}
LENGTHS = {"U": [5, 33, 70, 1, 47], "V": [2, 40, 77, 23], "W": [150, 64, 90]}


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp(f"bebulorn_{name}")
        write_random_model(cfg, str(d), seed=131 + i)
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
    """bfloat16 through a whole model.  Every sublayer's output is brought to unit size by a norm of its own, and a router's
    close call changes a token's experts, so small random models turn rounding into visible differences.  The measure is what
    rounding alone does: the same sequences through the reference kernels in bfloat16 (whole prompts, on the CPU), both
    against the float64 oracle.  The device's median and ninth-decile row errors may be twice the reference kernels' and
    0.03 / 0.06 more."""
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


# ---- configuration and plan ---------------------------------------------------------------------------------------------
def test_plan_of_parts_and_cache_groups():
    _typed, plan = resolve(CONFIGS["U"])
    assert plan.architecture == "Bebulorn" and [layer.block for layer in plan.layers] == ["sandwich"] * 4
    assert [layer.mixer.kind for layer in plan.layers] == ["retention", "gated_attention", "gated_delta", "retention"]
    assert [None if layer.feed_forward is None else layer.feed_forward.kind for layer in plan.layers] == \
        ["gated_mlp", "routed_experts", None, "routed_experts"]
    # the span runs twice: a slot per pass; before the second pass, and only there, the junction
    assert [e.layer for e in plan.run] == [0, 1, 2, 1, 2, 3]
    assert [e.before for e in plan.run] == [-1, -1, -1, 0, -1, -1] and [j.kind for j in plan.junctions] == ["readd"]
    groups = {g.name: g for g in plan.cache_groups}
    assert groups["attention_2x32_9"].slots == 2 and groups["attention_2x32_9"].kind == "window" and groups["attention_2x32_9"].window == 9
    # 4 heads of 8 x 12, then three rows of 2 x (2 x 8) + 48 channels
    assert groups["delta_state_624"].slots == 2 and groups["delta_state_624"].state_shape == (4 * 8 * 12 + 3 * (32 + 48),)
    assert groups["lightning_state_288"].slots == 1 and groups["lightning_state_192"].slots == 1
    assert plan.layers[0].block_params["residual_scale"] == 0.7
    _typed, plan = resolve(CONFIGS["V"])
    assert [e.layer for e in plan.run] == [0, 1, 2, 3] * 3 and [e.before for e in plan.run] == [-1] * 4 + [0, -1, -1, -1] * 2
    _typed, plan = resolve(CONFIGS["W"])
    assert not plan.junctions and sorted(g.window for g in plan.cache_groups if g.kind == "window") == [40, 70]
    names = {s.name for b in plan.bindings for s in b.sources}
    assert {"final.norm.b", "l0.mix.temp", "l2.mix.A_log", "l2.mix.q.conv", "l1.mlp.shared.up", "l3.mlp.e7.down", "head", "l1.mix.norm"} <= names
    assert "l4.norm2" not in names and "l1.mlp.e0.gate" not in names


def test_configuration_errors_are_named():
    def broken(change):
        cfg = json.loads(json.dumps(CONFIGS["U"]))
        change(cfg)
        return cfg

    cases = [
        (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
        (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
        (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
        (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
        (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
        (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
        (lambda c: c["layers"][2]["mixer"].update(conv=0), "conv"),
        (lambda c: c["layers"][2]["mixer"].pop("vdim"), "vdim"),
        (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "experts"),
        (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "shared.ff"),
        (lambda c: c["layers"][1]["mlp"].update(shared={}), "shared.ff"),
        (lambda c: c["layers"][0].update(type="mystery"), "mystery"),
        (lambda c: c["layers"][0]["mlp"].update(kind="mystery"), "mystery"),
        (lambda c: c["loop"].update(stop=7), "loop"),
        (lambda c: c["norm"].update(eps=0.0), "eps"),
    ]
    for change, word in cases:
        with pytest.raises(ConfigError, match=word):
            resolve(broken(change))


def test_tensors_of_absent_parts(tmp_path):
    """The norms around a feed-forward that a layer does not have may be there and are ignored; any other stranger is refused by
    name, as is a missing bias."""
    from flexengine_b200.weights.safetensors_io import write_safetensors
    write_random_model(CONFIGS["U"], str(tmp_path), seed=1)
    _c, weights = plain.read_model_folder(str(tmp_path))
    tensors = {k: v.to(torch.bfloat16) for k, v in weights.items()}

    def write():
        write_safetensors(str(tmp_path / "model.safetensors"), [(n, tuple(t.shape), t.dtype) for n, t in tensors.items()],
                          lambda n: tensors[n])
    for name in ("l2.norm2", "l2.norm2.b", "l2.norm2b", "l2.norm2b.b"):
        tensors[name] = torch.ones(64, dtype=torch.bfloat16)
    write()
    load_model(str(tmp_path), "float32", "cpu")
    tensors["l2.mlp.up"] = torch.ones(8, 64, dtype=torch.bfloat16)
    write()
    with pytest.raises(Exception, match="l2.mlp.up"):
        load_model(str(tmp_path), "float32", "cpu")
    del tensors["l2.mlp.up"], tensors["l1.norm1b.b"]
    write()
    with pytest.raises(Exception, match="l1.norm1b.b"):
        load_model(str(tmp_path), "float32", "cpu")


# ---- each mechanism alone -----------------------------------------------------------------------------------------
def run_mixer(mixer):
    entry = RunEntry(layer=0, cache_group=0, cache_slot=0, write_cache=True)
    return lambda ctx, rows: mixer.forward(ctx, rows, entry)


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("width", [40, 97, 192, 2052, 1030])
def test_layer_norms_around_a_branch(device, dtype, width):
    """x <- x + m norm_b(y) (+ rows a junction adds), then the next norm of the sum, in one kernel: all rows in place, chosen rows
    without writing, the branch in float32 and in the compute dtype; a mean far from zero, so that a variance taken the wrong
    way shows."""
    dt = getattr(torch, dtype)
    T, D, eps, m = 11, width, 1e-5, 0.37
    x = torch.randn(T, D, generator=torch.Generator().manual_seed(1)) + 30.0
    y, plus = bf16_exact(randn(T, D, seed=2, scale=3.0) + 16.0), torch.randn(T, D, generator=torch.Generator().manual_seed(3))
    vectors = [randn(D, seed=4) + 1.0, randn(D, seed=5), randn(D, seed=6) + 1.0, randn(D, seed=7)]
    post, after = (build_part("norm", PartSpec("layernorm", {"hidden_size": D, "eps": e})) for e in (3e-4, eps))
    post.bind({"weight": vectors[0].to(device), "bias": vectors[1].to(device)})
    after.bind({"weight": vectors[2].to(device), "bias": vectors[3].to(device)})
    ctx = simple_ctx(device, dt)
    w = [v.to(F64) for v in vectors]
    branch = m * plain.layer_norm(y.to(F64), 3e-4, w[0], w[1])
    for pending, into in ((lambda t: post.after(t, scale=m), branch),
                          (lambda t: PostNormed(t, post.weight, post.eps, None, norm_bias=post.bias, scale=m, plus=plus.to(device)), branch + plus.to(F64)),
                          (lambda t: t, y.to(F64)), (lambda t: PostNormed(None, None, 0.0, plus=plus.to(device)), plus.to(F64)),
                          (lambda t: None, torch.zeros(T, D, dtype=F64))):
        for branch_dtype in {dt, torch.float32}:
            residual = x.to(device).clone()
            rows = torch.tensor([7, 0, 10], dtype=torch.int32, device=device)
            want_stream = x.to(F64) + into
            want = plain.layer_norm(want_stream, eps, w[2], w[3])
            some = after.forward(ctx, residual, pending(y.to(device=device, dtype=branch_dtype)), rows=rows)
            assert torch.equal(residual, x.to(device))
            close(some.float().cpu(), want[rows.cpu().long()], dtype, "chosen rows", bars=(2e-5, 2e-2))
            got = after.forward(ctx, residual, pending(y.to(device=device, dtype=branch_dtype)))
            assert got.dtype == dt
            close(got.float().cpu(), want, dtype, "all rows", bars=(2e-5, 2e-2))
            assert (residual.cpu().double() - want_stream).abs().max() < 2e-5 * float(want_stream.abs().max())


def attention_weights(D, m, seed):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": randn(H * d, D, seed=seed, scale=D ** -0.5), "k": randn(G * d, D, seed=seed + 1, scale=D ** -0.5),
            "v": randn(G * dv, D, seed=seed + 2, scale=D ** -0.5), "o": randn(D, H * dv, seed=seed + 3, scale=(H * dv) ** -0.5),
            "temp": randn(H, seed=seed + 4) * 0.5 + 1.0}


ATTENTION_NAMES = {"qkvg.weight": ["q", "k", "v"], "o.weight": ["o"], "head_scales": ["temp"]}


def attention_part(D, m, weights, device, dt, eps=1e-5):
    window = (m.get("mask") or {"size": 0})["size"]
    mixer = build_part("mixer", PartSpec("gated_attention", {
        "hidden_size": D, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"], "eps": eps,
        "mask": "window" if window else "full", "mask_size": window, "value_norm": True, "head_scales": True, "softcap": m["softcap"],
        "gate": "none"}))
    bind_by_checkpoint_names(mixer, weights, ATTENTION_NAMES, device, dt)
    need = mixer.cache_need()
    return mixer, [CacheGroupSpec("kv", need["kind"], slots=1, kv_heads=need["kv_heads"], head_dim=need["head_dim"], window=need["window"])]


# heads, kv_heads, dim, vdim, window: values wider and narrower than keys, one head, groups of one, three and four, windows of one
# key, of a page, beyond the sequence; head sizes that are no multiples of 16, and 64 and 128 (tensor-core kernels in bfloat16)
ATTENTION_SHAPES = [(4, 2, 16, 24, 9), (2, 1, 32, 16, 4), (3, 3, 16, 16, 1), (8, 2, 64, 64, 20), (1, 1, 40, 8, 100), (6, 3, 64, 128, 13),
                    (6, 2, 128, 128, 17), (12, 4, 24, 64, 3), (5, 5, 48, 48, 32)]


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_alone(device, dtype, shape):
    """Scores spread several times as wide as the cap, one head's factor negative: a cap that is left out, applied before the
    factor or after the mask, or a factor of another head shows."""
    dt = getattr(torch, dtype)
    D, T = 48, 41
    m = attention(*shape, softcap=1.5, scale=2.0 * shape[2] ** -0.5)["mixer"]
    weights = attention_weights(D, m, seed=10)
    weights["temp"][-1] = -1.25
    mixer, specs = attention_part(D, m, weights, device, dt)
    h = randn(T, D, seed=11)
    want = plain.softmax_attention(h.to(F64), as64(weights), "", m, 1e-5)
    for cuts in ([T], [1] * T, [7, 2, 19, 2, 1, 10], [2, 37, 2], [1, 1, 2, 1, 36]):
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"attention {shape} cut {cuts[:5]}")


def peaked(D, m, seed, gain):
    """Weights under which queries and keys are channels 0..15 of the input, times ``gain``, the same for every head."""
    weights = attention_weights(D, m, seed)
    weights["temp"][:] = 1.0
    for name in ("q", "k"):
        weights[name][:] = 0.0
        for head in range(weights[name].shape[0] // m["dim"]):
            weights[name][head * m["dim"]:head * m["dim"] + 16, :16] = torch.eye(16) * gain
    return weights


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("back", [15, 16, 31, 32, 129, 130, 639])
@pytest.mark.parametrize("dim", [16, 64])
def test_a_key_just_inside_and_just_outside_the_window(device, dtype, decoded, back, dim):
    """The key ``back`` positions before the last query stands out so much that it decides the output where it is seen.  The window
    is ``back`` (just outside) or ``back`` + 1 (just inside): on both sides of a page border, far back, in prompts and decoded."""
    dt = getattr(torch, dtype)
    D, T = 32, 655
    h = randn(T, D, seed=31)
    direction = randn(16, seed=32)
    direction = direction / direction.norm() * 4.0
    h[:, :16] *= 0.2
    h[T - 1 - back, :16] = 2.0 * direction
    h[-1, :16] = direction
    last = {}
    for window in (back, back + 1):
        m = attention(4, 2, dim, 16, window, softcap=30.0, scale=1.0)["mixer"]
        weights = peaked(D, m, 30, 1.0)
        mixer, specs = attention_part(D, m, weights, device, dt)
        want = plain.softmax_attention(h.to(F64), as64(weights), "", m, 1e-5)
        last[window] = want[-1]
        cuts = [300, 354, 1] if decoded else [2, 330, 321, 2]
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, f"window {window}")
    # what the oracle says of the two windows differs by far more than the bars
    assert (last[back] - last[back + 1]).abs().max() > 0.25 * last[back + 1].abs().max()


def state_spec(mixer):
    need = mixer.cache_need()
    return [CacheGroupSpec("state", "state", slots=1, state_shape=need["state_shape"], state_dtype=need["state_dtype"])]


def lightning_weights(D, m, seed):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    return {"q": randn(H * d, D, seed=seed, scale=D ** -0.5), "k": randn(H * d, D, seed=seed + 1, scale=D ** -0.5),
            "v": randn(H * dv, D, seed=seed + 2, scale=D ** -0.5), "g": randn(H * dv, D, seed=seed + 3, scale=D ** -0.5),
            "o": randn(D, H * dv, seed=seed + 4, scale=(H * dv) ** -0.5), "norm": 1.0 + randn(H * dv, seed=seed + 5, scale=0.3)}


def lightning_part(D, m, weights, device, dt, eps=1e-5):
    mixer = build_part("mixer", PartSpec("retention", {
        "hidden_size": D, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "decay": m["decay"], "eps": eps, "activation": "silu",
        "key_scale": 1.0, "norm": "all_heads", "gate": "sigmoid"}))
    bind_by_checkpoint_names(mixer, weights, {"qkvg.weight": ["q", "k", "v", "g"], "o.weight": ["o"], "norm.weight": ["norm"]}, device, dt)
    return mixer, state_spec(mixer)


# heads, dim, vdim, decays: values narrower and wider than keys, one head, decays of exactly one and zero, sizes that are no
# multiples of four or eight, a head of 128, rows beyond 512 columns
@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(3, 16, 8, [0.9, 0.95, 0.99]), (2, 24, 40, [0.5, 0.999]), (1, 12, 12, [0.97]), (5, 6, 9, [0.9, 0.92, 0.0, 0.96, 1.0]),
                                   (2, 64, 64, [0.97, 0.999]), (1, 128, 72, [0.995]), (6, 64, 100, [0.98] * 6), (3, 36, 130, [0.9, 0.99, 0.999])])
def test_lightning_alone(device, dtype, shape):
    dt = getattr(torch, dtype)
    D, T = 48, 45
    m = lightning(*shape)["mixer"]
    weights = lightning_weights(D, m, seed=50)
    mixer, specs = lightning_part(D, m, weights, device, dt)
    h = randn(T, D, seed=51)
    want = plain.lightning(h.to(F64), as64(weights), "", m, 1e-5)
    for cuts in ([T], [1] * T, [7, 2, 19, 2, 1, 14], [2, 41, 2], [1, 1, 2, 1, 40]):
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"lightning {shape} cut {cuts[:5]}")


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("cuts", [[700], [2, 330, 366, 2], [300, 380] + [1] * 20])
def test_lightning_remembers_over_hundreds_of_tokens(device, dtype, cuts):
    """One token writes far more than the others; decays near 1 still know it hundreds of tokens later, a fast one does not."""
    dt = getattr(torch, dtype)
    D, T = 32, 700
    m = lightning(3, 16, 16, [1.0, 0.998, 0.9])["mixer"]
    weights = lightning_weights(D, m, seed=60)
    weights["k"][:, 0] = 2.0
    mixer, specs = lightning_part(D, m, weights, device, dt)
    h = randn(T, D, seed=61, scale=0.2)
    h[:, 0] = 0.0
    h[3, 0] = 8.0
    want = plain.lightning(h.to(F64), as64(weights), "", m, 1e-5)
    silent = h.clone()
    silent[3, 0] = 0.0
    other = plain.lightning(silent.to(F64), as64(weights), "", m, 1e-5)
    assert (other[-1] - want[-1]).abs().max() > 0.3 * want[-1].abs().max()
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, "far memory", bars=(1e-4, 0.12))


def delta_weights(D, m, seed):
    H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    w = {"q": randn(G * d, D, seed=seed, scale=D ** -0.5), "k": randn(G * d, D, seed=seed + 1, scale=D ** -0.5),
         "v": randn(H * dv, D, seed=seed + 2, scale=D ** -0.5), "g": randn(H * dv, D, seed=seed + 3, scale=D ** -0.5),
         "b": randn(H, D, seed=seed + 4, scale=2.0 * D ** -0.5), "a": randn(H, D, seed=seed + 5, scale=D ** -0.5),
         "o": randn(D, H * dv, seed=seed + 6, scale=(H * dv) ** -0.5), "A_log": randn(H, seed=seed + 7), "dt_bias": randn(H, seed=seed + 8) - 1.0,
         "norm": 1.0 + randn(dv, seed=seed + 9, scale=0.3)}
    for i, (name, rows) in enumerate((("q", G * d), ("k", G * d), ("v", H * dv))):
        w[name + ".conv"] = randn(rows, taps, seed=seed + 10 + i, scale=taps ** -0.5)
    return w


DELTA_NAMES = {"qkvgba.weight": ["q", "k", "v", "g", "b", "a"], "conv.weight": ["q.conv", "k.conv", "v.conv"], "A_log": ["A_log"],
               "dt_bias": ["dt_bias"], "norm.weight": ["norm"], "o.weight": ["o"]}


def delta_part(D, m, weights, device, dt, eps=1e-5):
    mixer = build_part("mixer", PartSpec("gated_delta", {"hidden_size": D, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"],
                                                         "vdim": m["vdim"], "conv": m["conv"], "eps": eps}))
    bind_by_checkpoint_names(mixer, weights, DELTA_NAMES, device, dt)
    return mixer, state_spec(mixer)


# heads, kv_heads, dim, vdim, taps: as many query/key heads as value heads, one for all, groups of two and three; one tap to six;
# values narrower and wider than keys, sizes that are no multiples of four, of a warp and of the threads' runs, up to 256 x 200
DELTA_SHAPES = [(4, 2, 8, 12, 4), (3, 3, 16, 8, 2), (6, 2, 10, 14, 1), (1, 1, 7, 5, 3), (4, 1, 32, 24, 4), (2, 2, 64, 64, 6), (4, 2, 128, 128, 3),
                (9, 3, 36, 40, 3), (2, 1, 256, 200, 4), (2, 1, 33, 300, 2)]


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_alone(device, dtype, shape):
    """Whole, token by token and in portions down to two tokens: the state and the convolutions' last rows are carried by the
    seat, in float32."""
    dt = getattr(torch, dtype)
    D, T = 48, 45
    m = delta(*shape)["mixer"]
    weights = delta_weights(D, m, seed=70)
    mixer, specs = delta_part(D, m, weights, device, dt)
    h = randn(T, D, seed=71)
    want = plain.gated_delta(h.to(F64), as64(weights), "", m, 1e-5)
    for cuts in ([T], [1] * T, [7, 2, 19, 2, 1, 14], [2, 41, 2], [1, 1, 2, 1, 40], [9, 3, 8, 4, 5, 16]):
        close(drive(run_mixer(mixer), specs, h, cuts, device, dt), want, dtype, f"delta {shape} cut {cuts[:5]}")


def slow_delta(D, m, seed):
    """Decays so near one that the state remembers for thousands of tokens."""
    weights = delta_weights(D, m, seed)
    weights["A_log"][:] = -6.0
    weights["a"][:] *= 0.1
    return weights


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("cuts", [[700], [2, 330, 366, 2], [300, 380] + [1] * 20])
def test_delta_remembers_over_hundreds_of_tokens(device, dtype, cuts):
    """Channels 0..7 of the input are the keys and queries (no token between reads or writes the direction the third token writes
    and the last one asks for): what was written comes back hundreds of tokens later.  A state that is lost, decayed twice or
    mixed up between seats shows at once."""
    dt = getattr(torch, dtype)
    D, T = 32, 700
    m = delta(2, 1, 8, 16, 1)["mixer"]
    weights = slow_delta(D, m, seed=80)
    for name in ("q", "k"):
        weights[name][:] = 0.0
        weights[name][:, :8] = torch.eye(8)
        weights[name + ".conv"][:] = 1.0
    weights["b"][:] = 0.0
    h = randn(T, D, seed=81)
    h[:, :8] = h[:, :8].abs() + 0.5
    h[:, 0] = 0.0                                          # silu(0) = 0: the direction is free
    h[3, :8] = 0.0
    h[3, 0] = 6.0
    h[-1, :8] = 0.0
    h[-1, 0] = 6.0
    weights["v"][:, 8:] *= 2.0
    mixer, specs = delta_part(D, m, weights, device, dt)
    want = plain.gated_delta(h.to(F64), as64(weights), "", m, 1e-5)
    other = h.clone()
    other[3, 8:] = -other[3, 8:]
    told = plain.gated_delta(other.to(F64), as64(weights), "", m, 1e-5)
    assert (told[-1] - want[-1]).abs().max() > 0.3 * want[-1].abs().max()
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=64), want, dtype, "far memory")


@pytest.mark.parametrize("device,dtype", CASES)
def test_recurrences_over_a_portion_of_thousands_of_tokens(device, dtype):
    dt = getattr(torch, dtype)
    D, T = 16, 2300
    cuts = [2200, 98, 1, 1]
    m = lightning(2, 16, 24, [0.999, 0.97])["mixer"]
    weights = lightning_weights(D, m, seed=90)
    mixer, specs = lightning_part(D, m, weights, device, dt)
    h = randn(T, D, seed=91)
    want = plain.lightning(h.to(F64), as64(weights), "", m, 1e-5)
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=160), want, dtype, "lightning, a long portion")
    m = delta(3, 1, 16, 20, 4)["mixer"]
    weights = slow_delta(D, m, seed=92)
    mixer, specs = delta_part(D, m, weights, device, dt)
    want = plain.gated_delta(h.to(F64), as64(weights), "", m, 1e-5)
    close(drive(run_mixer(mixer), specs, h, cuts, device, dt, page=16, pages=160), want, dtype, "delta, a long portion", bars=(2e-4, 6e-2))


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("sizes", [(48, 72), (40, 100), (64, 256)])
def test_dense_feed_forward_alone(device, dtype, sizes):
    dt = getattr(torch, dtype)
    D, F = sizes
    weights = {"gate": randn(F, D, seed=1, scale=D ** -0.5), "up": randn(F, D, seed=2, scale=D ** -0.5), "down": randn(D, F, seed=3, scale=F ** -0.5)}
    part = build_part("feed_forward", PartSpec("gated_mlp", {"hidden_size": D, "intermediate_size": F, "activation": "relu"}))
    bind_by_checkpoint_names(part, weights, {"gate_up.weight": ["gate", "up"], "down.weight": ["down"]}, device, dt)
    for T in (1, 5, 33):
        h = randn(T, D, seed=4 + T)
        got = part.forward(simple_ctx(device, dt), h.to(device=device, dtype=dt))
        close(got.float().cpu(), plain.dense_feed_forward(h.to(F64), as64(weights), ""), dtype, f"dense {sizes} rows {T}")


def routed_weights(D, mlp, seed):
    E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
    w = {"router": randn(E, D, seed=seed, scale=2.0 * D ** -0.5)}
    for e in range(E):
        w[f"e{e}.up"] = randn(F, D, seed=seed + 10 + e, scale=2.0 * D ** -0.5)
        w[f"e{e}.down"] = randn(D, F, seed=seed + 100 + e, scale=F ** -0.5)
    if mlp.get("shared"):
        S = mlp["shared"]["ff"]
        w["shared.up"], w["shared.down"] = randn(S, D, seed=seed + 200, scale=2.0 * D ** -0.5), randn(D, S, seed=seed + 201, scale=S ** -0.5)
    return w


def routed_part(D, mlp, weights, device, dt):
    E, shared = mlp["router"]["experts"], (mlp.get("shared") or {"ff": 0})["ff"]
    part = build_part("feed_forward", PartSpec("routed_experts", {
        "hidden_size": D, "experts": E, "top": mlp["router"]["top"], "expert_size": mlp["expert"]["ff"], "shared_size": shared,
        "router": "softmax_chosen", "activation": "gelu"}))
    names = {"router.weight": ["router"], "experts.up.weight": [f"e{e}.up" for e in range(E)], "experts.down.weight": [f"e{e}.down" for e in range(E)]}
    if shared:
        names.update({"shared.up.weight": ["shared.up"], "shared.down.weight": ["shared.down"]})
    bind_by_checkpoint_names(part, weights, names, device, dt)
    return part


@pytest.mark.parametrize("device,dtype", CASES)
@pytest.mark.parametrize("shape", [(5, 2, 24, 40), (6, 1, 40, 0), (4, 4, 64, 8), (8, 3, 32, 128), (1, 1, 16, 16), (12, 2, 64, 64), (40, 6, 8, 24)])
def test_routed_feed_forward_alone(device, dtype, shape):
    """The chosen experts and their weights are compared as well as the sum.  Rows whose choice is a close call are left out in
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
        got_chosen, got_share = ctx.ops.route_top(logits, part.top, 1.0, over_chosen=True)
        sure = gaps[0] > (1e-5 if dtype == "float32" else 2e-2) if gaps else torch.ones(T, dtype=torch.bool)
        if not bool(sure.any()):
            continue
        for row in sure.nonzero().flatten().tolist():
            mine = dict(zip(got_chosen[row].tolist(), got_share[row].tolist()))
            theirs = dict(zip(chosen[row].tolist(), share[row].tolist()))
            assert mine.keys() == theirs.keys() and all(abs(mine[e] - theirs[e]) < (1e-5 if dtype == "float32" else 2e-2) for e in mine)
        got = part.forward(ctx, h.to(device=device, dtype=dt))
        close(got.float().cpu()[sure], want[sure], dtype, f"routed {shape} rows {T}")


# ---- kernels alone (GPU) ---------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(4, 2, 64, 128, 4), (3, 3, 24, 40, 3), (2, 1, 130, 72, 2), (6, 2, 128, 200, 4), (2, 2, 17, 9, 5)])
def test_delta_kernels_against_the_references(heads, kv_heads, dim, vdim, taps):
    """One step of portions of 1, 2, 3, 4, 5, 8, 9, 63 and 130 tokens (every way a last block of four can be filled): seats that
    hold a state, fresh ones and a request without a seat; outputs, states and histories afterwards.  Then the decode kernel on
    one token a request over the same seats."""
    from flexengine_b200 import ops
    dev = "cuda:0"
    lengths, seats = [1, 2, 3, 4, 5, 8, 9, 63, 130], [2, 0, -1, 5, 1, 4, 8, 3, 6]
    T, n = sum(lengths), heads * dim * vdim
    C = 2 * kv_heads * dim + heads * vdim
    at = -(-n // 4) * 4
    gen = torch.Generator().manual_seed(7)
    projected = torch.randn(T, C + heads * vdim + 2 * heads + 3, generator=gen)
    conv = torch.randn(taps, C, generator=gen) * taps ** -0.5
    state = torch.randn(9, at + (taps - 1) * C + 5, generator=gen) * 0.5
    a_log, dt_bias = torch.randn(heads, generator=gen), torch.randn(heads, generator=gen)
    weight = torch.randn(vdim, generator=gen) + 1.0
    cu = torch.tensor([0] + list(np.cumsum(lengths)), dtype=torch.int32)
    slots = torch.tensor(seats, dtype=torch.int32)
    sizes = (heads, kv_heads, dim, vdim)
    token_request = torch.repeat_interleave(torch.arange(len(lengths), dtype=torch.int32), torch.tensor(lengths))
    want_state = state.clone()
    qkv, gates = kernel_refs.delta_prepare(projected, conv, want_state, at, slots, cu, token_request, a_log, dt_bias, 1e-6, dim ** -0.5, *sizes)
    want = kernel_refs.delta_scan(qkv, gates, want_state, slots, cu, *sizes)
    d = {k: v.to(dev) for k, v in dict(projected=projected, conv=conv, state=state, slots=slots, cu=cu, tr=token_request, a_log=a_log,
                                       dt_bias=dt_bias, weight=weight).items()}
    got_qkv, numbers = ops.delta_prepare(d["projected"], d["conv"], d["state"], at, d["slots"], d["cu"], d["tr"], d["a_log"], d["dt_bias"], 1e-6,
                                         dim ** -0.5, *sizes, max_q_len=max(lengths))
    got = ops.delta_scan(got_qkv, numbers, d["state"], d["slots"], d["cu"], *sizes, max_q_len=max(lengths))
    assert (got_qkv.cpu() - qkv).abs().max() <= 1e-5 * max(1.0, float(qkv.abs().max()))
    assert (got.cpu() - want).abs().max() <= 3e-5 * want.abs().max()
    assert (d["state"].cpu() - want_state).abs().max() <= 3e-5 * want_state.abs().max()
    R = len(lengths)
    rows = torch.randn(R, projected.shape[1], generator=gen)
    want = kernel_refs.delta_decode(rows, conv, want_state, at, slots, a_log, dt_bias, weight, 1e-5, 1e-6, dim ** -0.5, *sizes, torch.float32)
    got = ops.delta_decode(rows.to(dev), d["conv"], d["state"], at, d["slots"], d["a_log"], d["dt_bias"], d["weight"], 1e-5, 1e-6, dim ** -0.5,
                           *sizes, torch.float32)
    assert (got.cpu() - want).abs().max() <= 1e-4 * want.abs().max()
    assert (d["state"].cpu() - want_state).abs().max() <= 3e-5 * want_state.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(4, 2, 32, 8), (8, 2, 64, 16), (6, 6, 16, 16), (16, 1, 128, 16), (3, 1, 48, 4), (12, 3, 64, 16), (2, 1, 256, 16)])
@pytest.mark.parametrize("lengths", [[(0, 70)], [(299, 1), (37, 1), (1, 1)], [(40, 33), (130, 1), (0, 2), (15, 300)], [(1000, 1)] * 3, [(0, 1100)]])
def test_squashed_scores_in_every_attention_kernel(dtype, shape, lengths):
    """Decode steps (clustered and split), portions, mixed steps: the CUDA kernels against the reference, with factors per head far
    enough apart (one negative) that a head reading another's shows, a cap well inside the scores' range, none, and a window."""
    from flexengine_b200 import ops
    nq, nkv, d, page = shape
    dt = getattr(torch, dtype)
    dev = "cuda:0"
    gen = torch.Generator().manual_seed(5)
    R = len(lengths)
    starts, counts = [s for s, _ in lengths], [n for _, n in lengths]
    T = sum(counts)
    most = max(s + n for s, n in lengths)
    per = -(-most // page)
    pages = R * per + 3
    table = torch.randperm(pages, generator=gen)[:R * per].view(R, per).to(torch.int32).to(dev)
    kc = (torch.randn(pages, nkv, page, d, generator=gen) * 0.7).to(device=dev, dtype=dt)
    vc = torch.randn(pages, nkv, page, d, generator=gen).to(device=dev, dtype=dt)
    q = torch.randn(T, nq * d + 8, generator=gen).to(device=dev, dtype=dt)
    cu = torch.tensor([0] + list(np.cumsum(counts)), dtype=torch.int32, device=dev)
    ctx = types.SimpleNamespace(cu_q=cu, q_start=torch.tensor(starts, dtype=torch.int32, device=dev),
                                token_request=torch.repeat_interleave(torch.arange(R, dtype=torch.int32), torch.tensor(counts)).to(dev),
                                max_q_len=max(counts), max_ctx_len=most, host_lengths=counts, host_starts=starts)
    scales = (0.4 + torch.arange(nq, dtype=torch.float32) * 0.35).to(dev)
    scales[-1] = -1.5
    scale = 1.5 * d ** -0.5
    for window, score in ((0, dict(softcap=2.0, head_scales=scales)), (50, dict(softcap=25.0, head_scales=scales)), (0, dict(head_scales=scales)),
                          (0, dict(softcap=3.0))):
        want = kernel_refs.paged_attention(q, kc, vc, table, ctx, nq, nkv, d, page, scale, window, **score)
        runs = {"as the step would choose": lambda: ops.paged_attention(q, kc, vc, table, ctx, nq, nkv, d, page, scale, window, **score)}
        if dtype == "bfloat16":
            common = (q, q.stride(0), kc, vc, table, ctx.cu_q, ctx.q_start)
            if max(counts) == 1 and nq // nkv <= 16:
                for splits in (1, 3, 8):
                    runs[f"cluster of {splits}"] = lambda splits=splits: ops.paged_decode_cluster(
                        *common, R, nq, nkv, d, page, scale, window, splits, **score)
                for splits in (1, 5, 40):
                    runs[f"{splits} splits and a merge"] = lambda splits=splits: ops.paged_decode_mma(
                        *common, R, nq, nkv, d, page, scale, window, splits, **score)
            runs["mma.sync portions"] = lambda: ops.paged_prefill_mma(*common, T, R, max(counts), nq, nkv, d, page, scale, window, **score)
            if d in (64, 128):
                for splits in (1, 4):
                    runs[f"tcgen05 portions, keys split {splits} ways"] = lambda splits=splits: ops.paged_prefill_tcgen05(
                        *common, T, R, max(counts), nq, nkv, d, page, scale, window, splits=splits, **score)
        for what, run in runs.items():
            err = (run().float() - want.float()).abs().max()
            assert float(err) <= (2e-4 if dtype == "float32" else 3e-2) * max(1.0, float(want.float().abs().max())), f"{what} {score}: error {float(err):.3e}"
    ops.check_status(dev)


@pytest.mark.gpu
@pytest.mark.parametrize("rows,K,N", [(1, 128, 72), (8, 256, 520), (1100, 1024, 520), (2048, 1536, 1000), (37, 96, 40)])
def test_relu_gate_and_exact_gelu_in_the_products_epilogues(rows, K, N):
    """The weight-streaming kernel (a handful of rows), the tcgen05 kernel (a prompt's worth) and the product with the
    activation kernel behind it give the same rows."""
    from flexengine_b200 import ops
    x = randn(rows, K, seed=1).to(device="cuda:0", dtype=torch.bfloat16)
    w = randn(2 * N, K, seed=2, scale=2.0 * K ** -0.5).to(device="cuda:0", dtype=torch.bfloat16)
    for got, want in ((ops.linear_gated(x, w, N, "relu"), kernel_refs.linear_gated(x, w, N, "relu")),
                      (ops.linear_activated(x, w, "gelu"), kernel_refs.linear_activated(x, w, "gelu"))):
        assert (got.float() - want.float()).abs().max() <= 2e-2 * max(1.0, float(want.float().abs().max()))


@pytest.mark.gpu
@pytest.mark.parametrize("T,D,F,experts,top", [(700, 1024, 1024, 4, 2), (1500, 1024, 1536, 3, 1), (300, 256, 128, 6, 3), (6, 128, 64, 8, 2)])
def test_gelu_experts_on_the_grouped_products(T, D, F, experts, top):
    from flexengine_b200 import ops
    gen = torch.Generator().manual_seed(3)
    h = randn(T, D, seed=4).to(device="cuda:0", dtype=torch.bfloat16)
    up = randn(experts, F, D, seed=5, scale=2.0 * D ** -0.5).to(device="cuda:0", dtype=torch.bfloat16)
    down = randn(experts, D, F, seed=6, scale=F ** -0.5).to(device="cuda:0", dtype=torch.bfloat16)
    chosen = torch.stack([torch.randperm(experts, generator=gen)[:top] for _ in range(T)]).to(torch.int32).cuda()
    weights = torch.rand(T, top, generator=gen).cuda()
    got = ops.routed_experts(h, chosen, weights, up, down, activation="gelu")
    want = kernel_refs.routed_experts(h, chosen, weights, up, down, activation="gelu")
    assert (got.float() - want.float()).abs().max() <= 3e-2 * max(1.0, float(want.float().abs().max()))
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
@pytest.mark.parametrize("name", ["U", "V", "W"])
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


def test_the_stream_after_every_run_of_a_layer_against_plain(model_dirs):
    """The residual stream after every run of a layer, with what is pending put in: the plain implementation's."""
    for name in ("U", "V", "W"):
        ids = requests_for(name)["r1"]
        cfg, weights = plain.read_model_folder(model_dirs[name])
        after = []
        plain.forward_logits(cfg, weights, ids, after)
        _cfg, plan, model = load_model(model_dirs[name], "float32", "cpu")
        cache = CacheManager(plan.cache_groups, 16, 16, 1, torch.float32, "cpu")
        runner = ModelRunner(model, cache, ops=kernel_refs)
        cache.reserve("a", len(ids))
        ctx = runner.build_context([StepEntry("a", ids, [])])
        residual = model.embedding.forward(ctx)
        origin, pending = residual.clone(), None
        assert len(plan.run) == len(after)
        for at, entry in enumerate(plan.run):
            if entry.before >= 0:
                residual, pending = model.junctions[entry.before].forward(ctx, residual, pending, origin)
            pending = model.blocks[entry.layer].forward(ctx, residual, pending, entry)
            settled = residual.double() + pending.scale * plain.layer_norm(pending.y.double(), pending.eps, pending.weight.double(), pending.norm_bias.double())
            assert (settled - after[at]).abs().max() < 2e-5 * float(after[at].abs().max()), f"{name}: run {at}"


STACKS = {
    "one attention layer without a feed-forward": config(50, 32, 1e-5, 1.0, [(attention(2, 1, 16, 16, 5), None)]),
    "one delta layer that is the whole span": config(97, 48, 1e-5, 0.5, [(delta(2, 2, 8, 8, 3), dense(32))], loop=(0, 1, 4)),
    "lightning only, a span that runs once": config(64, 40, 1e-6, 2.0, [
        (lightning(2, 8, 16, [0.9, 0.99]), None), (lightning(4, 4, 4, [0.5, 0.8, 0.9, 1.0]), moe(3, 2, 16, shared=8))], loop=(0, 2, 1)),
    "a span at the end": config(83, 56, 1e-6, 0.25, [
        (delta(4, 1, 12, 8, 2), moe(2, 1, 8)), (attention(7, 7, 8, 8, 17, softcap=2.0), dense(24)), (lightning(1, 8, 24, [0.95]), dense(40))], loop=(1, 3, 3)),
    "no window, no cap": config(61, 32, 1e-5, 0.9, [
        ({"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 8, "scale": 0.4}}, dense(24))]),
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
    plain_cfg = json.loads(json.dumps(cfg))
    for layer in plain_cfg["layers"]:                        # the plain implementation wants every key: a cap and a window that do nothing
        if layer["type"] == "attention":
            layer["mixer"].setdefault("mask", {"size": 0})
            layer["mixer"].setdefault("softcap", 1e9)
    want = plain.forward_logits(plain_cfg, plain.read_model_folder(str(tmp_path))[1], ids)
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
    name = "W"
    requests = requests_for(name, seed=9)
    together = make_runner(model_dirs[name], dtype, device, 32, PAGE[name])
    logits = together.step([StepEntry(rid, ids, [len(ids) - 1]) for rid, ids in requests.items()])
    for row, (rid, ids) in enumerate(requests.items()):
        alone = make_runner(model_dirs[name], dtype, device, 16, PAGE[name])
        close(logits[row:row + 1], alone.step([StepEntry(rid, ids, [len(ids) - 1])]), dtype, rid, bars=(1e-4, 8e-2))


@pytest.mark.parametrize("device,dtype", CASES)
def test_first_tokens_and_long_decoding(model_dirs, device, dtype):
    """A prompt of one token, then 150 tokens decoded one by one beside a neighbour that arrives later and leaves: every row
    against the whole sequence.  The window passes over decoded tokens, pages fill and are given back."""
    name = "U"
    rng = random.Random(12)
    ids = helpers.random_prompt(rng, 151, CONFIGS[name]["vocab"])
    other = helpers.random_prompt(rng, 60, CONFIGS[name]["vocab"])
    runner = make_runner(model_dirs[name], dtype, device, 16, PAGE[name], seats=2)
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
@pytest.mark.parametrize("name", ["U", "V"])
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
    name = "U"
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
