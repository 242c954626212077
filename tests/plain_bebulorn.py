"""A plain, slow implementation of the Bebulorn decoder: one function per mechanism, whole sequences at once, float64.
It shares no code with the package: it reads ``config.json`` and the safetensors file itself and has no cache, no batches
and no state beyond a loop variable.

The model: x = embed[token].  A layer is x <- x + m N1b(mixer(N1(x))), then x <- x + m N2b(ff(N2(x))) where it has a
feed-forward; every N is a layer norm with weight and bias, m one constant.  Mixers: softmax attention without positions
(unit-norm values, a number per head on the scores, scores squashed by tanh, a sliding window), lightning attention (a
fixed decay per head, silu on q, k and v, one norm over all heads, a sigmoid gate) and the gated delta rule (short
convolutions, unit vectors, a decay and a step size per token and head).  Feed-forwards: dense with a relu gate, or routed
over experts without a gate, with a shared expert.  A span of layers may run several times with the same weights; before
every pass but the first the embedding's output is added to the stream.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

DT = torch.float64


# ---- reading a model folder ---------------------------------------------------------------------------------------
def read_model_folder(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        config = json.load(f)
    weights = {}
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        index = json.loads(f.read(n))
        base = 8 + n
        kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
        for name, meta in index.items():
            if name == "__metadata__":
                continue
            a, b = meta["data_offsets"]
            f.seek(base + a)
            t = torch.frombuffer(bytearray(f.read(b - a)), dtype=kinds[meta["dtype"]]).reshape(meta["shape"])
            weights[name] = t.to(DT) if t.is_floating_point() else t
    return config, weights


# ---- small pieces ---------------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, eps, weight, bias):
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt(centred.pow(2).mean(dim=-1, keepdim=True) + eps) * weight + bias


def silu(z):
    return z * torch.sigmoid(z)


def causal_convolution(u, table):
    """u [T, channels], table [channels, taps]: y_t = sum_j table[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], table.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            at = t - (taps - 1) + j
            if at >= 0:
                y[t] += table[:, j] * u[at]
    return y


# ---- mixers -----------------------------------------------------------------------------------------------------------
def visible(T, window):
    """[T, T]: whether query i sees key j, 0 <= i - j (< window where there is one)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax_attention(h, w, p, m, eps):
    """h [T, D]; ``p`` the tensors' prefix ('l0.mix.'), ``m`` the mixer's entry of the configuration."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d)
    k = (h @ w[p + "k"].T).view(T, G, d).repeat_interleave(H // G, dim=1)
    v = unit_rms((h @ w[p + "v"].T).view(T, G, dv), eps).repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] * w[p + "temp"][:, None, None]
    scores = m["softcap"] * torch.tanh(scores / m["softcap"])
    scores = scores.masked_fill(~visible(T, m["mask"]["size"]), float("-inf"))
    out = torch.einsum("hij,jhd->ihd", torch.softmax(scores, dim=-1), v)
    return out.reshape(T, H * dv) @ w[p + "o"].T


def lightning(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, d)
    k = silu(h @ w[p + "k"].T).view(T, H, d)
    v = silu(h @ w[p + "v"].T).view(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=DT)
    state = torch.zeros(H, d, dv, dtype=DT)
    rows = []
    for t in range(T):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", state, q[t]))
    out = unit_rms(torch.stack(rows).reshape(T, H * dv), eps) * w[p + "norm"]
    return (out * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_decay_and_step(h, w, p):
    """(g, beta) [T, heads]: what the state is multiplied by, and how much of a token's correction is written."""
    z = h @ w[p + "a"].T + w[p + "dt_bias"]
    softplus = torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))
    return torch.exp(-torch.exp(w[p + "A_log"]) * softplus), torch.sigmoid(h @ w[p + "b"].T)


def delta_rule(q, k, v, g, beta):
    """q, k [T, heads, dim], v [T, heads, vdim], g, beta [T, heads] -> o [T, heads, vdim]."""
    T, H, d = q.shape
    state = torch.zeros(H, d, v.shape[-1], dtype=DT)
    rows = []
    for t in range(T):
        state = g[t][:, None, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", state, k[t]))
        state = state + k[t][:, :, None] * u[:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(rows)


def gated_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def stream(name, heads, size):
        return silu(causal_convolution(h @ w[p + name].T, w[p + name + ".conv"])).view(T, heads, size)

    def unit(x):
        return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + 1e-6)

    q = (unit(stream("q", G, d)) * d ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(stream("k", G, d)).repeat_interleave(H // G, dim=1)
    v = stream("v", H, dv)
    g, beta = delta_decay_and_step(h, w, p)
    out = unit_rms(delta_rule(q, k, v, g, beta), eps) * w[p + "norm"]
    return (out.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": softmax_attention, "lightning": lightning, "delta": gated_delta}


# ---- feed-forwards ---------------------------------------------------------------------------------------------------
def dense_feed_forward(h, w, p):
    return (torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def expert(h, w, p):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def route(logits, top):
    """(chosen [T, top], weights [T, top]): the largest softmax scores, divided by their sum."""
    scores = torch.softmax(logits, dim=-1)
    order = torch.sort(scores, dim=-1, descending=True, stable=True)
    best = order.values[:, :top]
    return order.indices[:, :top], best / (best.sum(dim=-1, keepdim=True) + 1e-20)


def routed_feed_forward(h, w, p, mlp, gaps=None):
    """``gaps`` (a list) receives, per token, the gap between the last chosen and the first rejected router logit."""
    experts, top = mlp["router"]["experts"], mlp["router"]["top"]
    logits = h @ w[p + "router"].T
    if gaps is not None and top < experts:
        ranked = torch.sort(logits, dim=-1, descending=True).values
        gaps.append(ranked[:, top - 1] - ranked[:, top])
    chosen, weights = route(logits, top)
    out = torch.zeros_like(h)
    for e in range(experts):
        rows, places = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += weights[rows, places][:, None] * expert(h[rows], w, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------
def norm(x, w, name, eps):
    return layer_norm(x, eps, w[name], w[name + ".b"])


def layer_forward(x, w, i, spec, config, gaps=None):
    eps, m = config["norm"]["eps"], config["residual_mult"]
    name = f"l{i}"
    mixed = MIXERS[spec["type"]](norm(x, w, name + ".norm1", eps), w, name + ".mix.", spec["mixer"], eps)
    x = x + m * norm(mixed, w, name + ".norm1b", eps)
    mlp = spec.get("mlp")
    if mlp is not None:
        h = norm(x, w, name + ".norm2", eps)
        fed = dense_feed_forward(h, w, name + ".mlp.") if mlp["kind"] == "dense" else routed_feed_forward(h, w, name + ".mlp.", mlp, gaps)
        x = x + m * norm(fed, w, name + ".norm2b", eps)
    return x


def run_order(config):
    """[(layer, the embedding's output is added before it)]: the layers in the order they run."""
    count = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(count)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(start)]
    for turn in range(times):
        order += [(i, i == start and turn > 0) for i in range(start, stop)]
    return order + [(i, False) for i in range(stop, count)]


def forward_logits(config, weights, ids, after_layers=None, gaps=None):
    """float64 logits [T, vocab] of the whole sequence ``ids``; ``after_layers`` (a list) receives x after every layer run."""
    w = weights
    x0 = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    x = x0
    for i, again in run_order(config):
        if again:
            x = x + x0
        x = layer_forward(x, w, i, config["layers"][i], config, gaps)
        if after_layers is not None:
            after_layers.append(x)
    return norm(x, w, "final.norm", config["norm"]["eps"]) @ w["head"].T
