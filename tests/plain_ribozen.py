"""A plain, slow implementation of the Ribozen decoder: one function per mechanism, whole sequences at once, float64.
It shares no code with the package: it reads ``config.json`` and the safetensors file itself and has no cache, no batches
and no state beyond a loop variable.

The model: x = scale * embed[token].  A layer is x <- x + ls1 * mixer(N1(x)), then x <- x + ls2 * ff(N2(x)) where it has a
feed-forward; N is an RMS norm, ls1 and ls2 a learned number per channel.  Mixers: a matrix memory with exponential gates
(``mlstm``), the state-space layer with one decay per head (``mamba2``), and a pair of mixers side by side (``parallel``):
softmax attention under a window that keeps the first tokens, beside a selective scan with a decay per channel and state
entry.  Feed-forward: experts that read their input times their sigmoid score, and a shared expert.
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


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def causal_convolution(u, table, bias):
    """u [T, channels], table [channels, taps]: y_t = bias + sum_j table[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], table.shape[1]
    y = bias.repeat(T, 1)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += table[:, j] * u[:T - back]
    return y


# ---- rotation ---------------------------------------------------------------------------------------------------------
def rotation_frequencies(rot):
    """(frequencies [dims / 2], factor of cosine and sine) with the YaRN blend of slow and fast pairs where one is given."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return torch.tensor(plain, dtype=DT), 1.0

    def pair_that_turns(times):
        return dims * math.log(scaling["original"] / (2 * math.pi * times)) / (2 * math.log(base))

    lo = max(math.floor(pair_that_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * slow + f * (1.0 - slow))
    return torch.tensor(out, dtype=DT), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dim]: the first rot.dims entries of every head turned by the position, i paired with i + dims/2."""
    if not rot or not rot["dims"]:
        return x
    freq, gain = rotation_frequencies(rot)
    half = rot["dims"] // 2
    angle = torch.arange(x.shape[0], dtype=DT)[:, None, None] * freq
    cos, sin = torch.cos(angle) * gain, torch.sin(angle) * gain
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], dim=-1)


# ---- mixers -----------------------------------------------------------------------------------------------------------
def visible(T, window, keep_first):
    """[T, T]: whether query i sees key j: j <= i and (i - j < window or j < keep_first)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < window) | (j < keep_first)) if window else j <= i


def windowed_attention(h, w, p, m, eps):
    """h [T, D]; ``p`` the tensors' prefix ('l0.mix.left.'), ``m`` the sizes.  The gated heads through the output projection."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(name):
        return h @ w[p + name].T + w[p + name + ".b"]

    q = rotate(rms_norm(projected("q"), w[p + "q.norm"], eps).view(T, H, d), m.get("rot"))
    k = rotate(rms_norm(projected("k"), w[p + "k.norm"], eps).view(T, G, d), m.get("rot")).repeat_interleave(H // G, dim=1)
    v = projected("v").view(T, G, dv).repeat_interleave(H // G, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    if m.get("softcap"):
        scores = m["softcap"] * torch.tanh(scores / m["softcap"])
    mask = m.get("mask") or {}
    scores = scores.masked_fill(~visible(T, mask.get("size", 0), mask.get("keep_first", 0)), float("-inf"))
    out = torch.einsum("hij,jhd->ihd", torch.softmax(scores, dim=-1), v).reshape(T, H * dv)
    return (out * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def selective_scan(x, dt, A, B, C):
    """x, dt [T, channels], A [channels, state] (negative), B, C [T, state]: S <- exp(dt A) S + dt x B, y = S C."""
    state = torch.zeros_like(A)
    rows = []
    for t in range(x.shape[0]):
        state = torch.exp(dt[t][:, None] * A) * state + (dt[t] * x[t])[:, None] * B[t]
        rows.append(state @ C[t])
    return torch.stack(rows)


def mamba(h, w, p, m):
    inner, rank, N = m["inner"], m["dt_rank"], m["state"]
    x, z = (h @ w[p + "in"].T).split([inner, inner], dim=-1)
    x = silu(causal_convolution(x, w[p + "conv"], w[p + "conv.b"]))
    low, B, C = (x @ w[p + "x"].T).split([rank, N, N], dim=-1)
    dt = softplus(low @ w[p + "dt"].T + w[p + "dt.b"])
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), B, C) + w[p + "D"] * x
    return (y * silu(z)) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * windowed_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * mamba(h, w, p + "right.", m["right"])


def head_scan(q, k, v, decay, weight):
    """q, k [T, heads, N], v [T, heads, dv], decay, weight [T, heads]: S <- decay S + weight k v^T, o = S^T q [T, heads, dv]."""
    T, H, N = q.shape
    state = torch.zeros(H, N, v.shape[-1], dtype=DT)
    rows = []
    for t in range(T):
        state = decay[t][:, None, None] * state + weight[t][:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hnv,hn->hv", state, q[t]))
    return torch.stack(rows)


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xBC, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = silu(causal_convolution(xBC, w[p + "conv"], w[p + "conv.b"])).split([inner, G * N, G * N], dim=-1)
    x = x.view(T, H, dv)
    B, C = (t.view(T, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    y = head_scan(C, B, x, decay, dt) + w[p + "D"][:, None] * x
    y = y.reshape(T, inner) * silu(z)
    y = unit_rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def exponential_memory(q, k, v, log_forget, log_input):
    """q, k [T, heads, dim], v [T, heads, vdim], the gates' logarithms [T, heads]; a running maximum that starts at zero."""
    T, H, d = q.shape
    S, n, m = torch.zeros(H, d, v.shape[-1], dtype=DT), torch.zeros(H, d, dtype=DT), torch.zeros(H, dtype=DT)
    rows = []
    for t in range(T):
        new = torch.maximum(log_forget[t] + m, log_input[t])
        keep, add = torch.exp(log_forget[t] + m - new), torch.exp(log_input[t] - new)
        m = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        below = torch.maximum((n * q[t]).sum(dim=-1).abs(), torch.exp(-m)) + 1e-6
        rows.append(torch.einsum("hdv,hd->hv", S, q[t]) / below[:, None])
    return torch.stack(rows)


def mlstm(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)

    def capped(name):
        return cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)

    o = exponential_memory(q, k, v, log_sigmoid(capped("f")), capped("i"))
    out = unit_rms(o, eps).reshape(T, H * dv) * w[p + "norm"]
    return (out * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    return {"mlstm": mlstm, "mamba2": mamba2, "parallel": parallel}[kind](h, w, p, m, eps)


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(logits, top):
    """(chosen [T, top], weights [T, top]): the largest sigmoid scores, as they are."""
    order = torch.sort(torch.sigmoid(logits), dim=-1, descending=True, stable=True)
    return order.indices[:, :top], order.values[:, :top]


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
            out[rows] += expert(weights[rows, places][:, None] * h[rows], w, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------
def layer_forward(x, w, i, spec, config, gaps=None):
    eps, name = config["norm"]["eps"], f"l{i}."
    x = x + w[name + "ls1"] * mixer(spec["type"], rms_norm(x, w[name + "norm1"], eps), w, name + "mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        x = x + w[name + "ls2"] * routed_feed_forward(rms_norm(x, w[name + "norm2"], eps), w, name + "mlp.", spec["mlp"], gaps)
    return x


def forward_logits(config, weights, ids, after_layers=None, gaps=None):
    """float64 logits [T, vocab] of the whole sequence ``ids``; ``after_layers`` (a list) receives x after every layer."""
    w = weights
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)] * config["embedding"]["scale"]
    for i, spec in enumerate(config["layers"]):
        x = layer_forward(x, w, i, spec, config, gaps)
        if after_layers is not None:
            after_layers.append(x)
    return rms_norm(x, w["final.norm"], config["norm"]["eps"]) @ w["head"].T
