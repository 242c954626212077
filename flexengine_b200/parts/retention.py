"""Retention: linear attention with one fixed decay per head, no softmax and no denominator.

q, k = W_q h, W_k h in heads of ``dim``; v = W_v h in heads of ``vdim``.  The first ``rot_dims`` entries of every query
and key head turn by position * rot_base^(-2i/rot_dims), entry i paired with i + rot_dims/2; the keys are then multiplied
by dim^(-1/2).  Per head, with state S [dim, vdim]:
    S_t = decay_h S_(t-1) + k_t v_t^T ;   o_t = S_t^T q_t .
Each head's o is divided by its root mean square (no weight), the heads are concatenated, multiplied by silu(W_g h) and
projected.  S of a request lives in a state slot of the cache manager in float32, zero at admission; angles, the rotated
queries and keys, the decay, the recurrence and the head norm are float32 whatever the compute dtype.  The four
projections are one product.

Options: ``activation`` "silu" is applied to the projected q, k and v (before anything else; lightning attention);
``key_scale`` replaces dim^(-1/2); ``norm`` "all_heads" divides the concatenated heads by ONE root mean square and multiplies
them by a weight (``norm.weight``, heads * vdim numbers) in place of the unit norm per head; ``gate`` "sigmoid" takes sigmoid(W_g h).
"""
from __future__ import annotations

import torch

from .base import Mixer, register_mixer


class RetentionMixer(Mixer):
    NORMS = ("head", "all_heads")
    GATES = ("silu", "sigmoid")

    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, decay, rot_base: float = 10000.0, rot_dims: int = 0,
                 eps: float = 1e-6, activation: str | None = None, key_scale: float | None = None, norm: str = "head", gate: str = "silu"):
        self.hidden_size, self.heads, self.dim, self.vdim = int(hidden_size), int(heads), int(dim), int(vdim)
        self.decay = tuple(float(x) for x in decay)
        if len(self.decay) != self.heads:
            raise ValueError("one decay per head")
        self.rot_base, self.rot_dims, self.eps = float(rot_base), int(rot_dims), float(eps)
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            raise ValueError("rot_dims must be even and at most dim")
        if activation not in (None, "silu") or norm not in self.NORMS or gate not in self.GATES:
            raise ValueError(f"activation {activation!r} / norm {norm!r} / gate {gate!r}: known are None and 'silu', {self.NORMS}, {self.GATES}")
        if activation is not None and self.rot_dims:
            raise ValueError("activated queries and keys do not turn")
        self.activation, self.norm, self.gate = activation, norm, gate
        self.key_scale = float(key_scale) if key_scale is not None else self.dim ** -0.5
        self.qkvg_weight = self.o_weight = self.norm_weight = None
        self._tables = {}

    @property
    def input_width(self) -> int:
        return 2 * self.heads * self.dim + 2 * self.heads * self.vdim

    @property
    def inner_width(self) -> int:
        return self.heads * self.vdim

    def parameter_shapes(self) -> dict:
        shapes = {"qkvg.weight": ((self.input_width, self.hidden_size), "matrix"),
                  "o.weight": ((self.hidden_size, self.inner_width), "matrix")}
        if self.norm == "all_heads":
            shapes["norm.weight"] = ((self.inner_width,), "vector")
        return shapes

    def reads_first(self):
        return self.qkvg_weight

    @property
    def state_elements(self) -> int:
        return self.heads * self.dim * self.vdim

    def cache_need(self):
        return {"kind": "state", "state_shape": (self.state_elements,), "state_dtype": "float32"}

    def tables(self, device):
        """(inverse frequencies [rot_dims / 2] or None, decay [heads]) as float32 on ``device``, rounded once from float64."""
        key = str(device)
        if key not in self._tables:
            inv_freq = None
            if self.rot_dims:
                i = torch.arange(self.rot_dims // 2, dtype=torch.float64)
                inv_freq = torch.pow(torch.tensor(self.rot_base, dtype=torch.float64), -2.0 * i / self.rot_dims)
                inv_freq = inv_freq.to(torch.float32).to(device).contiguous()
            self._tables[key] = (inv_freq, torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(device))
        return self._tables[key]

    def forward(self, ctx, h, entry):
        projected = ctx.ops.linear(h, self.qkvg_weight)
        return ctx.ops.linear(self.mix(ctx, projected, entry), self.o_weight)

    def mix(self, ctx, projected, entry, out=None, scale=1.0):
        """``projected`` [T, >= input_width] = q | k | v | g (any row stride) -> the normed, gated heads [T, inner_width],
        times ``scale``, into ``out`` where given."""
        ops = ctx.ops
        H, d, dv = self.heads, self.dim, self.vdim
        state = ctx.groups[entry.cache_group].state(entry.cache_slot)        # [seats, H d dv] float32
        inv_freq, decay = self.tables(projected.device)
        plain = self.activation is None and self.norm == "head" and self.gate == "silu"
        if ctx.max_q_len == 1 and plain:
            # a step of one token a request: rotation, recurrence, head norm and gate in one kernel
            return ops.retention_decode(projected, H, d, dv, ctx.positions, inv_freq, self.rot_dims, self.key_scale, decay, state,
                                        ctx.state_slots, self.eps, ctx.dtype, scale=scale, into=out)
        gates = projected[:, 2 * H * d + H * dv:2 * H * d + 2 * H * dv]
        if ctx.max_q_len == 1 and self.norm == "all_heads":
            # activation (or rotation) and recurrence in one kernel; the norm reads all heads of a row
            o = ops.retention_decode(projected, H, d, dv, ctx.positions, inv_freq, self.rot_dims, self.key_scale, decay, state,
                                     ctx.state_slots, self.eps, ctx.dtype, activation=self.activation, raw=True)
        else:
            if self.activation is not None:
                # queries, keys and values through the activation: float32 from here on
                rows = ops.activate_rows(projected, 2 * H * d + H * dv, self.activation, ((H * d, 1.0), (H * d, self.key_scale)))
                qk, values = rows[:, :2 * H * d], rows[:, 2 * H * d:]
            else:
                # queries and keys, rotated, the keys scaled: float32 from here on
                qk = ops.rotate_heads(projected, 2 * H, d, ctx.positions, inv_freq, self.rot_dims, ((H, 1.0), (H, self.key_scale)))
                values = projected[:, 2 * H * d:2 * H * d + H * dv]
            o = ops.retention_scan(qk, values, decay, state, ctx.state_slots, ctx.cu_q, H, d, dv, max_q_len=ctx.max_q_len)
        if self.norm == "all_heads":
            return ops.head_rmsnorm_gate(o, self.norm_weight, gates, self.eps, 1, ctx.dtype, scale=scale, into=out, gate=self.gate)
        more = {} if self.gate == "silu" else {"gate": self.gate}
        return ops.head_rmsnorm_gate(o, None, gates, self.eps, H, ctx.dtype, scale=scale, into=out, **more)


register_mixer("retention", RetentionMixer)
