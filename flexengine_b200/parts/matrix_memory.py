"""A matrix memory with exponential gates (the mLSTM of xLSTM): linear attention whose decay and step size are a head's own
for every token, divided by what a memory of the keys alone answers.

q, k = W_q h, W_k h in heads of ``dim``, q times ``query_scale`` (dim^(-1/2) unless given); v = W_v h in heads of ``vdim``.  Per head
a log input gate i = cap tanh((W_i h + b_i) / cap) and a log forget gate f = log sigmoid(cap tanh((W_f h + b_f) / cap)).  With a
running maximum m (zero at the start):
    m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n <- exp(f + m - m') n + exp(i - m') k;  m <- m';
    o = S^T q / (max(|n . q|, exp(-m)) + floor).
Each head's o is divided by its root mean square, times a weight of all heads' size, times sigmoid(W_g h), and projected.

The step is the scan of ``ops.head_scan``: a decay a and a weight w per token and head, S <- a S + w k v^T, o = S^T q.  A state
slot of the cache manager (float32, zero at admission) holds S of every head, then the heads' n, then their m.  The six
projections are one product, kept in float32; gates, maximum, recurrence, divisor and head norm are float32 whatever the
compute dtype.
"""
from __future__ import annotations

from .base import Mixer, register_mixer


class MatrixMemoryMixer(Mixer):
    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float, query_scale: float | None = None,
                 floor: float = 1e-6):
        self.hidden_size, self.heads, self.dim, self.vdim = int(hidden_size), int(heads), int(dim), int(vdim)
        self.gate_cap, self.eps, self.floor = float(gate_cap), float(eps), float(floor)
        if not self.gate_cap > 0.0:
            raise ValueError("the cap of the gates is positive")
        self.query_scale = float(query_scale) if query_scale is not None else self.dim ** -0.5
        self.qkvgif_weight = self.gates_bias = self.norm_weight = self.o_weight = None

    @property
    def inner_width(self) -> int:
        return self.heads * self.vdim

    @property
    def input_width(self) -> int:
        return 2 * self.heads * self.dim + 2 * self.inner_width + 2 * self.heads

    @property
    def state_elements(self) -> int:
        """S of every head, the heads' memories of the keys, their running maxima; in steps of four."""
        return -(-self.heads * (self.dim * self.vdim + self.dim + 1) // 4) * 4

    def parameter_shapes(self) -> dict:
        return {"qkvgif.weight": ((self.input_width, self.hidden_size), "matrix"), "gates.bias": ((2 * self.heads,), "vector"),
                "norm.weight": ((self.inner_width,), "vector"), "o.weight": ((self.hidden_size, self.inner_width), "matrix")}

    def reads_first(self):
        return self.qkvgif_weight

    def cache_need(self):
        return {"kind": "state", "state_shape": (self.state_elements,), "state_dtype": "float32"}

    def forward(self, ctx, h, entry):
        ops = ctx.ops
        projected = ops.linear(h, self.qkvgif_weight, None, out_float32=True)          # q | k | v | g | i | f
        state = ctx.groups[entry.cache_group].state(entry.cache_slot)
        H, d, dv = self.heads, self.dim, self.vdim
        if ctx.max_q_len == 1:
            # a step of one token a request: everything between the two products in one kernel
            out = ops.memory_decode(projected, self.gates_bias, self.gate_cap, self.query_scale, self.floor, state, ctx.state_slots,
                                    self.norm_weight, self.eps, H, d, dv, ctx.dtype)
            return ops.linear(out, self.o_weight)
        qk, inner = H * d, H * dv
        gates = ops.memory_gates(projected[:, 2 * qk + 2 * inner:], self.gates_bias, self.gate_cap, state, H * (d * dv + d), ctx.state_slots,
                                 ctx.cu_q, H, max_q_len=ctx.max_q_len)
        o = ops.head_scan(projected[:, :qk], projected[:, qk:2 * qk], projected[:, 2 * qk:2 * qk + inner], gates, state, ctx.state_slots,
                          ctx.cu_q, H, H, d, dv, query_scale=self.query_scale, divided=self.floor, max_q_len=ctx.max_q_len)
        out = ops.head_rmsnorm_gate(o, self.norm_weight, projected[:, 2 * qk + inner:2 * qk + 2 * inner], self.eps, H, ctx.dtype, gate="sigmoid")
        return ops.linear(out, self.o_weight)


register_mixer("matrix_memory", MatrixMemoryMixer)
