"""The gated delta rule: a linear recurrence whose state a token first lets decay, then corrects.

q, k = W_q h, W_k h in ``kv_heads`` heads of ``dim``; v = W_v h in ``heads`` heads of ``vdim``; head h uses query/key head
h // (heads / kv_heads).  Every channel of q, k and v passes a causal convolution of ``conv`` taps over time (zeros before
the start) and silu; q and k become unit vectors per head, x / sqrt(sum(x^2) + unit_eps), and q is multiplied by
``query_scale`` (dim^(-1/2) unless given).  Per token and head a decay g = exp(-exp(A_log) softplus(W_a h + dt_bias)) and a
step size beta = sigmoid(W_b h).  With state S [dim, vdim] per head:
    S <- g S ;   u = beta (v - S^T k) ;   S <- S + k u^T ;   o = S^T q .
Each head's o is divided by its root mean square, times one weight of ``vdim`` numbers, times silu(W_g h), and projected.

A state slot of the cache manager (float32, zero at admission) holds S of every head and behind it the last conv - 1
projected rows of q | k | v.  The six projections are one product, kept in float32; convolutions, unit vectors, decay, step
size, the recurrence and the head norm are float32 whatever the compute dtype.
"""
from __future__ import annotations

from .base import Mixer, register_mixer


class GatedDeltaMixer(Mixer):
    def __init__(self, hidden_size: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, eps: float,
                 unit_eps: float = 1e-6, query_scale: float | None = None):
        if heads % kv_heads:
            raise ValueError("the heads must share the query/key heads out equally")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.dim, self.vdim, self.conv = int(dim), int(vdim), int(conv)
        if self.conv < 1:
            raise ValueError("a convolution has at least one tap")
        self.eps, self.unit_eps = float(eps), float(unit_eps)
        self.query_scale = float(query_scale) if query_scale is not None else self.dim ** -0.5
        self.qkvgba_weight = self.conv_weight = self.A_log = self.dt_bias = self.norm_weight = self.o_weight = None
        self._conv_by_tap = self._head_weight = None

    @property
    def channels(self) -> int:
        """Channels that pass a convolution: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def inner_width(self) -> int:
        return self.heads * self.vdim

    @property
    def input_width(self) -> int:
        return self.channels + self.inner_width + 2 * self.heads

    @property
    def matrix_elements(self) -> int:
        """Where the convolutions' history begins in a seat's row: behind the heads' states, on a 16-byte boundary."""
        return -(-self.heads * self.dim * self.vdim // 4) * 4

    @property
    def state_elements(self) -> int:
        return -(-(self.matrix_elements + (self.conv - 1) * self.channels) // 4) * 4

    def parameter_shapes(self) -> dict:
        return {"qkvgba.weight": ((self.input_width, self.hidden_size), "matrix"), "conv.weight": ((self.channels, self.conv), "vector"),
                "A_log": ((self.heads,), "vector"), "dt_bias": ((self.heads,), "vector"), "norm.weight": ((self.vdim,), "vector"),
                "o.weight": ((self.hidden_size, self.inner_width), "matrix")}

    def bind(self, tensors: dict) -> None:
        super().bind(tensors)
        # the table tap by tap, [taps, channels]: the kernels' lanes then read neighbouring numbers
        self._conv_by_tap = self.conv_weight.t().contiguous()
        self._head_weight = self.norm_weight.repeat(self.heads).contiguous()

    def reads_first(self):
        return self.qkvgba_weight

    def cache_need(self):
        return {"kind": "state", "state_shape": (self.state_elements,), "state_dtype": "float32"}

    def forward(self, ctx, h, entry):
        ops = ctx.ops
        projected = ops.linear(h, self.qkvgba_weight, None, out_float32=True)          # q | k | v | g | b | a
        state = ctx.groups[entry.cache_group].state(entry.cache_slot)                  # [seats, state | history] float32
        sizes = (self.heads, self.kv_heads, self.dim, self.vdim)
        if ctx.max_q_len == 1:
            # a step of one token a request: everything between the two products in one kernel
            out = ops.delta_decode(projected, self._conv_by_tap, state, self.matrix_elements, ctx.state_slots, self.A_log, self.dt_bias,
                                   self.norm_weight, self.eps, self.unit_eps, self.query_scale, *sizes, ctx.dtype)
            return ops.linear(out, self.o_weight)
        qkv, gates = ops.delta_prepare(projected, self._conv_by_tap, state, self.matrix_elements, ctx.state_slots, ctx.cu_q,
                                       ctx.token_request, self.A_log, self.dt_bias, self.unit_eps, self.query_scale, *sizes,
                                       max_q_len=ctx.max_q_len)
        o = ops.delta_scan(qkv, gates, state, ctx.state_slots, ctx.cu_q, *sizes, max_q_len=ctx.max_q_len)
        g = projected[:, self.channels:self.channels + self.inner_width]
        out = ops.head_rmsnorm_gate(o, self._head_weight, g, self.eps, self.heads, ctx.dtype)
        return ops.linear(out, self.o_weight)


register_mixer("gated_delta", GatedDeltaMixer)
