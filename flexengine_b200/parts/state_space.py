"""State-space mixers: recurrences whose decay and step size depend on the token.

``head_state_space`` (Mamba-2): one decay per head.  W_in h = z | x | B | C | dt with x, z in ``heads`` heads of ``vdim``, B and C
in ``groups`` groups of ``state`` (head h reads group h // (heads / groups)), dt one number per head.  x, B and C pass a
causal convolution of ``conv`` taps over time (with a bias, zeros before the start) and silu; dt <- softplus(dt + dt_bias).
Per head S <- exp(-exp(A_log) dt) S + dt B x^T (S is state x vdim), y = S^T C + D x.  y (all heads) times silu(z), then
divided in ``norm_groups`` equal parts by each part's root mean square, times a weight, and projected.

``selective_scan`` (Mamba): a decay per channel and state entry.  W_in h = x | z (``inner`` each); x passes the convolution and
silu; W_x x = low | B | C (``dt_rank``, ``state``, ``state``); dt = softplus(W_dt low + bias) per channel; A = -exp(A_log).  Per
channel c and entry n S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n, y_c = sum_n S[c, n] C_n + D_c x_c; y silu(z) is
projected.

A state slot of the cache manager (float32, zero at admission) holds S and behind it, on a 16-byte boundary, the last conv - 1
inputs of the convolution.  Step sizes, decays with their exponentials, the recurrences and the norm are float32 whatever
the compute dtype; so is the whole projection of ``head_state_space`` (its step sizes are rows of it).
"""
from __future__ import annotations

from .base import Mixer, register_mixer


class _ConvolvedState(Mixer):
    """What the two have in common: a seat of state and history, and the convolution's table tap by tap."""

    def matrix_elements(self) -> int:
        raise NotImplementedError

    @property
    def history_at(self) -> int:
        return -(-self.matrix_elements() // 4) * 4

    @property
    def state_elements(self) -> int:
        return -(-(self.history_at + (self.conv - 1) * self.channels) // 4) * 4

    def cache_need(self):
        return {"kind": "state", "state_shape": (self.state_elements,), "state_dtype": "float32"}

    def bind(self, tensors: dict) -> None:
        super().bind(tensors)
        # [taps, channels]: the kernels' lanes then read neighbouring numbers
        self._conv_by_tap = self.conv_weight.t().contiguous()
        # what a step size is multiplied by for the logarithm of the decay
        self._minus_a = -self.A_log.exp()


class HeadStateSpaceMixer(_ConvolvedState):
    def __init__(self, hidden_size: int, heads: int, vdim: int, state: int, groups: int, norm_groups: int, conv: int, eps: float):
        if heads % groups or (heads * vdim) % norm_groups:
            raise ValueError("groups must share the heads out equally, norm_groups the channels")
        self.hidden_size, self.heads, self.vdim, self.state = int(hidden_size), int(heads), int(vdim), int(state)
        self.groups, self.norm_groups, self.conv, self.eps = int(groups), int(norm_groups), int(conv), float(eps)
        if self.conv < 1:
            raise ValueError("a convolution has at least one tap")
        self.in_weight = self.conv_weight = self.conv_bias = self.dt_bias = self.A_log = self.D = self.norm_weight = self.o_weight = None

    @property
    def inner_width(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """What passes the convolution: x | B | C."""
        return self.inner_width + 2 * self.groups * self.state

    @property
    def input_width(self) -> int:
        return self.inner_width + self.channels + self.heads

    def matrix_elements(self) -> int:
        return self.heads * self.state * self.vdim

    def parameter_shapes(self) -> dict:
        H = self.heads
        return {"in.weight": ((self.input_width, self.hidden_size), "matrix"), "conv.weight": ((self.channels, self.conv), "vector"),
                "conv.bias": ((self.channels,), "vector"), "dt_bias": ((H,), "vector"), "A_log": ((H,), "vector"), "D": ((H,), "vector"),
                "norm.weight": ((self.inner_width,), "vector"), "o.weight": ((self.hidden_size, self.inner_width), "matrix")}

    def reads_first(self):
        return self.in_weight

    def forward(self, ctx, h, entry):
        ops = ctx.ops
        H, dv, N, G, inner, C = self.heads, self.vdim, self.state, self.groups, self.inner_width, self.channels
        projected = ops.linear(h, self.in_weight, None, out_float32=True)              # z | x | B | C | dt
        state = ctx.groups[entry.cache_group].state(entry.cache_slot)
        rows, gates = ops.conv_silu(projected[:, inner:inner + C], self._conv_by_tap, self.conv_bias, state, self.history_at, ctx.state_slots,
                                    ctx.cu_q, out_float32=True, steps=(projected[:, inner + C:], self.dt_bias, self._minus_a),
                                    max_q_len=ctx.max_q_len)
        x, B, Cq = rows[:, :inner], rows[:, inner:inner + G * N], rows[:, inner + G * N:]
        y = ops.head_scan(Cq, B, x, gates, state, ctx.state_slots, ctx.cu_q, H, G, N, dv, skip=self.D, max_q_len=ctx.max_q_len)
        out = ops.gated_group_rmsnorm(y, projected[:, :inner], self.norm_weight, self.eps, self.norm_groups, ctx.dtype)
        return ops.linear(out, self.o_weight)


class SelectiveScanMixer(_ConvolvedState):
    input_parameter = "in.weight"         # the side's input matrix, where it stands beside another mixer

    def __init__(self, hidden_size: int, inner: int, state: int, dt_rank: int, conv: int):
        self.hidden_size, self.inner, self.state, self.dt_rank, self.conv = int(hidden_size), int(inner), int(state), int(dt_rank), int(conv)
        if self.conv < 1:
            raise ValueError("a convolution has at least one tap")
        self.in_weight = self.conv_weight = self.conv_bias = self.x_weight = self.dt_weight = self.dt_bias = self.A_log = self.D = self.o_weight = None

    @property
    def inner_width(self) -> int:
        return self.inner

    @property
    def channels(self) -> int:
        return self.inner

    @property
    def input_width(self) -> int:
        return 2 * self.inner

    def matrix_elements(self) -> int:
        return self.inner * self.state

    def parameter_shapes(self) -> dict:
        D, I, N, R = self.hidden_size, self.inner, self.state, self.dt_rank
        return {"in.weight": ((2 * I, D), "matrix"), "conv.weight": ((I, self.conv), "vector"), "conv.bias": ((I,), "vector"),
                "x.weight": ((R + 2 * N, I), "matrix"), "dt.weight": ((I, R), "matrix"), "dt.bias": ((I,), "vector"),
                "A_log": ((I, N), "vector"), "D": ((I,), "vector"), "o.weight": ((D, I), "matrix")}

    def reads_first(self):
        return self.in_weight

    def forward(self, ctx, h, entry):
        return ctx.ops.linear(self.mix(ctx, ctx.ops.linear(h, self.in_weight), entry), self.o_weight)

    def mix(self, ctx, projected, entry, out=None, scale=1.0):
        """``projected`` [T, >= input_width] = x | z (any row stride) -> y silu(z) [T, inner], times ``scale``, into ``out`` where
        given."""
        ops = ctx.ops
        I = self.inner
        state = ctx.groups[entry.cache_group].state(entry.cache_slot)
        x, _ = ops.conv_silu(projected[:, :I], self._conv_by_tap, self.conv_bias, state, self.history_at, ctx.state_slots, ctx.cu_q,
                             max_q_len=ctx.max_q_len)
        low = ops.linear(x, self.x_weight)                                              # low | B | C
        z = projected[:, I:2 * I]
        if ctx.max_q_len == 1:
            # a step of one token a request: the step sizes' projection inside the scan's kernel
            return ops.selective_decode(x, low, self.dt_weight, self.dt_bias, self._minus_a, self.D, z, state, ctx.state_slots, scale=scale,
                                        into=out)
        dt = ops.linear(low[:, :self.dt_rank], self.dt_weight, None, out_float32=True)
        return ops.selective_scan(x, dt, self.dt_bias, self._minus_a, low[:, self.dt_rank:], self.D, z, state, ctx.state_slots, ctx.cu_q,
                                  scale=scale, into=out, max_q_len=ctx.max_q_len)


register_mixer("head_state_space", HeadStateSpaceMixer)
register_mixer("selective_scan", SelectiveScanMixer)
