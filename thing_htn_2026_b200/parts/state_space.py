"""State-space duality (Mamba-2): a recurrent token mixer with a matrix state per head and one decay
per head and token.  With ``n_heads`` heads of ``value_dim``, a state of N entries and G groups of
neighbouring heads that share B and C:

    [z | x | B | C | dt] = W_in h                     (heads * value_dim twice, G * N twice, heads)
    [x | B | C] <- silu(conv([x | B | C]) + b_conv)   (a causal convolution per channel over ``conv_taps`` tokens,
                                                       the last tap the current token's, zeros before the start)
    t = softplus(dt + dt_bias)                        (one step size per head)
    S <- exp(-exp(A_log) t) S + (t B) x^T             y = S^T C + D x           per head
    y <- y * silu(z), divided by its root mean square over ``norm_groups`` equal parts, * norm
    out = W_o y

``W_in`` is held as two weights: the rows of z, x, B and C, and the rows of dt, whose product keeps its
float32 result.  State per sequence, zero when a slot opens: ``S`` float32 ``[n_heads, value_dim, N]``
and a ring of the last ``conv_taps`` raw inputs of the convolution (position p at ``p mod conv_taps``).
Everything that enters the recurrence after the products and the convolution is float32.  Kernels:
csrc/state_space.cu, csrc/linear_attention.cu.
"""

from __future__ import annotations

from typing import List

import torch

from .. import ops
from ..cache.sequence_cache import CacheNeed, StateSpec
from ..config.base import PartSpec, ScheduleEntry
from ..weights.loader import GAIN, MATRIX, TensorSpec
from .registry import register_part
from .runtime import Runtime, StepContext


@register_part("mixer", "state_space")
class StateSpaceMixer:
    @staticmethod
    def _sizes(spec: PartSpec):
        p = spec.params
        return (int(p["hidden_size"]), int(p["n_heads"]), int(p["value_dim"]), int(p["state"]), int(p["groups"]),
                int(p["conv_taps"]))

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> List[TensorSpec]:
        hidden, h, e, n, g, taps = cls._sizes(spec)
        t, inner, channels = spec.tensors, h * e, h * e + 2 * g * n
        return [TensorSpec(t["in"], (inner + channels + h, hidden), MATRIX),
                TensorSpec(t["conv"], (channels, taps), GAIN, init="conv_taps"),
                TensorSpec(t["conv_bias"], (channels,), GAIN, init="small_normal"),
                TensorSpec(t["dt_bias"], (h,), GAIN, init="step_bias"),
                TensorSpec(t["A_log"], (h,), GAIN, init="log_rate"),
                TensorSpec(t["D"], (h,), GAIN),
                TensorSpec(t["norm"], (inner,), GAIN),
                TensorSpec(t["o"], (hidden, inner), MATRIX)]

    def __init__(self, spec: PartSpec, runtime: Runtime):
        _, h, e, n, g, self.taps = self._sizes(spec)
        self.parts = int(spec.params["norm_groups"])
        self.eps = float(spec.params["norm_eps"])
        self.inner = h * e
        if h % g or self.inner % self.parts:
            raise ValueError(f"state_space: {h} heads in {g} groups, {self.inner} entries in {self.parts} parts")
        self.dtype = runtime.dtype
        f32 = lambda t: t.to(torch.float32).contiguous()
        w_in = runtime.tensor(spec, "in")
        wide = 2 * self.inner + 2 * g * n
        self.w_in, self.w_dt = w_in[:wide].contiguous(), w_in[wide:].contiguous()
        rate = torch.exp(runtime.tensor(spec, "A_log").to(torch.float64)).to(torch.float32).contiguous()
        self.shape = ops.StateSpace(h, e, n, g, f32(runtime.tensor(spec, "conv")), f32(runtime.tensor(spec, "conv_bias")),
                                    f32(runtime.tensor(spec, "dt_bias")), rate, f32(runtime.tensor(spec, "D")))
        self.gain = f32(runtime.tensor(spec, "norm"))
        self.w_o = runtime.tensor(spec, "o")

    def cache_need(self) -> CacheNeed:
        s = self.shape
        return (StateSpec((s.n_heads, s.vdim, s.n_state), torch.float32), StateSpec((self.taps, s.channels), self.dtype))

    def forward(self, x: torch.Tensor, ctx: StepContext, entry: ScheduleEntry) -> torch.Tensor:
        state, ring = ctx.cache.state_view(entry.cache, 0), ctx.cache.state_view(entry.cache, 1)
        proj = ops.linear(x, self.w_in, err=ctx.err)
        dt = ops.linear(x, self.w_dt, out_dtype=torch.float32, err=ctx.err, rows_alone=False)
        y = ops.state_space(proj, self.inner, dt, self.shape, state, ring, ctx.rows, ctx.cache.seq_lens)
        n = ops.gated_group_norm(y, proj, 0, self.gain, self.eps, self.parts, self.dtype)
        return ops.linear(n, self.w_o, err=ctx.err)
