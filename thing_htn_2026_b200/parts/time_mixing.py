"""Time mixing (RWKV): a recurrent token mixer whose projections read blends of a token and the one
before it.  With ``x'`` the mixer's input at the previous token (zeros for the first), every one of
the five inputs s in (r, k, v, g, w) is ``x_s = x + (x' - x) * mu_s``, and

    r, k, v = W_r x_r, W_k x_k, W_v x_v               (``n_heads`` heads of ``dim``)
    w       = exp(-exp(W_w2 tanh(W_w1 x_w) + w0))     (a decay per head and key channel)
    o       = (S + diag(u) k v^T)^T r                 (the bonus u counts for the current token only)
    S      <- diag(w) S + k v^T
    out     = W_o (concat_h(o_h / sqrt(mean(o_h^2) + eps)) * norm * silu(W_g x_g))

``rank`` (the channels between W_w1 and W_w2; None: the shapes of the checkpoint's two tensors give
it).  The four wide products are one batched product over the blends; the decay's first product keeps
its float32 result.  State per sequence, zero when a slot opens: ``S`` float32 ``[n_heads, dim (value),
dim (key)]`` and the last input row ``[hidden]`` in the activation type.  Single-token steps run one
kernel between the first products and the last.  Everything that enters the recurrence after the
products is float32.  Kernels: csrc/wkv.cu, csrc/linear_attention.cu.
"""

from __future__ import annotations

from typing import List

import torch

from .. import ops
from ..cache.sequence_cache import CacheNeed, StateSpec
from ..config.base import PartSpec, ScheduleEntry
from ..weights.loader import GAIN, MATRIX, TensorSpec
from .linear_attention import pad_rank
from .registry import register_part
from .runtime import Runtime, StepContext

WIDE = ("r", "k", "v", "g")            # the order of the batched product
BLENDS = WIDE + ("w",)


@register_part("mixer", "time_mixing")
class TimeMixing:
    @staticmethod
    def _sizes(spec: PartSpec):
        p = spec.params
        return int(p["hidden_size"]), int(p["n_heads"]), int(p["dim"])

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> List[TensorSpec]:
        hidden, h, d = cls._sizes(spec)
        rank, t = spec.params.get("rank"), spec.tensors
        r = -1 if rank is None else int(rank)
        specs = [TensorSpec(t[f"mu_{s}"], (hidden,), GAIN, init="unit_interval") for s in BLENDS]
        specs += [TensorSpec(t[s], (h * d, hidden), MATRIX) for s in WIDE]
        specs += [TensorSpec(t["w1"], (r, hidden), MATRIX), TensorSpec(t["w2"], (h * d, r), MATRIX),
                  TensorSpec(t["w0"], (h * d,), GAIN, init="log_decay"), TensorSpec(t["u"], (h, d), GAIN, init="unit_normal"),
                  TensorSpec(t["norm"], (h * d,), GAIN), TensorSpec(t["o"], (hidden, h * d), MATRIX)]
        return specs

    def __init__(self, spec: PartSpec, runtime: Runtime):
        self.hidden, self.n_heads, self.dim = self._sizes(spec)
        self.dtype = runtime.dtype
        self.eps = float(spec.params["norm_eps"])
        f32 = lambda t: t.to(torch.float32).contiguous()
        if runtime.tensor(spec, "w1").shape[0] != runtime.tensor(spec, "w2").shape[1]:
            raise ValueError("time_mixing: the two projections of the decay do not meet in one rank")
        self.mu = torch.stack([f32(runtime.tensor(spec, f"mu_{s}")) for s in BLENDS]).contiguous()
        self.w_wide = torch.stack([runtime.tensor(spec, s) for s in WIDE]).contiguous()
        self.w1, self.w2 = pad_rank(runtime.tensor(spec, "w1"), runtime.tensor(spec, "w2"))
        self.w0, self.u = f32(runtime.tensor(spec, "w0")), f32(runtime.tensor(spec, "u"))
        self.gain = f32(runtime.tensor(spec, "norm"))
        self.w_o = runtime.tensor(spec, "o")

    def cache_need(self) -> CacheNeed:
        return (StateSpec((self.n_heads, self.dim, self.dim), torch.float32), StateSpec((self.hidden,), self.dtype))

    def forward(self, x: torch.Tensor, ctx: StepContext, entry: ScheduleEntry) -> torch.Tensor:
        state, shift = ctx.cache.state_view(entry.cache, 0), ctx.cache.state_view(entry.cache, 1)
        blends = ops.token_shift(x, self.mu, shift, ctx.rows, ctx.cache.seq_lens)
        planes = ops.linear_batched(blends[:len(WIDE)], self.w_wide)
        low = ops.linear(blends[len(WIDE)], self.w1, out_dtype=torch.float32, err=ctx.err, rows_alone=False)
        if ctx.rows.max_q_len == 1:
            y = ops.wkv_decode(planes, low, self.w2, self.w0, self.u, self.gain, self.eps, state, ctx.rows, self.n_heads, self.dim)
        else:
            z = ops.linear(ops.tanh_rows(low, self.dtype), self.w2, out_dtype=torch.float32, err=ctx.err)
            o = ops.wkv(planes, z, self.w0, self.u, state, ctx.rows, self.n_heads, self.dim)
            y = ops.gated_head_norm(o, planes[WIDE.index("g")], 0, self.gain, self.eps, self.n_heads, self.dim, self.dtype)
        return ops.linear(y, self.w_o, err=ctx.err)
