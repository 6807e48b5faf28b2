"""Parts that add something of their own to the stream behind a layer's sublayers.

``token_rows``: what the token itself brings to this layer.  With x the stream (rounded to the activation
type), t the row's token and ``dim`` columns of a table that all layers share, starting at ``column``:

    g = gelu(W_gate x) * table[t, column : column + dim]      (the tanh form of gelu)
    y = W_proj g,     x <- x + norm(y)

The norm is a part of its own; its output is added by the kernel that also computes the next layer's norm
(the result travels as a :class:`Branch`).  In steps of few rows the gate's kernel reads the stream and what is
pending on it, so that no kernel of its own has to add that first.  Kernels: csrc/token_side.cu."""

from __future__ import annotations

from dataclasses import replace
from typing import List

import torch

from .. import ops
from ..config.base import PartSpec
from ..weights.loader import MATRIX, TensorSpec
from .registry import part_class, register_part
from .runtime import Branch, Runtime, StepContext


@register_part("side", "token_rows")
class TokenRows:
    """Parameters: ``hidden_size, vocab_size, dim, column, table_width`` and ``norm`` (a norm's spec);
    tensors ``table`` [vocab, table_width], ``gate`` [dim, hidden], ``proj`` [hidden, dim]."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> List[TensorSpec]:
        p = spec.params
        hidden, dim = int(p["hidden_size"]), int(p["dim"])
        return [TensorSpec(spec.tensors["table"], (int(p["vocab_size"]), int(p["table_width"])), MATRIX, init="unit_normal"),
                TensorSpec(spec.tensors["gate"], (dim, hidden), MATRIX), TensorSpec(spec.tensors["proj"], (hidden, dim), MATRIX),
                *part_class("norm", p["norm"].kind).tensor_specs(p["norm"])]

    def __init__(self, spec: PartSpec, runtime: Runtime):
        p = spec.params
        self.column = int(p["column"])
        if self.column < 0 or self.column + int(p["dim"]) > int(p["table_width"]):
            raise ValueError(f"token_rows: {p['dim']} columns from {self.column} of a table of {p['table_width']}")
        self.table = runtime.tensor(spec, "table")
        self.w_gate, self.w_proj = runtime.tensor(spec, "gate"), runtime.tensor(spec, "proj")
        self.norm = part_class("norm", p["norm"].kind)(p["norm"], runtime)

    def forward(self, x: torch.Tensor, ctx: StepContext) -> Branch:
        g = ops.token_gate(x, self.w_gate, self.table, ctx.tokens, self.column, err=ctx.err)
        return Branch(ops.linear(g, self.w_proj, err=ctx.err), self.norm)

    def reads_pending(self, h: torch.Tensor) -> bool:
        """Whether ``forward_pending`` serves a step of these rows."""
        return h.shape[0] <= ops.TOKEN_GATE_FUSED_ROWS and ops.token_gate_pending_supported(h, self.w_gate)

    def forward_pending(self, h: torch.Tensor, d: Branch, ctx: StepContext) -> Branch:
        """The same from the stream and the scaled outputs that are still to be added to it: they are added
        in the gate's kernel for what it reads, and to the stream itself together with this part's output."""
        g = ops.token_gate_pending(h, d.scaled, self.w_gate, self.table, ctx.tokens, self.column, err=ctx.err)
        return replace(d, tensor=ops.linear(g, self.w_proj, err=ctx.err), norm=self.norm)
