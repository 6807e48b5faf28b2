"""Token embedding (a row gather, engine/engine.py:1101) and the LM head
(engine/engine.py:1120; with tied weights it is the embedding table, :225-226).
Logits are float32.

The embedding takes two optional parameters: ``scale`` (the rows are multiplied by it) and
``stream`` "float32" (the rows come out in float32, scaled in float32: the start of a residual
stream that is kept in float32).  ``positions`` (a mapping ``kind: "sinusoid", base``; float32
stream only): a position vector is added to every row, ``sin(p w_i)`` at entry 2i and
``cos(p w_i)`` at entry 2i + 1 with ``w_i = base^(-2i / hidden_size)`` and p the row's position
in its sequence; the frequencies are computed in double on the host, the angles and their sines
in double on the device.  ``positions`` with ``kind: "learned", size`` (float32 stream only): the row of
the tensor ``positions`` [size, hidden] at the row's position is added, unscaled; ``position_limit`` is
then the most positions a sequence can have.  ``pairs`` (a mapping ``buckets, mul_before, mul_token``;
float32 stream only): a row of the tensor ``pairs`` [buckets + 1, hidden] is added for every pair of
neighbouring tokens, number ``(before * mul_before + token * mul_token) mod buckets``, the last row for
a sequence's first token.  The token before the first one of a step is per-sequence state
(``previous_token``, registered through ``sequence_states``).  ``norm`` (the spec of an RMS norm; float32
stream only, without a scale, positions or pairs): the token's row passes this norm as it starts the stream.
``forward_kept`` gives the start of the stream twice, for a model that adds it again later.

The head takes ``scale`` (default 1): a constant factor on the logits."""

from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..config.base import PartSpec
from ..weights.loader import MATRIX, TensorSpec
from .registry import part_class, register_part
from .runtime import Runtime


@register_part("embedding", "embedding")
class Embedding:
    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> List[TensorSpec]:
        p, width = spec.params, int(spec.params["hidden_size"])
        specs = [TensorSpec(spec.tensors["weight"], (int(p["vocab_size"]), width), MATRIX)]
        if p.get("pairs") is not None:
            specs.append(TensorSpec(spec.tensors["pairs"], (int(p["pairs"]["buckets"]) + 1, width), MATRIX))
        if p.get("positions") is not None and p["positions"].get("kind") == "learned":
            specs.append(TensorSpec(spec.tensors["positions"], (int(p["positions"]["size"]), width), MATRIX))
        if p.get("norm") is not None:
            specs += part_class("norm", p["norm"].kind).tensor_specs(p["norm"])
        return specs

    def __init__(self, spec: PartSpec, runtime: Runtime):
        self.table = runtime.tensor(spec, "weight")
        self.scale = float(spec.params.get("scale", 1.0))
        self.float32_stream = spec.params.get("stream") == "float32"
        if self.scale != 1.0 and not self.float32_stream:
            raise ValueError("embedding: a scale needs stream 'float32'")
        self.frequencies = self.positions = self.pairs = None
        self.position_limit: Optional[int] = None
        positions, pairs = spec.params.get("positions"), spec.params.get("pairs")
        if (positions is not None or pairs is not None) and not self.float32_stream:
            raise ValueError("embedding: positions and pairs need stream 'float32'")
        if positions is not None:
            if positions.get("kind") == "sinusoid":
                width = int(spec.params["hidden_size"])
                pair = torch.arange((width + 1) // 2, dtype=torch.float64)
                self.frequencies = (float(positions["base"]) ** (-2.0 * pair / width)).to(runtime.device)
            elif positions.get("kind") == "learned":
                self.positions = runtime.tensor(spec, "positions")
                self.position_limit = self.positions.shape[0]
            else:
                raise ValueError(f"embedding: positions of kind {positions.get('kind')!r} (known: 'sinusoid', 'learned')")
        if pairs is not None:
            self.pairs = ops.PairTable(runtime.tensor(spec, "pairs"), int(pairs["mul_before"]), int(pairs["mul_token"]))
        if self.pairs is not None and self.frequencies is not None:
            raise ValueError("embedding: pairs go with learned positions or none")
        self.norm = None
        if spec.params.get("norm") is not None:
            if not self.float32_stream or self.scale != 1.0 or positions is not None or pairs is not None:
                raise ValueError("embedding: a norm needs stream 'float32', and no scale, positions or pairs")
            self.norm = part_class("norm", spec.params["norm"].kind)(spec.params["norm"], runtime)

    def sequence_states(self) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        """Per-sequence state by name (shape without the slots, dtype), zeroed when a slot opens."""
        return {"previous_token": ((), torch.int32)} if self.pairs is not None else {}

    def forward(self, tokens: torch.Tensor, err: torch.Tensor, rows: Optional[ops.StepRows] = None,
                cache=None) -> torch.Tensor:
        """``rows``: the step's rows, for an embedding that adds positions or pairs; ``cache``: the
        sequences' cache, for one that adds pairs or learned positions."""
        if self.norm is not None:
            return ops.embed_norm(self.table, tokens, self.norm.as_gain, err)[0]
        if self.pairs is not None or self.positions is not None:
            if rows is None or cache is None:
                raise ValueError("embedding: pairs or learned positions are added, the step's rows and cache are needed")
            previous = cache.sequence_state("previous_token") if self.pairs is not None else None
            return ops.embed_rows(self.table, tokens, self.scale, rows, cache.seq_lens, self.pairs, previous, self.positions, err)
        if self.frequencies is not None:
            if rows is None:
                raise ValueError("embedding: positions are added, the step's rows are needed")
            return ops.gather_rows_scaled(self.table, tokens, self.scale, err, rows.row_pos, self.frequencies)
        if self.float32_stream:
            return ops.gather_rows_scaled(self.table, tokens, self.scale, err)
        return ops.gather_rows(self.table, tokens, err)


    def forward_kept(self, tokens: torch.Tensor, err: torch.Tensor, rows: Optional[ops.StepRows] = None,
                     cache=None) -> Tuple[torch.Tensor, torch.Tensor]:
        """(the float32 stream's start, the same rows once more)."""
        if not self.float32_stream:
            raise ValueError("embedding: the start of a stream can be kept where the stream is float32")
        if self.norm is not None:
            return ops.embed_norm(self.table, tokens, self.norm.as_gain, err, copy=True)
        h = self.forward(tokens, err, rows, cache)
        return h, h.clone()


@register_part("head", "lm_head")
class LMHead:
    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> List[TensorSpec]:
        copies = (spec.tensors["stored_copy"],) if "stored_copy" in spec.tensors else ()
        return [TensorSpec(spec.tensors["weight"], (int(spec.params["vocab_size"]), int(spec.params["hidden_size"])),
                           MATRIX, copies=copies)]

    def __init__(self, spec: PartSpec, runtime: Runtime):
        self.weight = runtime.tensor(spec, "weight")
        self.vocab_size = int(spec.params["vocab_size"])
        self.scale = float(spec.params.get("scale", 1.0))

    def forward(self, x: torch.Tensor, err: Optional[torch.Tensor] = None) -> torch.Tensor:
        logits = ops.linear(x, self.weight, out_dtype=torch.float32, err=err)
        return ops.scale_(logits, self.scale) if self.scale != 1.0 else logits
