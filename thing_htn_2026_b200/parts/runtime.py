"""What a part gets from its surroundings: at construction the precision, the device and
its tensors; at every step the rows, the cache and the error word."""

from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Dict, List, Optional, Sequence

import torch

from .. import ops
from ..config.base import PartSpec, ScheduleEntry


@dataclass
class Runtime:
    """Construction-time surroundings of a part."""

    dtype: torch.dtype
    device: torch.device
    tensors: Dict[str, torch.Tensor]
    shared: Dict[str, object] = field(default_factory=dict)   # parts built once per model, by PartSpec.key()

    def tensor(self, spec: PartSpec, name: str) -> torch.Tensor:
        return self.tensors[spec.tensors[name]]


@dataclass
class Branch:
    """A sublayer's output that has not been added to the residual stream yet, with the norm
    it passes before the add (None: it is added as it is).  Blocks hand it on in place of a bare
    tensor when the add is to be fused into the next norm.  ``second``: the output of a sublayer
    that ran beside the first on the same input, added with it; ``factor``: what multiplies
    the branch as it is added.  ``write``: over a residual stream of several copies
    (hyper-connections), the numbers (:class:`ops.StreamNumbers`) by which the sublayer that
    produced the tensor remixes the copies and adds its output to each.  ``scaled``
    (:class:`ops.ScaledPair`): outputs with a factor per entry (layer scale), added ahead of the tensor,
    which may then be None; ``add_rows``: float32 rows that are added as they are."""

    tensor: Optional[torch.Tensor]
    norm: Optional[object] = None
    second: Optional[torch.Tensor] = None
    factor: float = 1.0
    write: Optional[object] = None
    scaled: Optional[object] = None
    add_rows: Optional[torch.Tensor] = None

    @property
    def plain(self) -> bool:
        """One output of a sublayer, with or without a norm of its own, and nothing else."""
        return self.second is None and self.factor == 1.0 and self.write is None and self.scaled is None and self.add_rows is None

    def at(self, rows: torch.Tensor) -> "Branch":
        """The branch at the given rows (int32 indices)."""
        def pick(t):
            return None if t is None else ops.gather_rows(t, rows)
        return replace(self, tensor=pick(self.tensor), second=pick(self.second), add_rows=pick(self.add_rows),
                       scaled=None if self.scaled is None else self.scaled.at(rows))


@dataclass(frozen=True)
class HostBatch:
    """What the host knows of a step before it runs: for each sequence its slot, the tokens
    it brings and the tokens it already holds, in the order of the packed rows."""

    slots: Sequence[int]
    counts: Sequence[int]
    held: Sequence[int]
    page_size: int

    @property
    def row_starts(self) -> List[int]:
        starts, at = [], 0
        for c in self.counts:
            starts.append(at)
            at += c
        return starts

    @property
    def max_count(self) -> int:
        return max(self.counts) if self.counts else 0


@dataclass
class StepContext:
    """Step-time surroundings of a part.  ``rows`` says, for each packed row, which slot it
    belongs to and its position; ``cache`` holds keys, values and per-sequence state;
    ``inputs`` holds, by name, the int32 device tensors that parts asked for through
    ``step_inputs`` (they travel in the step's one upload); ``tokens`` are the step's token ids (int32,
    one per row)."""

    rows: ops.StepRows
    cache: "object"
    err: torch.Tensor
    inputs: Dict[str, torch.Tensor] = field(default_factory=dict)
    extras: Dict[str, object] = field(default_factory=dict)
    tokens: Optional[torch.Tensor] = None
