"""Per-sequence recurrent state beside the paged KV cache: one slot per running sequence (the batcher's slot index).

A layer's state is a set of fp32 tensors [slots, ...]. Slots are never cleared: the kernels start a sequence whose rows
begin at position 0 from zero state, so a slot that changes hands needs no work on the host. A preempted sequence is
recomputed from position 0 in whatever slot it gets next.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch


class RecurrentState:
    """State tensors of one layer, by name."""

    def __init__(self, slots: int, shapes: Dict[str, Tuple[int, ...]], device):
        self.slots = int(slots)
        self.t = {name: torch.zeros((self.slots,) + tuple(shape), dtype=torch.float32, device=device)
                  for name, shape in shapes.items()}

    def __getitem__(self, name: str) -> torch.Tensor:
        return self.t[name]

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * 4 for t in self.t.values())


class PagedWithState:
    """Cache of a layer that has both: paged K / V and a recurrent state (attention behind a short convolution)."""

    def __init__(self, pages: torch.Tensor, state: RecurrentState):
        self.pages, self.state = pages, state

    @property
    def nbytes(self) -> int:
        return self.pages.numel() * self.pages.element_size() + self.state.nbytes
