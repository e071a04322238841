"""Recurrent states of live requests: what a layer that is no attention keeps per request instead of keys and values.

A request takes one slot when it is admitted and gives it back when it ends or is retracted. Per recurrent mixer the slot holds
a state (fp32) and, where the mixer has them, a ring of the convolution's inputs, by position modulo taps, and a normaliser with its
running maximum (``ops/delta.py``, ``ops/linear_scan.py``). Slots are not cleared: a sequence's first token starts from zeros whatever its slot holds.
"""

from __future__ import annotations

import heapq
from typing import NamedTuple

import torch

from slime_b200.ops.linear_scan import SlotState


class OutOfStateSlots(RuntimeError):
    pass


class StateShape(NamedTuple):
    """A recurrent mixer: heads, widths of a key and a value, channels and taps of its convolution (0: none), and whether it keeps a
    normaliser."""

    heads: int
    dim: int
    vdim: int
    channels: int = 0
    taps: int = 0
    normalised: bool = False


class RecurrentStates:
    def __init__(self, geometry: list[StateShape | tuple], slots: int, dtype, device):
        """``geometry``: ``StateShape`` of every recurrent mixer."""
        self.geometry, self.slots, self.dtype, self.device = [StateShape(*g) for g in geometry], slots, dtype, device
        self.free = list(range(slots))
        self.of: list[SlotState] = []
        self.allocate()

    def allocate(self):
        if self.of:
            return
        f32 = lambda *s: torch.zeros(self.slots, *s, dtype=torch.float32, device=self.device)  # noqa: E731
        for g in self.geometry:
            ring = torch.zeros(self.slots, g.taps, g.channels, dtype=self.dtype, device=self.device) if g.taps else None
            self.of.append(SlotState(f32(g.heads, g.dim, g.vdim), ring, f32(g.heads, g.dim) if g.normalised else None,
                                     f32(g.heads, 2) if g.normalised else None))  # fmt: skip

    @property
    def state(self) -> list[torch.Tensor]:
        return [s.state for s in self.of]

    @property
    def ring(self) -> list[torch.Tensor | None]:
        return [s.ring for s in self.of]

    def release(self):
        self.of = []

    def take(self) -> int:
        if not self.free:
            raise OutOfStateSlots(f"all {self.slots} state slots are taken")
        return heapq.heappop(self.free)

    def give(self, slot: int):
        assert 0 <= slot < self.slots and slot not in self.free, f"state slot {slot} given back twice"
        heapq.heappush(self.free, slot)

    def num_bytes(self) -> int:
        return sum(x.numel() * x.element_size() for s in self.of for x in (s.state, s.ring, s.norm, s.top) if x is not None)
