"""Recurrent states of live requests: what a layer that is no attention keeps per request instead of keys and values.

A request takes one slot when it is admitted and gives it back when it ends or is retracted. Per recurrent mixer the slot holds
the delta rule's state (fp32) and a ring of the convolution's inputs, by position modulo taps (``ops/delta.py``). Slots are
not cleared: a sequence's first token starts from zeros whatever its slot holds.
"""

from __future__ import annotations

import heapq

import torch


class OutOfStateSlots(RuntimeError):
    pass


class RecurrentStates:
    def __init__(self, geometry: list[tuple[int, int, int, int, int]], slots: int, dtype, device):
        """``geometry``: (heads, key width, value width, convolution channels, taps) of every recurrent mixer."""
        self.geometry, self.slots, self.dtype, self.device = [tuple(g) for g in geometry], slots, dtype, device
        self.free = list(range(slots))
        self.state: list[torch.Tensor] = []
        self.ring: list[torch.Tensor] = []
        self.allocate()

    def allocate(self):
        if self.state:
            return
        for h, d, dv, channels, taps in self.geometry:
            self.state.append(torch.zeros(self.slots, h, d, dv, dtype=torch.float32, device=self.device))
            self.ring.append(torch.zeros(self.slots, taps, channels, dtype=self.dtype, device=self.device))

    def release(self):
        self.state, self.ring = [], []

    def take(self) -> int:
        if not self.free:
            raise OutOfStateSlots(f"all {self.slots} state slots are taken")
        return heapq.heappop(self.free)

    def give(self, slot: int):
        assert 0 <= slot < self.slots and slot not in self.free, f"state slot {slot} given back twice"
        heapq.heappush(self.free, slot)

    def num_bytes(self) -> int:
        return sum(x.numel() * x.element_size() for x in self.state + self.ring)
