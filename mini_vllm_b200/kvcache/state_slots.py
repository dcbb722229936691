"""Slots of per-sequence recurrent state: a request holds one from admission until it finishes or is preempted.

A slot is an index into the state buffers of every recurrent layer.  It is handed out uncleared - a sequence starts from
zero at position 0 - and the lowest free slot goes first, so a freed slot is used again at once."""
from __future__ import annotations

import heapq


class StateSlots:
    def __init__(self, capacity: int):
        self.capacity = capacity
        self._free = list(range(capacity))

    @property
    def num_free(self) -> int:
        return len(self._free)

    def take(self) -> int:
        if not self._free:
            raise RuntimeError("no free state slot")
        return heapq.heappop(self._free)

    def give(self, slot: int) -> None:
        assert 0 <= slot < self.capacity and slot not in self._free
        heapq.heappush(self._free, slot)
