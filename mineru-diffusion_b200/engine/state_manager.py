"""Slots of the recurrent-state pools: one per request in flight.

The counterpart of the page allocator for state whose size does not grow with the sequence (matrix states, the last
inputs of short convolutions).  A slot is never cleared: a sequence that starts at position 0 starts from a zero state
whatever its slot holds.
"""
from __future__ import annotations

from collections import deque


class StateManager:

    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self.free: deque[int] = deque(range(num_slots))

    def can_allocate(self) -> bool:
        return bool(self.free)

    def allocate(self, seq) -> None:
        if seq.state_slot >= 0:
            raise AssertionError("sequence already holds a state slot")
        seq.state_slot = self.free.popleft()

    def deallocate(self, seq) -> None:
        if seq.state_slot >= 0:
            self.free.append(seq.state_slot)
            seq.state_slot = -1
