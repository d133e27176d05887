"""Slots for the state that sequences of recurrent models carry from token to token (recurrent state, the last inputs of
convolutions).  A slot belongs to one live sequence and has two halves: a step reads one half and writes the other, so
running the same step again (CUDA-graph capture does) gives the same result, and no kernel reads what another CTA of the
same launch has already replaced.  The tensors live in the model runner; this is the bookkeeping on the host.
"""
from __future__ import annotations

from typing import List, Tuple

from ..types import MemoryError_


class StateSlots:
    FRESH = -1          # read index of a sequence without history: zero state

    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self._free: List[int] = list(range(num_slots - 1, -1, -1))
        self._half = [0] * num_slots

    def allocate(self) -> int:
        if not self._free:
            raise MemoryError_(f"all {self.num_slots} state slots are in use")
        slot = self._free.pop()
        self._half[slot] = 0
        return slot

    def free(self, slot: int) -> None:
        if slot in self._free or not 0 <= slot < self.num_slots:
            raise MemoryError_(f"state slot {slot} is not in use")
        self._free.append(slot)

    def num_free(self) -> int:
        return len(self._free)

    def advance(self, slot: int, fresh: bool) -> Tuple[int, int]:
        """(half to read or FRESH, half to write) of the sequence's next step, as indices into 2 * num_slots rows."""
        cur = self._half[slot]
        self._half[slot] = cur ^ 1
        return (self.FRESH if fresh else 2 * slot + cur), 2 * slot + (cur ^ 1)
