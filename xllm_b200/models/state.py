"""Per-sequence recurrent state: slot bookkeeping and a pool for layers of differing state shapes.

The scheduler admits at most `n_slots` sequences at a time and slots return on finish, preemption and abort, so
`slot_of` finds a free slot whenever it needs one (the reference's LinearState block manager,
xllm/core/framework/block/)."""
from __future__ import annotations

from typing import Dict, Tuple

import torch


class StateSlots:
    """Slot numbers owned by the running sequences (keyed by the scheduler's sequence id: parallel samples of one
    request have their own state)."""

    def __init__(self, n_slots: int):
        self.free = list(range(n_slots - 1, -1, -1))
        self.owner = {}
        self.n_slots = n_slots

    def slot_of(self, seq_id) -> int:
        s = self.owner.get(seq_id)
        if s is None:
            if not self.free:
                raise RuntimeError("no free state slot: the scheduler admitted more sequences than the pool holds")
            s = self.owner[seq_id] = self.free.pop()
        return s

    def release(self, seq_id):
        s = self.owner.pop(seq_id, None)
        if s is not None:
            self.free.append(s)


class RecurrentStatePool(StateSlots):
    """fp32 matrix states of any set of layers: `shapes[layer] = (heads, key size, value size)`; the value size is
    stored rounded up to four.  One more slot than `n_slots` exists: `scratch_slot`, for passes outside the scheduler.
    Slots are not cleared: a layer ignores what a slot holds when a sequence starts at position 0."""

    def __init__(self, shapes: Dict[int, Tuple[int, int, int]], n_slots: int, device):
        super().__init__(n_slots)
        self.scratch_slot = n_slots
        self.layers = {i: torch.zeros(n_slots + 1, h, dk, (dv + 3) // 4 * 4, dtype=torch.float32, device=device)
                       for i, (h, dk, dv) in shapes.items()}

    @staticmethod
    def bytes_per_slot(shapes) -> int:
        return sum(h * dk * ((dv + 3) // 4 * 4) * 4 for h, dk, dv in shapes.values())
