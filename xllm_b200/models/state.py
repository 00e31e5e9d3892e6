"""Per-sequence recurrent state: slot bookkeeping and a pool for layers of differing state shapes.

The scheduler admits at most `n_slots` sequences at a time and slots return on finish, preemption and abort, so
`slot_of` finds a free slot whenever it needs one (the reference's LinearState block manager,
xllm/core/framework/block/)."""
from __future__ import annotations

import math
from typing import Dict, Tuple, Union

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
    """States of any set of layers, by layer: (heads, key size, value size) is one fp32 matrix state per head, the value
    size stored rounded up to four; a dict {name: (shape, dtype)} is a state of several named parts, of which a part with
    dtype None is such a matrix state.  One more slot than `n_slots` exists: `scratch_slot`, for passes outside the scheduler.
    Slots are not cleared: a layer ignores what a slot holds when a sequence starts at position 0."""

    def __init__(self, shapes: Dict[int, Union[Tuple[int, int, int], dict]], n_slots: int, device):
        super().__init__(n_slots)
        self.scratch_slot = n_slots

        def make(part):
            shape, dtype = self._stored(part)
            return torch.zeros(n_slots + 1, *shape, dtype=dtype, device=device)

        self.layers = {i: {n: make(p) for n, p in s.items()} if isinstance(s, dict) else make((s, None))
                       for i, s in shapes.items()}

    @staticmethod
    def _stored(part):
        shape, dtype = part
        if dtype is not None:
            return tuple(shape), dtype
        h, dk, dv = shape
        return (h, dk, (dv + 3) // 4 * 4), torch.float32

    @staticmethod
    def bytes_per_slot(shapes) -> int:
        parts = [p for s in shapes.values() for p in (s.values() if isinstance(s, dict) else [(s, None)])]
        return sum(math.prod(shape) * dtype.itemsize for shape, dtype in map(RecurrentStatePool._stored, parts))
