"""What a sequence leaves behind between steps: per-layer keys and values and the previous token's mixer input.

The state of `slots` sequences is allocated once; a sequence holds one slot from ``open`` to ``close``.
Nothing has to be cleared when a slot changes hands: a query sees only positions its own sequence has
written, and the kernels take the state before position 0 as zero.
"""
from __future__ import annotations

from typing import List, Optional

import torch


class StateError(RuntimeError):
    """No free slot, an unknown sequence, or a sequence longer than its slot."""


class SequenceState:
    def __init__(self, model, slots: int, capacity: int):
        """model: dense.DenseModel; capacity: tokens per slot."""
        from .dense import pad16
        if slots < 1 or capacity < 1:
            raise ValueError("slots and capacity must be positive")
        self.slots, self.capacity = slots, capacity
        dt, dev = model.dtype, model.device
        self.k: List[torch.Tensor] = []
        self.v: List[torch.Tensor] = []
        self.shift: List[Optional[torch.Tensor]] = []
        for spec, w in zip(model.spec.layers, model.layers):
            m = spec.mixer
            self.k.append(torch.zeros((slots, capacity, m.kv_heads * pad16(m.dim)), dtype=dt, device=dev))
            self.v.append(torch.zeros((slots, capacity, m.kv_heads * pad16(m.vdim)), dtype=dt, device=dev))
            # two rows, used in turn by the parity of the position: a step reads one while it writes the other
            self.shift.append(torch.zeros((slots, 2, model.width_pad), dtype=torch.float32, device=dev)
                              if w.get("shift") is not None else None)
        self._free = list(range(slots - 1, -1, -1))
        self._length = {}

    def open(self) -> int:
        if not self._free:
            raise StateError(f"all {self.slots} slots are taken")
        slot = self._free.pop()
        self._length[slot] = 0
        return slot

    def close(self, slot: int) -> None:
        if slot not in self._length:
            raise StateError(f"slot {slot} is not open")
        del self._length[slot]
        self._free.append(slot)

    @property
    def free_slots(self) -> int:
        return len(self._free)

    def length(self, slot: int) -> int:
        if slot not in self._length:
            raise StateError(f"slot {slot} is not open")
        return self._length[slot]

    def advance(self, slot: int, tokens: int) -> None:
        n = self.length(slot) + tokens
        if n > self.capacity:
            raise StateError(f"sequence of {n} tokens in a slot of {self.capacity}")
        self._length[slot] = n

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.k + self.v + [s for s in self.shift if s is not None])
