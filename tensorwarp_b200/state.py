"""What a sequence leaves behind between steps, for every run of a layer: keys and values and the previous token's mixer
input, latents, or a recurrent state.

The state of `slots` sequences is allocated once; a sequence holds one slot from ``open`` to ``close``.
Nothing has to be cleared when a slot changes hands: a query sees only positions its own sequence has
written, and the kernels take the state (recurrent or shifted) before position 0 as zero.
"""
from __future__ import annotations

from typing import Dict, List

import torch


class StateError(RuntimeError):
    """No free slot, an unknown sequence, or a sequence longer than its slot."""


class SequenceState:
    def __init__(self, model, slots: int, capacity: int):
        """model: dense.DenseModel; capacity: tokens per slot."""
        from .dense import AttentionSpec, LatentAttentionSpec, pad16
        if slots < 1 or capacity < 1:
            raise ValueError("slots and capacity must be positive")
        self.slots, self.capacity = slots, capacity
        dt, dev = model.dtype, model.device
        f32 = torch.float32
        self.runs: List[Dict[str, torch.Tensor]] = []       # by the name of the native layer's field

        def zeros(*shape, dtype=dt):
            return torch.zeros((slots,) + shape, dtype=dtype, device=dev)

        for i, _ in model.runs:
            m, run = model.spec.layers[i].mixer, {}
            if isinstance(m, AttentionSpec):
                run["k_cache"] = zeros(capacity, m.kv_heads * pad16(m.dim))
                run["v_cache"] = zeros(capacity, m.kv_heads * pad16(m.vdim))
                if model.layers[i].get("shift") is not None:
                    # two rows, used in turn by the parity of the position: a step reads one while it writes the other
                    run["shift_state"] = zeros(2, model.width_pad, dtype=f32)
            elif isinstance(m, LatentAttentionSpec):
                run["latent_cache"] = zeros(capacity, pad16(m.rank) + pad16(m.rot_dim))
            else:
                run["gla_state"] = zeros(m.heads, pad16(m.dim), pad16(m.vdim), dtype=f32)
            self.runs.append(run)
        self.k, self.v, self.shift = ([run.get(name) for run in self.runs] for name in ("k_cache", "v_cache", "shift_state"))
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
        return sum(t.numel() * t.element_size() for run in self.runs for t in run.values())
