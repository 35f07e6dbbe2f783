"""Device pools of models whose layers differ in what they cache.

A model lists its caching modules (``cache_owners``); each says what it needs (``cache_needs``) as
``(kind, attribute, row shape)`` entries: ``"paged"`` rows, one per token in the blocks of the scheduler's block
pool ``[num_blocks, block_size, *row]`` in the compute dtype, and ``"slot"`` rows, one fp32 row per live sequence
``[num_slots, *row]``.  All paged pools share the block ids and all slot pools the slot ids, so a sequence has one
block table and one slot whatever its layers look like.
"""
from __future__ import annotations

import math

import torch


class LayeredCache:
    def __init__(self, model, block_size: int, dtype: torch.dtype, device):
        self.block_size, self.dtype, self.device = block_size, dtype, device
        self.needs = [(owner, kind, attr, tuple(row)) for owner in model.cache_owners()
                      for kind, attr, row in owner.cache_needs()]
        for _, kind, attr, _ in self.needs:
            if kind not in ("paged", "slot"):
                raise ValueError(f"unknown cache kind {kind!r} for {attr}")
        self.buffers: list[torch.Tensor] = []

    def block_bytes(self) -> int:
        """Bytes of one KV block over all layers."""
        return sum(math.prod(row) for _, kind, _, row in self.needs if kind == "paged") * self.block_size * self.dtype.itemsize

    def slot_bytes(self) -> int:
        return sum(math.prod(row) for _, kind, _, row in self.needs if kind == "slot") * 4

    def allocate(self, num_blocks: int, num_slots: int) -> None:
        """One tensor per pool, injected into the module that asked for it."""
        for owner, kind, attr, row in self.needs:
            if kind == "paged":
                t = torch.zeros(num_blocks, self.block_size, *row, dtype=self.dtype, device=self.device)
            else:
                t = torch.zeros(num_slots, *row, dtype=torch.float32, device=self.device)
            setattr(owner, attr, t)
            self.buffers.append(t)
