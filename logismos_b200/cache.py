"""Host-side managers of what live sequences hold: blocks of the paged cache and per-sequence state slots.
The scheduler (serving.py), the trace replay and direct callers of the executors share them."""
from __future__ import annotations

from typing import Dict, List

import numpy as np

BLOCK = 16  # tokens per block of the paged cache


def blocks_for(n_tokens: int) -> int:
    return -(-n_tokens // BLOCK)


class BlockAllocator:
    """Hands out cache blocks of 16 tokens from a fixed pool; one table row per sequence. ``seed`` None
    hands them out in order, else in a seeded random order."""

    def __init__(self, n_pool_blocks: int, max_blocks_per_seq: int, seed=0):
        if seed is None:
            self.free: List[int] = list(range(n_pool_blocks - 1, -1, -1))
        else:
            self.free = np.random.default_rng(seed).permutation(n_pool_blocks).tolist()
        self.max_blocks = max_blocks_per_seq
        self.tables: Dict[object, List[int]] = {}
        self._rows: Dict[object, np.ndarray] = {}

    def ensure(self, seq_id, n_tokens: int) -> np.ndarray:
        """The table row of a sequence, grown to hold n_tokens (-1 beyond its blocks)."""
        need = blocks_for(n_tokens)
        if need > self.max_blocks:
            raise ValueError("sequence exceeds max_blocks_per_seq")
        t = self.tables.get(seq_id, [])
        if need - len(t) > len(self.free):
            raise MemoryError("KV pool exhausted")
        if seq_id not in self.tables:
            self.tables[seq_id], self._rows[seq_id] = t, np.full(self.max_blocks, -1, np.int32)
        while len(t) < need:
            self._rows[seq_id][len(t)] = self.free[-1]
            t.append(self.free.pop())
        return self.row(seq_id)

    def row(self, seq_id) -> np.ndarray:
        return self._rows[seq_id].copy()

    def release(self, seq_id):
        self.free.extend(reversed(self.tables.pop(seq_id, [])))
        self._rows.pop(seq_id, None)


class SlotAllocator:
    """Per-sequence state slots: one per live sequence."""

    def __init__(self, n_slots: int):
        self.free: List[int] = list(range(n_slots - 1, -1, -1))
        self.slots: Dict[object, int] = {}

    def get(self, seq_id) -> int:
        if seq_id not in self.slots:
            if not self.free:
                raise MemoryError("state slots exhausted")
            self.slots[seq_id] = self.free.pop()
        return self.slots[seq_id]

    def release(self, seq_id):
        s = self.slots.pop(seq_id, None)
        if s is not None:
            self.free.append(s)
