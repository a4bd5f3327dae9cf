"""Per-request state of the layer-list models (hybrid.py): slots, and what every layer keeps per slot.

A request owns one slot.  Recurrent layers keep fixed-size state per slot; an attention layer keeps a ring of pages per
slot, and pages for the first tokens where those stay visible, taken from the layer's pool when the slot is acquired and given back with it.  Nothing is cleared in between: the
kernels never read a slot's old contents for a sequence that starts at position 0.
"""
from __future__ import annotations

import numpy as np

from .device import CUDA, Tensor


class PageRing:
    """One layer's paged store: T [n_pages][page][ld], and the block table int32 [slots][pages_per_slot].  Position p of a
    slot lives on page table[slot][(p / page) % pages_per_slot], so `pages_per_slot` pages serve any length as long as the
    positions that are still looked at, and the tokens of one call, span no more than they hold.  The first `pinned` pages of a
    slot are no part of the ring: they keep the sequence's first positions, table[slot][p / page], and the ring runs over the
    others, table[slot][pinned + (p / page - pinned) % (pages_per_slot - pinned)]."""

    def __init__(self, dev: CUDA, slots: int, span: int, row: int, dtype: str, page: int, pinned: int = 0):
        self.page, self.row, self.pinned = page, row, pinned
        self.pages_per_slot = pinned + (span + page - 1) // page
        self.n_pages = slots * self.pages_per_slot
        self.pool = Tensor.zeros((self.n_pages, page, row), dtype, dev)
        self._free = list(range(self.n_pages))[::-1]
        self._table = np.zeros((slots, self.pages_per_slot), np.int32)
        self.table = Tensor.zeros(self._table.shape, "int32", dev)

    def acquire(self, slot: int) -> None:
        self._table[slot] = [self._free.pop() for _ in range(self.pages_per_slot)]
        self.table.assign(self._table)

    def release(self, slot: int) -> None:
        self._free.extend(int(p) for p in self._table[slot])

    def nbytes(self) -> int:
        return self.pool.nbytes + self.table.nbytes


class SlotStates:
    """Slots of one model: which are taken, how many tokens each has seen, and the layers' stores."""

    def __init__(self, dev: CUDA, slots: int, max_context: int, max_rows: int, page: int = 64):
        self.dev, self.slots, self.max_context, self.max_rows, self.page = dev, slots, max_context, max_rows, page
        self._free = list(range(slots))[::-1]
        self.length = [0] * slots
        self.rings: list[PageRing] = []
        self.tensors: list[Tensor] = []

    # ---- stores, made by the layers at construction
    def per_slot(self, shape: tuple, dtype: str) -> Tensor:
        t = Tensor.zeros((self.slots,) + shape, dtype, self.dev)
        self.tensors.append(t)
        return t

    def ring(self, row: int, dtype: str, window: int, keep: int = 0) -> PageRing:
        """Pages for rows of `row` elements, `window` positions looked back on (0: all of them), the first `keep` ones for good."""
        span = self.max_context if window <= 0 else min(self.max_context, window - 1 + self.max_rows)
        pinned = (keep + self.page - 1) // self.page
        if pinned * self.page + span >= self.max_context:  # every position has a place of its own
            span, pinned = self.max_context, 0
        r = PageRing(self.dev, self.slots, span, row, dtype, self.page, pinned)
        self.rings.append(r)
        return r

    # ---- requests
    def acquire(self) -> int:
        if not self._free:
            raise ValueError(f"all {self.slots} slots are taken")
        slot = self._free.pop()
        self.length[slot] = 0
        for r in self.rings:
            r.acquire(slot)
        return slot

    def release(self, slot: int) -> None:
        if slot in self._free:
            raise ValueError(f"slot {slot} is not taken")
        for r in self.rings:
            r.release(slot)
        self._free.append(slot)

    def advance(self, slot: int, start_pos: int, n: int) -> None:
        """Tokens start_pos .. start_pos + n - 1 are about to be fed; state can only go on from where it is, or start anew."""
        if start_pos + n > self.max_context:
            raise ValueError(f"start_pos {start_pos} + {n} tokens exceeds max_context {self.max_context}")
        if start_pos not in (0, self.length[slot]):
            raise ValueError(f"recurrent state of slot {slot} is at position {self.length[slot]}: it cannot go on from {start_pos}")
        self.length[slot] = start_pos + n

    def nbytes(self) -> int:
        return sum(t.nbytes for t in self.tensors) + sum(r.nbytes() for r in self.rings)
