"""Slots, pages and the device page table of a paged cache, shared by every model's cache.

Pages, reference counts and slot leases live in the host runtime's allocator (csrc/core/kvalloc.cc); this class only
mirrors each slot's page list into the device page table.  A page covers `page_tokens` token positions of every pool.
"""
from __future__ import annotations

from typing import List, Optional

import torch

I32 = torch.int32


class PagedSlots:
    def _init_pages(self, slots: int, max_ctx: int, device, page_tokens: int, n_pages: Optional[int]):
        self.slots, self.max_ctx, self.page_tokens = slots, max_ctx, page_tokens
        self.max_pages = (max_ctx + page_tokens - 1) // page_tokens
        self.n_pages = n_pages if n_pages is not None else self.max_pages * slots
        self.page_table_host = torch.full((slots, self.max_pages), -1, dtype=I32)
        self.page_table = self.page_table_host.to(device)
        from ..runtime import core as K
        self.alloc = K.KvAllocator(self.n_pages, slots, page_tokens)

    @property
    def free_pages(self) -> int:
        return self.alloc.free_pages

    def pages_of(self, slot: int) -> List[int]:
        return self.alloc.pages(slot)

    def admit(self):
        """Lease a free slot -> (slot, generation), or None when every slot is taken."""
        return self.alloc.admit()

    def _gen(self, slot: int) -> int:
        """Generation of the slot's lease; a slot used without admit() (single-request drivers) is leased here."""
        g = self.alloc.generation(slot)
        if g == 0:
            g = self.alloc.admit_slot(slot)
            assert g is not None
        return g

    def _publish(self, slot: int, first: int = 0):
        pages = self.alloc.pages(slot)
        n = len(pages)
        if n > first:
            self.page_table_host[slot, first:n] = torch.tensor(pages[first:], dtype=I32)
            self.page_table[slot, first:n].copy_(self.page_table_host[slot, first:n], non_blocking=True)

    def ensure(self, slot: int, n_tokens: int) -> bool:
        """Make sure `slot` has pages for positions [0, n_tokens).  Returns False when the pool is exhausted."""
        need = (n_tokens + self.page_tokens - 1) // self.page_tokens
        if need > self.max_pages:
            return False
        gen = self._gen(slot)
        have = self.alloc.page_count(slot)
        if need <= have:
            return True
        try:
            self.alloc.ensure(slot, gen, n_tokens)
        except MemoryError:
            return False
        self._publish(slot, have)
        return True

    def release(self, slot: int):
        g = self.alloc.generation(slot)
        if g:
            self.alloc.retire(slot, g)
        self.page_table_host[slot].fill_(-1)
        self.page_table[slot].fill_(-1)

    def drop_snapshot(self, snap):
        if snap.pages:
            self.alloc.release_pages(snap.pages)
        snap.pages = []
