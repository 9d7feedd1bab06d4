"""Page ownership shared by the KV pools of all model families.

A *page* is ``page_size`` consecutive token positions of one sequence; requests and the prefix tree hold references on
it, and it returns to the free list with the last one.  Families whose layers have sliding windows keep the window rows
in a second pool with its own lifetime (:class:`minisgl.kvcache.pool.DSV4KVPool`); the window operations of this base
class do nothing, so that the cache manager and the prefix tree treat both kinds alike.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List

import torch


@dataclass
class PoolSizes:
    num_pages: int
    num_swa_slots: int
    num_req_slots: int
    page_size: int


class PagedPool:
    """The last page id and the last table slot are reserved for the dummy request that pads CUDA-graph batches."""

    has_window = False        # some layers keep their rows in window slots with a lifetime of their own
    prefix_align = 1          # a prefix hit resumes at a multiple of lcm(this, page size) tokens
    prefix_reusable = True    # everything a later request needs to resume behind a cached page belongs to the page

    def __init__(self, sizes: PoolSizes, device):
        self.sizes, self.device = sizes, torch.device(device)
        self.page_size = sizes.page_size
        P, R = sizes.num_pages + 1, sizes.num_req_slots + 1
        self.dummy_page, self.dummy_slot = P - 1, R - 1
        self.free_pages: List[int] = list(range(sizes.num_pages - 1, -1, -1))
        self.page_ref = [0] * P
        self.counters = {"pages_taken": 0, "pages_released": 0}

    # ------------------------------------------------------------------ pages
    @property
    def num_free_pages(self) -> int:
        return len(self.free_pages)

    def alloc_pages(self, n: int, with_swa: bool = True) -> List[int]:
        if n > len(self.free_pages) or (with_swa and n > self.num_free_swa):
            raise RuntimeError(f"KV pool exhausted: want {n} pages, free {len(self.free_pages)} pages / "
                               f"{self.num_free_swa} SWA slots")
        pages = [self.free_pages.pop() for _ in range(n)]
        for p in pages:
            assert self.page_ref[p] == 0, f"page {p} handed out while referenced"
            self.page_ref[p] = 1
        self.counters["pages_taken"] += n
        if with_swa:
            self.attach_swa(pages)
        return pages

    def ref_pages(self, pages) -> None:
        for p in pages:
            assert self.page_ref[p] > 0, f"page {p} referenced while free"
            self.page_ref[p] += 1

    def unref_pages(self, pages) -> None:
        """Drops one reference; a page whose count reaches zero returns to the free list with its SWA slot."""
        freed = []
        for p in pages:
            assert self.page_ref[p] > 0, f"double free of page {p}"
            self.page_ref[p] -= 1
            if self.page_ref[p] == 0:
                freed.append(p)
        if freed:
            self._on_freed(freed)
            self.free_pages.extend(freed)
            self.counters["pages_released"] += len(freed)

    def _on_freed(self, pages: List[int]) -> None:
        pass

    # ------------------------------------------------------------------ window storage (none here)
    @property
    def num_free_swa(self) -> int:
        return self.num_free_pages

    def attach_swa(self, pages) -> None:
        pass

    def pin_swa(self, pages, owner: str = "req") -> None:
        pass

    def unpin_swa(self, pages, owner: str = "req") -> None:
        pass

    def drop_tree_pins(self, n_slots: int) -> int:
        return 0

    def has_swa(self, page: int) -> bool:
        return True

    def assert_no_leak(self) -> None:
        assert len(self.free_pages) == self.sizes.num_pages, (len(self.free_pages), self.sizes.num_pages)
        assert all(r == 0 for r in self.page_ref[:-1])
