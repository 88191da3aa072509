"""Paged key/value cache: fixed-size pages from one pool, a page table per lane, one table for every attention layer.

A page holds 64 consecutive positions of one lane for *all* attention layer runs (a looped layer has one run per pass), so the
page allocator (csrc/host_radix.cpp) is asked once per 64 tokens of a sequence.  Per run the pools are
``k [pages, kv_heads, 64, dim]`` and ``v [pages, kv_heads, 64, vdim]``: a head's page is one contiguous block.
"""
from __future__ import annotations

import numpy as np
import torch

from ..sched.core import Pager

PAGE = 64


class PagesExhausted(RuntimeError):
    pass


class PagedKV:
    def __init__(self, runs: list[tuple[int, int, int]], n_pages: int, lanes: int, max_context: int, dtype: torch.dtype, device):
        """``runs``: (kv_heads, dim, vdim) of every attention layer run."""
        self.lanes, self.n_pages, self.max_pages = lanes, n_pages, -(-max_context // PAGE)
        self.k = [torch.zeros((n_pages, g, PAGE, d), dtype=dtype, device=device) for g, d, _ in runs]
        self.v = [torch.zeros((n_pages, g, PAGE, v), dtype=dtype, device=device) for g, _, v in runs]
        self.pager = Pager(n_pages)
        self.pages: list[list[int]] = [[] for _ in range(lanes)]
        self.table = torch.zeros((lanes, self.max_pages), dtype=torch.int32, device=device)
        self._host = torch.zeros((lanes, self.max_pages), dtype=torch.int32)
        if torch.device(device).type == "cuda":
            self._host = self._host.pin_memory()
        self._np = self._host.numpy()
        self._dirty: set[int] = set()

    @property
    def free_pages(self) -> int:
        return self.pager.free

    def held(self, lane: int) -> int:
        return len(self.pages[lane])

    def ensure(self, lane: int, rows: int) -> None:
        """Back positions [0, rows) of a lane."""
        need, own = -(-rows // PAGE), self.pages[lane]
        if need > self.max_pages:
            raise ValueError(f"{rows} positions are beyond the context of {self.max_pages * PAGE}")
        if need - len(own) > self.pager.free:
            raise PagesExhausted(f"lane {lane} needs {need - len(own)} more pages, {self.pager.free} of {self.n_pages} are free")
        while len(own) < need:
            page = self.pager.alloc()
            self._np[lane, len(own)] = page
            own.append(page)
            self._dirty.add(lane)

    def truncate(self, lane: int, rows: int) -> None:
        """Give back the pages of a lane that hold no position below ``rows``."""
        own, keep = self.pages[lane], -(-rows // PAGE)
        while len(own) > keep:
            self.pager.release(own.pop())

    def upload(self) -> None:
        """Send the table rows that changed (the caller has made sure that the previous upload has left the host buffer)."""
        for lane in sorted(self._dirty):
            self.table[lane].copy_(self._host[lane], non_blocking=True)
        self._dirty.clear()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.k + self.v)
