"""Who holds which page and which row: the host-side allocator behind the engine.

A request owns one row of the page table (its ``table_idx``, also the row of its recurrent state) and the pages its
row names.  When every attention layer has a window, pages that have fallen behind the widest one are given back while
the request goes on; their entries in the page table are never read again.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

PAGE_SIZE = 16


class OutOfPages(RuntimeError):
    pass


class CacheManager:
    def __init__(self, num_pages: int, num_slots: int, max_len: int, window: Optional[int], device, spare_page: Optional[int] = None,
                 pages_needed: bool = True):
        """``window``: keys behind a token that may still be read (None: all; 0: no layer reads any).  ``spare_page``
        fills the extra last row of the page table, which padding requests use."""
        self.num_pages, self.num_slots, self.max_len, self.window = num_pages, num_slots, max_len, window
        self.needs_pages = pages_needed
        self._free_pages: List[int] = list(range(num_pages - 1, -1, -1))
        self._free_slots: List[int] = list(range(num_slots - 1, -1, -1))
        self._pages: Dict[int, Dict[int, int]] = {}              # slot -> page index in the sequence -> page id
        self._first: Dict[int, int] = {}                         # slot -> first page index not yet given back
        pitch = max(1, -(-max_len // PAGE_SIZE))
        self._host = torch.zeros((num_slots + 1, pitch), dtype=torch.int32)
        if spare_page is not None:
            self._host[num_slots] = spare_page
        self.page_table = self._host.to(device)
        self._dirty: set = set()

    @property
    def free_slots(self) -> int:
        return len(self._free_slots)

    @property
    def free_pages(self) -> int:
        return len(self._free_pages)

    def pages_for(self, tokens: int, portion: int) -> int:
        """Most pages a request of ``tokens`` tokens holds at once when it is fed at most ``portion`` at a time."""
        if not self.needs_pages:
            return 0
        live = tokens if self.window is None else min(tokens, self.window + portion + PAGE_SIZE)
        return -(-live // PAGE_SIZE) + (0 if self.window is None or live == tokens else 1)

    def allocate(self) -> int:
        if not self._free_slots:
            raise OutOfPages("no free request slot")
        slot = self._free_slots.pop()
        self._pages[slot] = {}
        self._first[slot] = 0
        return slot

    def extend(self, slot: int, start: int, end: int) -> None:
        """Pages for positions [start, end); all or nothing."""
        if end > self.max_len:
            raise ValueError(f"{end} tokens exceed the engine's max_len {self.max_len}")
        if not self.needs_pages or end <= start:
            return
        have = self._pages[slot]
        missing = [i for i in range(start // PAGE_SIZE, (end - 1) // PAGE_SIZE + 1) if i not in have]
        if len(missing) > len(self._free_pages):
            raise OutOfPages(f"{len(missing)} pages needed, {len(self._free_pages)} free")
        for i in missing:
            have[i] = self._free_pages.pop()
            self._host[slot, i] = have[i]
        if missing:
            self._dirty.add(slot)

    def trim(self, slot: int, length: int) -> None:
        """Gives back the pages that no token at position ``length`` or later can see."""
        if self.window is None:
            return
        first = max(0, length - self.window + 1) // PAGE_SIZE if self.window else length // PAGE_SIZE
        have = self._pages[slot]
        for i in range(self._first[slot], first):
            if i in have:
                self._free_pages.append(have.pop(i))
        self._first[slot] = max(first, self._first[slot])

    def free(self, slot: int) -> None:
        self._free_pages.extend(self._pages.pop(slot).values())
        self._free_slots.append(slot)
        self._dirty.discard(slot)

    def locations(self, slots: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """Cache rows (page * 16 + offset) of positions (host tensors)."""
        return self._host[slots, positions // PAGE_SIZE] * PAGE_SIZE + positions % PAGE_SIZE

    def sync(self) -> None:
        """Brings the device's page table up to date (one small copy)."""
        if not self._dirty:
            return
        rows = sorted(self._dirty)
        self._dirty.clear()
        src = self._host[rows]
        if self.page_table.is_cuda:
            src = src.pin_memory().to(self.page_table.device, non_blocking=True)
        self.page_table[torch.tensor(rows, device=self.page_table.device)] = src
