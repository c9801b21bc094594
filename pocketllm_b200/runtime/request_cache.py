"""Pages and slots of a batch of requests.

A request that is admitted gets one slot (its row of every recurrent state and of the page table) and, as its tokens come,
pages of `page` positions from a shared pool; both go back when it ends and are handed out again. The manager is host code:
the layers own the device memory ([pages, page, row] per paged layer, [slots, ...] per recurrent state) and index it with
what this class hands out. Nothing is cleared on reuse: a state is started from zero by position 0 of its new owner, a
page row is written before any query may see its position.
"""
from __future__ import annotations

import numpy as np


class CacheFull(RuntimeError):
    """No slot, or not enough pages, for what was asked; nothing was changed."""


class RequestCache:
    def __init__(self, max_requests: int, pages: int, page: int = 64, device: str | None = "cuda"):
        if max_requests < 1 or pages < 1:
            raise ValueError("at least one slot and one page")
        self.page, self.pages, self.max_requests = page, pages, max_requests
        self._free_pages = list(range(pages - 1, -1, -1))
        self._free_slots = list(range(max_requests - 1, -1, -1))
        self.table = np.zeros((max_requests, pages), dtype=np.int32)     # page of every `page` positions of a slot
        self._slot: dict[object, int] = {}
        self._held: dict[object, list[int]] = {}
        self.length: dict[object, int] = {}                             # tokens already run
        self._dirty: set[int] = set()
        self.device_table = None
        if device is not None:
            import torch
            self.device_table = torch.zeros(max_requests, pages, dtype=torch.int32, device=device)

    def __contains__(self, rid) -> bool:
        return rid in self._slot

    @property
    def live(self) -> list:
        return list(self._slot)

    @property
    def free_pages(self) -> int:
        return len(self._free_pages)

    @property
    def free_slots(self) -> int:
        return len(self._free_slots)

    def slot(self, rid) -> int:
        return self._slot[rid]

    def pages_for(self, tokens: int) -> int:
        return (tokens + self.page - 1) // self.page

    def missing_pages(self, rid, tokens: int) -> int:
        """Pages that request `rid` (known or not) lacks for `tokens` positions."""
        return max(0, self.pages_for(tokens) - len(self._held.get(rid, ())))

    def reserve(self, wanted: dict) -> None:
        """Room for `wanted` = {request: total positions}, admitting unknown requests; all or nothing."""
        new = [r for r in wanted if r not in self._slot]
        need = sum(self.missing_pages(r, n) for r, n in wanted.items())
        if len(new) > len(self._free_slots):
            raise CacheFull(f"{len(new)} new requests but {len(self._free_slots)} free slots")
        if need > len(self._free_pages):
            raise CacheFull(f"{need} pages needed but {len(self._free_pages)} free")
        for r, n in wanted.items():
            if r not in self._slot:
                self._slot[r] = self._free_slots.pop()
                self._held[r], self.length[r] = [], 0
            for _ in range(self.missing_pages(r, n)):
                pg = self._free_pages.pop()
                self.table[self._slot[r], len(self._held[r])] = pg
                self._held[r].append(pg)
                self._dirty.add(self._slot[r])

    def advance(self, rid, tokens: int) -> None:
        self.length[rid] += tokens

    def release(self, rid) -> None:
        self._free_pages.extend(reversed(self._held.pop(rid)))
        self._free_slots.append(self._slot.pop(rid))
        del self.length[rid]

    def sync(self) -> None:
        """Bring changed rows of the page table to the device."""
        if not self._dirty or self.device_table is None:
            self._dirty.clear()
            return
        import torch
        for s in self._dirty:
            self.device_table[s].copy_(torch.from_numpy(self.table[s]))
        self._dirty.clear()
