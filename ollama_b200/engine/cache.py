"""Paged cache and recurrent state of the sequences in a number of slots.

Keys and values live in pages of 64 positions taken from one pool: a slot owns the pages that cover its tokens and a table row says
where each block of 64 positions is.  The pool is shared by all layer runs (a page has a place in every run's storage), so that its
size is counted in tokens, not in sequences.  Recurrent layers keep a fixed-size state per slot.
"""
from __future__ import annotations

import numpy as np
import torch

PAGE = 64


class CacheFull(RuntimeError):
    """The pool has no page left for the tokens asked for."""


class PagedCache:
    def __init__(self, n_slots: int, n_ctx: int, pool_tokens: int | None = None, device="cuda"):
        """``n_ctx``: most tokens of one sequence; ``pool_tokens``: tokens the pool holds in all (default: every slot full)."""
        self.n_slots, self.n_ctx, self.device = n_slots, n_ctx, device
        self.max_pages = max(1, -(-n_ctx // PAGE))
        self.n_pages = max(1, -(-pool_tokens // PAGE) if pool_tokens is not None else n_slots * self.max_pages)
        self.free = list(range(self.n_pages - 1, -1, -1))
        self.owned: list[list[int]] = [[] for _ in range(n_slots)]
        self.table_np = np.zeros((n_slots, self.max_pages), np.int32)      # entries without a page hold 0: a valid index, never read unmasked
        self.table = torch.zeros(n_slots, self.max_pages, device=device, dtype=torch.int32)
        self._dirty = False
        self.paged: list[torch.Tensor] = []        # [n_pages, ...]
        self.states: list[torch.Tensor] = []       # [n_slots, ...]

    # -- storage --------------------------------------------------------------------------------------
    def add_pages(self, kv_heads: int, dim: int, dtype) -> torch.Tensor:
        """Storage of one layer run's keys or values: [page, kv head, position in the page, dim]."""
        t = torch.zeros(self.n_pages, kv_heads, PAGE, dim, device=self.device, dtype=dtype)
        self.paged.append(t)
        return t

    def add_state(self, *shape: int) -> torch.Tensor:
        t = torch.zeros(self.n_slots, *shape, device=self.device, dtype=torch.float32)
        self.states.append(t)
        return t

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.paged + self.states)

    # -- bookkeeping ----------------------------------------------------------------------------------
    def reserve(self, slot: int, n_tokens: int) -> None:
        """Give ``slot`` pages for positions 0 .. n_tokens - 1 (pages it has stay where they are)."""
        own, need = self.owned[slot], -(-n_tokens // PAGE)
        if need > self.max_pages:
            raise CacheFull(f"{n_tokens} tokens in a slot of {self.n_ctx}")
        if need - len(own) > len(self.free):
            raise CacheFull(f"{need - len(own)} pages wanted, {len(self.free)} free")
        while len(own) < need:
            page = self.free.pop()
            self.table_np[slot, len(own)] = page
            own.append(page)
            self._dirty = True

    def release(self, slot: int) -> None:
        """Give back what ``slot`` holds.  Its state needs no clearing: a sequence at position 0 does not read it."""
        if self.owned[slot]:
            self.free += reversed(self.owned[slot])
            self.owned[slot] = []
            self.table_np[slot] = 0
            self._dirty = True

    def sync(self) -> int:
        """Bring the device's page table up to date; returns the bytes copied."""
        if not self._dirty:
            return 0
        self._dirty = False
        self.table.copy_(torch.from_numpy(self.table_np))
        return self.table_np.nbytes

    def copy(self, src: int, dst: int, n_tokens: int) -> None:
        """Positions 0 .. n_tokens - 1 and the state of slot ``src`` become those of slot ``dst``."""
        self.reserve(dst, n_tokens)
        n = -(-n_tokens // PAGE)
        if n:
            a = torch.tensor(self.owned[src][:n], device=self.device)
            b = torch.tensor(self.owned[dst][:n], device=self.device)
            for t in self.paged:
                t[b] = t[a]
        for t in self.states:
            t[dst].copy_(t[src])
