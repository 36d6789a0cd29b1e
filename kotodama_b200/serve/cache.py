"""Paged caches of the serving engine: fixed-size pages from one free list that all layers share (a page index
means the same slot in every layer).  What a page holds is the model family's business."""
from __future__ import annotations

from typing import Any, Optional, Sequence

import torch

PAGE = 16                          # tokens per page


class PagePool:
    """The free list of pages and, for families whose layers carry a state from token to token, of state slots (one per
    live sequence)."""

    def __init__(self, num_pages: int, num_states: int = 0) -> None:
        self.num_pages = num_pages
        self.free = list(range(num_pages - 1, -1, -1))
        self.num_states = num_states
        self.free_states = list(range(num_states - 1, -1, -1))

    def can_take_state(self) -> bool:
        return not self.num_states or bool(self.free_states)

    def take_state(self) -> int:
        """A state slot (-1 in families without states).  What it holds is undefined: a sequence's first pass starts from zero."""
        if not self.num_states:
            return -1
        if not self.free_states:
            raise RuntimeError("no free state slot")
        return self.free_states.pop()

    def give_state(self, slot: int) -> None:
        self.free_states.append(slot)

    def pages_for(self, tokens: int) -> int:
        return (tokens + PAGE - 1) // PAGE

    def can_allocate(self, n: int) -> bool:
        return len(self.free) >= n

    def allocate(self, n: int) -> list[int]:
        if len(self.free) < n:
            raise RuntimeError("KV cache exhausted")
        return [self.free.pop() for _ in range(n)]

    def release(self, pages: list[int]) -> None:
        self.free.extend(reversed(pages))


class PagedKVCache(PagePool):
    """Keys and values per KV head."""

    def __init__(self, cfg: Any, num_pages: int, device: torch.device, dtype: torch.dtype,
                 n_kv_local: Optional[int] = None) -> None:
        super().__init__(num_pages)
        self.n_kv = n_kv_local or cfg.num_kv_heads
        self.hd = cfg.head_dim
        shape = (cfg.num_layers, num_pages, self.n_kv, PAGE, self.hd)      # 16 rows of one (page, head) are contiguous
        self.k = torch.zeros(shape, device=device, dtype=dtype)
        self.v = torch.zeros(shape, device=device, dtype=dtype)


class PagedLatentCache(PagePool):
    """One latent row per token and layer (the layers' widths may differ): the attention reads the same row as key and as
    value.  A page is ``[width / block, 16, block]``: ``block`` columns of its 16 tokens are contiguous."""

    def __init__(self, widths: Sequence[int], blocks: Sequence[int], num_pages: int, device: torch.device, dtype: torch.dtype) -> None:
        super().__init__(num_pages)
        self.c = [torch.zeros(num_pages, w // k, PAGE, k, device=device, dtype=dtype) for w, k in zip(widths, blocks)]


class HybridCache(PagePool):
    """Per attention layer run the keys and values of every token (head sizes may differ between layers and between keys
    and values), per recurrent layer run a matrix state and the convolutions' last inputs of every state slot.  Lists are indexed
    by layer run; the entries of the other kind of layer are None."""

    def __init__(self, kv: Sequence[Optional[tuple[int, int, int]]], rec: Sequence[Optional[tuple[int, int, int, int]]], num_pages: int,
                 num_states: int, device: torch.device, dtype: torch.dtype) -> None:
        """``kv``: (kv heads, key size, value size) per run; ``rec``: (heads, key size, value size, taps)."""
        super().__init__(num_pages, num_states if any(r is not None for r in rec) else 0)
        z = lambda *s, dt=dtype: torch.zeros(s, device=device, dtype=dt)
        n = self.num_states
        self.k = [z(num_pages, c[0], PAGE, c[1]) if c else None for c in kv]
        self.v = [z(num_pages, c[0], PAGE, c[2]) if c else None for c in kv]
        self.state = [z(n, c[0], c[1], (c[2] + 3) // 4 * 4, dt=torch.float32) if c else None for c in rec]
        self.ring = [z(n, c[0], max(c[3] - 1, 1), 2 * c[1] + c[2]) if c else None for c in rec]
