"""Paged caches of the serving engine: fixed-size pages from one free list that all layers share (a page index
means the same slot in every layer).  What a page holds is the model family's business."""
from __future__ import annotations

from typing import Any, Optional, Sequence

import torch

PAGE = 16                          # tokens per page


class PagePool:
    """The free list."""

    def __init__(self, num_pages: int) -> None:
        self.num_pages = num_pages
        self.free = list(range(num_pages - 1, -1, -1))

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
