"""Paged KV cache for decode: fixed-size pages handed out by a free-list allocator, a block
table per sequence, and per-sequence lengths (padding tokens are never stored).  The contiguous
cache in ``cache.py`` keeps the reference's semantics; this one feeds the decode kernels."""
from __future__ import annotations

import torch

from ..paged_sequences import PageAllocator, PagedSequences  # noqa: F401


class PagedKVCache(PagedSequences):
    def __init__(self, cfg, batch_size: int, max_tokens_per_seq: int, *, page_size: int = 64,
                 dtype=torch.bfloat16, device=None, num_pages: int | None = None):
        super().__init__(batch_size, max_tokens_per_seq, page_size=page_size, device=device, num_pages=num_pages)
        self.cfg = cfg
        G, K = cfg.num_kv_heads, cfg.head_dim
        shape = (self.num_pages, page_size, G, K)
        self.k_pages = [torch.zeros(shape, dtype=dtype, device=device) for _ in range(cfg.num_layers)]
        self.v_pages = [torch.zeros(shape, dtype=dtype, device=device) for _ in range(cfg.num_layers)]
