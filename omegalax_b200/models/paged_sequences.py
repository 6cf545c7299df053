"""Page bookkeeping shared by the decode caches: a free list of fixed-size pages, a block table and a
length per sequence.  What a page holds (keys and values, latents) is the subclass's business.

``HybridCache`` is the cache of decoders whose layers differ: pages of latents or of keys and values for
attention layers, one fp32 state per sequence for recurrent layers, and layers that read another layer's
pages.  When every paged layer looks back over a window only, pages that have left the widest window
return to the allocator while the sequence goes on.
"""
from __future__ import annotations

import dataclasses

import torch


class PageAllocator:
    """Host-side free list of physical pages."""

    def __init__(self, num_pages: int):
        self.free = list(range(num_pages - 1, -1, -1))
        self.num_pages = num_pages

    def alloc(self) -> int:
        if not self.free:
            raise RuntimeError("paged KV cache is out of pages")
        return self.free.pop()

    def release(self, pages) -> None:
        self.free.extend(int(p) for p in pages)


class PagedSequences:
    """``batch_size`` sequences over ``num_pages`` pages of ``page_size`` tokens."""

    def __init__(self, batch_size: int, max_tokens_per_seq: int, *, page_size: int = 64, device=None,
                 num_pages: int | None = None):
        self.B, self.page_size, self.device = batch_size, page_size, device
        self.max_blocks = -(-max_tokens_per_seq // page_size)
        self.num_pages = num_pages or batch_size * self.max_blocks
        self.allocator = PageAllocator(self.num_pages)
        self.block_table_host = torch.full((batch_size, self.max_blocks), -1, dtype=torch.int32)
        self.block_table = torch.zeros(batch_size, self.max_blocks, dtype=torch.int32, device=device)
        self.blocks_held = [0] * batch_size
        self.blocks_dropped = [0] * batch_size      # leading blocks given back by drop_before
        self.seq_lens_host = [0] * batch_size
        self.seq_lens = torch.zeros(batch_size, dtype=torch.int32, device=device)

    @property
    def capacity(self) -> int:
        """Most tokens one sequence can hold."""
        return self.max_blocks * self.page_size

    def reserve(self, new_tokens: list[int]) -> None:
        """Make sure every sequence has pages for ``new_tokens[b]`` more tokens."""
        changed = False
        for b, n in enumerate(new_tokens):
            need = -(-(self.seq_lens_host[b] + n) // self.page_size)
            if need > self.max_blocks:
                raise RuntimeError(f"sequence {b} exceeds the cache capacity of {self.capacity} tokens")
            for j in range(self.blocks_held[b], need):
                self.block_table_host[b, j] = self.allocator.alloc()
                self.blocks_held[b] = j + 1
                changed = True
        if changed:
            self.block_table.copy_(self.block_table_host.clamp_min(0))

    def advance(self, new_tokens: list[int]) -> None:
        for b, n in enumerate(new_tokens):
            self.seq_lens_host[b] += n
        self.seq_lens.copy_(torch.tensor(self.seq_lens_host, dtype=torch.int32))

    def drop_before(self, b: int, slot: int) -> None:
        """Give back the pages of sequence b whose slots all lie before ``slot`` and are read no more."""
        first = min(max(slot, 0) // self.page_size, self.blocks_held[b])
        if first > self.blocks_dropped[b]:
            gone = slice(self.blocks_dropped[b], first)
            self.allocator.release(self.block_table_host[b, gone].tolist())
            self.block_table_host[b, gone] = -1
            self.blocks_dropped[b] = first

    def free_sequence(self, b: int) -> None:
        pages = self.block_table_host[b][self.block_table_host[b] >= 0].tolist()
        self.allocator.release(pages)
        self.block_table_host[b] = -1
        self.blocks_held[b] = 0
        self.blocks_dropped[b] = 0
        self.seq_lens_host[b] = 0
        self.seq_lens.copy_(torch.tensor(self.seq_lens_host, dtype=torch.int32))

    def flat_rows(self, seq_of_token, slot_of_token):
        """Row index into pages.view(num_pages * page_size, ...) of (sequence, slot) pairs (device tensors)."""
        blk = self.block_table[seq_of_token.long(), (slot_of_token // self.page_size).long()].long()
        return blk * self.page_size + (slot_of_token % self.page_size).long()

    def flat_row_host(self, b: int, slot: int) -> int:
        return int(self.block_table_host[b, slot // self.page_size]) * self.page_size + slot % self.page_size

    def flat_rows_host(self, b: int, start: int, n: int) -> torch.Tensor:
        """int32 rows of slots [start, start + n) of sequence b."""
        slots = torch.arange(start, start + n, dtype=torch.int32)
        return self.block_table_host[b][(slots // self.page_size).long()] * self.page_size + slots % self.page_size


@dataclasses.dataclass(frozen=True)
class LatentPages:
    """Paged rows of [latent | rotated key part]."""
    rank: int
    rot: int

    @property
    def pitch(self) -> int:      # rows start on 16-byte boundaries in both dtypes
        return -(-(self.rank + self.rot) // 8) * 8


@dataclasses.dataclass(frozen=True)
class KeyValuePages:
    """Paged rows of [value | key] per key/value head, of which a query reads the last ``window`` (0: all)."""
    kv_heads: int
    dim: int
    vdim: int
    window: int = 0

    @property
    def pitch(self) -> int:
        return -(-self.kv_heads * (self.dim + self.vdim) // 8) * 8


@dataclasses.dataclass(frozen=True)
class RecurrentState:
    """One fp32 state [heads, key_dim, value_dim] per sequence."""
    heads: int
    key_dim: int
    value_dim: int


@dataclasses.dataclass(frozen=True)
class SharedWith:
    """The layer reads what layer ``layer`` stores."""
    layer: int


class HybridCache(PagedSequences):
    """``specs[i]`` says what layer i keeps; ``stores[i]`` is the tensor: [num_pages * page_size, pitch]
    for latents or keys and values, [batch, heads, K, V] fp32 for states.  A sequence without tokens starts from a zero
    state whatever its slot held before, so freeing a sequence clears nothing."""

    def __init__(self, specs, batch_size: int, max_tokens_per_seq: int, *, page_size: int = 64, dtype=torch.bfloat16,
                 device=None, num_pages: int | None = None):
        super().__init__(batch_size, max_tokens_per_seq, page_size=page_size, device=device, num_pages=num_pages)
        self.dtype = dtype
        self.stores: list[torch.Tensor] = []
        for i, s in enumerate(specs):
            if isinstance(s, (LatentPages, KeyValuePages)):
                self.stores.append(torch.zeros(self.num_pages * page_size, s.pitch, dtype=dtype, device=device))
            elif isinstance(s, RecurrentState):
                self.stores.append(torch.zeros(batch_size, s.heads, s.key_dim, s.value_dim, dtype=torch.float32, device=device))
            elif isinstance(s, SharedWith):
                if not 0 <= s.layer < i or not isinstance(specs[s.layer], LatentPages):
                    raise ValueError(f"layer {i} cannot share the cache of layer {s.layer}")
                self.stores.append(self.stores[s.layer])
            else:
                raise TypeError(f"layer {i}: unknown cache spec {s!r}")
        windows = [getattr(s, "window", 0) for s in specs if not isinstance(s, RecurrentState)]
        self.horizon = max(windows) if windows and min(windows) > 0 else 0      # 0: every cached token may be read
        self.decode_graph = None     # recorded single-token step (see decode_graph.py)

    def advance(self, new_tokens: list[int]) -> None:
        super().advance(new_tokens)
        if self.horizon:
            for b, n in enumerate(new_tokens):
                if n:
                    self.drop_before(b, self.seq_lens_host[b] + 1 - self.horizon)
