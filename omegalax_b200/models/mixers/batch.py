"""What one call of a serving decoder processes, as device tensors."""
from __future__ import annotations

import dataclasses

import torch


@dataclasses.dataclass
class TokenBatch:
    """N rows.  Prompts: the new tokens of all sequences, packed.  ``single``: row b is sequence b's one
    new token (id and position -1 where it has none), N = batch size, so the shapes are those of the
    cache and a recorded step can be replayed."""
    ids: torch.Tensor           # int32 [N]
    pos: torch.Tensor           # int32 [N] position in the sequence
    row: torch.Tensor           # int32 [N] cache row the token goes to
    seq: torch.Tensor           # int32 [N] sequence of the token
    seen: torch.Tensor          # int32 [N] tokens of the sequence visible to this one (pos + 1, 0 if idle)
    cu: torch.Tensor            # int32 [B+1] packed rows of the sequences
    history: torch.Tensor       # int32 [B] tokens cached before the call
    block_table: torch.Tensor   # int32 [B, max_blocks]
    page_size: int
    max_new: int                # longest run of new tokens
    single: bool
    fresh: bool                 # every sequence with new tokens starts here
    positions: int              # bound on positions, for the rotary tables
    flat: torch.Tensor          # the buffer the tensors above are slices of
    shared: dict = dataclasses.field(default_factory=dict)   # layer -> rows of this call that later layers read

    @staticmethod
    def build(cache, tokens: list) -> "TokenBatch":
        """``tokens[b]``: 1-D int32 CPU tensor of sequence b's new tokens (possibly empty).  Pages must
        be reserved.  One host -> device copy."""
        B, lens = cache.B, cache.seq_lens_host
        n = [int(t.numel()) for t in tokens]
        single = max(n) == 1
        i32 = torch.int32
        if single:
            ids = torch.tensor([int(t[0]) if k else -1 for t, k in zip(tokens, n)], dtype=i32)
            pos = torch.tensor([lens[b] if n[b] else -1 for b in range(B)], dtype=i32)
            row = torch.tensor([cache.flat_row_host(b, lens[b]) if n[b] else -1 for b in range(B)], dtype=i32)
            seq = torch.arange(B, dtype=i32)
            cu = torch.arange(B + 1, dtype=i32)
        else:
            ids = torch.cat([t.to(i32) for t in tokens])
            pos = torch.cat([torch.arange(lens[b], lens[b] + n[b], dtype=i32) for b in range(B)])
            row = torch.cat([cache.flat_rows_host(b, lens[b], n[b]) for b in range(B)])
            seq = torch.repeat_interleave(torch.arange(B, dtype=i32), torch.tensor(n))
            cu = torch.tensor([0] + n, dtype=i32).cumsum(0).to(i32)
        hist = torch.tensor(lens, dtype=i32)
        parts = [ids, pos, row, seq, pos + 1, cu, hist]
        # every part starts on a 16-byte boundary of the one buffer that travels
        padded = [torch.cat([p, p.new_zeros(-p.numel() % 4)]) for p in parts]
        flat = torch.cat(padded).to(cache.device)
        out, at = [], 0
        for p, q in zip(parts, padded):
            out.append(flat[at:at + p.numel()])
            at += q.numel()
        fresh = all(lens[b] == 0 for b in range(B) if n[b])
        return TokenBatch(*out, block_table=cache.block_table, page_size=cache.page_size, max_new=max(n), single=single,
                          fresh=fresh, positions=cache.capacity, flat=flat)
