"""Latent attention: keys and values are expanded from one low-rank latent per token, next to a rotated
key part that all heads share; only the two are cached.

Prompts expand keys and values and run the tcgen05 attention kernel on [unrotated | rotated] heads.
Decoding moves the expansion to the query side (q W_uk, W_uv o) and attends to the cached latents
directly.  A layer with ``kv_from`` has no latent of its own and reads that layer's rows.
"""
from __future__ import annotations

import dataclasses

import torch
from torch import nn

from ...ops import serving as S
from ..paged_sequences import LatentPages, SharedWith
from ..rope_scaling import RotaryConfig, RotaryTable
from .batch import TokenBatch
from .layers import Projection


@dataclasses.dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int            # unrotated query / key channels per head
    rot_dim: int        # rotated ones
    vdim: int
    kv_rank: int
    scale: float
    rot: RotaryConfig
    kv_from: int | None = None

    def cache_spec(self):
        return LatentPages(self.kv_rank, self.rot_dim) if self.kv_from is None else SharedWith(self.kv_from)


class LatentAttention(nn.Module):
    def __init__(self, cfg: LatentAttentionConfig, layer: int, width: int, eps: float, rotary: RotaryTable, device=None,
                 dtype=None):
        super().__init__()
        self.cfg, self.eps, self.rotary, self.layer = cfg, eps, rotary, layer
        kw = dict(device=device, dtype=dtype)
        self.q_rows = cfg.heads * (cfg.dim + cfg.rot_dim)
        own = cfg.kv_from is None
        self.in_proj = Projection(width, self.q_rows + (cfg.kv_rank + cfg.rot_dim if own else 0), **kw)   # [q | latent | rotated key]
        if own:
            self.latent_norm = nn.Parameter(torch.ones(cfg.kv_rank, **kw))
        self.kv_proj = Projection(cfg.kv_rank, cfg.heads * (cfg.dim + cfg.vdim), **kw)                    # [W_uk | W_uv]
        self.out_proj = Projection(cfg.heads * cfg.vdim, width, **kw)

    def forward(self, h, batch: TokenBatch, store, x):
        c = self.cfg
        proj = self.in_proj(h)
        N, H, hd, uk_rows = proj.shape[0], c.heads, c.dim + c.rot_dim, c.heads * c.dim
        expand = not batch.single and batch.fresh and S.two_part_fits(proj.dtype, c.dim, c.rot_dim, c.vdim, c.kv_rank)
        cos, sin = self.rotary.get(batch.positions, proj.device)
        if c.kv_from is None:
            packed = None
            if expand:
                packed = torch.empty(N, store.shape[1], dtype=proj.dtype, device=proj.device)
                batch.shared[self.layer] = packed
            S.latent_prepare(proj, batch.pos, batch.row, cos, sin, H, c.dim, c.rot_dim, c.kv_rank, dkv_off=self.q_rows,
                             norm_w=self.latent_norm, cache=store, eps=self.eps, packed=packed)
        else:
            S.latent_prepare(proj, batch.pos, batch.row, cos, sin, H, c.dim, c.rot_dim, c.kv_rank)
        w = self.kv_proj.weight
        if expand:
            packed = batch.shared.get(self.layer if c.kv_from is None else c.kv_from)
            if packed is None:      # the owner's head sizes kept it off this path: read the rows back from its pages
                packed = store.index_select(0, batch.row.long())
            kv = S.project(packed[:, :c.kv_rank], w)
            y = S.attn_two_part(proj, kv, packed[:, c.kv_rank:], kv[:, uk_rows:], batch.cu, batch.max_new, H, c.dim, c.rot_dim,
                                c.vdim, c.scale)
        else:
            q = proj[:, :self.q_rows]
            if batch.single and S.latent_decode_fits(proj.dtype, c.dim, c.rot_dim, c.kv_rank):
                q_lat = S.latent_absorb(q, hd, w[:uk_rows], H, c.dim, c.kv_rank, torch.bfloat16)
                o = S.latent_decode(q_lat, q, hd, c.dim, c.rot_dim, store, batch.seen, batch.block_table, batch.page_size, c.scale)
            else:
                q_lat = S.latent_absorb(q, hd, w[:uk_rows], H, c.dim, c.kv_rank, torch.float32)
                o = S.latent_attn_any(q_lat, q, hd, c.dim, c.rot_dim, store, batch.seq, batch.seen, batch.block_table,
                                      batch.page_size, c.scale)
            y = S.latent_expand(o, w[uk_rows:], c.vdim)
        self.out_proj(y, into=x)
