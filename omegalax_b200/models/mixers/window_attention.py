"""Grouped-query softmax attention over a sliding window, with a learned sink per head, query and key norms
taken over whole projections and values mixed with those of an earlier layer.

    q, k = rotate(rms_norm(W_q h)), rotate(rms_norm(W_k h))     (each norm over all heads at once)
    v = (1 - lambda) W_v h + lambda v_first                     (v_first: W_v h of layer ``v_from``)
    y = W_o sum_j softmax_j(q k_j scale) v_j                    (denominator + exp(sink), last ``window`` tokens)

q, k and v are rows of one projection, which the prepare kernel turns into attention operands in place
while it stores key and value.  Fresh prompts then run the tcgen05 attention kernel on the packed rows,
single tokens the split decode kernel on the pages; other portions and other types the any-size kernel.
"""
from __future__ import annotations

import dataclasses

import torch
from torch import nn

from ...ops import serving as S
from ..paged_sequences import KeyValuePages
from ..rope_scaling import RotaryConfig, RotaryTable
from .batch import TokenBatch
from .layers import Projection


@dataclasses.dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int            # query / key channels per head, the first rot.dims of them rotated
    vdim: int
    scale: float
    rot: RotaryConfig
    window: int         # tokens a query sees, itself included; 0: all
    v_from: int | None = None      # layer whose values are mixed in; its own index: it hands its values on
    sink: bool = True

    def cache_spec(self):
        return KeyValuePages(self.kv_heads, self.dim, self.vdim, self.window)


class WindowAttention(nn.Module):
    def __init__(self, cfg: WindowAttentionConfig, layer: int, width: int, eps: float, rotary: RotaryTable, device=None,
                 dtype=None):
        super().__init__()
        self.cfg, self.eps, self.rotary, self.layer = cfg, eps, rotary, layer
        kw = dict(device=device, dtype=dtype)
        c = cfg
        self.k_at, self.v_at = c.heads * c.dim, (c.heads + c.kv_heads) * c.dim
        self.in_proj = Projection(width, self.v_at + c.kv_heads * c.vdim, **kw)      # [q | k | v]
        self.qk_norm = nn.Parameter(torch.ones(self.v_at, **kw))                     # [q | k]
        self.value_mix = nn.Parameter(torch.zeros((), **kw)) if c.v_from is not None else None
        self.sink = nn.Parameter(torch.zeros(c.heads, **kw)) if c.sink else None
        self.out_proj = Projection(c.heads * c.vdim, width, **kw)

    def forward(self, h, batch: TokenBatch, store, x):
        c = self.cfg
        proj = self.in_proj(h)
        cos, sin = self.rotary.get(batch.positions, proj.device)
        v = proj[:, self.v_at:]
        mix = v_first = None
        if c.v_from == self.layer:
            batch.shared[self.layer] = v
        elif c.v_from is not None:
            mix, v_first = self.value_mix, batch.shared[c.v_from]
        S.window_prepare(proj, batch.pos, batch.row, cos, sin, c.heads, c.kv_heads, c.dim, c.vdim, self.qk_norm, store, self.eps,
                         mix=mix, v_first=v_first)
        q, sizes = proj[:, :self.k_at], (c.heads, c.kv_heads, c.dim, c.vdim, c.scale, c.window, self.sink)
        if not batch.single and batch.fresh and S.window_prompt_fits(proj.dtype, c.dim, c.vdim):
            y = S.attn_window(q, proj[:, self.k_at:], v, batch.cu, batch.max_new, *sizes)
        elif batch.single and S.window_decode_fits(proj.dtype, c.dim, c.vdim):
            y = S.window_decode(q, store, batch.seen, batch.block_table, batch.page_size, *sizes)
        else:
            y = S.window_attn_any(q, store, batch.seq, batch.seen, batch.block_table, batch.page_size, *sizes)
        self.out_proj(y, into=x)
