"""Gated linear attention with a decay per key channel.

    q = W_q h dim^-1/2,  k = W_k h,  v = W_v h,  alpha = sigmoid(W_a2 W_a1 h + b)^(1/tau)
    S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t
    y = W_o (rms_norm(o) * w * silu(W_g h))        (norm over each head's value channels)

q, k, v, g and the low-rank half of the decay are rows of one projection.  The recurrence runs in
fp32 with its state in the cache; a single-token step is one fused kernel after the projections.
"""
from __future__ import annotations

import dataclasses

import torch
from torch import nn

from ...ops import serving as S
from ..paged_sequences import RecurrentState
from .batch import TokenBatch
from .layers import Projection


@dataclasses.dataclass(frozen=True)
class GatedLinearAttentionConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int

    def cache_spec(self):
        return RecurrentState(self.heads, self.dim, self.vdim)


class GatedLinearAttention(nn.Module):
    def __init__(self, cfg: GatedLinearAttentionConfig, width: int, eps: float, device=None, dtype=None):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        kw = dict(device=device, dtype=dtype)
        self.qk, self.vg = cfg.heads * cfg.dim, cfg.heads * cfg.vdim
        self.in_proj = Projection(width, 2 * self.qk + 2 * self.vg + cfg.decay_rank, **kw)    # [q | k | v | g | a1]
        self.decay_proj = Projection(cfg.decay_rank, self.qk, **kw)
        self.decay_bias = nn.Parameter(torch.zeros(self.qk, **kw))
        self.norm_weight = nn.Parameter(torch.ones(cfg.vdim, **kw))
        self.out_proj = Projection(self.vg, width, **kw)

    def forward(self, h, batch: TokenBatch, store, x):
        c = self.cfg
        proj = self.in_proj(h)
        z = self.decay_proj(proj[:, 2 * (self.qk + self.vg):], out_dtype=torch.float32).contiguous()
        scale = c.dim ** -0.5
        if batch.single:
            y = S.gla_step(proj, z, self.decay_bias, self.norm_weight, store, batch.seen, c.heads, c.dim, c.vdim, scale,
                           c.tau, self.eps)
        else:
            o = S.gla_scan(proj, S.gla_decay_(z, self.decay_bias, c.tau), store, batch.cu, batch.history, c.heads, c.dim,
                           c.vdim, scale)
            y = S.gla_norm_gate(o, proj[:, 2 * self.qk + self.vg:2 * (self.qk + self.vg)], self.norm_weight, self.eps)
        self.out_proj(y, into=x)
