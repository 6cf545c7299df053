"""The Letitar decoder: fp32 residual rows, layer norms with bias, a mixer and a squared-relu
feed-forward per layer, soft-capped logits.  Inference only, on CUDA, in bf16 or fp32."""
from __future__ import annotations

import torch
from torch import nn

from ...ops import serving as S
from ..decode_graph import DecodeGraph
from ..mixers import (GatedLinearAttention, GatedLinearAttentionConfig, LatentAttention, LayerNorm, Projection,
                      SquaredReluMLP, TokenBatch)
from ..paged_sequences import HybridCache
from ..rope_scaling import RotaryTable
from .config import LayerConfig, LetitarConfig


class TokenTable(nn.Module):
    def __init__(self, num: int, dim: int, device=None, dtype=None):
        super().__init__()
        self.weight = nn.Parameter(torch.empty(num, dim, device=device, dtype=dtype))
        if self.weight.device.type != "meta":
            nn.init.normal_(self.weight)

    def forward(self, ids32):
        return S.embed_rows(ids32, self.weight)


class LetitarLayer(nn.Module):
    def __init__(self, cfg: LetitarConfig, lc: LayerConfig, index: int, rotary, device=None, dtype=None):
        super().__init__()
        kw = dict(device=device, dtype=dtype)
        self.norm1 = LayerNorm(cfg.width, cfg.norm_eps, **kw)
        if isinstance(lc.mixer, GatedLinearAttentionConfig):
            self.mixer = GatedLinearAttention(lc.mixer, cfg.width, cfg.norm_eps, **kw)
        else:
            self.mixer = LatentAttention(lc.mixer, index, cfg.width, cfg.norm_eps, rotary(lc.mixer.rot), **kw)
        self.norm2 = LayerNorm(cfg.width, cfg.norm_eps, **kw) if lc.mlp is not None else None
        self.mlp = SquaredReluMLP(lc.mlp, cfg.width, **kw) if lc.mlp is not None else None

    def forward(self, x, batch: TokenBatch, store):
        self.mixer(self.norm1(x), batch, store, x)
        if self.mlp is not None:
            self.mlp(self.norm2(x), x)


class Letitar(nn.Module):
    def __init__(self, cfg: LetitarConfig, device=None, dtype=None):
        super().__init__()
        dtype = dtype or torch.float32
        kw = dict(device=device, dtype=dtype)
        self.cfg = cfg
        tables: dict = {}
        rotary = lambda rot: tables.setdefault(rot, RotaryTable(rot))  # noqa: E731  one table per rotation
        self.embedder = TokenTable(cfg.vocab_size, cfg.width, **kw)
        self.layers = nn.ModuleList(LetitarLayer(cfg, lc, i, rotary, **kw) for i, lc in enumerate(cfg.layers))
        self.final_norm = LayerNorm(cfg.width, cfg.norm_eps, **kw)
        self.lm_head = Projection(cfg.width, cfg.vocab_size, **kw)

    @staticmethod
    def make_cache_for(cfg: LetitarConfig, batch_size: int, max_tokens_per_seq: int, *, page_size: int = 64, num_pages=None,
                       dtype=torch.bfloat16, device=None) -> HybridCache:
        return HybridCache([layer.mixer.cache_spec() for layer in cfg.layers], batch_size, max_tokens_per_seq,
                           page_size=page_size, dtype=dtype, device=device, num_pages=num_pages)

    @torch.no_grad()
    def run_layers(self, batch: TokenBatch, cache: HybridCache, after_layer=None):
        """fp32 residual rows [N, width] of the batch's tokens after the last layer."""
        x = self.embedder(batch.ids)
        for i, layer in enumerate(self.layers):
            layer(x, batch, cache.stores[i])
            if after_layer is not None:
                after_layer(i, x)
        return x

    @torch.no_grad()
    def decode_paged(self, token_ids, segment_ids, cache: HybridCache, select=None):
        """Run the new tokens of a [B, T] batch (padding anywhere) against the cache and store what the
        layers keep.  Returns normed hidden rows: of every sequence's last new token [B, D] (zeros for
        sequences without one), or, with the bool mask ``select`` [B, T], of the marked tokens in order."""
        ids, real = token_ids.cpu(), segment_ids.cpu() != 0
        tokens = [ids[b][real[b]].to(torch.int32) for b in range(cache.B)]
        new = [int(t.numel()) for t in tokens]
        cache.reserve(new)
        if max(new, default=0) == 0:
            rows = 0 if select is not None else cache.B
            return torch.zeros(rows, self.cfg.width, dtype=self.lm_head.weight.dtype, device=cache.device)
        batch = TokenBatch.build(cache, tokens)
        x = DecodeGraph.step(self, cache, batch) if batch.single else self.run_layers(batch, cache)
        cache.advance(new)
        if select is None:
            if batch.single:
                h = self.final_norm(x)
                return h if min(new) > 0 else h * torch.tensor(new, device=h.device, dtype=h.dtype)[:, None]
            out = torch.zeros(cache.B, x.shape[1], dtype=self.lm_head.weight.dtype, device=x.device)
            has = [b for b in range(cache.B) if new[b]]
            end = torch.tensor(new).cumsum(0) - 1
            out[has] = self.final_norm(x[end[has].to(x.device)])
            return out
        sel = select.cpu() & real
        if batch.single:
            rows = torch.nonzero(sel.any(-1)).reshape(-1)
        else:
            rows = torch.nonzero(sel[real]).reshape(-1)
        return self.final_norm(x[rows.to(x.device)])

    def logits(self, hidden):
        """fp32 logits of normed hidden rows."""
        y = self.lm_head(hidden.reshape(-1, hidden.shape[-1]), out_dtype=torch.float32).contiguous()
        return S.soft_cap_(y, self.cfg.logit_softcap).view(*hidden.shape[:-1], self.cfg.vocab_size)

    @torch.no_grad()
    def forward(self, token_ids, segment_ids, cache=None, num_right_pads: int = 0):
        """Normed hidden states [B, T, D] (zeros at padding) and the auxiliary loss (none)."""
        B, T = token_ids.shape
        if cache is None:
            w = self.lm_head.weight
            cache = self.make_cache_for(self.cfg, B, T, dtype=w.dtype, device=w.device)
        real = segment_ids != 0
        rows = self.decode_paged(token_ids, segment_ids, cache, select=real)
        out = torch.zeros(B, T, self.cfg.width, dtype=rows.dtype, device=rows.device)
        out[real.to(rows.device)] = rows
        return out, torch.zeros((), dtype=torch.float32, device=rows.device)
