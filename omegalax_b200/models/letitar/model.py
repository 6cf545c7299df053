"""The Letitar decoder: layer norms with bias, a mixer and a squared-relu feed-forward per layer, a head of
its own and soft-capped logits."""
from __future__ import annotations

import torch

from ...ops import serving as S
from ..mixers import GatedLinearAttention, GatedLinearAttentionConfig, LatentAttention, LayerNorm, Projection, SquaredReluMLP
from ..stream_decoder import DecoderLayer, StreamDecoder
from .config import LayerConfig, LetitarConfig


class Letitar(StreamDecoder):
    norm = LayerNorm

    def __init__(self, cfg: LetitarConfig, device=None, dtype=None):
        super().__init__(cfg, device, dtype)
        self.lm_head = Projection(cfg.width, cfg.vocab_size, device=device, dtype=dtype or torch.float32)

    @staticmethod
    def make_layer(cfg: LetitarConfig, lc: LayerConfig, index: int, rotary, device=None, dtype=None) -> DecoderLayer:
        kw = dict(device=device, dtype=dtype)
        norm1 = LayerNorm(cfg.width, cfg.norm_eps, **kw)
        if isinstance(lc.mixer, GatedLinearAttentionConfig):
            mixer = GatedLinearAttention(lc.mixer, cfg.width, cfg.norm_eps, **kw)
        else:
            mixer = LatentAttention(lc.mixer, index, cfg.width, cfg.norm_eps, rotary(lc.mixer.rot), **kw)
        if lc.mlp is None:
            return DecoderLayer(norm1, mixer)
        return DecoderLayer(norm1, mixer, LayerNorm(cfg.width, cfg.norm_eps, **kw), SquaredReluMLP(lc.mlp, cfg.width, **kw))

    def logits(self, hidden):
        """fp32 logits of normed hidden rows."""
        y = self.lm_head(hidden.reshape(-1, hidden.shape[-1]), out_dtype=torch.float32).contiguous()
        return S.soft_cap_(y, self.cfg.logit_softcap).view(*hidden.shape[:-1], self.cfg.vocab_size)
