"""The Difedra decoder: RMS norms, windowed attention and a gated feed-forward or routed experts per layer,
logits of the embedding table."""
from __future__ import annotations

from ..mixers import GatedMLP, GatedMLPConfig, MixtureOfExperts, RMSNorm, WindowAttention
from ..stream_decoder import DecoderLayer, StreamDecoder
from .config import DifedraConfig, LayerConfig


class Difedra(StreamDecoder):
    norm = RMSNorm

    @staticmethod
    def make_layer(cfg: DifedraConfig, lc: LayerConfig, index: int, rotary, device=None, dtype=None) -> DecoderLayer:
        kw = dict(device=device, dtype=dtype)
        norm1 = RMSNorm(cfg.width, cfg.norm_eps, **kw)
        mixer = WindowAttention(lc.mixer, index, cfg.width, cfg.norm_eps, rotary(lc.mixer.rot), **kw)
        if lc.mlp is None:
            return DecoderLayer(norm1, mixer)
        mlp = (GatedMLP if isinstance(lc.mlp, GatedMLPConfig) else MixtureOfExperts)(lc.mlp, cfg.width, **kw)
        return DecoderLayer(norm1, mixer, RMSNorm(cfg.width, cfg.norm_eps, **kw), mlp)
