"""Letitar configuration: the layer list of a config.json, one mixer and at most one feed-forward each."""
from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from ..mixers import DenseMLPConfig, GatedLinearAttentionConfig, LatentAttentionConfig
from ..rope_scaling import RotaryConfig, YarnScaling
from ..stream_decoder import StreamDecoderConfig

ARCHITECTURE = "Letitar"
DEFAULT_DECAY_RANK = 32      # of random-initialised models; a checkpoint's tensor shape decides otherwise

MixerConfig = GatedLinearAttentionConfig | LatentAttentionConfig


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    mixer: MixerConfig
    mlp: DenseMLPConfig | None


@dataclasses.dataclass(frozen=True, kw_only=True)
class LetitarConfig(StreamDecoderConfig):
    logit_softcap: float

    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if not isinstance(m, LatentAttentionConfig):
                continue
            if m.rot.dims > m.rot_dim or m.rot.dims % 2:
                raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.rot_dim} channels")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, LatentAttentionConfig) or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {m.kv_from} is not an earlier latent-attention layer with a latent of its own")
                if (src.kv_rank, src.rot_dim, src.rot) != (m.kv_rank, m.rot_dim, m.rot):
                    raise ValueError(f"layer {i}: latent size or rotation differs from layer {m.kv_from}, whose cache it reads")


def _rotary(d: Mapping) -> RotaryConfig:
    s = d.get("scaling")
    scaling = None if s is None else YarnScaling(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"]))
    return RotaryConfig(int(d["dims"]), float(d["base"]), scaling)


def _layer(i: int, d: Mapping, shapes: Mapping[str, tuple]) -> LayerConfig:
    m, kind = d["mixer"], d["type"]
    if kind == "gla":
        rank = shapes.get(f"l{i}.mix.a1", (DEFAULT_DECAY_RANK,))[0]
        mixer = GatedLinearAttentionConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]),
                                           int(m.get("decay_rank", rank)))
    elif kind == "latent_attention":
        mixer = LatentAttentionConfig(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                      float(m["scale"]), _rotary(m["rot"]), m.get("kv_from"))
    else:
        raise ValueError(f"layer {i}: unknown mixer type '{kind}'")
    mlp = d.get("mlp")
    if mlp is not None:
        if mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind '{mlp.get('kind')}'")
        mlp = DenseMLPConfig(int(mlp["ff"]))
    return LayerConfig(mixer, mlp)


def make_config_from_hf(hf_cfg: Mapping[str, Any], shapes: Mapping[str, tuple] | None = None) -> LetitarConfig:
    """Parse a config.json dict.  ``shapes`` (tensor name -> shape of the checkpoint) gives the sizes that
    only the tensors know."""
    if hf_cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture is {hf_cfg.get('architecture')!r}")
    return LetitarConfig(
        vocab_size=int(hf_cfg["vocab"]), width=int(hf_cfg["width"]), norm_eps=float(hf_cfg["norm"]["eps"]),
        logit_softcap=float(hf_cfg["logit_softcap"]),
        layers=tuple(_layer(i, d, shapes or {}) for i, d in enumerate(hf_cfg["layers"])))


def config_to_hf(cfg: LetitarConfig) -> dict:
    """The config.json dict of ``cfg``."""
    layers = []
    for layer in cfg.layers:
        m = dataclasses.asdict(layer.mixer)
        if isinstance(layer.mixer, LatentAttentionConfig):
            kind = "latent_attention"
            m = {k: v for k, v in m.items() if not (k == "kv_from" and v is None)}
            m["rot"] = {k: v for k, v in m["rot"].items() if not (k == "scaling" and v is None)}
        else:
            kind = "gla"
            m.pop("decay_rank")
        layers.append({"type": kind, "mixer": m, "mlp": None if layer.mlp is None else {"kind": "dense", "ff": layer.mlp.ff}})
    return {"architecture": ARCHITECTURE, "vocab": cfg.vocab_size, "width": cfg.width, "norm": {"eps": cfg.norm_eps},
            "logit_softcap": cfg.logit_softcap, "layers": layers}


# ---------------------------------------------------------------------------------------------- presets
def _gla(heads, dim, vdim, tau=8.0, rank=DEFAULT_DECAY_RANK):
    return GatedLinearAttentionConfig(heads, dim, vdim, tau, rank)


def _latent(heads, dim, rot_dim, vdim, rank, kv_from=None, base=10000.0, factor=8.0, original=4096):
    return LatentAttentionConfig(heads, dim, rot_dim, vdim, rank, (dim + rot_dim) ** -0.5,
                                 RotaryConfig(rot_dim, base, YarnScaling(factor, original, 16.0, 1.0)), kv_from)


def _preset(vocab, width, ff, mixers) -> LetitarConfig:
    return LetitarConfig(vocab_size=vocab, width=width, norm_eps=1e-6, logit_softcap=25.0,
                         layers=tuple(LayerConfig(m, DenseMLPConfig(ff)) for m in mixers))


PRESETS = {
    "letitar-smoke": lambda: _preset(512, 128, 384, [_gla(2, 32, 64), _latent(4, 32, 16, 32, 64), _gla(2, 32, 64),
                                                     _latent(4, 32, 16, 32, 64, kv_from=1)]),
    # layers of production size: 4096 wide, 32 heads, as many multiply-adds in the feed-forward as a
    # gated one of width 12288
    "letitar-8layer-4096": lambda: _preset(151936, 4096, 18432, [
        _latent(32, 128, 64, 128, 512), _gla(32, 128, 128), _gla(32, 128, 128), _gla(32, 128, 128),
        _latent(32, 128, 64, 128, 512), _gla(32, 128, 128), _gla(32, 128, 128), _latent(32, 128, 64, 128, 512, kv_from=4)]),
}
