"""Difedra configuration: the layer list of a config.json, windowed attention and at most one feed-forward
(dense, or routed experts) each."""
from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from ..mixers import GatedMLPConfig, MixtureOfExpertsConfig, WindowAttentionConfig
from ..rope_scaling import RotaryConfig, WavelengthScaling
from ..stream_decoder import StreamDecoderConfig

ARCHITECTURE = "Difedra"
DENSE_ACT, EXPERT_ACT = "gelu_tanh", "silu"


@dataclasses.dataclass(frozen=True)
class LayerConfig:
    mixer: WindowAttentionConfig
    mlp: GatedMLPConfig | MixtureOfExpertsConfig | None


@dataclasses.dataclass(frozen=True, kw_only=True)
class DifedraConfig(StreamDecoderConfig):
    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} query heads do not share {m.kv_heads} key/value heads evenly")
            if m.rot.dims > m.dim or m.rot.dims % 2:
                raise ValueError(f"layer {i}: cannot rotate {m.rot.dims} of {m.dim} channels")
            if m.window < 1:
                raise ValueError(f"layer {i}: a window of {m.window} tokens")
            if m.v_from is not None and m.v_from != i:
                src = self.layers[m.v_from].mixer if 0 <= m.v_from < i else None
                if src is None or src.v_from != m.v_from or (src.kv_heads, src.vdim) != (m.kv_heads, m.vdim):
                    raise ValueError(f"layer {i}: its values cannot be mixed with those of layer {m.v_from}")


def _rotary(d: Mapping) -> RotaryConfig:
    s = d.get("scaling")
    scaling = None if s is None else WavelengthScaling(float(s["factor"]), float(s["original"]), float(s["low"]), float(s["high"]))
    return RotaryConfig(int(d["dims"]), float(d["base"]), scaling)


def _layer(i: int, d: Mapping, first_mix: int | None) -> LayerConfig:
    m, mlp = d["mixer"], d.get("mlp")
    if d["type"] != "attention":
        raise ValueError(f"layer {i}: unknown mixer type '{d['type']}'")
    mixer = WindowAttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                  _rotary(m["rot"]), int(m["mask"]["size"]), first_mix if m.get("v_mix") else None)
    if mlp is not None:
        if mlp.get("kind") == "dense":
            mlp = GatedMLPConfig(int(mlp["ff"]), DENSE_ACT)
        elif mlp.get("kind") == "moe":
            mlp = MixtureOfExpertsConfig(int(mlp["router"]["experts"]), int(mlp["router"]["top"]),
                                         GatedMLPConfig(int(mlp["expert"]["ff"]), EXPERT_ACT))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind '{mlp.get('kind')}'")
    return LayerConfig(mixer, mlp)


def make_config_from_hf(hf_cfg: Mapping[str, Any], shapes: Mapping[str, tuple] | None = None) -> DifedraConfig:
    """Parse a config.json dict, which gives every size."""
    if hf_cfg.get("architecture") != ARCHITECTURE:
        raise ValueError(f"not a {ARCHITECTURE} config: architecture is {hf_cfg.get('architecture')!r}")
    layers = hf_cfg["layers"]
    first_mix = next((i for i, d in enumerate(layers) if d["mixer"].get("v_mix")), None)
    return DifedraConfig(vocab_size=int(hf_cfg["vocab"]), width=int(hf_cfg["width"]), norm_eps=float(hf_cfg["norm"]["eps"]),
                         layers=tuple(_layer(i, d, first_mix) for i, d in enumerate(layers)))


def config_to_hf(cfg: DifedraConfig) -> dict:
    """The config.json dict of ``cfg``."""
    layers = []
    for layer in cfg.layers:
        m = layer.mixer
        rot = {k: v for k, v in dataclasses.asdict(m.rot).items() if not (k == "scaling" and v is None)}
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot,
                 "mask": {"size": m.window}, "v_mix": m.v_from is not None}
        mlp = layer.mlp
        if isinstance(mlp, GatedMLPConfig):
            mlp = {"kind": "dense", "ff": mlp.ff}
        elif mlp is not None:
            mlp = {"kind": "moe", "router": {"experts": mlp.experts, "top": mlp.top}, "expert": {"ff": mlp.expert.ff}}
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "vocab": cfg.vocab_size, "width": cfg.width, "norm": {"eps": cfg.norm_eps},
            "layers": layers}


# ---------------------------------------------------------------------------------------------- presets
def _preset(vocab, width, heads, kv_heads, dim, vdim, window, mlps, rot=None) -> DifedraConfig:
    rot = RotaryConfig(dim, 500000.0, WavelengthScaling(8.0, 8192, 1.0, 4.0)) if rot is None else rot
    mixer = WindowAttentionConfig(heads, kv_heads, dim, vdim, dim ** -0.5, rot, window, 0)
    return DifedraConfig(vocab_size=vocab, width=width, norm_eps=1e-6, layers=tuple(LayerConfig(mixer, m) for m in mlps))


def _dense(ff):
    return GatedMLPConfig(ff, DENSE_ACT)


def _moe(experts, top, ff):
    return MixtureOfExpertsConfig(experts, top, GatedMLPConfig(ff, EXPERT_ACT))


PRESETS = {
    "difedra-smoke": lambda: _preset(512, 128, 4, 2, 32, 48, 24, [_dense(384), _moe(8, 2, 64), _moe(8, 2, 64)],
                                     RotaryConfig(16, 10000.0, WavelengthScaling(4.0, 256, 1.0, 4.0))),
    # layers of production size: 2048 wide, 32 heads over 4, 8 of 128 experts of 768
    "difedra-8layer-2048": lambda: _preset(151936, 2048, 32, 4, 128, 128, 4096, [_dense(6144)] + [_moe(128, 8, 768)] * 7),
}
