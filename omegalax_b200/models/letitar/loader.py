"""Load a Letitar checkpoint (config.json + model.safetensors)."""
from __future__ import annotations

import torch

from ..mixers import GatedLinearAttentionConfig
from ..params_utils import Rule, StateAssembler, native_state, rows, stream_safetensors
from .config import LetitarConfig, make_config
from .model import Letitar


def _fused(i: int, target: str, parts) -> list[Rule]:
    """Rules for checkpoint tensors that are consecutive row ranges of one parameter."""
    out, at = [], 0
    for name, n in parts:
        out.append(Rule(rf"l{i}\.mix\.{name}", lambda m, t=target: t, lambda m, lo=at, hi=at + n: rows(lo, hi)))
        at += n
    return out


def key_rules(cfg: LetitarConfig) -> list[Rule]:
    """Checkpoint key -> native slice."""
    def whole(key, target):
        return Rule(key.replace(".", r"\."), lambda m, t=target: t)

    out = [whole("embed", "embedder.weight"), whole("head", "lm_head.weight"),
           whole("final.norm", "final_norm.weight"), whole("final.norm.b", "final_norm.bias")]
    for i, layer in enumerate(cfg.layers):
        n, m = f"layers.{i}", layer.mixer
        for norm in ("norm1", "norm2"):
            if norm == "norm1" or layer.mlp is not None:
                out += [whole(f"l{i}.{norm}", f"{n}.{norm}.weight"), whole(f"l{i}.{norm}.b", f"{n}.{norm}.bias")]
        if layer.mlp is not None:
            out += [whole(f"l{i}.mlp.up", f"{n}.mlp.up.weight"), whole(f"l{i}.mlp.down", f"{n}.mlp.down.weight")]
        out.append(whole(f"l{i}.mix.o", f"{n}.mixer.out_proj.weight"))
        if isinstance(m, GatedLinearAttentionConfig):
            qk, vg = m.heads * m.dim, m.heads * m.vdim
            out += _fused(i, f"{n}.mixer.in_proj.weight", [("q", qk), ("k", qk), ("v", vg), ("g", vg), ("a1", m.decay_rank)])
            out += [whole(f"l{i}.mix.a2", f"{n}.mixer.decay_proj.weight"), whole(f"l{i}.mix.a2.b", f"{n}.mixer.decay_bias"),
                    whole(f"l{i}.mix.norm", f"{n}.mixer.norm_weight")]
        else:
            own = m.kv_from is None
            out += _fused(i, f"{n}.mixer.in_proj.weight",
                          [("q", m.heads * (m.dim + m.rot_dim))] + ([("dkv", m.kv_rank + m.rot_dim)] if own else []))
            out += _fused(i, f"{n}.mixer.kv_proj.weight", [("uk", m.heads * m.dim), ("uv", m.heads * m.vdim)])
            if own:
                out.append(whole(f"l{i}.mix.dkv.norm", f"{n}.mixer.latent_norm"))
    return out


def load_into(model: Letitar, cfg: LetitarConfig, file_dir) -> None:
    asm = StateAssembler(native_state(model), key_rules(cfg))
    for key, tensor in stream_safetensors(file_dir):
        asm.assign(key, tensor)
    asm.finish()


def create_letitar_from_safetensors(file_dir, *, device="cpu", dtype=torch.bfloat16) -> Letitar:
    """Every checkpoint key must map and every parameter be filled, otherwise a RuntimeError lists them."""
    cfg = make_config(str(file_dir))
    model = Letitar(cfg, device=device, dtype=dtype)
    load_into(model, cfg, file_dir)
    return model
