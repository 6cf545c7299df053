"""Letitar checkpoint tensors -> parameters."""
from __future__ import annotations

from ..mixers import GatedLinearAttentionConfig
from ..params_utils import Rule
from ..stream_decoder import stacked, whole
from .config import LetitarConfig


def key_rules(cfg: LetitarConfig) -> list[Rule]:
    """Checkpoint key -> native slice."""
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
            out += stacked(f"l{i}.mix.", f"{n}.mixer.in_proj.weight", [("q", qk), ("k", qk), ("v", vg), ("g", vg), ("a1", m.decay_rank)])
            out += [whole(f"l{i}.mix.a2", f"{n}.mixer.decay_proj.weight"), whole(f"l{i}.mix.a2.b", f"{n}.mixer.decay_bias"),
                    whole(f"l{i}.mix.norm", f"{n}.mixer.norm_weight")]
        else:
            own = m.kv_from is None
            out += stacked(f"l{i}.mix.", f"{n}.mixer.in_proj.weight",
                           [("q", m.heads * (m.dim + m.rot_dim))] + ([("dkv", m.kv_rank + m.rot_dim)] if own else []))
            out += stacked(f"l{i}.mix.", f"{n}.mixer.kv_proj.weight", [("uk", m.heads * m.dim), ("uv", m.heads * m.vdim)])
            if own:
                out.append(whole(f"l{i}.mix.dkv.norm", f"{n}.mixer.latent_norm"))
    return out
