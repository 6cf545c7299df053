"""Difedra checkpoint tensors -> parameters."""
from __future__ import annotations

from ..mixers import GatedMLPConfig
from ..params_utils import Rule
from ..stream_decoder import part, stacked, whole
from .config import DifedraConfig


def key_rules(cfg: DifedraConfig) -> list[Rule]:
    """Checkpoint key -> native slice."""
    out = [whole("embed", "embedder.weight"), whole("final.norm", "final_norm.weight")]
    for i, layer in enumerate(cfg.layers):
        p, n, m, mlp = f"l{i}.", f"layers.{i}.", layer.mixer, layer.mlp
        q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        out += stacked(p + "mix.", n + "mixer.in_proj.weight", [("q", q), ("k", k), ("v", v)])
        out += stacked(p + "mix.", n + "mixer.qk_norm", [("q.norm", q), ("k.norm", k)])
        out += [whole(p + "norm1", n + "norm1.weight"), whole(p + "mix.o", n + "mixer.out_proj.weight")]
        if m.sink:
            out.append(whole(p + "mix.sink", n + "mixer.sink"))
        if m.v_from is not None:
            out.append(whole(p + "mix.vmix", n + "mixer.value_mix"))
        if mlp is None:
            continue
        out.append(whole(p + "norm2", n + "norm2.weight"))
        if isinstance(mlp, GatedMLPConfig):
            out += stacked(p + "mlp.", n + "mlp.gate_up.weight", [("gate", mlp.ff), ("up", mlp.ff)])
            out.append(whole(p + "mlp.down", n + "mlp.down.weight"))
            continue
        out.append(whole(p + "mlp.router", n + "mlp.router.weight"))
        for e in range(mlp.experts):
            out += stacked(p + f"mlp.e{e}.", n + "mlp.experts_gate_up", [("gate", mlp.expert.ff), ("up", mlp.expert.ff)], (e,))
            out.append(part(p + f"mlp.e{e}.down", n + "mlp.experts_down", (e,)))
    return out
