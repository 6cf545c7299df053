"""Write a Letitar model as a checkpoint folder: the loader's rules walked backwards."""
from __future__ import annotations

from pathlib import Path

import torch

from ..hf_io import save_hf_config
from ..params_utils import native_state, save_safetensors
from .config import LetitarConfig, config_to_hf
from .loader import key_rules
from .model import Letitar


def letitar_to_tensors(model: Letitar, cfg: LetitarConfig) -> dict[str, torch.Tensor]:
    state, out = native_state(model), {}
    for rule in key_rules(cfg):
        key = rule.pattern.replace("\\.", ".")
        m = rule.regex.fullmatch(key)
        t, idx = state[rule.target(m)].detach(), rule.index(m)
        out[key] = (t if idx is None else t[idx]).to(torch.bfloat16).contiguous()
    return out


def export_letitar_to_safetensors(model: Letitar, cfg: LetitarConfig, out_dir) -> Path:
    save_safetensors(letitar_to_tensors(model, cfg), out_dir)
    save_hf_config(config_to_hf(cfg), out_dir)
    return Path(out_dir)
