"""Difedra family description."""
from __future__ import annotations

from ..stream_decoder import Family
from .config import ARCHITECTURE, PRESETS, DifedraConfig, config_to_hf, make_config_from_hf
from .loader import key_rules
from .model import Difedra

FAMILY = Family(architecture=ARCHITECTURE, config_cls=DifedraConfig, config_from_hf=make_config_from_hf, config_to_hf=config_to_hf,
                key_rules=key_rules, model_cls=Difedra, presets=PRESETS, kernels="window_serving")
