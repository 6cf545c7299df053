"""Letitar: decoder-only models of gated-linear-attention and latent-attention layers."""
from .config import LetitarConfig, LayerConfig, is_supported_letitar_model_id, make_config, make_config_from_hf
from .model import Letitar

__all__ = ["Letitar", "LetitarConfig", "LayerConfig", "is_supported_letitar_model_id", "make_config", "make_config_from_hf"]
