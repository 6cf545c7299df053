"""Letitar: decoder-only models of gated-linear-attention and latent-attention layers."""
from .config import LayerConfig, LetitarConfig, make_config_from_hf
from .model import Letitar
from .registry import FAMILY

__all__ = ["FAMILY", "Letitar", "LetitarConfig", "LayerConfig", "make_config_from_hf"]
