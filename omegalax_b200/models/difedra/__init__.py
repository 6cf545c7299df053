"""Difedra: decoder-only models of windowed attention layers with dense or routed feed-forwards."""
from .config import DifedraConfig, LayerConfig, make_config_from_hf
from .model import Difedra
from .registry import FAMILY

__all__ = ["FAMILY", "Difedra", "DifedraConfig", "LayerConfig", "make_config_from_hf"]
