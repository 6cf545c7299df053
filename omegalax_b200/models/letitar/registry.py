"""Letitar family registry."""
from __future__ import annotations

from .config import LetitarConfig, is_supported_letitar_model_id, list_letitar_model_ids, make_config, make_config_from_hf


def build_config(model_id: str) -> LetitarConfig:
    return make_config(model_id)


def get_model_cls(model_id: str | None = None):
    from .model import Letitar

    return Letitar


__all__ = ["LetitarConfig", "build_config", "get_model_cls", "is_supported_letitar_model_id", "list_letitar_model_ids",
           "make_config", "make_config_from_hf"]
