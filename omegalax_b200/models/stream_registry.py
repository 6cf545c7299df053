"""The serving decoder designs by name, config.json and configuration type."""
from __future__ import annotations

from typing import Mapping

from .difedra.registry import FAMILY as DIFEDRA
from .letitar.registry import FAMILY as LETITAR
from .stream_decoder import Family, StreamDecoder, StreamDecoderConfig

FAMILIES: tuple[Family, ...] = (LETITAR, DIFEDRA)


def family_of(cfg) -> Family:
    """The family of a configuration object."""
    for f in FAMILIES:
        if isinstance(cfg, f.config_cls):
            return f
    raise ValueError(f"no serving decoder has a configuration of type {type(cfg).__name__}")


def family_for(hf_cfg: Mapping) -> Family | None:
    """The family a config.json dict belongs to."""
    return next((f for f in FAMILIES if f.owns(hf_cfg)), None)


def family_of_preset(model_id: str) -> Family | None:
    return next((f for f in FAMILIES if model_id in f.presets), None)


def list_model_ids() -> list[str]:
    return sorted(name for f in FAMILIES for name in f.presets)


__all__ = ["FAMILIES", "Family", "StreamDecoder", "StreamDecoderConfig", "family_for", "family_of", "family_of_preset",
           "list_model_ids"]
