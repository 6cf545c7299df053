"""Rotary frequencies, scaled for long contexts in one of two ways, and the cos / sin tables the kernels read.

Frequencies and angles are formed in double precision and rounded once, so a table entry is good to
fp32 at any position.
"""
from __future__ import annotations

import dataclasses
import math

import torch


@dataclasses.dataclass(frozen=True)
class YarnScaling:
    """Frequencies whose wavelength fits ``fast`` or more turns into ``original`` positions are kept,
    those below ``slow`` turns are divided by ``factor``, with a linear ramp over the pair index
    between; cos and sin grow by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    def apply(self, freq, rot: "RotaryConfig"):
        def pair_index(turns: float) -> float:
            return rot.dims * math.log(self.original / (turns * 2 * math.pi)) / (2 * math.log(rot.base))

        lo = max(math.floor(pair_index(self.fast)), 0)
        hi = min(math.ceil(pair_index(self.slow)), rot.dims - 1)
        i = torch.arange(rot.dims // 2, dtype=torch.float64)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return freq / self.factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(self.factor) + 1.0


@dataclasses.dataclass(frozen=True)
class WavelengthScaling:
    """Frequencies that make more than ``high`` turns in ``original`` positions are kept, those that make
    fewer than ``low`` are divided by ``factor``, with a ramp linear in the turns between; the amplitude
    stays 1 (the scheme of Llama 3.1)."""
    factor: float
    original: float
    low: float
    high: float

    def apply(self, freq, rot: "RotaryConfig"):
        turns = self.original * freq / (2 * math.pi)
        if self.high > self.low:
            keep = ((turns - self.low) / (self.high - self.low)).clamp(0.0, 1.0)
        else:
            keep = (turns >= self.low).to(freq.dtype)
        return (1.0 - keep) * freq / self.factor + keep * freq, 1.0


@dataclasses.dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    scaling: YarnScaling | WavelengthScaling | None = None

    def frequencies(self) -> tuple[torch.Tensor, float]:
        """(float64 [dims/2] radians per position, amplitude of cos and sin)."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        freq = torch.exp(i * (-2.0 / self.dims * math.log(self.base)))
        return (freq, 1.0) if self.scaling is None else self.scaling.apply(freq, self)


class RotaryTable:
    """fp32 (cos, sin) [positions, dims/2] on one device, rebuilt larger when a caller needs more."""

    def __init__(self, cfg: RotaryConfig):
        self.cfg = cfg
        self._tables: dict = {}

    def get(self, positions: int, device) -> tuple[torch.Tensor, torch.Tensor]:
        have = self._tables.get(device)
        if have is None or have[0].shape[0] < positions:
            freq, amp = self.cfg.frequencies()
            n = 1 << max(positions - 1, 255).bit_length()
            ang = torch.arange(n, dtype=torch.float64, device=device)[:, None] * freq.to(device)
            have = ((torch.cos(ang) * amp).float().contiguous(), (torch.sin(ang) * amp).float().contiguous())
            self._tables[device] = have
        return have
