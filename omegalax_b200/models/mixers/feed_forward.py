"""Feed-forward blocks of the serving decoders."""
from __future__ import annotations

import dataclasses

from torch import nn

from ...ops import serving as S
from .layers import Projection


@dataclasses.dataclass(frozen=True)
class DenseMLPConfig:
    ff: int


class SquaredReluMLP(nn.Module):
    """down(relu(up(h))^2), added into the residual rows."""

    def __init__(self, cfg: DenseMLPConfig, width: int, device=None, dtype=None):
        super().__init__()
        self.up = Projection(width, cfg.ff, device=device, dtype=dtype)
        self.down = Projection(cfg.ff, width, device=device, dtype=dtype)

    def forward(self, h, x):
        self.down(S.relu_squared(self.up(h).contiguous()), into=x)
