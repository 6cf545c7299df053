"""Feed-forward blocks of the serving decoders."""
from __future__ import annotations

import dataclasses
import math

import torch
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


@dataclasses.dataclass(frozen=True)
class GatedMLPConfig:
    ff: int
    act: str            # "silu" or "gelu_tanh"


class GatedMLP(nn.Module):
    """down(act(gate(h)) * up(h)), added into the residual rows."""

    def __init__(self, cfg: GatedMLPConfig, width: int, device=None, dtype=None):
        super().__init__()
        self.act = cfg.act
        self.gate_up = Projection(width, 2 * cfg.ff, device=device, dtype=dtype)      # [gate | up]
        self.down = Projection(cfg.ff, width, device=device, dtype=dtype)

    def forward(self, h, x):
        self.down(S.gated_act(self.gate_up(h).contiguous(), self.act), into=x)


@dataclasses.dataclass(frozen=True)
class MixtureOfExpertsConfig:
    experts: int
    top: int
    expert: GatedMLPConfig

    def __post_init__(self):
        if not 0 < self.top <= min(self.experts, 16) or self.experts > 512:
            raise ValueError(f"cannot route to {self.top} of {self.experts} experts (at most 16 of 512)")


class MixtureOfExperts(nn.Module):
    """Gated feed-forwards of which each token uses the ``top`` with the largest router logits; the sigmoid of
    its logit scales an expert's input.  The outputs are added into the residual rows."""

    def __init__(self, cfg: MixtureOfExpertsConfig, width: int, device=None, dtype=None):
        super().__init__()
        self.cfg = cfg
        kw = dict(device=device, dtype=dtype)
        self.router = Projection(width, cfg.experts, **kw)
        self.experts_gate_up = nn.Parameter(torch.empty(cfg.experts, 2 * cfg.expert.ff, width, **kw))
        self.experts_down = nn.Parameter(torch.empty(cfg.experts, width, cfg.expert.ff, **kw))
        for w in (self.experts_gate_up, self.experts_down):
            if w.device.type != "meta":
                nn.init.normal_(w, std=1.0 / math.sqrt(w.shape[2]))

    def forward(self, h, x):
        weight, idx = S.route_sigmoid(self.router(h, out_dtype=torch.float32), self.cfg.top)
        S.experts_into(h, weight, idx, self.experts_gate_up, self.experts_down, self.cfg.expert.act, x)
