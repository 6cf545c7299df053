"""Parameter holders of the serving decoders: projections and norms of fp32 rows."""
from __future__ import annotations

import math

import torch
from torch import nn

from ...ops import serving as S


class Projection(nn.Module):
    """Weight [out, in] without bias."""

    def __init__(self, in_dim: int, out_dim: int, device=None, dtype=None):
        super().__init__()
        self.weight = nn.Parameter(torch.empty(out_dim, in_dim, device=device, dtype=dtype))
        self.reset_parameters()

    def reset_parameters(self):
        if self.weight.device.type != "meta":
            nn.init.normal_(self.weight, std=1.0 / math.sqrt(self.weight.shape[1]))

    def forward(self, x, out_dtype=None, into=None):
        return S.project(x, self.weight, out_dtype=out_dtype, into=into)


class LayerNorm(nn.Module):
    """Layer norm with weight and bias, fp32 rows in, weight dtype out."""

    def __init__(self, dim: int, eps: float, device=None, dtype=None):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim, device=device, dtype=dtype))
        self.bias = nn.Parameter(torch.zeros(dim, device=device, dtype=dtype))
        self.eps = eps

    def forward(self, x):
        return S.layernorm_rows(x, self.weight, self.bias, self.eps)


class RMSNorm(nn.Module):
    """x / sqrt(mean(x^2) + eps) * weight, fp32 rows in, weight dtype out."""

    def __init__(self, dim: int, eps: float, device=None, dtype=None):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim, device=device, dtype=dtype))
        self.eps = eps

    def forward(self, x):
        return S.rms_rows(x, self.weight, self.eps)
