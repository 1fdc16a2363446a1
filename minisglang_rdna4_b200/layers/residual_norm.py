"""Norm of a layer with an fp32 residual stream: residual add and layer norm (no bias) or RMS norm in one pass."""
from __future__ import annotations

import torch

from .. import ops
from .base import BaseOP


class ResidualNorm(BaseOP):
    """``center``: subtract the mean (layer norm). Outputs have ``out_cols`` columns (zero past the width)."""

    def __init__(self, width: int, eps: float, center: bool, dtype, device, out_cols: int) -> None:
        self.weight = torch.empty((width,), dtype=torch.float32, device=device)
        self._eps, self._center, self._dtype, self._cols = eps, center, dtype, out_cols

    def forward(self, x: torch.Tensor, delta):
        """``(x + delta, norm)``; ``delta`` None: nothing to add."""
        return ops.add_norm(x, delta, self.weight, self._eps, self._center, self._dtype, self._cols)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.weight = torch.ones_like(self.weight)
