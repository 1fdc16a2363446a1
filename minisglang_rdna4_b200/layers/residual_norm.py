"""Norms of a layer with an fp32 residual stream, in one pass with the residual add: layer norm (no bias) or RMS norm
(``ResidualNorm``); layer norms with a bias on both sides of a sublayer, pairs of sublayers, depth averages
(``BiasedNorm``, ``LayerHistory``; ``ops.residual_step`` does them together)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import BaseOP


class ResidualNorm(BaseOP):
    """``center``: subtract the mean (layer norm). Outputs have ``out_cols`` columns (zero past the width). The norm of a
    sublayer's output (``post`` of the next one's ``forward``) is one of these that is never called itself."""

    def __init__(self, width: int, eps: float, center: bool, dtype, device, out_cols: int) -> None:
        self.weight = torch.empty((width,), dtype=torch.float32, device=device)
        self._eps, self._center, self._dtype, self._cols = eps, center, dtype, out_cols

    def forward(self, x: torch.Tensor, delta, post: Optional["ResidualNorm"] = None, mult: float = 1.0):
        """``(x + delta, norm)``; ``delta`` None: nothing to add. ``post``: ``mult`` times that RMS norm of ``delta`` is
        what is added."""
        return ops.add_norm(x, delta, self.weight, self._eps, self._center, self._dtype, self._cols,
                            None if post is None else post.weight, mult)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.weight = torch.ones_like(self.weight)

class BiasedNorm(BaseOP):
    """Weight and bias of a layer norm; ``residual_step`` applies it."""

    def __init__(self, width: int, device) -> None:
        self.weight = torch.empty((width,), dtype=torch.float32, device=device)
        self.bias = torch.empty((width,), dtype=torch.float32, device=device)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.weight, self.bias = torch.ones_like(self.weight), torch.zeros_like(self.bias)


class LayerHistory:
    """The results of the layers so far in a step, ``[layers + 1, rows, width]`` fp32; row 0 is the embedding output."""

    def __init__(self, layers: int, rows: int, width: int, device) -> None:
        self.rows = torch.empty((layers + 1, rows, width), dtype=torch.float32, device=device)
        self.count = 0
