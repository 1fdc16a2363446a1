"""Dense gated feed-forward of a model with an fp32 residual stream."""
from __future__ import annotations

import torch

from .. import ops
from ..parallel.info import get_tp_info
from ..utils import div_even
from .base import BaseOP
from .linear import ReplicatedLinear, RowParallelLinear


class DenseGatedMLP(BaseOP):
    """silu-gated feed-forward with an fp32 result."""

    def __init__(self, ff: int, width_pad: int, dtype, device) -> None:
        tp = get_tp_info().size
        self._ff = (div_even(ff, tp) + 15) // 16 * 16
        self.gate_up = ReplicatedLinear(width_pad, 2 * self._ff, dtype, device)
        self.down = RowParallelLinear(self._ff * tp, width_pad, dtype, device)

    def forward_partial32(self, x: torch.Tensor):
        return self.down.forward_partial32(ops.silu_and_mul(self.gate_up.forward(x)))
