"""Pre-norm of a layer with an fp32 residual stream: residual add, RMS norm with one gain for all coordinates, and
a short causal depthwise convolution ahead of each sublayer (``h + conv(h)``).

The sublayers of a parallel layer read the same normalised rows, so their convolutions share one tail of ``taps - 1``
rows per request. The tail lives in the recurrent-state cache (``ctx.gdn_state``, one slot per request row)."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from .. import ops
from ..core import get_global_ctx
from .base import BaseOP


class ScalarNormConv(BaseOP):
    """``filters``: how many sublayers get a convolved copy (0: the norm alone). ``state_id``: the layer's row in the
    state cache. Outputs have ``out_cols`` columns (zero past the width: the GEMM kernels want a multiple of 8)."""

    def __init__(self, width: int, taps: int, filters: int, state_id: int, eps: float, dtype, device,
                 out_cols: int) -> None:
        self.gain = torch.empty((1,), dtype=torch.float32, device=device)
        self._taps, self._state_id, self._eps = taps, state_id, eps
        self._dtype, self._cols = dtype, out_cols
        if filters > 0:
            self.conv1 = torch.empty((taps, width), dtype=torch.float32, device=device)
        if filters > 1:
            self.conv2 = torch.empty((taps, width), dtype=torch.float32, device=device)
        self._filters = filters

    def forward(self, x: torch.Tensor, delta) -> Tuple[torch.Tensor, torch.Tensor, Optional[torch.Tensor]]:
        """``(x + delta, y1, y2)``; the tails of the step's requests advance."""
        if self._filters == 0:
            return ops.add_scalar_norm_conv(x, delta, self.gain, self._eps, None, None, None, None, None, None, 0,
                                            self._dtype, self._cols)
        ctx = get_global_ctx()
        batch = ctx.batch
        md = batch.attn_metadata
        out = self._apply(x, delta, md.cu_q, batch.gdn_slots, batch.gdn_has_state, md.max_q)
        if ctx.recurrent_journal is not None:
            ctx.recurrent_journal.append((self, out[0]))
        return out

    def _apply(self, x, delta, cu_q, slots, has_state, max_q: int):
        # the cache keeps [slots, width * (taps - 1)] values per layer; here they are taps - 1 rows
        state = get_global_ctx().gdn_state.conv_state(self._state_id)
        state = state.view(state.shape[0], self._taps - 1, self.conv1.shape[1])
        return ops.add_scalar_norm_conv(x, delta, self.gain, self._eps, self.conv1, getattr(self, "conv2", None),
                                        state, cu_q, slots, has_state, max_q, self._dtype, self._cols)

    def replay(self, x: torch.Tensor, cu_q, slots, has_state) -> None:
        """Re-advance the (restored) tails over the kept residual rows of a verify step."""
        self._apply(x, None, cu_q, slots, has_state, x.shape[0])

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.gain = torch.ones_like(self.gain)
        for name in ("conv1", "conv2"):
            w = getattr(self, name, None)
            if w is not None:
                r = torch.randn(w.shape, generator=gen, device=gen.device, dtype=torch.float32) * 0.3
                setattr(self, name, r.to(w.device))
