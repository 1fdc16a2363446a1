"""Selective state-space mixer (Mamba): one projection to ``[x ‖ z]``, a causal convolution with silu over ``x``, a
projection of that to ``[dt (low rank) ‖ B ‖ C]``, the recurrence on the request's state slot, gated by ``silu(z)``. Sizes
in ``models.config.ScanLayer``."""
from __future__ import annotations

import torch

from .. import ops
from ..core import get_global_ctx
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from .base import BaseOP
from .linear import ReplicatedLinear


class SelectiveScanLayer(BaseOP):
    """``state_row``: the layer's row in the state cache. Channels are padded with zeros to a multiple of 16, the state to
    a multiple of 4; under tensor parallelism a rank has a share of the channels."""

    def __init__(self, spec, state_row: int, width_pad: int, dtype, device) -> None:
        tp = get_tp_info()
        if spec.inner % tp.size:
            raise ValueError(f"{spec.inner} scan channels over {tp.size} ranks")
        self._spec, self._state_row, self._dtype = spec, state_row, dtype
        self._c, self._n, self._r = spec.inner_pad(tp.size), spec.state_pad, spec.rank_pad

        def fp32(*shape):
            return torch.empty(shape, dtype=torch.float32, device=device)

        self.in_proj = ReplicatedLinear(width_pad, 2 * self._c, dtype, device)
        self.conv, self.conv_bias = fp32(self._c, spec.taps), fp32(self._c)
        self.x_proj = ReplicatedLinear(self._c, self._r + 2 * self._n, dtype, device)
        self.dt_proj = ReplicatedLinear(self._r, self._c, dtype, device)
        self.dt_bias, self.skip = fp32(self._c), fp32(self._c)
        self.a_log = fp32(self._c, self._n)
        self._a = None

    @property
    def out_width(self) -> int:
        return self._c

    def _post_load_self(self) -> None:
        self._a = -torch.exp(self.a_log)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ctx = get_global_ctx()
        batch = ctx.batch
        proj = self.in_proj.forward(x)
        if ctx.recurrent_journal is not None:
            ctx.recurrent_journal.append((self, proj))
        md = batch.attn_metadata
        chunked = batch.is_prefill and not batch.spec_verify and md.max_q >= 8
        return self._mix(proj, md.cu_q, batch.gdn_slots, batch.gdn_has_state, chunked, md.max_q)

    def _mix(self, proj: torch.Tensor, cu_q, slots, has_state, chunked: bool, max_q: int = 0) -> torch.Tensor:
        """Convolution and recurrence over the projected rows; advances both states."""
        st, c, r, n = get_global_ctx().gdn_state, self._c, self._r, self._n
        x = ops.causal_conv_silu(proj[:, :c], self.conv, self.conv_bias, st.conv_state(self._state_row), cu_q, slots,
                                 has_state, max_q)
        y = self.x_proj.forward(x)
        if get_tp_info().size > 1:             # the other ranks hold the other channels
            y = get_comm().all_reduce(y)
        dt = ops.gemm(y[:, :r], self.dt_proj.weight, None, torch.float32)
        return ops.selective_scan(x, dt, self.dt_bias, self._a, y[:, r:r + n], y[:, r + n:r + 2 * n], self.skip,
                                  proj[:, c:], st.ssm_state(self._state_row), cu_q, slots, has_state, chunked)

    def replay(self, proj: torch.Tensor, cu_q, slots, has_state) -> None:
        """Re-advance the (restored) states over the kept rows of a verify step."""
        self._mix(proj, cu_q, slots, has_state, False)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        def draw(t, scale):
            return (torch.randn(t.shape, generator=gen, device=gen.device) * scale).to(t.device, t.dtype)

        self.conv, self.conv_bias = draw(self.conv, 0.3), torch.zeros_like(self.conv_bias)
        self.dt_bias, self.skip = draw(self.dt_bias, 0.5) - 3.0, torch.ones_like(self.skip)
        steps = torch.arange(1, self._n + 1, dtype=torch.float32, device=self.a_log.device)
        self.a_log = torch.log(steps).expand(self._c, self._n).contiguous()
