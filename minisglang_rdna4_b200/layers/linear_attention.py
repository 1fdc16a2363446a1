"""Linear attention with a decaying state per head (no delta rule, no convolution): one projection to
``[q ‖ k ‖ v ‖ output gate (‖ low-rank decay input)]``, the recurrence on the request's state slot, a norm of the
result (per head or over all heads) with the gate. ``models.config.LinearAttnLayer`` says which decay, activation,
rotation, norm and gate a layer has."""
from __future__ import annotations

import torch

from .. import ops
from ..core import get_global_ctx
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from ..utils import div_even
from .base import BaseOP
from .linear import ReplicatedLinear
from .rotary import get_rope_cache


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class LinearAttentionLayer(BaseOP):
    """``state_row``: the layer's row in the state cache. Heads are padded with zero channels to multiples of 16."""

    def __init__(self, spec, state_row: int, width_pad: int, eps: float, dtype, device) -> None:
        self._h = div_even(spec.heads, get_tp_info().size)
        self._spec, self._state_row, self._eps = spec, state_row, eps
        self._dk, self._dv = spec.dim_pad, spec.vdim_pad
        self._kd, self._vd = self._h * self._dk, self._h * self._dv
        self._rank = spec.gate_rank
        self.in_proj = ReplicatedLinear(width_pad, 2 * self._kd + 2 * self._vd + _pad16(self._rank), dtype, device)
        self.norm = torch.empty((self._vd if spec.joint_norm else self._dv,), dtype=torch.float32, device=device)
        if spec.decay is None:
            self.decay_up = torch.empty((self._kd, self._rank), dtype=dtype, device=device)
            self.decay_bias = torch.empty((self._kd,), dtype=torch.float32, device=device)
            self._decay = None
        else:
            tp = get_tp_info()
            mine = spec.decay[tp.rank * self._h:(tp.rank + 1) * self._h]
            self._decay = torch.tensor(mine, dtype=torch.float32, device=device)
        # neighbouring channels are pairs (checkpoints with half-split pairs are loaded in that order)
        self._cos_sin = get_rope_cache(spec.rotary, device) if spec.rotary is not None else None

    @property
    def out_width(self) -> int:
        return _pad16(self._vd)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ctx = get_global_ctx()
        batch = ctx.batch
        proj = self.in_proj.forward(x)
        if ctx.recurrent_journal is not None:
            ctx.recurrent_journal.append((self, proj, batch.positions))
        md = batch.attn_metadata
        chunked = batch.is_prefill and not batch.spec_verify and md.max_q >= 8
        return self._mix(proj, md.cu_q, batch.gdn_slots, batch.gdn_has_state, batch.positions, chunked)

    def _mix(self, proj: torch.Tensor, cu_q, slots, has_state, positions, chunked: bool) -> torch.Tensor:
        """The recurrence over the projected rows (advances the state), norm and gate."""
        spec, kd, vd = self._spec, self._kd, self._vd
        q, k = (proj[:, i * kd:(i + 1) * kd].unflatten(1, (self._h, self._dk)) for i in range(2))
        v = proj[:, 2 * kd:2 * kd + vd].unflatten(1, (self._h, self._dv))
        g = proj[:, 2 * kd + vd:2 * kd + 2 * vd]
        gate = None
        if self._decay is None:
            low = proj[:, 2 * kd + 2 * vd:2 * kd + 2 * vd + self._rank]
            gate = (low, self.decay_up, self.decay_bias)
        state = get_global_ctx().gdn_state.ssm_state(self._state_row)
        o = ops.linear_attention(q, k, v, state, cu_q, slots, has_state, decay=self._decay, gate=gate, tau=spec.tau,
                                 q_scale=spec.q_scale, act=spec.act, chunked=chunked,
                                 rope=None if self._cos_sin is None else (self._cos_sin, positions))
        total = None
        if spec.joint_norm and get_tp_info().size > 1:      # the other ranks hold the other heads
            total = get_comm().all_reduce(o.float().pow(2).sum((1, 2)))
        return ops.norm_gate(o, g, self.norm, self._eps, spec.vdim, spec.joint_norm, spec.gate_act, self.out_width,
                             total, spec.heads)

    def replay(self, proj: torch.Tensor, cu_q, slots, has_state, positions) -> None:
        """Re-advance the (restored) states over the kept rows of a verify step."""
        self._mix(proj, cu_q, slots, has_state, positions, False)

    def _post_load_self(self) -> None:
        if not self._spec.weighted:
            self.norm = torch.ones_like(self.norm)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.norm = torch.ones_like(self.norm)
        if self._decay is None:
            w = torch.randn(self.decay_up.shape, generator=gen, device=gen.device) * std
            self.decay_up = w.to(self.decay_up.device, self.decay_up.dtype)
            self.decay_bias = torch.full_like(self.decay_bias, 2.0)
