"""Grouped-query attention of a layer with a geometry of its own (``models.config.HeadLayer``): head counts, widths, rotation,
reach (window or chunk), soft cap, norms of queries and keys, output gate; a layer may read the keys and values of an
earlier one and then projects queries alone. Further forms: scores with a logarithmic distance bias, a softmax that counts
a zero score besides, and heads that apply a mixture of all heads' weights.

One projection gives queries, keys, values and gates; every head takes ``row_pad`` columns of it, zeros past its
channels, which change no dot product."""
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


class HeadAttentionLayer(BaseOP):
    """``row``: index in the pool of the layer whose keys and values are read."""

    def __init__(self, spec, row: int, width_pad: int, eps: float, dtype, device, max_positions: int = 0) -> None:
        """``max_positions``: the longest sequence, for distance biases without a window."""
        self._max_distance = max_positions
        tp = get_tp_info().size
        self._spec, self._row, self._eps = spec, row, eps
        # heads whose weights are mixed are all on every rank; a rank hands on its share of them
        self._h = spec.heads if spec.talk else div_even(spec.heads, tp)
        self._hk = spec.kv_heads if spec.talk else div_even(spec.kv_heads, tp, allow_replicate=True)
        self._mine = div_even(spec.heads, tp)
        self._own, self._d = spec.kv_from is None, spec.row_pad
        if torch.device(device).type == "cuda" and dtype != torch.float32 and self._d > 256:
            raise NotImplementedError(f"heads of {max(spec.dim, spec.vdim)} channels: the 16-bit attention kernels take 256")
        # columns: query heads, then (a layer with keys and values of its own) those, then the gates
        self._gate_at = (self._h + (2 * self._hk if self._own else 0)) * self._d
        self.in_proj = ReplicatedLinear(width_pad, self._gate_at + (self._h * self._d if spec.gate else 0), dtype, device)
        if spec.joint_norm:
            self.q_norm = torch.empty((self._h * self._d,), dtype=torch.float32, device=device)
            if self._own:
                self.k_norm = torch.empty((self._hk * self._d,), dtype=torch.float32, device=device)
        self._cos_sin = get_rope_cache(spec.rotary, device) if spec.rotary is not None else None
        self._extra = {}
        if spec.log_bias:
            self.r1 = torch.empty((self._h,), dtype=torch.float32, device=device)
            self.r2 = torch.empty((self._h,), dtype=torch.float32, device=device)
        if spec.talk:
            self.talk = torch.empty((self._h, self._h), dtype=torch.float32, device=device)

    @property
    def out_width(self) -> int:
        return self._mine * self._d

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """``x [T, width]`` -> the heads' values, gated, ``[T, heads * row_pad]``."""
        ctx = get_global_ctx()
        batch, spec = ctx.batch, self._spec
        y = self.in_proj.forward(x)
        pool = ctx.kv_cache
        store = (pool.k_cache(self._row), pool.v_cache(self._row), batch.out_loc) if self._own else None
        q = ops.heads_rope_store(
            y, self._h, self._hk, self._d, spec.dim, batch.positions, self._cos_sin,
            spec.rotary is not None and spec.rotary.interleaved, self._eps,
            self.q_norm if spec.joint_norm else None, self.k_norm if spec.joint_norm and self._own else None,
            self._totals(y), spec.unit_norm, store)
        out = ctx.attn_backend.forward_heads(q, self._row, batch, scale=spec.scale, window=spec.window, chunk=spec.chunk,
                                             softcap=spec.softcap, gate=y[:, self._gate_at:] if spec.gate else None,
                                             **self._extra)
        if self._mine < self._h:
            out = out[:, get_tp_info().rank * self._mine:][:, :self._mine]
        return out.reshape(out.shape[0], self.out_width)

    def _totals(self, y: torch.Tensor):
        """Sums of squares over the heads of all ranks, for the norm over all heads together."""
        tp, spec = get_tp_info().size, self._spec
        if tp == 1 or not spec.joint_norm:
            return None
        nq, nk = self._h * self._d, self._hk * self._d
        sums = torch.stack([y[:, :nq].float().pow(2).sum(-1),
                            y[:, nq:nq + (nk if self._own else 0)].float().pow(2).sum(-1)], 1)
        copies = tp * self._hk // spec.kv_heads        # ranks that hold the same key head
        return get_comm().all_reduce(sums), spec.heads * spec.dim, spec.kv_heads * spec.dim * copies

    def _post_load_self(self) -> None:
        # what the kernels read past a head's channels is zero, whatever filled the weights
        spec, d, weight = self._spec, self._d, self.in_proj.weight
        own = self._hk if self._own else 0
        for at, n, used in ((0, self._h, spec.dim), (self._h, own, spec.dim), (self._h + own, own, spec.vdim)):
            weight[at * d:(at + n) * d].view(n, d, weight.shape[1])[:, used:] = 0
        if spec.log_bias:       # one number per head and distance in reach
            far = torch.arange(spec.window or self._max_distance + 256, dtype=torch.float64, device=weight.device)
            bias = self.r1.double()[:, None] * torch.log1p(self.r2.double()[:, None] * far)
            self._extra["bias"] = bias.float().contiguous()
        if spec.zero_sink:
            self._extra["sink"] = torch.zeros(self._h, dtype=torch.float32, device=weight.device)
        if spec.talk:
            self._extra["talk"] = self.talk

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        for name in ("q_norm", "k_norm"):
            if hasattr(self, name):
                setattr(self, name, torch.ones_like(getattr(self, name)))
        if self._spec.log_bias:
            self.r1, self.r2 = torch.ones_like(self.r1), torch.full_like(self.r2, 0.5)
        if self._spec.talk:
            mix = torch.randn(self.talk.shape, generator=gen, device=gen.device) * 0.1
            self.talk = mix.to(self.talk.device) + torch.eye(self._h, device=self.talk.device)
