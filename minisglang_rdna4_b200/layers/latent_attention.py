"""Latent attention without positions: a layer caches one latent per token (its own, or it reads another layer's),
and its per-head keys and values are linear in that latent.

The decoding form is absorbed: queries move into the latent space through the key half (``q W_uk``), every head attends
to the same latent rows, and the attended latents come back through the value half (``W_uv``). Each layer has sizes,
scale, window and heads of its own."""
from __future__ import annotations

import torch

from ..core import get_global_ctx
from ..parallel.info import get_tp_info
from ..utils import div_even
from .base import BaseOP
from .linear import ReplicatedLinear


class LatentAttentionLayer(BaseOP):
    """``spec`` gives the sizes (``models.config.LatentLayer``); ``row`` is the index in the latent pool of the layer
    whose latent is read. Weights are padded with zeros to the widths the kernels take."""

    def __init__(self, spec, row: int, width_pad: int, eps: float, dtype, device) -> None:
        self._h = div_even(spec.heads, get_tp_info().size)
        self._spec, self._row, self._eps = spec, row, eps
        self._own = spec.kv_from is None
        self._dim, self._vdim, self._rank = spec.dim_pad, spec.vdim_pad, spec.rank_pad
        # one projection: the heads' queries, then (a layer with a latent of its own) the latent
        self.q_proj = ReplicatedLinear(width_pad, self._h * self._dim + (self._rank if self._own else 0), dtype, device)
        if self._own:
            self.latent_norm = torch.empty((self._rank,), dtype=torch.float32, device=device)
        self.up_k = torch.empty((self._h, self._rank, self._dim), dtype=dtype, device=device)
        self.up_v = torch.empty((self._h, self._vdim, self._rank), dtype=dtype, device=device)
        self._expand_k = None        # up_k as [heads * dim, rank]: the expanded prefill form (16-bit, GPU)

    @property
    def out_width(self) -> int:
        return self._h * self._vdim

    def forward(self, x: torch.Tensor, out: torch.Tensor) -> None:
        """``x [T, width]`` -> the heads' values, concatenated, into ``out [T, heads * vdim]`` (any row stride)."""
        ctx = get_global_ctx()
        batch = ctx.batch
        t, nq = x.shape[0], self._h * self._dim
        qc = self.q_proj.forward(x)
        store = (qc[:, nq:], self.latent_norm, self._spec.kv_rank, self._eps) if self._own else None
        q = qc[:, :nq].unflatten(1, (self._h, self._dim))
        ctx.attn_backend.latent_forward(q, self.up_k, self.up_v, self._row, batch, scale=self._spec.scale,
                                        window=self._spec.window, out=out.unflatten(1, (self._h, self._vdim)),
                                        expand_k=self._expand_k, store=store)

    def _post_load_self(self) -> None:
        if self.up_k.is_cuda and self.up_k.dtype == torch.bfloat16:
            self._expand_k = self.up_k.transpose(1, 2).reshape(self._h * self._dim, self._rank).contiguous()

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        for name in ("up_k", "up_v"):
            w = getattr(self, name)
            setattr(self, name, (torch.randn(w.shape, generator=gen, device=gen.device) * std).to(w.device, w.dtype))
        if self._own:
            self.latent_norm = torch.ones_like(self.latent_norm)
