"""Latent attention: a layer caches one latent per token (its own, or it reads another layer's), and its per-head keys
and values are linear in that latent. A layer may have a rotary part besides (a few query channels per head against one
rotated key that all heads share, cached behind the latent), a sink logit per head in the softmax denominator and a
sigmoid gate per head on the output.

The decoding form is absorbed: queries move into the latent space through the key half (``q W_uk``), every head attends
to the same latent rows, and the attended latents come back through the value half (``W_uv``). Each layer has sizes,
scale, window and heads of its own. The rotary channels pass ``up_k`` through an identity block (and meet zeros in
``up_v``), so that both forms treat a pool row ``[latent ‖ rotated key]`` as one vector."""
from __future__ import annotations

import torch

from ..core import get_global_ctx
from ..parallel.info import get_tp_info
from ..utils import div_even
from .base import BaseOP
from .linear import ReplicatedLinear
from .rotary import get_rope_cache


class LatentAttentionLayer(BaseOP):
    """``spec`` gives the sizes (``models.config.LatentLayer``); ``row`` is the index in the latent pool of the layer
    whose latent is read. Weights are padded with zeros to the widths the kernels take."""

    def __init__(self, spec, row: int, width_pad: int, eps: float, dtype, device) -> None:
        self._h = div_even(spec.heads, get_tp_info().size)
        self._spec, self._row, self._eps = spec, row, eps
        self._own = spec.kv_from is None
        self._dim, self._vdim, self._rank = spec.dim_pad, spec.vdim_pad, spec.rank_pad
        # one projection: the heads' queries, then (a layer with a latent of its own) the latent and the shared rotary
        # key, then the heads' gates
        self._gate_at = self._h * self._dim + (self._rank if self._own else 0)
        self.q_proj = ReplicatedLinear(width_pad, self._gate_at + (-(-self._h // 16) * 16 if spec.gate else 0), dtype, device)
        if spec.sink:
            self.sink = torch.empty((self._h,), dtype=torch.float32, device=device)
        self._cos_sin = get_rope_cache(spec.rotary, device) if spec.rotary is not None else None
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
        spec = self._spec
        store = (qc[:, nq:nq + self._rank], self.latent_norm, spec.kv_rank, self._eps) if self._own else None
        q = qc[:, :nq].unflatten(1, (self._h, self._dim))
        rope = None
        if spec.rotary is not None:
            rope = (spec.dim, spec.rotary.rotary_dim, self._cos_sin, spec.rot_dim)
        ctx.attn_backend.latent_forward(q, self.up_k, self.up_v, self._row, batch, scale=spec.scale,
                                        window=spec.window, out=out.unflatten(1, (self._h, self._vdim)),
                                        expand_k=self._expand_k, store=store, rope=rope,
                                        sink=self.sink if spec.sink else None,
                                        gate=qc[:, self._gate_at:self._gate_at + self._h] if spec.gate else None)

    def _post_load_self(self) -> None:
        if self.up_k.is_cuda and self.up_k.dtype == torch.bfloat16:
            self._expand_k = self.up_k.transpose(1, 2).reshape(self._h * self._dim, self._rank).contiguous()

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        for name in ("up_k", "up_v"):
            w = getattr(self, name)
            setattr(self, name, (torch.randn(w.shape, generator=gen, device=gen.device) * std).to(w.device, w.dtype))
        spec, r = self._spec, self._spec.kv_rank
        self.up_k[:, r:] = 0
        self.up_k[:, :, spec.dim:] = 0
        self.up_v[:, :, r:] = 0
        self.rotary_identity()
        if self._own:
            self.latent_norm = torch.ones_like(self.latent_norm)
        if spec.sink:
            self.sink = torch.zeros_like(self.sink)

    def rotary_identity(self) -> None:
        """The block of ``up_k`` that hands the rotary channels through."""
        spec = self._spec
        for j in range(spec.rot_dim):
            self.up_k[:, spec.kv_rank + j, spec.dim + j] = 1
