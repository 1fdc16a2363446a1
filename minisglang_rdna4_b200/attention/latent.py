"""Attention backend of models that cache latents instead of per-head keys and values
(``layers/latent_attention.py``). Prefill, portions of prompts, decode and draft verification in one batch: every row
reads the paged latent pool after the step's latents were stored."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..core import Batch, get_global_ctx
from .base import AttnMetadata, BaseAttnBackend


class LatentAttentionBackend(BaseAttnBackend):
    def __init__(self, device, max_seq_len: int, single_split: bool = False) -> None:
        self.device = torch.device(device)
        self.max_seq_len = max_seq_len
        self.single_split = single_split

    def prepare_metadata(self, batch: Batch, block_table, cu_q, seq_lens, max_q: int, max_kv: int,
                         causal: bool = True, mask: Optional[torch.Tensor] = None, host_cu_q=None,
                         host_seq_lens=None, mask_window: int = 0, mask_swa=None) -> None:
        if mask is not None or not causal:
            raise NotImplementedError("latent attention is causal and takes no mask")
        batch.attn_metadata = AttnMetadata(cu_q=cu_q, seq_lens=seq_lens, block_table=block_table, max_q=max_q,
                                           max_kv=max_kv, decode=max_q == 1)

    def forward(self, q, layer: int, batch: Batch, *, scale: float, window: int = 0, swa: bool = False):
        raise NotImplementedError("models with a latent pool call latent_forward")

    def latent_forward(self, q, up_k, up_v, row: int, batch: Batch, *, scale: float, window: int, out) -> None:
        """``q [T, H, dim]``, ``up_k [H, rank, dim]``, ``up_v [H, vdim, rank]`` -> ``out [T, H, vdim]``."""
        md = batch.attn_metadata
        q_lat = ops.head_gemm(q, up_k)
        o_lat = ops.latent_attention(q_lat, get_global_ctx().kv_cache.rows(row), md.block_table, md.cu_q, md.seq_lens,
                                     scale, window, md.max_q, md.max_kv, self._splits(q, md, window))
        ops.head_gemm(o_lat, up_v, out)

    def _splits(self, q, md: AttnMetadata, window: int) -> int:
        """Key ranges per query tile of a decode step. Depends on the batch size and on what the window or the pool
        can hold, never on the lengths in the batch: a captured graph and an eager step reduce in the same order."""
        if not md.decode or self.single_split or not q.is_cuda:
            return 1
        from ..ops.cuda import latent_splits

        reach = min(window, self.max_seq_len) if window > 0 else self.max_seq_len
        return latent_splits(md.seq_lens.numel(), q.shape[1], up_to=reach)
