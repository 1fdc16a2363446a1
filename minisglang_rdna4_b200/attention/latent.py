"""Attention backend of models that cache latents instead of per-head keys and values
(``layers/latent_attention.py``). Prefill, portions of prompts, decode and draft verification in one batch: every row
reads the paged latent pool after the step's latents were stored.

Two forms of the same sum. Absorbed: queries go into the latent space and attend to the latents themselves; any mix of
rows. Expanded (16-bit prefill steps on a GPU, ``ops.cuda.LatentPrefillPlan``): per-head keys and values of the latents
in sight are computed first, which takes fewer operations when a step has many rows, and runs on tcgen05."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..core import Batch, get_global_ctx
from .base import AttnMetadata, BaseAttnBackend


class LatentAttentionBackend(BaseAttnBackend):
    def __init__(self, layers, device, max_seq_len: int, single_split: bool = False) -> None:
        self.device = torch.device(device)
        windows = [s.window for s in layers if s is not None]
        self.reach = max(windows) if windows and min(windows) > 0 else 0
        self.max_seq_len = max_seq_len
        self.single_split = single_split       # speculative verification must reproduce decode rows bit for bit

    def prepare_metadata(self, batch: Batch, block_table, cu_q, seq_lens, max_q: int, max_kv: int,
                         causal: bool = True, mask: Optional[torch.Tensor] = None, host_cu_q=None,
                         host_seq_lens=None, mask_window: int = 0, mask_swa=None) -> None:
        if mask is not None or not causal:
            raise NotImplementedError("latent attention is causal and takes no mask")
        plan = None
        if host_cu_q is not None and batch.is_prefill and not batch.spec_verify and self.device.type == "cuda":
            from ..env import ENV
            from ..ops.cuda import LatentPrefillPlan

            if not ENV.DISABLE_TC_PREFILL.value and LatentPrefillPlan.pays(host_cu_q, host_seq_lens, self.reach):
                plan = LatentPrefillPlan(host_cu_q, host_seq_lens, self.reach, self.device)
        batch.attn_metadata = AttnMetadata(cu_q=cu_q, seq_lens=seq_lens, block_table=block_table, max_q=max_q,
                                           max_kv=max_kv, decode=max_q == 1, prefill_plan=plan)

    def forward(self, q, layer: int, batch: Batch, *, scale: float, window: int = 0, swa: bool = False):
        raise NotImplementedError("models with a latent pool call latent_forward")

    def latent_forward(self, q, up_k, up_v, row: int, batch: Batch, *, scale: float, window: int, out,
                       expand_k=None, store=None, rope=None, sink=None, gate=None) -> None:
        """``q [T, H, dim]``, ``up_k [H, rank, dim]``, ``up_v [H, vdim, rank]`` -> ``out [T, H, vdim]``. ``expand_k``:
        ``up_k`` as ``[H * dim, rank]``, where the expanded form may be used. ``store`` (a layer with latents of its own):
        ``(raw latents [T, rank], norm weight, rank, eps)`` to norm and store ahead of the attention. ``rope``: ``(first
        rotary channel of a query head, rotated channels, cos / sin table, width of the shared key part)``. ``sink [H]``,
        ``gate [T, H]``: logits in the softmax denominator and of the sigmoid on the output."""
        md = batch.attn_metadata
        rows = get_global_ctx().kv_cache.rows(row)
        if rope is not None:
            dim, dims, table, rot_dim = rope
            ops.latent_rope(q, dim, dims, table, batch.positions,
                            None if store is None else (*store, rows, batch.out_loc, rot_dim))
            store = None
        if store is not None:
            store = (*store, rows, batch.out_loc)
            if not (md.decode and q.is_cuda and q.dtype == torch.bfloat16):
                ops.latent_norm_store(*store)
                store = None
        if md.prefill_plan is not None and expand_k is not None:
            from ..ops import cuda as K

            if K.latent_prefill_ok(q.shape[2], up_v.shape[1], scale):
                K.latent_prefill(q, expand_k, up_v, rows, row, md.block_table,
                                 md.prefill_plan, scale, window, out, sink=sink, gate=gate)
                return
        q_lat = ops.head_gemm(q, up_k, store=store)
        splits = self._splits(q_lat, md, window)
        if 1 < splits and q.shape[0] <= 32:   # few rows: the value projection merges the key ranges itself
            from ..ops import cuda as K

            parts = K.latent_attention(q_lat, rows, md.block_table, md.cu_q, md.seq_lens, scale, window, md.max_q,
                                       md.max_kv, splits, merge=False, sink=sink)
            K.head_gemm_combine(parts, up_v, out, gate=gate)
            return
        o_lat = ops.latent_attention(q_lat, rows, md.block_table, md.cu_q, md.seq_lens, scale, window, md.max_q,
                                     md.max_kv, splits, one_form=self.single_split, sink=sink)
        ops.head_gemm(o_lat, up_v, out, gate=gate)

    def _splits(self, q, md: AttnMetadata, window: int) -> int:
        """Key ranges per query tile of a decode step. Depends on the batch size and on what the window or the pool
        can hold, never on the lengths in the batch: a captured graph and an eager step reduce in the same order."""
        if (not md.decode or self.single_split or not q.is_cuda or q.dtype != torch.bfloat16
                or q.shape[2] > 576):
            return 1
        from ..ops.cuda import latent_splits

        reach = min(window, self.max_seq_len) if window > 0 else self.max_seq_len
        return latent_splits(md.seq_lens.numel(), q.shape[1], q.shape[2], up_to=reach)
