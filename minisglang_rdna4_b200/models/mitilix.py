"""Mitilix: a decoder of parallel layers (attention and feed-forward read the same norm and are added together) over an
fp32 residual stream.

* token embedding plus a learned position vector; no other positional information;
* every sublayer reads ``h + conv(h)``, ``h`` the layer's scalar-gain RMS norm, ``conv`` a short causal depthwise
  convolution of its own (``layers/norm_conv.py``);
* sliding-window latent attention, a layer may read the latents of an earlier one (``layers/latent_attention.py``);
* a dense exact-gelu feed-forward, or none.

The two output projections of a layer are one matrix product over the concatenated rows ``[heads' values ‖ activated
feed-forward]``; its fp32 result is added to the residual by the next layer's norm."""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .. import ops
from ..core import get_global_ctx
from ..layers import BaseOP, ParallelLMHead, ReplicatedLinear, RowParallelLinear, VocabParallelEmbedding
from ..layers.latent_attention import LatentAttentionLayer
from ..layers.norm_conv import ScalarNormConv
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from ..utils import div_even
from .config import LatentLayer, ModelConfig


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class MitilixLayer(BaseOP):
    def __init__(self, cfg: ModelConfig, layer_id: int, dtype, device) -> None:
        spec = cfg.latent_layers[layer_id]
        wp, tp = _pad16(cfg.hidden_size), get_tp_info().size
        self._dtype = dtype
        self.norm = ScalarNormConv(cfg.hidden_size, cfg.input_conv_taps, 2 if spec.ff else 1, layer_id,
                                   cfg.rms_norm_eps, dtype, device, wp)
        self.attn = LatentAttentionLayer(spec, cfg.latent_row(layer_id), wp, cfg.rms_norm_eps, dtype, device)
        self._n_attn = self.attn.out_width
        self._ff = _pad16(div_even(spec.ff, tp)) if spec.ff else 0
        if self._ff:
            self.up_proj = ReplicatedLinear(wp, self._ff, dtype, device)
        self.out_proj = RowParallelLinear((self._n_attn + self._ff) * tp, wp, dtype, device)

    def forward(self, x: torch.Tensor, delta):
        x, h1, h2 = self.norm.forward(x, delta)
        rows = torch.empty((x.shape[0], self._n_attn + self._ff), dtype=self._dtype, device=x.device)
        self.attn.forward(h1, rows[:, :self._n_attn])
        if self._ff:
            ops.gelu_erf(self.up_proj.forward(h2), rows[:, self._n_attn:])
        return x, self.out_proj.forward_partial32(rows)


class MitilixBody(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype, device) -> None:
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, dtype, device)
        self.positions = torch.empty((cfg.max_position_embeddings, cfg.hidden_size), dtype=dtype, device=device)
        self.layers: List[MitilixLayer] = [MitilixLayer(cfg, i, dtype, device) for i in range(cfg.num_layers)]
        self.norm = ScalarNormConv(cfg.hidden_size, 0, 0, 0, cfg.rms_norm_eps, dtype, device, _pad16(cfg.hidden_size))

    def embed(self, ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        e = self.embed_tokens
        tp = get_tp_info()
        x = ops.embed_positions(ids, e.weight, self.positions if tp.rank == 0 else None, positions, e._start, e._len)
        return get_comm().all_reduce(x) if tp.size > 1 else x

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        w = torch.randn(self.positions.shape, generator=gen, device=gen.device) * std
        self.positions = w.to(self.positions.device, self.positions.dtype)


class MitilixForCausalLM(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype: torch.dtype, device) -> None:
        if cfg.quant is not None:
            raise NotImplementedError("Mitilix runs unquantised")
        self._cfg = cfg
        self.model = MitilixBody(cfg, dtype, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, _pad16(cfg.hidden_size), dtype, device, align=8)

    @property
    def config(self) -> ModelConfig:
        return self._cfg

    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        comm = get_comm()
        comm.row_shard_ok = False
        comm.split_k_ok = False
        x = self.model.embed(input_ids, get_global_ctx().batch.positions)
        delta = None
        for layer in self.model.layers:
            x, delta = layer.forward(x, delta)
        return self.model.norm.forward(x, delta)[1]

    # ---- checkpoint names ----
    def checkpoint_map(self) -> Dict[str, Tuple]:
        """Checkpoint tensor -> ``(shape, owner, attribute, fill)``; ``fill(param, tensor)`` writes this rank's share of
        the tensor into its place in the (zero-initialised) parameter."""
        cfg, tp = self._cfg, get_tp_info()
        w = cfg.hidden_size
        out: Dict[str, Tuple] = {}

        def whole(p, t):
            p.view(-1)[:t.numel()].copy_(t.reshape(-1))

        def corner(p, t):
            p[:t.shape[0], :t.shape[1]].copy_(t)

        def taps_first(p, t):
            p.copy_(t.t())

        def vocab(start):
            def fill(p, t):
                rows = t[start:start + p.shape[0]]
                p[:rows.shape[0], :rows.shape[1]].copy_(rows)
            return fill

        def mine(t, dim):
            n = t.shape[dim] // tp.size
            return t.narrow(dim, tp.rank * n, n)

        body = self.model
        v, taps = cfg.vocab_size, cfg.input_conv_taps
        out["embed"] = ((v, w), body.embed_tokens, "weight", vocab(body.embed_tokens._start))
        out["pos"] = ((cfg.max_position_embeddings, w), body, "positions", corner)
        out["final.norm"] = ((), body.norm, "gain", whole)
        out["head"] = ((v, w), self.lm_head, "weight", vocab(self.lm_head._start))
        for i, layer in enumerate(body.layers):
            s: LatentLayer = cfg.latent_layers[i]
            a, h = layer.attn, layer.attn._h
            nq = h * s.dim_pad

            def q(p, t, s=s, h=h, nq=nq):
                p[:nq].view(h, s.dim_pad, -1)[:, :s.dim, :w].copy_(mine(t, 0).reshape(h, s.dim, w))

            def dkv(p, t, nq=nq):
                p[nq:nq + t.shape[0], :w].copy_(t)

            def uk(p, t, s=s, h=h):
                p[:, :s.kv_rank, :s.dim].copy_(mine(t, 0).reshape(h, s.dim, s.kv_rank).transpose(1, 2))

            def uv(p, t, s=s, h=h):
                p[:, :s.vdim, :s.kv_rank].copy_(mine(t, 0).reshape(h, s.vdim, s.kv_rank))

            def o(p, t, s=s, h=h):
                p[:w, :h * s.vdim_pad].unflatten(1, (h, s.vdim_pad))[:, :, :s.vdim].copy_(
                    mine(t, 1).reshape(w, h, s.vdim))

            def up(p, t):
                corner(p, mine(t, 0))

            def down(p, t, n=layer._n_attn):
                part = mine(t, 1)
                p[:w, n:n + part.shape[1]].copy_(part)

            name = f"l{i}."
            out[name + "norm1"] = ((), layer.norm, "gain", whole)
            out[name + "canon1"] = ((w, taps), layer.norm, "conv1", taps_first)
            out[name + "mix.q"] = ((s.heads * s.dim, w), a.q_proj, "weight", q)
            out[name + "mix.uk"] = ((s.heads * s.dim, s.kv_rank), a, "up_k", uk)
            out[name + "mix.uv"] = ((s.heads * s.vdim, s.kv_rank), a, "up_v", uv)
            out[name + "mix.o"] = ((w, s.heads * s.vdim), layer.out_proj, "weight", o)
            if s.kv_from is None:
                out[name + "mix.dkv"] = ((s.kv_rank, w), a.q_proj, "weight", dkv)
                out[name + "mix.dkv.norm"] = ((s.kv_rank,), a, "latent_norm", whole)
            if s.ff:
                out[name + "canon2"] = ((w, taps), layer.norm, "conv2", taps_first)
                out[name + "mlp.up"] = ((s.ff, w), layer.up_proj, "weight", up)
                out[name + "mlp.down"] = ((w, s.ff), layer.out_proj, "weight", down)
        return out

    def init_dummy(self, seed: int, std: float = 0.02, gen_device: str = "cpu") -> None:
        gen = torch.Generator(device=gen_device)
        gen.manual_seed(seed)
        for mod in self.modules():
            if mod is not self and hasattr(mod, "init_dummy"):
                mod.init_dummy(gen, std)
