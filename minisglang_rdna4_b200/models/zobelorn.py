"""Zobelorn: a decoder of sequential layers over an fp32 residual stream with a norm before and after every sublayer,
``x <- x + m norm_b(sublayer(norm_a(x)))``; every layer with attention and a feed-forward of its own kind and size
(``models.config.LayerSpec`` with ``HeadLayer`` mixers):

* token embedding times a constant; RMS norms whose weights are stored around zero (``layers/residual_norm.py``);
* attention in a sliding window, with queries and keys normed over all heads together, capped scores and a gated output,
  or attention in chunks, with unit-normed queries and keys after the rotation; a layer may read the keys and values of
  an earlier one (``layers/head_attention.py``);
* a dense gated feed-forward, a mixture of experts whose weights multiply their inputs, with a shared one
  (``layers/moe.py``), or none.

Every sublayer hands an fp32 result (or the K ranges of its last product) to the next norm, which norms it, scales it,
adds it to the stream and norms the sum, in one pass."""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .. import ops
from ..core import get_global_ctx
from ..layers import BaseOP, ParallelLMHead, RowParallelLinear, VocabParallelEmbedding
from ..layers.gated_mlp import DenseGatedMLP
from ..layers.head_attention import HeadAttentionLayer
from ..layers.moe import ResidualExperts
from ..layers.residual_norm import ResidualNorm
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from .config import ModelConfig


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class ZobelornLayer(BaseOP):
    def __init__(self, cfg: ModelConfig, layer_id: int, dtype, device) -> None:
        spec = cfg.layer_specs[layer_id]
        w, wp, tp = cfg.hidden_size, _pad16(cfg.hidden_size), get_tp_info().size
        self._mult = cfg.residual_multiplier

        def norm() -> ResidualNorm:
            return ResidualNorm(w, cfg.rms_norm_eps, False, dtype, device, wp)

        self.norm1, self.norm1b = norm(), norm()
        self.mixer = HeadAttentionLayer(spec.mixer, cfg.head_row(layer_id), wp, cfg.rms_norm_eps, dtype, device)
        self.out_proj = RowParallelLinear(self.mixer.out_width * tp, wp, dtype, device)
        self._has_mlp = bool(spec.ff or spec.moe)
        if self._has_mlp:
            self.norm2, self.norm2b = norm(), norm()
            self.mlp = (ResidualExperts(spec.moe, w, wp, dtype, device) if spec.moe is not None
                        else DenseGatedMLP(spec.ff, wp, dtype, device))

    def forward(self, x: torch.Tensor, delta, post):
        """``(residual, last sublayer's output, its norm)`` -> the same after this layer."""
        x, h = self.norm1.forward(x, delta, post, self._mult)
        delta, post = self.out_proj.forward_partial32(self.mixer.forward(h)), self.norm1b
        if self._has_mlp:
            x, h = self.norm2.forward(x, delta, post, self._mult)
            delta, post = self.mlp.forward_partial32(h), self.norm2b
        return x, delta, post


class ZobelornBody(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype, device) -> None:
        self._scale = cfg.embedding_multiplier
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, dtype, device)
        self.layers: List[ZobelornLayer] = [ZobelornLayer(cfg, i, dtype, device) for i in range(cfg.num_layers)]
        self.norm = ResidualNorm(cfg.hidden_size, cfg.rms_norm_eps, False, dtype, device, _pad16(cfg.hidden_size))

    def embed(self, ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        e = self.embed_tokens
        x = ops.embed_positions(ids, e.weight, None, positions, e._start, e._len, scale=self._scale)
        return get_comm().all_reduce(x) if get_tp_info().size > 1 else x


class ZobelornForCausalLM(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype: torch.dtype, device) -> None:
        if cfg.quant is not None:
            raise NotImplementedError("Zobelorn runs unquantised")
        self._cfg = cfg
        self.model = ZobelornBody(cfg, dtype, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, _pad16(cfg.hidden_size), dtype, device, align=8)

    @property
    def config(self) -> ModelConfig:
        return self._cfg

    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        comm = get_comm()
        comm.row_shard_ok = False
        comm.split_k_ok = False
        x = self.model.embed(input_ids, get_global_ctx().batch.positions)
        delta = post = None
        for layer in self.model.layers:
            x, delta, post = layer.forward(x, delta, post)
        return self.model.norm.forward(x, delta, post, self._cfg.residual_multiplier)[1]

    # ---- checkpoint names ----
    def checkpoint_map(self) -> Dict[str, Tuple]:
        """Checkpoint tensor -> ``(shape, owner, attribute, fill)``, see ``models.weight._load_mapped``."""
        cfg, tp = self._cfg, get_tp_info()
        w, v, body = cfg.hidden_size, cfg.vocab_size, self.model
        out: Dict[str, Tuple] = {}

        def around_zero(p, t):
            p.copy_(t + 1.0)

        def vocab(start):
            def fill(p, t):
                rows = t[start:start + p.shape[0]]
                p[:rows.shape[0], :rows.shape[1]].copy_(rows)
            return fill

        def mine(t, dim=0):
            n = t.shape[dim] // tp.size
            return t.narrow(dim, tp.rank * n, n)

        def heads_of_rank(t, total, local, n):
            """``[total * n, ...]`` -> this rank's heads ``[local, n, ...]`` (fewer heads than ranks: copies)."""
            first = tp.rank * total // tp.size
            return t.reshape(total, n, *t.shape[1:])[first:first + local]

        def heads_at(at, total, local, n, d):
            """Rows of this rank's heads into blocks of ``d`` rows from ``at`` on."""
            def fill(p, t):
                p[at:at + local * d].view(local, d, -1)[:, :n, :t.shape[1]].copy_(heads_of_rank(t, total, local, n))
            return fill

        def head_weights(total, local, n, d):
            def fill(p, t):
                p.view(local, d)[:, :n].copy_(heads_of_rank(t, total, local, n))
            return fill

        def head_columns(total, local, n, d):
            def fill(p, t):
                part = heads_of_rank(t.t(), total, local, n)               # [local, n, width]
                p[:w, :local * d].unflatten(1, (local, d))[:, :, :n].copy_(part.permute(2, 0, 1))
            return fill

        def rows_at(at, share=True):
            """Rows of a matrix (this rank's share of them) into the rows from ``at`` on."""
            def fill(p, t):
                t = mine(t) if share else t
                p[at:at + t.shape[0], :t.shape[1]].copy_(t)
            return fill

        def columns(p, t):
            part = mine(t, 1)
            p[:w, :part.shape[1]].copy_(part)

        def expert(e, at):
            def fill(p, t):
                rows_at(at)(p[e], t)
            return fill

        def expert_down(e):
            def fill(p, t):
                columns(p[e], t)
            return fill

        out["embed"] = ((v, w), body.embed_tokens, "weight", vocab(body.embed_tokens._start))
        out["final.norm"] = ((w,), body.norm, "weight", around_zero)
        out["head"] = ((v, w), self.lm_head, "weight", vocab(self.lm_head._start))
        for i, layer in enumerate(body.layers):
            n, spec = f"l{i}.", cfg.layer_specs[i]
            for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer._has_mlp else ()):
                out[n + name] = ((w,), getattr(layer, name), "weight", around_zero)
            m, s, name = layer.mixer, spec.mixer, n + "mix."
            h, hk, d = m._h, m._hk, m._d
            out[name + "q"] = ((s.heads * s.dim, w), m.in_proj, "weight", heads_at(0, s.heads, h, s.dim, d))
            out[name + "o"] = ((w, s.heads * s.vdim), layer.out_proj, "weight", head_columns(s.heads, h, s.vdim, d))
            if m._own:
                out[name + "k"] = ((s.kv_heads * s.dim, w), m.in_proj, "weight", heads_at(h * d, s.kv_heads, hk, s.dim, d))
                out[name + "v"] = ((s.kv_heads * s.vdim, w), m.in_proj, "weight",
                                   heads_at((h + hk) * d, s.kv_heads, hk, s.vdim, d))
            if s.gate:
                out[name + "g"] = ((s.heads * s.vdim, w), m.in_proj, "weight", heads_at(m._gate_at, s.heads, h, s.vdim, d))
            if s.joint_norm:
                out[name + "q.norm"] = ((s.heads * s.dim,), m, "q_norm", head_weights(s.heads, h, s.dim, d))
                if m._own:
                    out[name + "k.norm"] = ((s.kv_heads * s.dim,), m, "k_norm", head_weights(s.kv_heads, hk, s.dim, d))
            if not layer._has_mlp:
                continue
            mlp, name = layer.mlp, n + "mlp."
            if spec.moe is None:
                out[name + "gate"] = ((spec.ff, w), mlp.gate_up, "weight", rows_at(0))
                out[name + "up"] = ((spec.ff, w), mlp.gate_up, "weight", rows_at(mlp._ff))
                out[name + "down"] = ((w, spec.ff), mlp.down, "weight", columns)
                continue
            e = spec.moe
            out[name + "router"] = ((e.experts, w), mlp, "router", rows_at(0, share=False))
            for j in range(e.experts):
                out[f"{name}e{j}.gate"] = ((e.ff, w), mlp, "w13", expert(j, 0))
                out[f"{name}e{j}.up"] = ((e.ff, w), mlp, "w13", expert(j, mlp._ff))
                out[f"{name}e{j}.down"] = ((w, e.ff), mlp, "w2", expert_down(j))
            if e.shared_ff:
                out[name + "shared.gate"] = ((e.shared_ff, w), mlp.shared_up, "weight", rows_at(0))
                out[name + "shared.up"] = ((e.shared_ff, w), mlp.shared_up, "weight", rows_at(mlp._shared_ff))
                out[name + "shared.down"] = ((w, e.shared_ff), mlp.shared_down, "weight", columns)
        return out

    def init_dummy(self, seed: int, std: float = 0.02, gen_device: str = "cpu") -> None:
        gen = torch.Generator(device=gen_device)
        gen.manual_seed(seed)
        for mod in self.modules():
            if mod is not self and hasattr(mod, "init_dummy"):
                mod.init_dummy(gen, std)
