"""Rafodra: a decoder of sequential layers over an fp32 residual stream, every layer with a mixer and a feed-forward of
its own kind and size (``models.config.LayerSpec``):

* token embedding times a constant; layer norms without a bias (``layers/residual_norm.py``);
* latent attention with a rotary part, a sink and a head gate; a layer may read the latents of an earlier one
  (``layers/latent_attention.py``);
* linear attention with a decaying state, one decay per head or one per key channel and token
  (``layers/linear_attention.py``);
* a dense gated feed-forward, a mixture of clamped experts with a gated shared one (``layers/moe.py``), or none.

Every sublayer hands an fp32 result (or the K ranges of its last product) to the next norm, which adds it."""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .. import ops
from ..core import get_global_ctx
from ..layers import BaseOP, ParallelLMHead, ReplicatedLinear, RowParallelLinear, VocabParallelEmbedding
from ..layers.gated_mlp import DenseGatedMLP
from ..layers.latent_attention import LatentAttentionLayer
from ..layers.linear_attention import LinearAttentionLayer
from ..layers.moe import ResidualExperts
from ..layers.residual_norm import ResidualNorm
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from .config import LatentLayer, ModelConfig


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class RafodraLayer(BaseOP):
    def __init__(self, cfg: ModelConfig, layer_id: int, dtype, device) -> None:
        spec = cfg.layer_specs[layer_id]
        w, wp, tp = cfg.hidden_size, _pad16(cfg.hidden_size), get_tp_info().size
        self._dtype, self._latent = dtype, isinstance(spec.mixer, LatentLayer)
        self.norm1 = ResidualNorm(w, cfg.rms_norm_eps, True, dtype, device, wp)
        if self._latent:
            self.mixer = LatentAttentionLayer(spec.mixer, cfg.latent_row(layer_id), wp, cfg.rms_norm_eps, dtype, device)
        else:
            self.mixer = LinearAttentionLayer(spec.mixer, cfg.state_row(layer_id), wp, cfg.rms_norm_eps, dtype, device)
        self.out_proj = RowParallelLinear(self.mixer.out_width * tp, wp, dtype, device)
        self._has_mlp = bool(spec.ff or spec.moe)
        if self._has_mlp:
            self.norm2 = ResidualNorm(w, cfg.rms_norm_eps, True, dtype, device, wp)
            self.mlp = (ResidualExperts(spec.moe, w, wp, dtype, device) if spec.moe is not None
                        else DenseGatedMLP(spec.ff, wp, dtype, device))

    def forward(self, x: torch.Tensor, delta):
        x, h = self.norm1.forward(x, delta)
        if self._latent:
            rows = torch.empty((x.shape[0], self.mixer.out_width), dtype=self._dtype, device=x.device)
            self.mixer.forward(h, rows)
        else:
            rows = self.mixer.forward(h)
        delta = self.out_proj.forward_partial32(rows)
        if self._has_mlp:
            x, h = self.norm2.forward(x, delta)
            delta = self.mlp.forward_partial32(h)
        return x, delta


class RafodraBody(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype, device) -> None:
        self._scale = cfg.embedding_multiplier
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, dtype, device)
        self.layers: List[RafodraLayer] = [RafodraLayer(cfg, i, dtype, device) for i in range(cfg.num_layers)]
        self.norm = ResidualNorm(cfg.hidden_size, cfg.rms_norm_eps, True, dtype, device, _pad16(cfg.hidden_size))

    def embed(self, ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        e = self.embed_tokens
        x = ops.embed_positions(ids, e.weight, None, positions, e._start, e._len, scale=self._scale)
        return get_comm().all_reduce(x) if get_tp_info().size > 1 else x


class RafodraForCausalLM(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype: torch.dtype, device) -> None:
        if cfg.quant is not None:
            raise NotImplementedError("Rafodra runs unquantised")
        self._cfg = cfg
        self.model = RafodraBody(cfg, dtype, device)
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
        """Checkpoint tensor -> ``(shape, owner, attribute, fill)``, see ``models.weight._load_mapped``."""
        cfg, tp = self._cfg, get_tp_info()
        w, v, body = cfg.hidden_size, cfg.vocab_size, self.model
        out: Dict[str, Tuple] = {}

        def whole(p, t):
            p.view(-1)[:t.numel()].copy_(t.reshape(-1))

        def vocab(start):
            def fill(p, t):
                rows = t[start:start + p.shape[0]]
                p[:rows.shape[0], :rows.shape[1]].copy_(rows)
            return fill

        def mine(t, dim=0):
            n = t.shape[dim] // tp.size
            return t.narrow(dim, tp.rank * n, n)

        def rows_at(at, share=True):
            """Rows of a matrix (this rank's share of them) into the rows from ``at`` on."""
            def fill(p, t):
                t = mine(t) if share else t
                p[at:at + t.shape[0], :t.shape[1]].copy_(t)
            return fill

        def heads_at(at, h, n, n_pad):
            """``[heads * n, width]`` into blocks of ``n_pad`` rows from ``at`` on."""
            def fill(p, t):
                p[at:at + h * n_pad].view(h, n_pad, -1)[:, :n, :t.shape[1]].copy_(mine(t).reshape(h, n, -1))
            return fill

        def head_columns(h, n, n_pad):
            """``[width, heads * n]`` into blocks of ``n_pad`` columns."""
            def fill(p, t):
                p[:w, :h * n_pad].unflatten(1, (h, n_pad))[:, :, :n].copy_(mine(t, 1).reshape(w, h, n))
            return fill

        def per_head(h, n, n_pad):
            def fill(p, t):
                p[:h * n_pad].view(h, n_pad)[:, :n].copy_(mine(t).reshape(h, n))
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
        out["final.norm"] = ((w,), body.norm, "weight", whole)
        out["head"] = ((v, w), self.lm_head, "weight", vocab(self.lm_head._start))
        for i, layer in enumerate(body.layers):
            n, spec = f"l{i}.", cfg.layer_specs[i]
            out[n + "norm1"] = ((w,), layer.norm1, "weight", whole)
            m, s = layer.mixer, spec.mixer
            h, name = m._h, n + "mix."
            out[name + "o"] = ((w, s.heads * s.vdim), layer.out_proj, "weight", head_columns(h, s.vdim, s.vdim_pad))
            if layer._latent:
                nq = h * s.dim_pad

                def uk(p, t, s=s, h=h, m=m):
                    p[:, :s.kv_rank, :s.dim].copy_(mine(t).reshape(h, s.dim, s.kv_rank).transpose(1, 2))
                    m.rotary_identity()

                def uv(p, t, s=s, h=h):
                    p[:, :s.vdim, :s.kv_rank].copy_(mine(t).reshape(h, s.vdim, s.kv_rank))

                def share(p, t):
                    p.copy_(mine(t))

                dq = s.dim + s.rot_dim
                out[name + "q"] = ((s.heads * dq, w), m.q_proj, "weight", heads_at(0, h, dq, s.dim_pad))
                out[name + "uk"] = ((s.heads * s.dim, s.kv_rank), m, "up_k", uk)
                out[name + "uv"] = ((s.heads * s.vdim, s.kv_rank), m, "up_v", uv)
                out[name + "sink"] = ((s.heads,), m, "sink", share)
                out[name + "g"] = ((s.heads, w), m.q_proj, "weight", rows_at(m._gate_at))
                if s.kv_from is None:
                    out[name + "dkv"] = ((s.kv_rank + s.rot_dim, w), m.q_proj, "weight", rows_at(nq, share=False))
                    out[name + "dkv.norm"] = ((s.kv_rank,), m, "latent_norm", whole)
            else:
                kd, vd = m._kd, m._vd
                for part, at, d, pad in (("q", 0, s.dim, s.dim_pad), ("k", kd, s.dim, s.dim_pad),
                                         ("v", 2 * kd, s.vdim, s.vdim_pad), ("g", 2 * kd + vd, s.vdim, s.vdim_pad)):
                    out[name + part] = ((s.heads * d, w), m.in_proj, "weight", heads_at(at, h, d, pad))
                if s.joint_norm:
                    out[name + "norm"] = ((s.heads * s.vdim,), m, "norm", per_head(h, s.vdim, s.vdim_pad))
                else:
                    out[name + "norm"] = ((s.vdim,), m, "norm", whole)
                if s.decay is None:
                    r = s.gate_rank
                    out[name + "a1"] = ((r, w), m.in_proj, "weight", rows_at(2 * kd + 2 * vd, share=False))
                    out[name + "a2"] = ((s.heads * s.dim, r), m, "decay_up", heads_at(0, h, s.dim, s.dim_pad))
                    out[name + "a2.b"] = ((s.heads * s.dim,), m, "decay_bias", per_head(h, s.dim, s.dim_pad))
            if not layer._has_mlp:
                continue
            out[n + "norm2"] = ((w,), layer.norm2, "weight", whole)
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
                out[name + "shared.sg"] = ((1, w), mlp, "router", rows_at(e.experts, share=False))
        return out

    def init_dummy(self, seed: int, std: float = 0.02, gen_device: str = "cpu") -> None:
        gen = torch.Generator(device=gen_device)
        gen.manual_seed(seed)
        for mod in self.modules():
            if mod is not self and hasattr(mod, "init_dummy"):
                mod.init_dummy(gen, std)
