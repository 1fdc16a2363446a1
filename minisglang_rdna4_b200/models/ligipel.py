"""Ligipel: a decoder of sequential layers over an fp32 residual stream, with a layer norm (weight and bias) before and after
every sublayer, ``x <- x + norm_b(sublayer(norm_a(x)))``, and a depth average after every layer: what goes on is a weighted
sum of the results of all layers so far (``layers/residual_norm.py``). Every layer has a mixer and a feed-forward of its own
kind and size (``models.config.LayerSpec``):

* two mixers side by side on the same rows, half the sum of their normed outputs: attention in a sliding window with a
  logarithmic distance bias, a zero score in the softmax denominator and mixed heads (``layers/head_attention.py``), and a
  selective scan (``layers/selective_scan.py``);
* or retention: linear attention with one decay per head and rotary positions (``layers/linear_attention.py``);
* a mixture of experts chosen by corrected scores, with a shared one (``layers/moe.py``), or none.

Every sublayer hands an fp32 result (or the K ranges of its last product) to the step that norms it, adds it, averages over
the depth and norms the sum for the next sublayer, in one pass."""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .. import ops
from ..core import get_global_ctx
from ..layers import BaseOP, ParallelLMHead, RowParallelLinear, VocabParallelEmbedding
from ..layers.head_attention import HeadAttentionLayer
from ..layers.linear_attention import LinearAttentionLayer
from ..layers.moe import ResidualExperts
from ..layers.residual_norm import BiasedNorm, LayerHistory
from ..layers.selective_scan import SelectiveScanLayer
from ..parallel.comm import get_comm
from ..parallel.info import get_tp_info
from .config import ModelConfig, PairMixer


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class LigipelLayer(BaseOP):
    def __init__(self, cfg: ModelConfig, layer_id: int, dtype, device) -> None:
        spec = cfg.layer_specs[layer_id]
        w, wp, tp = cfg.hidden_size, _pad16(cfg.hidden_size), get_tp_info().size
        self._pair = isinstance(spec.mixer, PairMixer)
        self.norm1, self.norm1b = BiasedNorm(w, device), BiasedNorm(w, device)
        if self._pair:
            self.mixer = HeadAttentionLayer(spec.mixer.left, cfg.head_row(layer_id), wp, cfg.rms_norm_eps, dtype, device,
                                            cfg.max_position_embeddings)
            self.scan = SelectiveScanLayer(spec.mixer.right, cfg.state_row(layer_id), wp, dtype, device)
            self.scan_out = RowParallelLinear(self.scan.out_width * tp, wp, dtype, device)
            self.left_weight = torch.empty((w,), dtype=torch.float32, device=device)
            self.right_weight = torch.empty((w,), dtype=torch.float32, device=device)
        else:
            self.mixer = LinearAttentionLayer(spec.mixer, cfg.state_row(layer_id), wp, cfg.rms_norm_eps, dtype, device)
        self.out_proj = RowParallelLinear(self.mixer.out_width * tp, wp, dtype, device)
        self._has_mlp = spec.moe is not None
        if self._has_mlp:
            self.norm2, self.norm2b = BiasedNorm(w, device), BiasedNorm(w, device)
            self.mlp = ResidualExperts(spec.moe, w, wp, dtype, device)
        self.dwa = torch.empty((layer_id + 2,), dtype=torch.float32, device=device)

    def mix(self, h: torch.Tensor):
        """The mixer's output and, for two of them, the weights of their norms."""
        out = self.out_proj.forward_partial32(self.mixer.forward(h))
        if not self._pair:
            return out, None
        return (out, self.scan_out.forward_partial32(self.scan.forward(h))), (self.left_weight, self.right_weight)

    def init_dummy(self, gen: torch.Generator, std: float = 0.02) -> None:
        self.dwa = torch.zeros_like(self.dwa)
        self.dwa[-1] = 1.0
        if self._pair:
            self.left_weight, self.right_weight = torch.ones_like(self.left_weight), torch.ones_like(self.right_weight)


class LigipelBody(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype, device) -> None:
        w = cfg.hidden_size
        self._dtype, self._eps, self._cols, self._scale = dtype, cfg.rms_norm_eps, _pad16(w), cfg.output_multiplier
        self.embed_tokens = VocabParallelEmbedding(cfg.vocab_size, w, dtype, device)
        self.embed_norm = BiasedNorm(w, device)
        self.layers: List[LigipelLayer] = [LigipelLayer(cfg, i, dtype, device) for i in range(cfg.num_layers)]
        self.norm = BiasedNorm(w, device)

    def _post_load_self(self) -> None:
        # the logits' factor, taken ahead of the product
        self._last = (self.norm.weight * self._scale, self.norm.bias * self._scale)

    def embed(self, ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        e = self.embed_tokens
        x = ops.embed_positions(ids, e.weight, None, positions, e._start, e._len)
        return get_comm().all_reduce(x) if get_tp_info().size > 1 else x

    def step(self, x, delta, norm, **more):
        return ops.residual_step(x, delta, norm, self._eps, self._dtype, self._cols, **more)

    def forward(self, ids: torch.Tensor) -> torch.Tensor:
        x = self.embed(ids, get_global_ctx().batch.positions)
        history = LayerHistory(len(self.layers), x.shape[0], x.shape[1], x.device)
        entry = [(layer.norm1.weight, layer.norm1.bias) for layer in self.layers] + [self._last]
        x, h = self.step(None, x, entry[0], post=(self.embed_norm.weight, self.embed_norm.bias), history=history)
        for i, layer in enumerate(self.layers):
            delta, pair = layer.mix(h)
            end = dict(history=history, coef=layer.dwa)
            post = (layer.norm1b.weight, layer.norm1b.bias)
            if layer._has_mlp:
                x, h = self.step(x, delta, (layer.norm2.weight, layer.norm2.bias), pair=pair, post=post)
                delta, pair, post = layer.mlp.forward_partial32(h), None, (layer.norm2b.weight, layer.norm2b.bias)
            x, h = self.step(x, delta, entry[i + 1], pair=pair, post=post, **end)
        return h


class LigipelForCausalLM(BaseOP):
    def __init__(self, cfg: ModelConfig, dtype: torch.dtype, device) -> None:
        if cfg.quant is not None:
            raise NotImplementedError("Ligipel runs unquantised")
        self._cfg = cfg
        self.model = LigipelBody(cfg, dtype, device)
        self.lm_head = ParallelLMHead(cfg.vocab_size, _pad16(cfg.hidden_size), dtype, device, align=8)

    @property
    def config(self) -> ModelConfig:
        return self._cfg

    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        comm = get_comm()
        comm.row_shard_ok = False
        comm.split_k_ok = False
        return self.model.forward(input_ids)

    # ---- checkpoint names ----
    def checkpoint_map(self) -> Dict[str, Tuple]:
        """Checkpoint tensor -> ``(shape, owner, attribute, fill)``, see ``models.weight._load_mapped``."""
        cfg, tp = self._cfg, get_tp_info()
        w, v, body = cfg.hidden_size, cfg.vocab_size, self.model
        out: Dict[str, Tuple] = {}

        def mine(t, dim=0):
            n = t.shape[dim] // tp.size
            return t.narrow(dim, tp.rank * n, n)

        def whole(p, t):
            p.copy_(t)

        def vocab(start):
            def fill(p, t):
                rows = t[start:start + p.shape[0]]
                p[:rows.shape[0], :rows.shape[1]].copy_(rows)
            return fill

        def rows_at(at, share=True):
            """Rows of a matrix (this rank's share of them) into the rows from ``at`` on."""
            def fill(p, t):
                t = mine(t) if share else t
                p[at:at + t.shape[0], :t.shape[1]].copy_(t)
            return fill

        def heads_at(at, n, width, order=None, share=False):
            """``[heads * n, width]`` into blocks of ``width`` rows from ``at`` on; ``order``: where its rows come from."""
            def fill(p, t):
                t = (mine(t) if share else t).reshape(-1, n, t.shape[1])
                t = t if order is None else t[:, order]
                p[at:at + t.shape[0] * width].view(t.shape[0], width, -1)[:, :n, :t.shape[2]].copy_(t)
            return fill

        def head_columns(n, width):
            """This rank's share of ``[width, heads * n]`` into blocks of ``width`` columns."""
            def fill(p, t):
                t = mine(t, 1).reshape(w, -1, n)
                p[:w, :t.shape[1] * width].unflatten(1, (t.shape[1], width))[:, :, :n].copy_(t)
            return fill

        def columns(p, t):
            part = mine(t, 1)
            p[:part.shape[0], :part.shape[1]].copy_(part)

        def columns_at(at, rows):
            def fill(p, t):
                columns(p[at:at + rows], t)
            return fill

        def front(p, t):
            """This rank's share of the first dimension; zeros past it."""
            t = mine(t)
            p[tuple(slice(0, n) for n in t.shape)].copy_(t)

        def expert(e, at):
            return lambda p, t: rows_at(at)(p[e], t)

        def expert_down(e):
            return lambda p, t: columns(p[e], t)

        def norm(name, owner):
            out[name], out[name + ".b"] = ((w,), owner, "weight", whole), ((w,), owner, "bias", whole)

        out["embed"] = ((v, w), body.embed_tokens, "weight", vocab(body.embed_tokens._start))
        norm("embed.norm", body.embed_norm)
        norm("final.norm", body.norm)
        out["head"] = ((v, w), self.lm_head, "weight", vocab(self.lm_head._start))
        for i, layer in enumerate(body.layers):
            n, spec = f"l{i}.", cfg.layer_specs[i]
            for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer._has_mlp else ()):
                norm(n + name, getattr(layer, name))
            out[n + "dwa"] = ((i + 2,), layer, "dwa", whole)
            m = layer.mixer
            if layer._pair:
                a, s = spec.mixer.left, spec.mixer.right
                name, h, d = n + "mix.left.", m._h, m._d
                out[name + "q"] = ((a.heads * a.dim, w), m.in_proj, "weight", heads_at(0, a.dim, d))
                out[name + "k"] = ((a.kv_heads * a.dim, w), m.in_proj, "weight", heads_at(h * d, a.dim, d))
                out[name + "v"] = ((a.kv_heads * a.vdim, w), m.in_proj, "weight", heads_at((h + m._hk) * d, a.vdim, d))
                out[name + "r1"], out[name + "r2"] = ((a.heads,), m, "r1", whole), ((a.heads,), m, "r2", whole)
                out[name + "talk"] = ((a.heads, a.heads), m, "talk", whole)
                out[name + "o"] = ((w, a.heads * a.vdim), layer.out_proj, "weight", head_columns(a.vdim, d))
                out[name + "out"] = ((w,), layer, "left_weight", whole)
                name, c, scan = n + "mix.right.", s.inner, layer.scan
                # x and z channels: this rank's share of each half
                out[name + "in"] = ((2 * c, w), scan.in_proj, "weight",
                                    lambda p, t, c=c, cp=scan._c: (rows_at(0)(p, t[:c]), rows_at(cp)(p, t[c:])))
                out[name + "conv"], out[name + "conv.b"] = ((c, s.taps), scan, "conv", front), ((c,), scan, "conv_bias", front)

                def x_proj(p, t, s=s, r=scan._r, ns=scan._n):
                    for at, part in ((0, t[:s.dt_rank]), (r, t[s.dt_rank:s.dt_rank + s.state]),
                                     (r + ns, t[s.dt_rank + s.state:])):
                        columns_at(at, part.shape[0])(p, part)

                out[name + "x"] = ((s.dt_rank + 2 * s.state, c), scan.x_proj, "weight", x_proj)
                out[name + "dt"] = ((c, s.dt_rank), scan.dt_proj, "weight", front)
                out[name + "dt.b"] = ((c,), scan, "dt_bias", front)
                out[name + "A_log"], out[name + "D"] = ((c, s.state), scan, "a_log", front), ((c,), scan, "skip", front)
                out[name + "o"] = ((w, c), layer.scan_out, "weight", columns)
                out[name + "out"] = ((w,), layer, "right_weight", whole)
            else:
                s, name = spec.mixer, n + "mix."
                # a pair of the rotation (i, i + dims / 2) becomes neighbours (2 i, 2 i + 1)
                half = (s.rotary.rotary_dim if s.rotary else 0) // 2
                order = [x for j in range(half) for x in (j, j + half)] + list(range(2 * half, s.dim))
                kd, vd = m._kd, m._vd
                for part, at, size, pad, rows in (("q", 0, s.dim, s.dim_pad, order), ("k", kd, s.dim, s.dim_pad, order),
                                                  ("v", 2 * kd, s.vdim, s.vdim_pad, None),
                                                  ("g", 2 * kd + vd, s.vdim, s.vdim_pad, None)):
                    out[name + part] = ((s.heads * size, w), m.in_proj, "weight", heads_at(at, size, pad, rows, True))
                out[name + "o"] = ((w, s.heads * s.vdim), layer.out_proj, "weight", head_columns(s.vdim, s.vdim_pad))
            if not layer._has_mlp:
                continue
            e, mlp, name = spec.moe, layer.mlp, n + "mlp."
            out[name + "router"] = ((e.experts, w), mlp, "router", rows_at(0, share=False))
            out[name + "correction"] = ((e.experts,), mlp, "correction", whole)
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
