"""The Zobelorn design beside the closest family at equal size: Laguna (sliding-window and global layers, weighted head
norms, gated attention output, sigmoid-routed experts with a plain shared one). Configurations and the time of every kernel of
both against its roofline; ``benchmark.design`` runs them. The chunks are as long as the longest sequence, so that a chunked
layer of one model sees what a global layer of the other sees."""
from __future__ import annotations

import gc
from typing import Dict, List

import torch

from ..models.config import ExpertSpec, HeadLayer, LayerSpec, ModelConfig, RotaryConfig, heads_config

# two blocks of (chunk) (window) (chunk) (chunk that reads the one before it); the first feed-forward is dense
SIZES = {
    "small": dict(width=2048, heads=16, kv_heads=4, dim=128, window=1024, ff=5632, experts=32, top=4, eff=768, layers=8,
                  vocab=32768),
    "large": dict(width=4096, heads=32, kv_heads=8, dim=128, window=1024, ff=11264, experts=32, top=4, eff=1536, layers=8,
                  vocab=32768),
}
MAX_POS = 4096
LLAMA = {"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
         "original_max_position_embeddings": 8192.0}


def _mixers(s: Dict):
    d = s["dim"]
    sizes = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5)
    window = HeadLayer(**sizes, rotary=RotaryConfig(d, d, MAX_POS, 2e5, {"rope_type": "linear", "factor": 2.0}),
                       window=s["window"], softcap=30.0, joint_norm=True, gate=True)
    chunk = HeadLayer(**sizes, rotary=RotaryConfig(d, d, MAX_POS, 5e5, LLAMA, interleaved=True), chunk=MAX_POS,
                      unit_norm=True)
    return window, chunk


def zobelorn_config(s: Dict) -> ModelConfig:
    from dataclasses import replace

    window, chunk = _mixers(s)
    moe = ExpertSpec(experts=s["experts"], top=s["top"], ff=s["eff"], shared_ff=s["eff"], act="silu", scoring="sigmoid",
                     on_input=True, shared_gated=False)
    specs: List[LayerSpec] = []
    for i in range(s["layers"]):
        mixer = (chunk, window, chunk, replace(chunk, kv_from=i - 1))[i % 4]
        specs.append(LayerSpec(mixer, ff=s["ff"]) if i == 0 else LayerSpec(mixer, moe=moe))
    return heads_config(specs, width=s["width"], vocab=s["vocab"], eps=1e-5, residual_multiplier=0.8, max_positions=MAX_POS)


def laguna_config(s: Dict) -> ModelConfig:
    n, d = s["layers"], s["dim"]
    return ModelConfig(
        num_layers=n, num_qo_heads=s["heads"], num_kv_heads=s["kv_heads"], head_dim=d, hidden_size=s["width"],
        vocab_size=s["vocab"], intermediate_size=s["ff"], rms_norm_eps=1e-6, rotary_config=RotaryConfig(d, d, MAX_POS, 5e5),
        model_type="laguna", architectures=("LagunaForCausalLM",), qk_norm=True, num_experts=s["experts"],
        num_experts_per_tok=s["top"], moe_intermediate_size=s["eff"], shared_expert_intermediate_size=s["eff"],
        first_k_dense_replace=1, scoring_func="sigmoid", sliding_window=s["window"],
        layer_types=tuple("sliding_attention" if i % 4 == 1 else "full_attention" for i in range(n)),
        max_position_embeddings=MAX_POS)


def kernels(s: Dict) -> List[Dict]:
    """Prefill (8192 rows: four prompts of 2048) and decode (64 requests at 2048 tokens)."""
    from .. import ops
    from ..attention.paged import PagedAttentionBackend
    from ..core import Batch, Context, set_global_ctx
    from ..kvcache import LayeredKVCache, MHAKVCache
    from ..layers.rotary import get_rope_cache
    from ..ops import cuda as K
    from ..ops import moe_kernels as M
    from .design import _peaks, _time

    w, h, hk, d, win, ff, e, top, eff = (s[k] for k in ("width", "heads", "kv_heads", "dim", "window", "ff", "experts", "top",
                                                        "eff"))
    window, chunk = _mixers(s)
    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    hbm, tc = _peaks()
    rows: List[Dict] = []
    g = torch.Generator(device=dev).manual_seed(0)

    def rnd(*shape, dtype=bf):
        return torch.randn(*shape, generator=g, device=dev, dtype=f32).mul_(0.1).to(dtype)

    def add(model, kernel, phase, fn, nbytes, flops=0):
        us = _time(fn)
        floor = max(nbytes / hbm, flops / tc) * 1e6
        rows.append({"model": model, "kernel": kernel, "phase": phase, "us": round(us, 2), "roofline_us": round(floor, 2),
                     "of_measured": round(floor / us, 3)})

    ps, ctx_len = 16, 2048
    for phase, b, n in (("prefill", 4, 2048), ("decode", 64, 1)):
        t = b * n
        cu = (torch.arange(b + 1, device=dev) * n).to(torch.int32)
        seq = torch.full((b,), ctx_len, dtype=torch.int32, device=dev)
        per = ctx_len // ps
        bt = torch.randperm(b * per, generator=g, device=dev).to(torch.int32).view(b, per)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(b).to(torch.int32)
        loc = (bt[torch.arange(b, device=dev).repeat_interleave(n), pos.long() // ps].long() * ps + pos % ps).to(torch.int32)
        # keys a row sees on average, and the distinct keys a step reads
        seen = {0: (n + 1) / 2 if n > 1 else ctx_len,
                win: sum(min(i + 1, win) for i in range(n)) / n if n > 1 else min(win, ctx_len)}
        distinct = {0: b * ctx_len, win: b * (ctx_len if n > 1 else min(win, ctx_len))}

        def attn_cost(reach, gated=False):
            return t * h * d * (6 if gated else 4) + distinct[reach] * hk * d * 4, 2 * t * h * seen[reach] * 2 * d

        # ---- Zobelorn: norms, heads, attention
        x, y, nw = rnd(t, w, dtype=f32), rnd(t, w, dtype=f32), torch.ones(w, device=dev)
        add("zobelorn", "norm of the output + add + norm (fp32 residual)", phase,
            lambda: ops.add_norm(x, y, nw, 1e-5, False, bf, w, nw, 0.8), t * w * 14)
        pool = LayeredKVCache(b * per, ps, [(hk, d)], bf, dev)
        pool._planes[0].copy_(rnd(*pool._planes[0].shape))
        set_global_ctx(None)
        ctx = Context(page_size=ps)
        ctx.kv_cache = pool
        set_global_ctx(ctx)
        be = PagedAttentionBackend(h, hk, d, dev, b, MAX_POS, heads=[(h, d)])
        batch = Batch(reqs=[], phase="prefill" if n > 1 else "decode")
        batch.positions, batch.out_loc = pos, loc
        be.prepare_metadata(batch, bt, cu, seq, n, ctx_len, host_cu_q=cu.cpu().numpy(), host_seq_lens=seq.cpu().numpy())
        proj = rnd(t, (2 * h + 2 * hk) * d)
        qw, kw = torch.ones(h * d, device=dev), torch.ones(hk * d, device=dev)
        store = (pool.k_cache(0), pool.v_cache(0), loc)
        q = rnd(t, h, d)
        for name, spec, weights in (("window", window, (qw, kw)), ("chunk", chunk, (None, None))):
            table = get_rope_cache(spec.rotary, torch.device(dev))
            inter = spec.rotary.interleaved
            add("zobelorn", f"head norms + rotation + store, {name}", phase,
                lambda: ops.heads_rope_store(proj, h, hk, d, d, pos, table, inter, 1e-5, *weights, None, spec.unit_norm, store),
                t * (2 * h + 4 * hk) * d * 2)
        add("zobelorn", "head norm + rotation, queries alone", phase,
            lambda: ops.heads_rope_store(proj, h, hk, d, d, pos, table, True, 1e-5, None, None, None, True, None),
            t * 2 * h * d * 2)
        gate = proj[:, (h + 2 * hk) * d:]
        add("zobelorn", "attention, window + soft cap + gate", phase,
            lambda: be.forward_heads(q, 0, batch, scale=d ** -0.5, window=win, softcap=30.0, gate=gate), *attn_cost(win, True))
        add("zobelorn", "attention, chunk", phase, lambda: be.forward_heads(q, 0, batch, scale=d ** -0.5, chunk=MAX_POS),
            *attn_cost(0))
        # ---- feed-forward
        hx = rnd(t, w)
        logits = rnd(t, e, dtype=f32)
        counts = torch.empty(e, dtype=torch.int32, device=dev)
        add("zobelorn", "routing", phase, lambda: M.moe_route(logits, top, False, "sigmoid", 1.0, counts), t * (e * 4 + top * 8))
        w13, w2, sh = rnd(e, 2 * eff, w), rnd(e, w, eff), rnd(t, w)
        tw, ids = M.moe_route(logits, top, False, "sigmoid", 1.0, counts)
        moe_bytes = min(e, t * top) * 3 * w * eff * 2 + t * w * 2
        moe_flops = 6 * t * top * w * eff
        add("zobelorn", "experts + shared sum (fp32)", phase,
            lambda: M.experts_partial32(hx, w13, w2, tw, ids, 0.0, 0.0, sh, None, counts, "silu", True),
            moe_bytes + t * w * 6, moe_flops)
        gu, gs = rnd(t, 2 * ff), rnd(t, 2 * eff)
        add("both", "silu x mul", phase, lambda: ops.silu_and_mul(gu), t * ff * 6)
        add("both", "silu x mul, shared expert", phase, lambda: ops.silu_and_mul(gs), t * eff * 6)

        def gemm(model, name, nn, kk, dt=bf):
            a, wt = rnd(t, kk), rnd(nn, kk)

            def run():
                K.set_next_gemm_planes(n == 1 and dt == f32)
                return K.gemm(a, wt, None, dt)
            add(model, name, phase, run, (t * kk + nn * kk) * 2 + t * nn * (4 if dt == f32 else 2), 2 * t * nn * kk)

        gemm("zobelorn", "gemm q + k + v + gates", (2 * h + 2 * hk) * d, w)
        gemm("zobelorn", "gemm q + k + v", (h + 2 * hk) * d, w)
        gemm("zobelorn", "gemm q", h * d, w)
        gemm("zobelorn", "gemm out (fp32)", w, h * d, f32)
        gemm("zobelorn", "gemm down (fp32)", w, ff, f32)
        gemm("zobelorn", "gemm router (fp32)", e, w, f32)
        gemm("both", "gemm gate + up", 2 * ff, w)
        gemm("both", "gemm gate + up, shared expert", 2 * eff, w)
        gemm("both", "gemm down, shared expert", w, eff)
        del pool, x, y, proj, gu
        # ---- Laguna
        kv = MHAKVCache(1, b * per, ps, hk, d, bf, torch.device(dev))
        kv._buf.copy_(rnd(*kv._buf.shape))
        rd, nb = rnd(t, w), rnd(w)
        add("laguna", "rms norm (the residual sum is a launch of its own)", phase, lambda: ops.rms_norm(rd, nb, 1e-6), t * w * 4)
        add("laguna", "residual sum", phase, lambda: rd + hx, t * w * 6)
        cs = get_rope_cache(RotaryConfig(d, d, MAX_POS, 1e4), torch.device(dev))
        qkv, hw = rnd(t, (h + 2 * hk) * d), rnd(d)
        add("laguna", "head norms + rotation + store", phase,
            lambda: ops.qk_norm_rope_store(qkv, hw, hw, pos, cs, h, hk, d, d, 1e-6, kv.k_cache(0), kv.v_cache(0), loc),
            t * (2 * h + 4 * hk) * d * 2)
        plan = K.PrefillPlan(cu.cpu().numpy(), seq.cpu().numpy(), dev) if n > 1 else None
        spl = None if n > 1 else K.choose_splits(b, hk, MAX_POS, True)
        for name, reach, p in (("paged attention, window", win, None), ("paged attention, global", 0, plan)):
            add("laguna", name, phase,
                lambda: K.paged_attention(q, kv.k_cache(0), kv.v_cache(0), bt, cu, seq, d ** -0.5, window=reach, max_q=n,
                                          max_kv=ctx_len, decode=n == 1, splits=spl, plan=p), *attn_cost(reach))
        hg = rnd(t, h)
        add("laguna", "output gate (tensor ops)", phase,
            lambda: (q * torch.nn.functional.softplus(hg.float()).to(bf).unsqueeze(-1)), t * h * d * 4)
        lb = rnd(t, e)
        add("laguna", "routing", phase, lambda: M.moe_route(lb, top, True, "sigmoid", 1.0, counts), t * (e * 2 + top * 8))
        tw, ids = M.moe_route(lb, top, True, "sigmoid", 1.0, counts)
        add("laguna", "experts", phase, lambda: K.moe_forward(hx, w13, w2, tw, ids, 0, counts), moe_bytes + t * w * 2, moe_flops)
        for name, nn, kk in (("gemm qkv", (h + 2 * hk) * d, w), ("gemm o", w, h * d), ("gemm down", w, ff), ("gemm router", e, w)):
            gemm("laguna", name, nn, kk)
        del kv, w13, w2
        gc.collect()
        torch.cuda.empty_cache()
    set_global_ctx(None)
    return rows
