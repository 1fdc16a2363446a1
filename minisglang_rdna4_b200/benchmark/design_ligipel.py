"""The Ligipel design beside the closest family at equal size: Nemotron-H (attention, state-space mixers and experts in layers
of their own). Configurations and the time of every kernel of both against its roofline; ``benchmark.design`` runs them. Where
another family's kernel is more alike (windowed attention, linear attention with a decay per head), it stands beside, too."""
from __future__ import annotations

import gc
from typing import Dict, List

import torch

from ..models.config import (
    ExpertSpec, HeadLayer, LayerSpec, LinearAttnLayer, ModelConfig, PairMixer, RotaryConfig, ScanLayer, pair_config,
)

# two blocks of (pair) (pair) (pair) (retention), experts in every layer
SIZES = {
    "small": dict(width=2048, heads=16, kv_heads=2, dim=128, window=1024, inner=4096, state=16, rank=128, rheads=8, rdim=128,
                  rvdim=256, experts=32, top=4, eff=768, layers=8, vocab=32768),
    "large": dict(width=4096, heads=32, kv_heads=2, dim=128, window=1024, inner=8192, state=16, rank=256, rheads=16, rdim=128,
                  rvdim=256, experts=32, top=4, eff=1536, layers=8, vocab=32768),
}
MAX_POS = 4096
MAMBA2 = dict(head=64, state=128, groups=8)


def ligipel_config(s: Dict) -> ModelConfig:
    d = s["dim"]
    pair = PairMixer(HeadLayer(heads=s["heads"], kv_heads=s["kv_heads"], dim=d, vdim=d, scale=d ** -0.5, window=s["window"],
                               log_bias=True, zero_sink=True, talk=True),
                     ScanLayer(inner=s["inner"], state=s["state"], dt_rank=s["rank"], taps=4))
    keep = LinearAttnLayer(heads=s["rheads"], dim=s["rdim"], vdim=s["rvdim"],
                           decay=tuple(1 - 2.0 ** -(5 + 7 * i / s["rheads"]) for i in range(s["rheads"])),
                           q_scale=s["rdim"] ** -0.5, rotary=RotaryConfig(s["rdim"], s["rdim"], MAX_POS, 1e4, interleaved=True),
                           weighted=False)
    moe = ExpertSpec(experts=s["experts"], top=s["top"], ff=s["eff"], shared_ff=s["eff"], act="silu", shared_gated=False,
                     correction=True, renorm=True)
    specs = [LayerSpec(keep if i % 4 == 3 else pair, moe=moe) for i in range(s["layers"])]
    return pair_config(specs, width=s["width"], vocab=s["vocab"], eps=1e-5, logit_scale=0.5, logit_softcap=30.0,
                       max_positions=MAX_POS)


def nemotron_config(s: Dict) -> ModelConfig:
    """A pair becomes an attention layer and a state-space layer, a retention a state-space layer; experts without a gate half
    are half as wide again."""
    kinds: List[str] = []
    for i in range(s["layers"]):
        kinds += (["mamba"] if i % 4 == 3 else ["attention", "mamba"]) + ["moe"]
    d = s["dim"]
    return ModelConfig(
        num_layers=len(kinds), num_qo_heads=s["heads"], num_kv_heads=s["kv_heads"], head_dim=d, hidden_size=s["width"],
        vocab_size=s["vocab"], intermediate_size=s["eff"] * 3 // 2 * s["top"], rms_norm_eps=1e-5,
        rotary_config=RotaryConfig(d, 0, MAX_POS, 1e4), model_type="nemotron_h", architectures=("NemotronHForCausalLM",),
        num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=s["eff"] * 3 // 2,
        shared_expert_intermediate_size=s["eff"] * 3 // 2, scoring_func="sigmoid", mlp_hidden_act="relu2",
        mamba_num_heads=s["inner"] // MAMBA2["head"], mamba_head_dim=MAMBA2["head"], ssm_state_size=MAMBA2["state"],
        mamba_n_groups=MAMBA2["groups"], layer_types=tuple(kinds), max_position_embeddings=MAX_POS)


def kernels(s: Dict) -> List[Dict]:
    """Prefill (8192 rows: four prompts of 2048) and decode (64 requests at 2048 tokens)."""
    from .. import ops
    from ..attention.paged import PagedAttentionBackend
    from ..core import Batch, Context, set_global_ctx
    from ..kvcache import LayeredKVCache, MHAKVCache
    from ..layers.residual_norm import LayerHistory
    from ..layers.rotary import get_rope_cache
    from ..ops import cuda as K
    from ..ops import moe_kernels as M
    from .design import _peaks, _time

    w, h, hk, d, win, c, ns, rank = (s[k] for k in ("width", "heads", "kv_heads", "dim", "window", "inner", "state", "rank"))
    rh, rd, rv, e, top, eff = (s[k] for k in ("rheads", "rdim", "rvdim", "experts", "top", "eff"))
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
        t, prompt = b * n, n > 1
        cu = (torch.arange(b + 1, device=dev) * n).to(torch.int32)
        seq = torch.full((b,), ctx_len, dtype=torch.int32, device=dev)
        per = ctx_len // ps
        bt = torch.randperm(b * per, generator=g, device=dev).to(torch.int32).view(b, per)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(b).to(torch.int32)
        loc = (bt[torch.arange(b, device=dev).repeat_interleave(n), pos.long() // ps].long() * ps + pos % ps).to(torch.int32)
        slots, has = torch.arange(b, dtype=torch.int32, device=dev), torch.ones(b, dtype=torch.int32, device=dev)
        # keys a row sees on average, and the distinct keys a step reads
        seen = {0: (n + 1) / 2 if prompt else ctx_len,
                win: sum(min(i + 1, win) for i in range(n)) / n if prompt else min(win, ctx_len)}
        distinct = {0: b * ctx_len, win: b * (ctx_len if prompt else min(win, ctx_len))}

        def attn_cost(reach, mixed=False):
            return (t * h * d * 4 + distinct[reach] * hk * d * 4,
                    2 * t * h * seen[reach] * (2 * d + (h if mixed else 0)))

        # ---- norms around the sublayers
        x, y, z = (rnd(t, w, dtype=f32) for _ in range(3))
        one, none = torch.ones(w, device=dev), torch.zeros(w, device=dev)
        norm = (one, none)
        add("ligipel", "residual step: pair of outputs, norm, add, norm", phase,
            lambda: ops.residual_step(x, (y, z), norm, 1e-5, bf, w, pair=(one, one), post=norm), t * w * 18)
        hist, coef = LayerHistory(6, t, w, dev), torch.ones(5, device=dev)

        def end():
            hist.count = 4
            ops.residual_step(x, y, norm, 1e-5, bf, w, post=norm, history=hist, coef=coef)
        add("ligipel", "residual step: norm, add, average over 5 results, norm", phase, end, t * w * (8 + 4 * 4 + 4 + 4 + 2))
        # ---- attention with mixed heads
        pool = LayeredKVCache(b * per, ps, [(hk, d)], bf, dev)
        pool._planes[0].copy_(rnd(*pool._planes[0].shape))
        set_global_ctx(None)
        ctx = Context(page_size=ps)
        ctx.kv_cache = pool
        set_global_ctx(ctx)
        be = PagedAttentionBackend(h, hk, d, dev, b, MAX_POS, heads=[(h, d)], talk=[(h, hk, d)])
        batch = Batch(reqs=[], phase="prefill" if prompt else "decode")
        batch.positions, batch.out_loc = pos, loc
        be.prepare_metadata(batch, bt, cu, seq, n, ctx_len, host_cu_q=cu.cpu().numpy(), host_seq_lens=seq.cpu().numpy())
        proj, q = rnd(t, (h + 2 * hk) * d), rnd(t, h, d)
        store = (pool.k_cache(0), pool.v_cache(0), loc)
        add("ligipel", "heads + store", phase,
            lambda: ops.heads_rope_store(proj, h, hk, d, d, pos, None, False, 1e-5, None, None, None, False, store),
            t * (2 * h + 4 * hk) * d * 2)
        bias = (0.5 * torch.log1p(0.5 * torch.arange(win, device=dev)))[None].repeat(h, 1).contiguous()
        extra = dict(bias=bias, sink=torch.zeros(h, device=dev), talk=torch.eye(h, device=dev) + rnd(h, h, dtype=f32))
        add("ligipel", "attention, window + distance bias + mixed heads", phase,
            lambda: be.forward_heads(q, 0, batch, scale=d ** -0.5, window=win, **extra), *attn_cost(win, True))
        add("zobelorn", "attention, window", phase, lambda: be.forward_heads(q, 0, batch, scale=d ** -0.5, window=win),
            *attn_cost(win))
        add("nemotron", "attention, global", phase, lambda: be.forward_heads(q, 0, batch, scale=d ** -0.5), *attn_cost(0))
        # ---- state-space mixers
        xz, cw, cb = rnd(t, 2 * c), rnd(c, 4, dtype=f32), rnd(c, dtype=f32)
        tail = torch.zeros(b, c, 3, dtype=bf, device=dev)
        add("ligipel", "convolution + silu", phase,
            lambda: ops.causal_conv_silu(xz[:, :c], cw, cb, tail, cu, slots, has, n), t * c * 4 + b * c * 12)
        xc, dt, bcd = rnd(t, c), rnd(t, c, dtype=f32), rnd(t, rank + 2 * ns)
        a, st = -torch.rand(c, ns, generator=g, device=dev) * 8 - 0.1, torch.zeros(b, 1, c, ns, device=dev)
        add("ligipel", "selective scan (softplus, skip and gate included)", phase,
            lambda: ops.selective_scan(xc, dt, cb - 3, a, bcd[:, rank:rank + ns], bcd[:, rank + ns:], cb, xz[:, c:], st, cu, slots,
                                       has, prompt), t * c * 10 + t * ns * 4 + 2 * b * c * ns * 4)
        mh, mp, mn, mg = c // MAMBA2["head"], MAMBA2["head"], MAMBA2["state"], MAMBA2["groups"]
        wide = c + 2 * mg * mn
        zx, cw2, cb2 = rnd(t, c + wide + mh), rnd(wide, 4), rnd(wide)
        tail2 = torch.zeros(b, wide, 3, dtype=bf, device=dev)
        add("nemotron", "convolution + silu", phase,
            lambda: ops.gdn_conv1d(zx[:, c:c + wide], cw2, tail2, cu, slots, has, cb2), t * wide * 4 + b * wide * 12)
        xbc, mst, hp = rnd(t, wide), torch.zeros(b, mh, mp, mn, device=dev), rnd(mh, dtype=f32)
        add("nemotron", "state-space recurrence", phase,
            lambda: ops.mamba2_scan(xbc, zx[:, c + wide:], hp, hp, hp, mst, cu, slots, has, mh, mg, mp, mn), t * wide * 2 + t * c * 2
            + 2 * b * c * mn * 4)
        nw = rnd(c)
        add("nemotron", "norm + gate", phase, lambda: ops.rms_norm_gate_first(xc, xz[:, c:], nw, 1e-5, c // mg), t * c * 6)
        # ---- retention
        lin, rst = rnd(t, rh * (2 * rd + 2 * rv)), torch.zeros(b, rh, rd, rv, device=dev)
        rq, rk = (lin[:, i * rh * rd:(i + 1) * rh * rd].unflatten(1, (rh, rd)) for i in range(2))
        rvv, decay = lin[:, 2 * rh * rd:2 * rh * rd + rh * rv].unflatten(1, (rh, rv)), torch.full((rh,), 0.99, device=dev)
        table = get_rope_cache(RotaryConfig(rd, rd, MAX_POS, 1e4), torch.device(dev))
        cost = (t * rh * (2 * rd + 2 * rv) * 2 + 2 * b * rh * rd * rv * 4, 4 * t * rh * rd * rv)
        add("ligipel", "retention (rotation included)", phase,
            lambda: ops.linear_attention(rq, rk, rvv, rst, cu, slots, has, decay=decay, chunked=prompt, rope=(table, pos)),
            cost[0] + t * rd * 4, cost[1])
        add("rafodra", "linear attention, decay per head", phase,
            lambda: ops.linear_attention(rq, rk, rvv, rst, cu, slots, has, decay=decay, chunked=prompt), *cost)
        o, gw = rnd(t, rh, rv), torch.ones(rv, device=dev)
        add("both", "norm per head + gate", phase,
            lambda: ops.norm_gate(o, lin[:, 2 * rh * rd + rh * rv:], gw, 1e-5, rv, False, "silu", rh * rv), t * rh * rv * 6)
        # ---- feed-forward
        hx, logits = rnd(t, w), rnd(t, e, dtype=f32)
        counts, corr = torch.empty(e, dtype=torch.int32, device=dev), rnd(e, dtype=f32) * 0.01
        add("ligipel", "routing", phase, lambda: M.moe_route(logits, top, True, "softmax", 1.0, counts, bias=corr),
            t * (e * 4 + top * 8))
        lb = rnd(t, e)
        add("nemotron", "routing", phase, lambda: M.moe_route(lb, top, True, "sigmoid", 1.0, counts, bias=corr),
            t * (e * 2 + top * 8))
        tw, ids = M.moe_route(logits, top, True, "softmax", 1.0, counts, bias=corr)
        w13, w2, sh = rnd(e, 2 * eff, w), rnd(e, w, eff), rnd(t, w)
        cost = (min(e, t * top) * 3 * w * eff * 2 + t * w * 2, 6 * t * top * w * eff)
        add("ligipel", "experts + shared sum (fp32)", phase,
            lambda: M.experts_partial32(hx, w13, w2, tw, ids, 0.0, 0.0, sh, None, counts, "silu"), cost[0] + t * w * 6, cost[1])
        del w13, w2
        n1, n2 = rnd(e, eff * 3 // 2, w), rnd(e, w, eff * 3 // 2)
        add("nemotron", "experts", phase, lambda: ops.moe_forward_plain(hx, n1, n2, tw, ids, 0, counts, "relu2"),
            cost[0] + t * w * 2, cost[1])
        del n1, n2
        gs, gp = rnd(t, 2 * eff), rnd(t, eff * 3 // 2)
        add("ligipel", "silu x mul, shared expert", phase, lambda: ops.silu_and_mul(gs), t * eff * 6)
        add("nemotron", "squared relu, shared expert", phase, lambda: ops.relu2(gp), t * eff * 6)
        rb, nb = rnd(t, w), rnd(w)
        add("nemotron", "rms norm (the residual sum is a launch of its own)", phase, lambda: ops.rms_norm(rb, nb, 1e-5), t * w * 4)
        add("nemotron", "residual sum", phase, lambda: rb + hx, t * w * 6)
        kv = MHAKVCache(1, b * per, ps, hk, d, bf, torch.device(dev))
        cs = get_rope_cache(RotaryConfig(d, d, MAX_POS, 1e4), torch.device(dev))
        add("nemotron", "heads + store", phase,
            lambda: ops.qk_norm_rope_store(proj, None, None, pos, cs, h, hk, d, 0, 1e-6, kv.k_cache(0), kv.v_cache(0), loc),
            t * (2 * h + 4 * hk) * d * 2)

        def gemm(model, name, nn, kk, dt=bf):
            am, wt = rnd(t, kk), rnd(nn, kk)

            def run():
                K.set_next_gemm_planes(n == 1 and dt == f32 and nn == w)
                return K.gemm(am, wt, None, dt)
            add(model, name, phase, run, (t * kk + nn * kk) * 2 + t * nn * (4 if dt == f32 else 2), 2 * t * nn * kk)

        gemm("both", "gemm q + k + v", (h + 2 * hk) * d, w)
        gemm("ligipel", "gemm attention out (fp32)", w, h * d, f32)
        gemm("ligipel", "gemm scan in", 2 * c, w)
        gemm("ligipel", "gemm scan dt + B + C", rank + 2 * ns, c)
        gemm("ligipel", "gemm scan dt up (fp32)", c, rank, f32)
        gemm("ligipel", "gemm scan out (fp32)", w, c, f32)
        gemm("ligipel", "gemm retention in", rh * (2 * rd + 2 * rv), w)
        gemm("ligipel", "gemm retention out (fp32)", w, rh * rv, f32)
        gemm("ligipel", "gemm router (fp32)", e, w, f32)
        gemm("ligipel", "gemm gate + up, shared expert", 2 * eff, w)
        gemm("ligipel", "gemm down, shared expert", w, eff)
        gemm("nemotron", "gemm attention out", w, h * d)
        gemm("nemotron", "gemm state-space in", c + wide + (mh + 7) // 8 * 8, w)
        gemm("nemotron", "gemm state-space out", w, c)
        gemm("nemotron", "gemm router", e, w)
        gemm("nemotron", "gemm up, shared expert", eff * 3 // 2, w)
        gemm("nemotron", "gemm down, shared expert", w, eff * 3 // 2)
        del pool, kv, x, y, z, hist, xz, zx, xbc, mst, st, rst
        gc.collect()
        torch.cuda.empty_cache()
    set_global_ctx(None)
    return rows
