"""The Rafodra design beside the closest family at equal size: the Qwen3-Next hybrid (gated delta net + gated full
attention, dense and mixture-of-experts feed-forwards with a gated shared expert). Configurations and the time of every
kernel of both against its roofline; ``benchmark.design`` runs them."""
from __future__ import annotations

import gc
from typing import Dict, List

import torch

from ..models.config import ExpertSpec, LatentLayer, LayerSpec, LinearAttnLayer, ModelConfig, RotaryConfig, layered_config

# two blocks of (attention, dense) (linear, experts) (linear, dense) (linear, experts)
SIZES = {
    "small": dict(width=2048, heads=16, kv_heads=4, dim=96, rot=32, rank=224, ff=5632, experts=32, top=4, eff=768, layers=8,
                  vocab=32768),
    "large": dict(width=4096, heads=32, kv_heads=8, dim=64, rot=64, rank=512, ff=11264, experts=32, top=4, eff=1536, layers=8,
                  vocab=32768),
}
MAX_POS = 4096
HD = 128          # value heads, linear-attention heads and the Qwen3-Next model's heads


def _mixers(s: Dict):
    lat = LatentLayer(heads=s["heads"], dim=s["dim"], vdim=HD, kv_rank=s["rank"], scale=HD ** -0.5, rot_dim=s["rot"],
                      rotary=RotaryConfig(s["rot"], s["rot"], MAX_POS, 1e4, interleaved=True), sink=True, gate=True)
    sizes = dict(heads=s["heads"], dim=HD, vdim=HD)
    decay = tuple(1 - 2.0 ** -(1 + 9 * i / s["heads"]) for i in range(s["heads"]))
    lightning = LinearAttnLayer(**sizes, decay=decay, act=True, joint_norm=True, gate_act="sigmoid")
    return lat, lightning, LinearAttnLayer(**sizes, gate_rank=16, tau=16.0, q_scale=HD ** -0.5)


def rafodra_config(s: Dict) -> ModelConfig:
    lat, lightning, gla = _mixers(s)
    moe = ExpertSpec(experts=s["experts"], top=s["top"], ff=s["eff"], limit=7.0, groups=8, keep=4, scale=2.0,
                     shared_ff=s["eff"], shared_limit=7.0)
    block = [LayerSpec(lat, ff=s["ff"]), LayerSpec(lightning, moe=moe), LayerSpec(lightning, ff=s["ff"]), LayerSpec(gla, moe=moe)]
    return layered_config(block * (s["layers"] // 4), width=s["width"], vocab=s["vocab"], eps=1e-5, max_positions=MAX_POS)


def qwen_config(s: Dict) -> ModelConfig:
    n = s["layers"]
    return ModelConfig(
        num_layers=n, num_qo_heads=s["heads"], num_kv_heads=s["kv_heads"], head_dim=HD, hidden_size=s["width"],
        vocab_size=s["vocab"], intermediate_size=s["ff"], rms_norm_eps=1e-6,
        rotary_config=RotaryConfig(HD, HD // 4, MAX_POS, 1e4), model_type="qwen3_next",
        architectures=("Qwen3NextForCausalLM",), qk_norm=True, num_experts=s["experts"], num_experts_per_tok=s["top"],
        moe_intermediate_size=s["eff"], shared_expert_intermediate_size=s["eff"], shared_expert_gate=True,
        decoder_sparse_step=2, linear_num_key_heads=s["heads"], linear_num_value_heads=s["heads"], linear_key_head_dim=HD,
        linear_value_head_dim=HD, attn_output_gate=True, norm_plus_one=True,
        layer_types=tuple("full_attention" if i % 4 == 0 else "linear_attention" for i in range(n)),
        max_position_embeddings=MAX_POS)


def kernels(s: Dict) -> List[Dict]:
    """Prefill (8192 rows: four prompts of 2048) and decode (64 requests at 2048 tokens)."""
    from .. import ops
    from ..attention.latent import LatentAttentionBackend
    from ..core import Batch, Context, set_global_ctx
    from ..kvcache import MHAKVCache
    from ..kvcache.mla_pool import MLALatentCache
    from ..layers.rotary import get_rope_cache
    from ..ops import cuda as K
    from ..ops import moe_kernels as M
    from .design import _peaks, _time

    w, h, hk, ff, e, top, eff = (s[k] for k in ("width", "heads", "kv_heads", "ff", "experts", "top", "eff"))
    lat, _, _ = _mixers(s)
    r, dq = lat.rank_pad, lat.dim_pad
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
        slots, has = torch.arange(b, dtype=torch.int32, device=dev), torch.ones(b, dtype=torch.int32, device=dev)
        seen = (n + 1) / 2 if n > 1 else ctx_len
        distinct = b * ctx_len
        # ---- Rafodra: norms, attention
        x, y, nw = rnd(t, w, dtype=f32), rnd(t, w, dtype=f32), torch.ones(w, device=dev)
        add("rafodra", "add + layer norm (fp32 residual)", phase, lambda: ops.add_norm(x, y, nw, 1e-5, True, bf, w), t * w * 14)
        pool = MLALatentCache(1, b * per, ps, r, 0, bf, dev)
        pool._buf.copy_(rnd(*pool._buf.shape))
        set_global_ctx(None)
        ctx = Context(page_size=ps)
        ctx.kv_cache = pool
        set_global_ctx(ctx)
        be = LatentAttentionBackend([lat], dev, MAX_POS)
        batch = Batch(reqs=[], phase="prefill" if n > 1 else "decode")
        batch.positions, batch.out_loc = pos, loc
        be.prepare_metadata(batch, bt, cu, seq, n, ctx_len, host_cu_q=cu.cpu().numpy(), host_seq_lens=seq.cpu().numpy())
        qc = rnd(t, h * dq + r + 16)
        q, c, gate = qc[:, :h * dq].unflatten(1, (h, dq)), qc[:, h * dq:h * dq + r], qc[:, h * dq + r:h * dq + r + h]
        uk, uv, sink = rnd(h, r, dq), rnd(h, HD, r), torch.zeros(h, device=dev)
        uk_rows = uk.transpose(1, 2).reshape(h * dq, r).contiguous()
        table, ones = get_rope_cache(lat.rotary, torch.device(dev)), torch.ones(r, device=dev)
        out = torch.empty(t, h, HD, dtype=bf, device=dev)
        store = (c, ones, s["rank"], 1e-5, pool.rows(0), loc, s["rot"])
        add("rafodra", "rotation + latent norm + store", phase,
            lambda: ops.latent_rope(q, s["dim"], s["rot"], table, pos, store), t * (h * s["rot"] * 4 + r * 4))

        def attend():
            if batch.attn_metadata.prefill_plan is not None:
                batch.attn_metadata.prefill_plan.dense = None
            be.latent_forward(q, uk, uv, 0, batch, scale=lat.scale, window=0, out=out, expand_k=uk_rows, sink=sink, gate=gate)

        expand = 2 * distinct * r * h * (dq + HD) + 2 * t * h * seen * (dq + HD)
        absorb = 2 * t * h * r * (dq + HD) + 2 * t * h * seen * 2 * r
        add("rafodra", "latent attention (projections in and out included)", phase, attend,
            t * h * (dq + HD) * 2 + distinct * r * 2 + h * r * (dq + HD) * 2, min(expand, absorb))
        if n == 1:
            q_lat = rnd(t, h, r)
            sp = be._splits(q_lat, batch.attn_metadata, 0)
            add("rafodra", "latent_attention", phase,
                lambda: K.latent_attention(q_lat, pool.rows(0), bt, cu, seq, lat.scale, 0, n, ctx_len, sp, merge=t > 32, sink=sink),
                t * h * r * 4 + distinct * r * 2, 2 * t * h * seen * 2 * r)
        # ---- Rafodra: linear attention
        kd = h * HD
        proj = rnd(t, 4 * kd + 16)
        lq, lk, lv = (proj[:, i * kd:(i + 1) * kd].unflatten(1, (h, HD)) for i in range(3))
        lg, low = proj[:, 3 * kd:4 * kd], proj[:, 4 * kd:]
        state = torch.zeros(b, h, HD, HD, device=dev)
        decay = torch.linspace(0.6, 0.999, h, device=dev)
        up, bias = rnd(kd, 16), torch.full((kd,), 2.0, device=dev)
        lin_bytes = t * kd * 2 * 4 + b * h * HD * HD * 8
        lin_flops = 4 * t * h * HD * HD
        args = (lq, lk, lv, state, cu, slots, has)
        add("rafodra", "linear attention, head decay", phase,
            lambda: ops.linear_attention(*args, decay=decay, act=True, chunked=n > 1), lin_bytes, lin_flops)
        add("rafodra", "linear attention, channel decay", phase,
            lambda: ops.linear_attention(*args, gate=(low, up, bias), tau=16.0, chunked=n > 1), lin_bytes, lin_flops)
        o = rnd(t, h, HD)
        wj = torch.ones(kd, device=dev)
        add("rafodra", "norm + gate, all heads", phase, lambda: ops.norm_gate(o, lg, wj, 1e-5, HD, True, "sigmoid", kd), t * kd * 6)
        add("rafodra", "norm + gate, per head", phase, lambda: ops.norm_gate(o, lg, wj[:HD], 1e-5, HD, False, "silu", kd), t * kd * 6)
        # ---- Rafodra: feed-forward
        hx = rnd(t, w)
        logits = rnd(t, e + 8, dtype=f32)
        counts = torch.empty(e, dtype=torch.int32, device=dev)
        add("rafodra", "routing (groups)", phase,
            lambda: M.moe_route(logits[:, :e], top, False, "softmax", 2.0, counts, groups=8, keep=4), t * (e * 4 + top * 8))
        w13, w2 = rnd(e, 2 * eff, w), rnd(e, w, eff)
        sh, sg = rnd(t, w), logits[:, e]
        tw, ids = M.moe_route(logits[:, :e], top, False, "softmax", 2.0, counts, groups=8, keep=4)
        moe_bytes = min(e, t * top) * 3 * w * eff * 2 + t * w * 2
        moe_flops = 6 * t * top * w * eff
        add("rafodra", "experts + shared sum (fp32)", phase,
            lambda: M.experts_partial32(hx, w13, w2, tw, ids, 7.0, 1.702, sh, sg, counts), moe_bytes + t * w * 6, moe_flops)
        up2 = rnd(t, 2 * eff)
        add("rafodra", "clamped activation", phase, lambda: ops.clamped_glu(up2, 7.0, 1.702), t * eff * 6)
        gu = rnd(t, 2 * ff)
        add("both", "silu x mul", phase, lambda: ops.silu_and_mul(gu), t * ff * 6)

        def gemm(model, name, nn, kk, dt=bf):
            a, wt = rnd(t, kk), rnd(nn, kk)

            def run():
                K.set_next_gemm_planes(n == 1 and dt == f32)
                return K.gemm(a, wt, None, dt)
            add(model, name, phase, run, (t * kk + nn * kk) * 2 + t * nn * (4 if dt == f32 else 2), 2 * t * nn * kk)

        gemm("rafodra", "gemm q + latent + gates", h * dq + r + -(-h // 16) * 16, w)
        gemm("rafodra", "gemm linear attention in", 4 * kd + 16, w)
        gemm("rafodra", "gemm out (fp32)", w, kd, f32)
        gemm("rafodra", "gemm down (fp32)", w, ff, f32)
        gemm("rafodra", "gemm router (fp32)", -(-(e + 1) // 8) * 8, w, f32)
        gemm("both", "gemm gate + up", 2 * ff, w)
        del pool, x, y, proj, gu, up2
        # ---- Qwen3-Next
        kv = MHAKVCache(1, b * per, ps, hk, HD, bf, torch.device(dev))
        kv._buf.copy_(rnd(*kv._buf.shape))
        rd, nb = rnd(t, w), rnd(w)
        add("qwen3_next", "rms norm (the residual sum is a launch of its own)", phase, lambda: ops.rms_norm(rd, nb, 1e-6), t * w * 4)
        cs = get_rope_cache(RotaryConfig(HD, HD // 4, MAX_POS, 1e4), torch.device(dev))
        qkv, qw = rnd(t, (h + 2 * hk) * HD), rnd(HD)
        add("qwen3_next", "head norms + rotation + store", phase,
            lambda: ops.qk_norm_rope_store(qkv, qw, qw, pos, cs, h, hk, HD, HD // 4, 1e-6, kv.k_cache(0), kv.v_cache(0), loc),
            t * (2 * h + 4 * hk) * HD * 2)
        q3 = rnd(t, h, HD)
        plan = K.PrefillPlan(cu.cpu().numpy(), seq.cpu().numpy(), dev) if n > 1 else None
        spl = K.choose_splits(b, hk, MAX_POS, n == 1)
        add("qwen3_next", "paged_attention", phase,
            lambda: K.paged_attention(q3, kv.k_cache(0), kv.v_cache(0), bt, cu, seq, HD ** -0.5, max_q=n, max_kv=ctx_len,
                                      decode=n == 1, splits=None if n > 1 else spl, plan=plan),
            t * h * HD * 4 + distinct * hk * HD * 4, 2 * t * h * seen * 2 * HD)
        mixed, cw = rnd(t, 3 * kd), rnd(3 * kd, 4)
        conv_state = torch.zeros(b, 3 * kd, 3, dtype=bf, device=dev)
        add("qwen3_next", "gdn convolution", phase, lambda: ops.gdn_conv1d(mixed, cw, conv_state, cu, slots, has), t * 3 * kd * 4)
        ab, al = rnd(t, 2 * h), torch.zeros(h, device=dev)
        add("qwen3_next", "gdn recurrence", phase,
            lambda: ops.gdn_recurrent(mixed, ab[:, :h], ab[:, h:], al, al, state, cu, slots, has, h, h, HD, HD),
            lin_bytes, 6 * t * h * HD * HD)
        z, gw = rnd(t, kd), rnd(HD)
        add("qwen3_next", "gated norm, per head", phase, lambda: ops.rms_norm_gated(o, z, gw, 1e-6), t * kd * 6)
        lb = rnd(t, e)
        add("qwen3_next", "routing", phase,
            lambda: M.moe_route(lb, top, True, "softmax", 1.0, counts), t * (e * 2 + top * 8))
        tw, ids = M.moe_route(lb, top, True, "softmax", 1.0, counts)
        add("qwen3_next", "experts", phase, lambda: K.moe_forward(hx, w13, w2, tw, ids, 0, counts), moe_bytes + t * w * 2, moe_flops)
        for name, nn, kk in (("gemm qkv", (h + 2 * hk) * HD, w), ("gemm o", w, kd), ("gemm gdn in", 4 * kd + -(-2 * h // 8) * 8, w),
                             ("gemm down", w, ff)):
            gemm("qwen3_next", name, nn, kk)
        del kv, w13, w2
        gc.collect()
        torch.cuda.empty_cache()
    set_global_ctx(None)
    return rows
