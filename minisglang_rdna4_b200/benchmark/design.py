"""Prefill and decode throughput of a design beside the closest family at equal size, and the time of every kernel of
both against its roofline: Mitilix beside a Mistral-shaped decoder (grouped-query sliding-window attention, gated MLP);
Rafodra beside the Qwen3-Next hybrid (``design_rafodra.py``); Zobelorn beside Laguna (``design_zobelorn.py``); Ligipel beside
Nemotron-H (``design_ligipel.py``).

``python bench.py --design mitilix|rafodra|zobelorn|ligipel [--size small|large]`` prints one JSON line per (size, model) and one per kernel.
Random weights, synthetic token ids, one GPU. Throughput comes from CUDA events around every engine step of
``LLM.generate``; a kernel is timed with CUDA events over many launches of which each flushes L2 first."""
from __future__ import annotations

import gc
import json
import multiprocessing as mp
import os
import statistics
from typing import Callable, Dict, List, Tuple

import torch

from ..models.config import LatentLayer, ModelConfig, RotaryConfig

# width, heads, head dim, latent rank, feed-forward, window; the pair's parameter counts per layer agree within 5 %
SIZES = {
    "small": dict(width=2048, heads=16, kv_heads=4, dim=128, rank=256, ff=7680, window=1024, layers=8, vocab=32768),
    "large": dict(width=4096, heads=32, kv_heads=8, dim=128, rank=512, ff=15360, window=1024, layers=8, vocab=32768),
}
MAX_POS = 4096


def mitilix_config(s: Dict) -> ModelConfig:
    n = s["layers"]
    spec = dict(heads=s["heads"], dim=s["dim"], vdim=s["dim"], kv_rank=s["rank"], scale=s["dim"] ** -0.5,
                window=s["window"], ff=s["ff"])
    layers = tuple(LatentLayer(**spec, kv_from=None if i < n // 2 else n // 2 - 1) for i in range(n))
    return ModelConfig(
        num_layers=n, num_qo_heads=s["heads"], num_kv_heads=1, head_dim=s["rank"], hidden_size=s["width"],
        vocab_size=s["vocab"], intermediate_size=max(s["ff"], s["heads"] * s["rank"]), rms_norm_eps=1e-5,
        rotary_config=RotaryConfig(s["rank"], 0, MAX_POS, 1e4), model_type="mitilix",
        architectures=("MitilixForCausalLM",), latent_layers=layers, input_conv_taps=4, linear_conv_kernel_dim=4,
        max_position_embeddings=MAX_POS)


def mistral_config(s: Dict) -> ModelConfig:
    return ModelConfig(
        num_layers=s["layers"], num_qo_heads=s["heads"], num_kv_heads=s["kv_heads"], head_dim=s["dim"],
        hidden_size=s["width"], vocab_size=s["vocab"], intermediate_size=s["ff"] * 2 // 3, rms_norm_eps=1e-5,
        rotary_config=RotaryConfig(s["dim"], s["dim"], MAX_POS, 1e4), model_type="mistral",
        architectures=("MistralForCausalLM",), sliding_window=s["window"], max_position_embeddings=MAX_POS)


# ------------------------------------------------------------------------------------------ end to end
def throughput(cfg: ModelConfig, batches=(1, 16, 64, 256), prompt: int = 2048, out: int = 48) -> Dict:
    from ..core import SamplingParams
    from ..llm import LLM
    from ..ops import cuda as K

    llm = LLM(model_config=cfg, use_dummy_weight=True, device="cuda", max_running_req=max(batches),
              max_extend_tokens=8192, memory_ratio=0.6, seed=1, cache_type="naive")
    eng, steps = llm.engine, []
    inner = eng.forward_batch

    def timed(batch, plan, args, return_logits=False):
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record(eng.stream)
        r = inner(batch, plan, args, return_logits)
        e.record(eng.stream)
        steps.append((s, e, batch.phase, plan.num_tokens))
        return r

    eng.forward_batch = timed
    g = torch.Generator().manual_seed(3)
    res: Dict = {"decode": {}, "prefill": {}}
    launches = K.LAUNCHES
    for b in (max(batches), *batches):              # the first pass warms up
        for _ in range(2):                          # ... and so does the first of two at every batch size
            steps.clear()
            prompts = [torch.randint(0, cfg.vocab_size, (prompt,), generator=g).tolist() for _ in range(b)]
            llm.generate(prompts, SamplingParams(max_tokens=out, ignore_eos=True))
        torch.cuda.synchronize()
        dec = [s.elapsed_time(e) for s, e, ph, n in steps if ph == "decode" and n == b][4:]
        pre = [(s.elapsed_time(e), n) for s, e, ph, n in steps if ph == "prefill"]
        ms = statistics.median(dec)
        res["decode"][b] = {"ms": round(ms, 4), "tok_s": round(b / ms * 1e3)}
        res["prefill"][b] = {"tok_s": round(sum(n for _, n in pre) / sum(t for t, _ in pre) * 1e3)}
    res["launches"] = K.LAUNCHES - launches
    res["params_m"] = round(sum(t.numel() for _, t, _, _ in llm.engine.model.named_parameters()) / 1e6)
    llm.shutdown()
    del llm, eng, inner
    gc.collect()
    torch.cuda.empty_cache()
    return res


# ------------------------------------------------------------------------------------------ kernels
def _time(fn: Callable[[], None], iters: int = 20) -> float:
    """Median device time in microseconds; L2 is flushed ahead of every launch."""
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(3):
        fn()
    times = []
    for _ in range(iters):
        flush.zero_()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record()
        fn()
        e.record()
        e.synchronize()
        times.append(s.elapsed_time(e) * 1e3)
    return statistics.median(times)


def _peaks() -> Tuple[float, float]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as fh:
            p = json.load(fh)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except (OSError, KeyError):
        return 6.65e12, 1.59e15


def kernels(s: Dict) -> List[Dict]:
    """Every kernel of a Mitilix layer and the like one of the Mistral layer: prefill (8192 rows: four prompts of
    2048) and decode (64 requests at 2048 tokens)."""
    from .. import ops
    from ..attention.latent import LatentAttentionBackend
    from ..core import Batch, Context, set_global_ctx
    from ..kvcache import MHAKVCache
    from ..kvcache.mla_pool import MLALatentCache
    from ..layers.rotary import get_rope_cache
    from ..ops import cuda as K

    w, h, hk, d, r, ff, win = (s[k] for k in ("width", "heads", "kv_heads", "dim", "rank", "ff", "window"))
    dev, bf = "cuda", torch.bfloat16
    hbm, tc = _peaks()
    rows: List[Dict] = []
    g = torch.Generator(device=dev).manual_seed(0)

    def rnd(*shape, dtype=bf):
        return torch.randn(*shape, generator=g, device=dev, dtype=torch.float32).mul_(0.1).to(dtype)

    def add(model, kernel, phase, us, nbytes, flops):
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
        slots = torch.arange(b, dtype=torch.int32, device=dev)
        # keys a query row sees on average, and the distinct keys a step reads
        if n > 1:
            seen = sum(min(i + 1, win) for i in range(n)) / n
            distinct = b * n
        else:
            seen, distinct = min(win, ctx_len), b * min(win, ctx_len)
        # ---- Mitilix
        x, y = rnd(t, w, dtype=torch.float32), rnd(t, w, dtype=torch.float32)
        c1, c2 = rnd(4, w, dtype=torch.float32), rnd(4, w, dtype=torch.float32)
        gain, state = torch.ones(1, device=dev), torch.zeros(b, 3, w, device=dev)
        has = torch.ones(b, dtype=torch.int32, device=dev)
        us = _time(lambda: ops.add_scalar_norm_conv(x, y, gain, 1e-5, c1, c2, state, cu, slots, has, n, bf, w))
        add("mitilix", "norm_conv", phase, us, t * w * (4 + 4 + 4 + 2 + 2) + 2 * b * w * 12, 0)
        pool = MLALatentCache(1, b * per, ps, r, 0, bf, dev)
        pool._buf.copy_(rnd(*pool._buf.shape))
        set_global_ctx(None)
        ctx = Context(page_size=ps)
        ctx.kv_cache = pool
        set_global_ctx(ctx)
        be = LatentAttentionBackend(mitilix_config(s).latent_layers, dev, MAX_POS)
        batch = Batch(reqs=[], phase="prefill" if n > 1 else "decode")
        be.prepare_metadata(batch, bt, cu, seq, n, ctx_len, host_cu_q=cu.cpu().numpy(), host_seq_lens=seq.cpu().numpy())
        q, uk, uv = rnd(t, h, d), rnd(h, r, d), rnd(h, d, r)
        out = torch.empty(t, h, d, dtype=bf, device=dev)
        uk_rows = uk.transpose(1, 2).reshape(h * d, r).contiguous()
        ones = torch.ones(r, device=dev)
        lat = rnd(t, r)
        us = _time(lambda: ops.latent_norm_store(lat, ones, r, 1e-5, pool.rows(0), loc))
        add("mitilix", "latent_norm_store", phase, us, t * r * 4, 0)
        # all of q -> latent space -> attention -> values: fewest operations of the absorbed and expanded forms
        def forward():
            if batch.attn_metadata.prefill_plan is not None:
                batch.attn_metadata.prefill_plan.dense = None
            be.latent_forward(q, uk, uv, 0, batch, scale=d ** -0.5, window=win, out=out, expand_k=uk_rows)

        us = _time(forward)
        expand = 2 * distinct * r * h * 2 * d + 2 * t * h * seen * 2 * d
        absorb = 2 * 2 * t * h * r * d + 2 * t * h * seen * 2 * r
        add("mitilix", "latent attention (projections in and out included)", phase, us,
            t * h * d * 2 * 2 + distinct * r * 2 + 2 * h * r * d * 2, min(expand, absorb))
        if n == 1:
            q_lat = rnd(t, h, r)
            sp = be._splits(q_lat, batch.attn_metadata, win)
            us = _time(lambda: K.latent_attention(q_lat, pool.rows(0), bt, cu, seq, d ** -0.5, win, n, ctx_len, sp, merge=t > 32))
            add("mitilix", "latent_attention", phase, us, t * h * r * 4 + distinct * r * 2, 2 * t * h * seen * 2 * r)
            us = _time(lambda: ops.head_gemm(q, uk))
            add("mitilix", "head_gemm (keys)", phase, us, t * h * (d + r) * 2 + h * r * d * 2, 2 * t * h * r * d)
            us = _time(lambda: ops.head_gemm(q_lat, uv, out))
            add("mitilix", "head_gemm (values)", phase, us, t * h * (d + r) * 2 + h * r * d * 2, 2 * t * h * r * d)
        else:
            plan = batch.attn_metadata.prefill_plan
            dense = plan.dense[1]
            k_all, vt = K.gemm(dense, uk_rows), torch.empty(h * d, plan.t_pad, dtype=bf, device=dev).normal_()
            from ..ops._lib import lib

            base = plan.tables.data_ptr()
            us = _time(lambda: lib().msgl_attn_prefill_pos(
                q.data_ptr(), q.stride(0), q.stride(1), k_all.data_ptr(), vt.data_ptr(), plan.t_pad, out.data_ptr(),
                out.stride(0), out.stride(1), base, plan.n_items, t, h, d, d, win, d ** -0.5, None, None, 0, 0,
                torch.cuda.current_stream().cuda_stream))
            add("mitilix", "expanded attention (window, tcgen05)", phase, us, t * h * d * 2 * 4, 2 * t * h * seen * 2 * d)
            del k_all, vt
        u, cat = rnd(t, ff), torch.empty(t, h * d + ff, dtype=bf, device=dev)
        us = _time(lambda: ops.gelu_erf(u, cat[:, h * d:]))
        add("mitilix", "gelu_erf", phase, us, t * ff * 4, 0)
        for name, nn, kk, dt in (("gemm q+latent", h * d + r, w, bf), ("gemm up", ff, w, bf),
                                 ("gemm out+down (fp32 out)", w, h * d + ff, torch.float32)):
            a, wt = rnd(t, kk), rnd(nn, kk)
            planes = n == 1 and dt == torch.float32

            def run(a=a, wt=wt, dt=dt, planes=planes):
                K.set_next_gemm_planes(planes)
                return K.gemm(a, wt, None, dt)
            us = _time(run)
            add("mitilix", name, phase, us, (t * kk + nn * kk) * 2 + t * nn * (4 if dt == torch.float32 else 2), 2 * t * nn * kk)
        del pool, x, y, cat, u
        # ---- Mistral
        inter = ff * 2 // 3
        kv = MHAKVCache(1, b * per, ps, hk, d, bf, torch.device(dev))
        kv._buf.copy_(rnd(*kv._buf.shape))
        rx, rd, nw = rnd(t, w), rnd(t, w), rnd(w)
        us = _time(lambda: ops.rms_norm_add(rd, rx, nw, 1e-5))
        add("mistral", "rms_norm_add", phase, us, t * w * 2 * 4, 0)
        cs = get_rope_cache(RotaryConfig(d, d, MAX_POS, 1e4), torch.device(dev))
        qkv = rnd(t, (h + 2 * hk) * d)
        us = _time(lambda: ops.qk_norm_rope_store(qkv, None, None, pos, cs, h, hk, d, d, 1e-5, kv.k_cache(0), kv.v_cache(0), loc))
        add("mistral", "rope + store", phase, us, t * (2 * h + 4 * hk) * d * 2, 0)
        q3 = rnd(t, h, d)
        spl = K.choose_splits(b, hk, MAX_POS, n == 1)
        us = _time(lambda: ops.paged_attention(q3, kv.k_cache(0), kv.v_cache(0), bt, cu, seq, d ** -0.5, window=win, max_q=n,
                                               max_kv=ctx_len, decode=n == 1, splits=spl))
        add("mistral", "paged_attention (window)", phase, us, t * h * d * 4 + distinct * hk * d * 4, 2 * t * h * seen * 2 * d)
        gu = rnd(t, 2 * inter)
        us = _time(lambda: ops.silu_and_mul(gu))
        add("mistral", "silu_and_mul", phase, us, t * inter * 6, 0)
        for name, nn, kk in (("gemm qkv", (h + 2 * hk) * d, w), ("gemm o", w, h * d), ("gemm gate+up", 2 * inter, w),
                             ("gemm down", w, inter)):
            a, wt = rnd(t, kk), rnd(nn, kk)
            us = _time(lambda a=a, wt=wt: K.gemm(a, wt))
            add("mistral", name, phase, us, (t * kk + nn * kk + t * nn) * 2, 2 * t * nn * kk)
        del kv
        gc.collect()
        torch.cuda.empty_cache()
    set_global_ctx(None)
    return rows


def run(design: str, size: str, what: str, clocks) -> None:
    if design == "rafodra":
        from . import design_rafodra as d

        sizes, pair, kernel_rows = d.SIZES, (("rafodra", d.rafodra_config), ("qwen3_next", d.qwen_config)), d.kernels
    elif design == "zobelorn":
        from . import design_zobelorn as d

        sizes, pair, kernel_rows = d.SIZES, (("zobelorn", d.zobelorn_config), ("laguna", d.laguna_config)), d.kernels
    elif design == "ligipel":
        from . import design_ligipel as d

        sizes, pair, kernel_rows = d.SIZES, (("ligipel", d.ligipel_config), ("nemotron_h", d.nemotron_config)), d.kernels
    else:
        sizes, pair, kernel_rows = SIZES, (("mitilix", mitilix_config), ("mistral", mistral_config)), kernels
    names = list(sizes) if size == "all" else [size]
    for name in names:
        s = sizes[name]
        clocks.start()
        lines = []
        if what in ("all", "throughput"):
            for model, make in pair:
                # a process per model: the device memory of one is gone when the next sizes its pool
                with mp.get_context("spawn").Pool(1) as pool:
                    lines.append({"design": model, "size": name, "shape": s, "prompt": 2048, "dtype": "bf16",
                                  "data": "synthetic", **pool.apply(throughput, (make(s),))})
        if what in ("all", "kernels"):
            lines += [{"size": name, **r} for r in kernel_rows(s)]
        seen = clocks.stop()
        for ln in lines:
            print(json.dumps({**ln, "clocks": {k: seen[k] for k in ("sm_mhz", "sm_max_mhz", "reasons")}}), flush=True)
