"""Kernels of the Zobelorn design against plain fp32 restatements of the same step, and the engine on the GPU."""
import pytest
import torch

import plain_zobelorn as plain
import zobelorn_util as U
from minisglang_rdna4_b200 import LLM, SamplingParams, ops
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.models.config import RotaryConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer
from test_mitilix_gpu import _batch, _gen

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF = torch.bfloat16


# ---------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("width,cols", [(320, 320), (200, 208), (97, 112), (4096, 4096), (1000, 1008), (16384, 16384)])
@pytest.mark.parametrize("rows", [3, 600])
@pytest.mark.parametrize("mult", [1.0, 0.45])
def test_norm_of_the_output_scaled_and_added(width, cols, rows, mult):
    from minisglang_rdna4_b200.ops.cuda import SplitPartial

    g = _gen(width)
    x, planes = torch.randn(rows, width, generator=g) * 2 + 1, torch.randn(3, rows, cols, generator=g)
    w, wb = torch.randn(width, generator=g), torch.randn(width, generator=g)
    for dtype, tol in ((torch.float32, 3e-5), (BF, 1e-2)):
        for delta, added in ((planes[0], planes[0]), (planes, planes.sum(0))):
            want = ref.add_norm(x, added, w, 1e-3, False, dtype, cols, wb, mult)
            dd = delta.to(DEV)
            got = ops.add_norm(x.to(DEV), SplitPartial(dd, torch.float32) if delta is planes else dd, w.to(DEV), 1e-3, False,
                               dtype, cols, wb.to(DEV), mult)
            torch.testing.assert_close(got[0].cpu(), want[0], rtol=2e-5, atol=2e-5)
            torch.testing.assert_close(got[1].float().cpu(), want[1].float(), rtol=tol, atol=tol)


@pytest.mark.parametrize("hq,hk,dim,rot,width", [
    (4, 2, 64, 64, 64), (5, 1, 40, 16, 64), (3, 1, 20, 12, 64), (16, 4, 128, 128, 128), (48, 8, 112, 96, 128), (6, 6, 72, 34, 128),
    (2, 1, 256, 256, 256), (40, 8, 250, 64, 256), (1, 1, 1, 0, 64), (7, 1, 80, 0, 128), (200, 4, 64, 32, 64), (2, 2, 300, 300, 512)])
@pytest.mark.parametrize("interleaved", [True, False])
def test_head_norms_rotation_and_store(hq, hk, dim, rot, width, interleaved):
    g = _gen(hq + dim + rot)
    t, ps, pages = (37, 16, 9) if hq != 3 and hk != 2 else (2500, 16, 160)     # more rows than CTAs
    pos = torch.randint(0, 900, (t,), generator=g).int()
    loc = torch.randperm(pages * ps, generator=g)[:t].int()
    loc[5] = -1                                             # a row that stores nothing
    table = get_rope_cache(RotaryConfig(dim, rot, 900, 1e4), "cpu") if rot else None
    proj = torch.zeros(t, hq + 2 * hk + 1, width)
    proj[..., :dim] = torch.randn(t, hq + 2 * hk + 1, dim, generator=g) * 3
    qw, kw = torch.zeros(hq, width), torch.zeros(hk, width)
    qw[:, :dim], kw[:, :dim] = torch.randn(hq, dim, generator=g), torch.randn(hk, dim, generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (BF, 1e-2)):
        x = proj.view(t, -1).to(dtype)
        for joint, unit, own in ((True, False, True), (False, True, True), (True, True, True), (False, False, True),
                                 (False, True, False), (True, False, False)):
            ws = (qw.view(-1), kw.view(-1) if own else None) if joint else (None, None)
            pools = [[torch.full((pages, hk, ps, width), 3.0, dtype=dtype, device=d) for _ in range(2)] for d in ("cpu", DEV)]
            keep = loc >= 0
            want = ref.heads_rope_store(x, hq, hk, width, dim, pos, table, interleaved, 1e-3, *ws, None, unit, None)
            if own:
                ref.heads_rope_store(x[keep], hq, hk, width, dim, pos[keep], table, interleaved, 1e-3, *ws, None, unit,
                                     (*pools[0], loc[keep]))
            got = ops.heads_rope_store(x.to(DEV), hq, hk, width, dim, pos.to(DEV), None if table is None else table.to(DEV),
                                       interleaved, 1e-3, *(None if w is None else w.to(DEV) for w in ws), None, unit,
                                       (*pools[1], loc.to(DEV)) if own else None)
            torch.testing.assert_close(got.float().cpu(), want.float(), rtol=tol, atol=tol)
            for a, b in zip(*pools):
                torch.testing.assert_close(b.float().cpu(), a.float(), rtol=tol, atol=tol)


def test_joint_norm_from_sums_of_other_ranks():
    g = _gen(1)
    x, w = torch.randn(9, 6 * 64, generator=g), torch.randn(4 * 64, generator=g)
    sums = torch.rand(9, 2, generator=g) * 500
    pools = [[torch.zeros(2, 1, 16, 64, device=d) for _ in range(2)] for d in ("cpu", DEV)]
    loc, pos = torch.arange(9).int(), torch.arange(9).int()
    kw = torch.randn(64, generator=g)
    for d, pool in zip(("cpu", DEV), pools):
        args = [z.to(d) for z in (x, pos, w, kw, sums, loc)]
        out = ops.heads_rope_store(args[0], 4, 1, 64, 64, args[1], None, False, 1e-5, args[2], args[3], (args[4], 512, 128), False,
                                   (*pool, args[5]))
        if d == "cpu":
            want = out
    torch.testing.assert_close(out.cpu(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(pools[1][0].cpu(), pools[0][0], rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("t", [1, 37, 300])
@pytest.mark.parametrize("shared", [True, False])
def test_experts_weighted_on_their_input(t, shared):
    g = _gen(t)
    e, k, width, wp, ff = 6, 3, 72, 80, 48
    x = torch.randn(t, wp, generator=g)
    w13, w2 = torch.randn(e, 2 * ff, wp, generator=g) * 0.3, torch.randn(e, 96, ff, generator=g) * 0.3
    logits = torch.randn(t, 8, generator=g)
    from minisglang_rdna4_b200.ops import moe_kernels

    counts = torch.empty(e, dtype=torch.int32, device=DEV)
    tw, ids = moe_kernels.moe_route(logits.to(DEV)[:, :e], k, False, "sigmoid", 1.0, counts)
    ww, wi = ref.moe_route(logits[:, :e], k, False, "sigmoid")
    assert torch.equal(ids.cpu(), wi)
    torch.testing.assert_close(tw.cpu(), ww, rtol=1e-5, atol=1e-7)
    sh = torch.randn(t, wp, generator=g)
    for dtype, tol in ((torch.float32, 1e-6), (BF, 1e-2)):
        a = [z.to(dtype) for z in (x, w13, w2)]
        extra = sh.to(dtype) if shared else None
        want = ref.experts_partial32(*a, ww, wi, 0.0, 0.0, extra, None, "silu", True)
        got = ops.experts_partial32(*[z.to(DEV) for z in a], tw, ids, 0.0, 0.0, None if extra is None else extra.to(DEV), None,
                                    counts, "silu", True)
        assert float((got.cpu() - want).abs().max() / want.abs().max()) < tol


# ---------------------------------------------------------------------------------- attention
REACHES = [("window", 1), ("window", 64), ("window", 100), ("window", 129), ("window", 3000), ("chunk", 1), ("chunk", 64),
           ("chunk", 100), ("chunk", 130), ("chunk", 3000)]


def _run(q, pool, bt, cu, seq, scale, kind, size, cap, gate, form):
    """``form``: general, split (decode rows over several key ranges) or tc (tcgen05)."""
    from minisglang_rdna4_b200.ops import cuda as K

    reach = dict(window=size if kind == "window" else 0, chunk=size if kind == "chunk" else 0)
    k, v = pool
    max_q = int((cu[1:] - cu[:-1]).max())
    extra = dict(softcap=cap, gate=gate, **reach)
    if form == "tc":
        assert K.prefill_heads_tc_ok(q, k, scale)
        group = q.shape[1] // k.shape[1]
        plan = K.PrefillPlan(cu.cpu().numpy(), seq.cpu().numpy(), q.device, reach["window"], reach["chunk"], 256 if group % 2 else 128)
        return K.prefill_attention_tc(q, k, v, bt, plan, scale, **extra)
    return K.paged_attention(q, k, v, bt, cu, seq, scale, max_q=max_q, max_kv=int(seq.max()), decode=max_q == 1,
                             splits=4 if form == "split" else 1, **extra)


@pytest.mark.parametrize("hq,hk,d,form", [
    (4, 2, 64, "general"), (6, 2, 64, "general"), (10, 1, 128, "general"), (3, 3, 256, "general"), (24, 1, 64, "general"),
    (4, 2, 64, "tc"), (3, 1, 64, "tc"), (8, 2, 128, "tc"), (6, 2, 128, "tc"), (2, 2, 128, "tc")])
@pytest.mark.parametrize("kind,size", REACHES)
def test_prompt_attention(hq, hk, d, form, kind, size):
    g = _gen(size + d)
    lens, starts, ps = [300, 2, 129, 1, 65], [0, 200, 77, 64, 190], 16
    cu, seq, bt = _batch(lens, starts, ps, 80, g)
    k, v = (torch.randn(80, hk, ps, d, generator=g).to(BF) for _ in range(2))
    q = (torch.randn(sum(lens), hq, d, generator=g) * 2).to(BF)
    wide = (torch.randn(sum(lens), hq * d + 64, generator=g) * 2).to(BF)
    pool = [z.to(DEV) for z in (q, bt, cu, seq, wide)]
    planes = U.split_planes(k.to(DEV), v.to(DEV))
    scale = d ** -0.5
    for cap, gated in ((0.0, False), (2.5, True)):
        gate, dgate = (wide[:, 64:], pool[4][:, 64:]) if gated else (None, None)
        want = ref.paged_attention(q.float(), k.float(), v.float(), bt, cu, seq, scale, window=size if kind == "window" else 0,
                                   chunk=size if kind == "chunk" else 0, softcap=cap,
                                   gate=None if gate is None else gate.float())
        got = _run(pool[0], planes, *pool[1:4], scale, kind, size, cap, dgate, form)
        torch.testing.assert_close(got.float().cpu(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("hq,hk,d", [(4, 2, 64), (8, 1, 128), (3, 1, 128), (12, 1, 64), (5, 5, 256), (40, 2, 64)])
@pytest.mark.parametrize("kind,size", REACHES)
def test_decode_attention(hq, hk, d, kind, size):
    g = _gen(size + d)
    ps = 16
    starts = [0, 62, 63, 64, 99, 100, 129, 255, 400]
    cu, seq, bt = _batch([1] * len(starts), starts, ps, 120, g)
    k, v = (torch.randn(120, hk, ps, d, generator=g).to(BF) for _ in range(2))
    q = (torch.randn(len(starts), hq, d, generator=g) * 2).to(BF)
    gate = (torch.randn(len(starts), hq * d, generator=g) * 2).to(BF)
    dq, dbt, dcu, dseq, dgate = (z.to(DEV) for z in (q, bt, cu, seq, gate))
    planes = U.split_planes(k.to(DEV), v.to(DEV))
    for cap, gated in ((0.0, False), (2.5, True)):
        want = ref.paged_attention(q.float(), k.float(), v.float(), bt, cu, seq, d ** -0.5, window=size if kind == "window" else 0,
                                   chunk=size if kind == "chunk" else 0, softcap=cap, gate=gate.float() if gated else None)
        for form in ("general", "split"):
            got = _run(dq, planes, dbt, dcu, dseq, d ** -0.5, kind, size, cap, dgate if gated else None, form)
            torch.testing.assert_close(got.float().cpu(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("hq,hk,d", [(4, 2, 64), (3, 1, 128), (6, 2, 256), (2, 1, 512)])
@pytest.mark.parametrize("kind,size", REACHES)
def test_fp32_attention(hq, hk, d, kind, size):
    g = _gen(size + d)
    lens, starts, ps = [300, 2, 1, 1], [0, 130, 64, 255], 16
    cu, seq, bt = _batch(lens, starts, ps, 60, g)
    k, v = (torch.randn(60, hk, ps, d, generator=g) for _ in range(2))
    q, gate = torch.randn(sum(lens), hq, d, generator=g) * 2, torch.randn(sum(lens), hq * d, generator=g) * 2
    dev = [z.to(DEV) for z in (q, k, v, bt, cu, seq, gate)]
    reach = dict(window=size if kind == "window" else 0, chunk=size if kind == "chunk" else 0)
    for cap, gated in ((0.0, False), (2.5, True)):
        want = ref.paged_attention(q.double(), k.double(), v.double(), bt, cu, seq, d ** -0.5, softcap=cap,
                                   gate=gate if gated else None, **reach)
        got = ops.paged_attention(*dev[:6], d ** -0.5, softcap=cap, gate=dev[6] if gated else None, max_q=300, max_kv=300, **reach)
        torch.testing.assert_close(got.cpu(), want.float(), rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("form", ["general", "tc", "decode", "split", "fp32"])
@pytest.mark.parametrize("kind,size", [("window", 64), ("window", 70), ("window", 128), ("window", 131), ("chunk", 64), ("chunk", 70),
                                       ("chunk", 128), ("chunk", 131)])
@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 127, 128, 143, 144, 255])
def test_a_loud_key_is_seen_exactly_within_reach(form, kind, size, at):
    """At the borders of pages, tiles, windows and chunks; every row of a prompt, and rows decoded one by one."""
    n, d, ps = 300, 64, 16
    q, k, v, bt = U.loud_key(n, at, n, d, ps)
    want = [p in U.seen_rows(kind, at, size, n) for p in range(n)]
    reach = dict(window=size if kind == "window" else 0, chunk=size if kind == "chunk" else 0)
    dt = torch.float32 if form == "fp32" else BF
    q, k, v = q.to(DEV, dt), k.to(DEV, dt), v.to(DEV, dt)
    planes = U.split_planes(k, v)
    if form in ("decode", "split"):
        rows = sorted({p for p in (at - 1, at, at + 1, at + size - 2, at + size - 1, at + size, at // size * size + size - 1,
                                   at // size * size + size, at // size * size - 1) if 0 <= p < n})
        m = len(rows)
        seq = torch.tensor([p + 1 for p in rows], dtype=torch.int32, device=DEV)
        cu = torch.arange(m + 1, dtype=torch.int32, device=DEV)
        got = _run(q[:m].contiguous(), planes, bt.repeat(m, 1).to(DEV), cu, seq, 1.0, kind, size, 0.0, None,
                   "split" if form == "split" else "general")
        assert [bool(x) for x in got[:, 0, 0] > 4.5] == [want[p] for p in rows]
        return
    cu, seq = torch.tensor([0, n], dtype=torch.int32, device=DEV), torch.tensor([n], dtype=torch.int32, device=DEV)
    if form == "fp32":
        got = ops.paged_attention(q, *planes, bt.to(DEV), cu, seq, 1.0, max_q=n, max_kv=n, **reach)
    else:
        got = _run(q, planes, bt.to(DEV), cu, seq, 1.0, kind, size, 0.0, None, form)
    assert [bool(x) for x in got[:, 0, 0] > 4.5] == want


@pytest.mark.parametrize("cap", [0.25, 4.0, 50.0, 60.0, 300.0])
@pytest.mark.parametrize("form", ["general", "tc"])
def test_capped_scores_far_out(form, cap):
    """Scores many times the cap (and of its size), of both signs, in both kernels: the weights are those of the capped
    scores, also where a row's keys all score close to the negative cap."""
    n, d, ps = 130, 64, 16
    g = _gen(3)
    k, v = (torch.randn(9, 1, ps, d, generator=g).to(BF) for _ in range(2))
    q = (torch.randn(n, 2, d, generator=g) * torch.tensor([0.1, 1.0, 8.0, 60.0, 200.0]).repeat(26)[:, None, None]).to(BF)
    k[..., 0] = 3.0
    q[7::10, :, 0] = -cap
    bt = torch.randperm(9, generator=g).int()[None]
    cu, seq = torch.tensor([0, n], dtype=torch.int32), torch.tensor([n], dtype=torch.int32)
    want = ref.paged_attention(q.float(), k.float(), v.float(), bt, cu, seq, 1.0, softcap=cap)
    got = _run(q.to(DEV), U.split_planes(k.to(DEV), v.to(DEV)), bt.to(DEV), cu.to(DEV), seq.to(DEV), 1.0, "window", 0, cap, None,
               form)
    torch.testing.assert_close(got.float().cpu(), want, rtol=2e-2, atol=2e-2)


def test_rows_do_not_depend_on_how_a_prompt_was_cut():
    """The tensor-core form sees keys in absolute blocks: a row is the same bit for bit whatever came with it."""
    g = _gen(5)
    n, d, ps = 400, 128, 16
    k, v = (torch.randn(25, 2, ps, d, generator=g).to(DEV, BF) for _ in range(2))
    q = torch.randn(n, 4, d, generator=g).to(DEV, BF)
    bt = torch.randperm(25, generator=g).int()[None].to(DEV)
    planes = U.split_planes(k, v)

    def rows(lo, hi, kind, size):
        cu = torch.tensor([0, hi - lo], dtype=torch.int32, device=DEV)
        return _run(q[lo:hi].contiguous(), planes, bt, cu, torch.tensor([hi], dtype=torch.int32, device=DEV), 0.1, kind, size, 3.0,
                    None, "tc")

    for kind, size in (("window", 100), ("chunk", 150)):
        whole = rows(0, n, kind, size)
        for cuts in ([0, 128, 256, 400], [0, 37, 300, 302, 400]):
            parts = torch.cat([rows(a, b, kind, size) for a, b in zip(cuts, cuts[1:])])
            torch.testing.assert_close(parts, whole, rtol=1e-2, atol=1e-2)


# ---------------------------------------------------------------------------------- the engine on the GPU
# rows of 64, 128 and 256, groups of odd and even size, experts beyond one tile
BIG = U.config([
    U.chunk(6, 2, 64, 48, 100, mlp=U.dense(96)), U.window(5, 1, 80, 96, 76, rot=64, cap=9.0, scale=0.1, mlp=U.moe(16, 4, 48)),
    U.chunk(12, 2, 64, 48, 130, scale=0.9, kv_from=0, mlp=U.moe(5, 5, 33, shared=0)), U.window(2, 2, 128, 128, 128, cap=20.0, scale=0.09),
    U.chunk(3, 3, 136, 72, 60, rot=48, mlp=U.dense(130)),
], width=96, vocab=131)
CASES = {"mixed": (U.MIXED, U.SEQS), "plain": (U.PLAIN, U.SEQS), "big": (BIG, {"a": 330, "b": 140, "c": 201, "d": 70})}
LIMITS = {"float32": 2e-4, "bfloat16": 0.05}


@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    cfg, lengths = CASES[request.param]
    w = U.weights(cfg, 1, sharp=1.5)
    path = U.save(tmp_path_factory.mktemp(request.param), cfg, w)
    seqs = U.clear_choices(cfg, path, {n: U.tokens(cfg, k, i) for i, (n, k) in enumerate(lengths.items())})
    return cfg, w, path, seqs, U.reference(cfg, w, seqs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_engine_portions_batches_and_reuse(model, dtype):
    cfg, w, path, seqs, want = model
    limit = LIMITS[dtype]
    rep = make_replayer(path, dtype, 896, "cuda")
    for sizes in ([1000], [100, 1, 2, 63], [2, 65]):
        for name in seqs:
            U.play(rep, seqs, [[(name, n)] for n in U.cuts(len(seqs[name]), sizes)], want, limit)
    # decoding alone (captured graphs) after most of the prompt
    n = len(seqs["c"]) - 24
    U.play(rep, seqs, [[("c", n)]] + [[("c", 1)]] * 24, want, limit)
    # everyone together, then mixed portions and single tokens with slots and pages taken again
    U.play(rep, seqs, [[(n, len(s)) for n, s in seqs.items()]], want, limit)
    at = {n: 0 for n in seqs}
    plan, k = [], 0
    while any(at[n] < len(seqs[n]) for n in seqs):
        step = []
        for j, n in enumerate(seqs):
            left = len(seqs[n]) - at[n]
            if left and (k + j) % 5:
                size = min(left, (1, 37, 2, 64, 1)[(k + 2 * j) % 5])
                step.append((n, size))
                at[n] += size
        k += 1
        if step:
            plan.append(step)
    U.play(rep, seqs, plan, want, limit)
    assert rep.engine.graph_runner is None or rep.engine.graph_runner.replays > 0
    rep.engine.shutdown()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg", [
    # (a norm over one channel is a sign: the smallest sizes are compared in 32 bits on the CPU)
    U.config([U.window(1, 1, 4, 5, 3), U.chunk(1, 1, 6, 3, 2), U.chunk(1, 1, 6, 3, 5, kv_from=1, mlp=U.moe(2, 1, 3, shared=2))],
             width=20, vocab=7, scale=1.0),
    U.config([U.window(7, 7, 130, 150, 300, mlp=U.dense(33)), U.chunk(6, 1, 70, 130, 40, rot=64)], width=40, vocab=64),
    U.config([U.window(20, 1, 48, 16, 50), U.chunk(32, 2, 64, 64, 31, mlp=U.moe(24, 6, 40, shared=100))], width=98, vocab=100),
    U.config([U.window(mlp=U.dense(7)), U.window()], vocab=100, mult=2.0),
], ids=["small", "wide", "many-heads", "windows-only"])
def test_engine_other_sizes(cfg, dtype, tmp_path):
    w = U.weights(cfg, 2, sharp=1.0)
    path = U.save(tmp_path, cfg, w)
    seqs = U.clear_choices(cfg, path, {"a": U.tokens(cfg, 90, 1), "b": U.tokens(cfg, 3, 2)})
    rep = make_replayer(path, dtype, 256, "cuda")
    steps = [[("a", 70)], [("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 1)], [("a", 1)], [("a", 14)]]
    U.play(rep, seqs, steps, U.reference(cfg, w, seqs), LIMITS[dtype])
    rep.engine.shutdown()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,at", [("window", 64, 63), ("window", 40, 30), ("chunk", 64, 63), ("chunk", 64, 64),
                                          ("chunk", 40, 79)])
def test_a_planted_token_shows_exactly_where_it_is_seen(tmp_path, kind, size, at, dtype):
    cfg, w = U.planted_token_model(kind, size)
    without = [3] * 200
    planted = list(without)
    planted[at] = 7
    rep = make_replayer(U.save(tmp_path, cfg, w), dtype, 256, "cuda")
    for sizes in ([200], [31, 2, 1], [90] + [1] * 110):
        rows = []
        for seq in (without, planted):
            lo, got = 0, []
            for n in U.cuts(200, sizes):
                got.append(rep.step([("a", seq[lo:lo + n], list(range(n)))], ["a"] if lo + n == 200 else []))
                lo += n
            rows.append(torch.cat(got))
        moved = (rows[0] - rows[1]).abs().amax(-1)
        seen = U.seen_rows(kind, at, size, 200)
        assert set((moved > 0).nonzero().flatten().tolist()) <= set(seen)
        assert float(moved[seen].min()) > (0 if dtype == "float32" else -1) and float(moved[seen].max()) > 0.1
    rep.engine.shutdown()


def test_long_decoding_follows_the_graphs(tmp_path):
    cfg = U.config([U.chunk(size=64), U.window(size=50), U.chunk(size=100, kv_from=0)])
    w = U.weights(cfg, 4)
    rep = make_replayer(U.save(tmp_path, cfg, w), "float32", 320, "cuda")
    seqs = {"a": U.tokens(cfg, 300, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 295, U.reference(cfg, w, seqs), LIMITS["float32"])
    rep.engine.shutdown()


def test_engine_generates_the_greedy_tokens(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cuda", dtype="fp32", page_size=16, max_running_req=4, num_page_override=128,
              max_extend_tokens=48)
    prompts = [seqs["a"][:59], seqs["b"], seqs["c"][:1], seqs["d"][:64]]
    n = 6 if len(seqs["a"]) < 100 else 2
    outs = llm.generate(prompts, SamplingParams(max_tokens=n, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.token_ids == U.greedy(cfg, w, p, n)
    again = seqs["d"][:64] + seqs["b"][:5]          # a prefix the cache holds
    o = llm.generate([again], SamplingParams(max_tokens=3, ignore_eos=True))[0]
    assert o.cached_tokens > 0
    assert o.token_ids[0] == int(plain.logits(cfg, w, again)[-1].argmax())
    llm.shutdown()


def test_draft_verification_keeps_the_greedy_tokens(model):
    cfg, w, path, seqs, _ = model
    prompts = [(seqs["b"][:20] * 4), seqs["c"][:12] * 6, seqs["d"]]
    sp = SamplingParams(max_tokens=24, ignore_eos=True)
    outs = []
    for spec in ({}, dict(spec_algorithm="ngram", spec_num_draft=4)):
        # without drafts, but on the code path that verification rows share
        llm = LLM(path, device="cuda", dtype="bf16", page_size=16, max_running_req=4, num_page_override=128,
                  spec_algorithm=spec.get("spec_algorithm", "ngram"), spec_num_draft=spec.get("spec_num_draft", 0) or 1)
        if not spec:
            llm.proposer = None
        outs.append([o.token_ids for o in llm.generate(prompts, sp)])
        assert not spec or llm.stats["spec_steps"] > 0
        llm.shutdown()
    assert outs[0] == outs[1]


def test_which_kernels_serve_a_step(model):
    """Prompts take the tcgen05 form where rows are 64 or 128 wide; 16-bit decoding never takes the fp32 one."""
    from minisglang_rdna4_b200.ops import cuda as K

    cfg, w, path, seqs, _ = model
    K.LEDGER.clear()
    rep = make_replayer(path, "bfloat16", 512, "cuda")
    rep.step([("a", seqs["a"], [0])], [])
    rep.step([("a", [1], [0])], ["a"])
    assert {"prefill_attention", "paged_attention", "heads_rope_store", "add_norm"} <= set(K.LEDGER)
    assert "paged_attention_f32" not in K.LEDGER and "gemm_f32" not in K.LEDGER
    rep.engine.shutdown()
