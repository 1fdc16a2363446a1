"""Kernels of the Ligipel design against plain fp32 restatements of the same step, and the engine on the GPU."""
import pytest
import torch

import ligipel_util as U
import plain_ligipel as plain
from minisglang_rdna4_b200 import LLM, SamplingParams, ops
from minisglang_rdna4_b200.layers.residual_norm import LayerHistory
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.models.config import RotaryConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer
from test_mitilix_gpu import _batch, _gen
from test_rafodra_gpu import LENS, _linear_case, _linear_run

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF = torch.bfloat16


def _dev(*ts):
    out = [t.to(DEV) for t in ts]
    torch.cuda.synchronize()
    return out


# ---------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("width,cols", [(320, 320), (200, 208), (97, 112), (4096, 4096), (1000, 1008), (7, 16), (8192, 8192)])
@pytest.mark.parametrize("rows", [3, 600])
@pytest.mark.parametrize("n", [0, 1, 4, 9])
def test_residual_step(width, cols, rows, n):
    """All forms: one or two outputs, with and without earlier residual, post norm, history and average; split products."""
    from minisglang_rdna4_b200.ops.cuda import SplitPartial

    g = _gen(width + n)
    r = lambda *s: torch.randn(*s, generator=g)
    x, planes, other = r(rows, width) * 2 + 1, r(3, rows, cols), r(rows, cols + 4)
    pw, post, norm, coef = (r(width), r(width)), (r(width), r(width)), (r(width), r(width)), r(n + 1)
    earlier = r(n, rows, width)
    on = lambda v: None if v is None else tuple(map(on, v)) if isinstance(v, tuple) else v.to(DEV)
    for dtype, tol in ((torch.float32, 5e-5), (BF, 1.5e-2)):
        for two, has_x, has_post, average in ((True, True, True, True), (False, True, True, True), (True, True, True, None),
                                              (False, False, True, False), (False, True, False, None)):
            hists = []
            for dev in ("cpu", DEV):
                h = LayerHistory(n, rows, width, dev) if average is not None else None
                if h is not None:
                    h.rows[:n], h.count = earlier.to(dev), n
                hists.append(h)
            kw = dict(pair=pw if two else None, post=post if has_post else None)
            d = (planes.sum(0), other) if two else planes.sum(0)
            want = ref.residual_step(x if has_x else None, d, norm, 1e-3, dtype, cols, history=hists[0],
                                     coef=coef if average else None, **kw)
            sp = SplitPartial(planes.to(DEV), torch.float32)
            got = ops.residual_step(x.to(DEV) if has_x else None, (sp, other.to(DEV)) if two else sp, on(norm), 1e-3, dtype, cols,
                                    history=hists[1], coef=on(coef) if average else None, **{k: on(v) for k, v in kw.items()})
            torch.testing.assert_close(got[0].cpu(), want[0], rtol=3e-5, atol=5e-5)
            torch.testing.assert_close(got[1].float().cpu(), want[1].float(), rtol=tol, atol=tol)
            if average is not None:
                assert hists[1].count == n + 1
                torch.testing.assert_close(hists[1].rows[n].cpu(), hists[0].rows[n], rtol=3e-5, atol=5e-5)
                assert torch.equal(hists[1].rows[:n].cpu(), earlier)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("c", [16, 272])
def test_convolution(taps, c):
    g = _gen(taps + c)
    lens = [1, 2, 63, 64, 65, 3, 200, 1, 129]
    t, has = sum(lens), torch.tensor([1, 1, 0, 1, 1, 0, 1, 0, 1], dtype=torch.int32)
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    slots = torch.randperm(11, generator=g)[:9].int()
    x, w, b = torch.randn(t, c + 24, generator=g), torch.randn(c, taps, generator=g), torch.randn(c, generator=g)
    flat = torch.randn(11, 8 + c * (taps - 1), generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (BF, 2e-2)):
        states = [flat.to(dtype).to(dev) for dev in ("cpu", DEV)]
        views = [s[:, 8:].unflatten(1, (c, taps - 1)) if taps > 1 else s.new_zeros(11, c, 0) for s in states]
        xd = x.to(dtype)
        want = ref.causal_conv_silu(xd[:, :c], w, b, views[0], cu, slots, has)
        got = ops.causal_conv_silu(xd.to(DEV)[:, :c], *_dev(w, b), views[1], *_dev(cu, slots, has), max(lens))
        torch.testing.assert_close(got.float().cpu(), want.float(), rtol=tol, atol=tol)
        assert torch.equal(states[1].cpu(), states[0])


@pytest.mark.parametrize("c,n", [(16, 4), (48, 8), (272, 16), (64, 12), (80, 32), (32, 36), (48, 64), (16, 128), (32, 200),
                                 (16, 256), (16, 300)])
def test_selective_scan_forms(c, n):
    lens = [1, 31, 32, 33, 2, 130, 5, 64]
    for dtype, tol in ((torch.float32, 3e-5), (BF, 1e-2)):
        case, cu, slots, has, state = U.scan_case(c, n, lens, c + n, dtype)
        st = state.clone()
        want = ref.selective_scan(**{k: v.float() for k, v in case.items()}, state=st[:, 16:].unflatten(1, (1, c, n)), cu_q=cu,
                                  slots=slots, has_state=has)
        rows = torch.cat([case["z"], torch.zeros(sum(lens), 16, dtype=dtype), case["b"], case["c"]], 1).to(DEV)
        dev = {k: v.to(DEV) for k, v in case.items() if k not in ("z", "b", "c")}
        dev.update(z=rows[:, :c], b=rows[:, c + 16:c + 16 + n], c=rows[:, c + 16 + n:])
        for chunked in (False, True):
            sd = state.clone().to(DEV)
            got = ops.selective_scan(**dev, state=sd[:, 16:].unflatten(1, (1, c, n)), cu_q=cu.to(DEV), slots=slots.to(DEV),
                                     has_state=has.to(DEV), chunked=chunked)
            scale = float(want.pow(2).mean().sqrt())
            torch.testing.assert_close(got.float().cpu() / scale, want / scale, rtol=tol, atol=tol)
            torch.testing.assert_close(sd.cpu(), st, rtol=1e-4, atol=1e-4)
            unused = [i for i in range(len(lens) + 2) if i not in slots.tolist()]
            assert torch.equal(sd[unused].cpu(), state[unused]) and torch.equal(sd[:, :16].cpu(), state[:, :16])


def test_selective_scan_with_extreme_steps():
    """Steps from nothing to far beyond what a state survives."""
    c, n, lens = 32, 16, [70, 3]
    case, cu, slots, has, state = U.scan_case(c, n, lens, 3)
    case["dt"] = case["dt"] * 40
    st = state.clone()
    want = ref.selective_scan(**case, state=st[:, 16:].unflatten(1, (1, c, n)), cu_q=cu, slots=slots, has_state=has)
    for dtype in (torch.float32, BF):
        dev = {k: v.to(DEV, dtype if k in ("x", "z", "b", "c") else torch.float32).contiguous() for k, v in case.items()}
        bc = torch.cat([dev["b"], dev["c"]], 1)
        dev["b"], dev["c"] = bc[:, :n], bc[:, n:]
        for chunked in (False, True):
            sd = state.clone().to(DEV)
            got = ops.selective_scan(**dev, state=sd[:, 16:].unflatten(1, (1, c, n)), cu_q=cu.to(DEV), slots=slots.to(DEV),
                                     has_state=has.to(DEV), chunked=chunked).float().cpu()
            assert bool(torch.isfinite(got).all())
            scale = float(want.pow(2).mean().sqrt())
            torch.testing.assert_close(got / scale, want / scale, rtol=2e-2, atol=1e-4 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("h,dk,dv,rot", [(3, 16, 16, 16), (2, 32, 48, 20), (2, 64, 64, 64), (4, 80, 80, 34), (2, 128, 128, 128),
                                         (1, 256, 256, 256), (2, 256, 96, 2)])
def test_linear_attention_with_rotation(h, dk, dv, rot):
    """Rotated in fp32 ahead of the recurrence: every form follows the restatement to the rounding of its output."""
    table = get_rope_cache(RotaryConfig(dk, rot, 700, 1e3), "cpu")
    g = _gen(dk)
    starts = torch.randint(0, 600, (len(LENS),), generator=g)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts.tolist(), LENS)]).int()
    for dtype, chunked in ((torch.float32, False), (BF, False), (BF, True)):
        case = _linear_case(h, dk, dv, 0, LENS, dtype, dk + rot)
        want, st_want = _linear_run(case, h, dk, dv, 0, "cpu", False, dtype=torch.float32, q_scale=dk ** -0.5, rope=(table, pos))
        got, st = _linear_run(case, h, dk, dv, 0, DEV, chunked, q_scale=dk ** -0.5, rope=(table.to(DEV), pos.to(DEV)))
        scale = float(want.pow(2).mean().sqrt())
        tol = 5e-5 if dtype == torch.float32 else 1e-2
        torch.testing.assert_close(got / scale, want / scale, rtol=tol, atol=tol)
        torch.testing.assert_close(st, st_want, rtol=5e-4, atol=2e-3)


@pytest.mark.parametrize("experts,top", [(6, 2), (16, 4), (128, 8), (5, 5)])
def test_routing_by_corrected_scores(experts, top):
    from minisglang_rdna4_b200.ops import moe_kernels as M

    g = _gen(experts)
    logits, corr = torch.randn(70, experts, generator=g) * 2, torch.randn(experts, generator=g) * 0.1
    want_w, want_i = ref.moe_route(logits, top, True, "softmax", corr)
    counts = torch.empty(experts, dtype=torch.int32, device=DEV)
    w, ids = M.moe_route(logits.to(DEV), top, True, "softmax", 1.0, counts, bias=corr.to(DEV))
    order, want_order = ids.cpu().long().argsort(-1), want_i.long().argsort(-1)
    assert torch.equal(ids.cpu().gather(1, order), want_i.gather(1, want_order))
    torch.testing.assert_close(w.cpu().gather(1, order), want_w.gather(1, want_order), rtol=1e-5, atol=1e-6)


# ---------------------------------------------------------------------------------- attention
def _attention_case(hq, hk, width, window, lens, starts, ps, seed):
    g = _gen(seed)
    cu, seq, bt = _batch(lens, starts, ps, 400, g)
    k, v = (torch.randn(401, hk, ps, width, generator=g) for _ in range(2))
    q = torch.randn(sum(lens), hq, width, generator=g)
    r1, r2 = torch.rand(hq, generator=g), torch.rand(hq, generator=g) * 2
    reach = window or 2000
    bias = r1[:, None] * torch.log1p(r2[:, None] * torch.arange(reach))
    sink, talk = torch.randn(hq, generator=g) * 2, torch.randn(hq, hq, generator=g) * 0.4 + torch.eye(hq)
    return q, k, v, bt, cu, seq, bias, sink, talk


@pytest.mark.parametrize("hq,hk,width,window,ps", [
    (6, 2, 64, 96, 16), (4, 1, 64, 1, 16), (3, 3, 64, 17, 8), (16, 4, 128, 200, 16), (32, 4, 128, 0, 16), (20, 5, 64, 130, 64),
    (64, 8, 128, 70, 16), (64, 4, 64, 300, 32), (7, 1, 128, 64, 16), (24, 3, 128, 65, 16), (4, 2, 256, 40, 16), (66, 2, 64, 40, 16)])
def test_single_rows_of_mixed_heads(hq, hk, width, window, ps):
    """Decode batches whole and in ranges, verification rows and short portions; sizes of the plain kernel too."""
    for lens, starts in (([1] * 5, [0, 63, 64, 700, 129]), ([1, 3, 2, 9], [300, 0, 64, 127])):
        q, k, v, bt, cu, seq, bias, sink, talk = _attention_case(hq, hk, width, window, lens, starts, ps, hq + window)
        scale = width ** -0.5
        for dtype, tol in ((torch.float32, 1e-4), (BF, 3e-2)):
            qd, kd, vd = (x.to(dtype) for x in (q, k, v))
            want = ref.paged_attention(qd.float(), kd.float(), vd.float(), bt, cu, seq, scale, window=window, bias=bias, sink=sink,
                                       talk=talk)
            kg, vg = U.split_planes(kd.to(DEV), vd.to(DEV))
            args = _dev(bt, cu, seq)
            extra = dict(zip(("bias", "sink", "talk"), _dev(bias, sink, talk)))
            decode = max(lens) == 1
            for splits in ((1, 2, 5, 16) if decode else (1,)):
                got = ops.paged_attention(qd.to(DEV), kg, vg, *args, scale, window=window, max_q=max(lens), max_kv=int(seq.max()),
                                          decode=decode, splits=splits, **extra)
                torch.testing.assert_close(got.float().cpu(), want, rtol=tol, atol=tol * float(want.pow(2).mean().sqrt() + 1))


@pytest.mark.parametrize("hq,hk,width,window", [(6, 2, 64, 96), (4, 2, 64, 1), (3, 3, 64, 300), (16, 4, 128, 200), (5, 1, 128, 127),
                                                (10, 5, 64, 129), (8, 2, 128, 0), (9, 3, 128, 64)])
def test_prompts_of_mixed_heads(hq, hk, width, window):
    from minisglang_rdna4_b200.ops import cuda as K

    lens, starts = [257, 70, 300, 1, 640], [0, 200, 129, 63, 511]
    q, k, v, bt, cu, seq, bias, sink, talk = _attention_case(hq, hk, width, window, lens, starts, 16, hq)
    q, k, v, scale = q.to(BF), k.to(BF), v.to(BF), 1.5 * width ** -0.5
    want = ref.paged_attention(q.float(), k.float(), v.float(), bt, cu, seq, scale, window=window, bias=bias, sink=sink, talk=talk)
    kg, vg = U.split_planes(k.to(DEV), v.to(DEV))
    plan = K.PrefillPlan(cu.numpy(), seq.numpy(), DEV, window)
    got = K.prefill_attention_tc(q.to(DEV), kg, vg, bt.to(DEV), plan, scale, window=window,
                                 **dict(zip(("bias", "sink", "talk"), _dev(bias, sink, talk))))
    torch.testing.assert_close(got.float().cpu(), want, rtol=3e-2, atol=3e-2 * float(want.pow(2).mean().sqrt() + 1))
    assert K.attn_status() == 0


@pytest.mark.parametrize("window", [64, 100, 128])
@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 398, 399])
def test_a_loud_key_is_seen_exactly_within_the_window(at, window):
    from minisglang_rdna4_b200.ops import cuda as K

    bias = (0.001 * torch.log1p(torch.arange(window).float()))[None].repeat(2, 1).contiguous()
    extra = dict(bias=bias.to(DEV), sink=torch.zeros(2, device=DEV), talk=torch.eye(2, device=DEV))
    seen = list(range(at, min(at + window, 400)))
    q, k, v, bt = U.loud_key(400, at, 400, 64, 16, g=2)
    args = _dev(bt, torch.tensor([0, 400], dtype=torch.int32), torch.tensor([400], dtype=torch.int32))
    for dtype in (BF, torch.float32):
        kg, vg = U.split_planes(k.to(DEV, dtype), v.to(DEV, dtype))
        rows = [ops.paged_attention(q.to(DEV, dtype), kg, vg, *args, 1.0, window=window, max_q=400, max_kv=400, **extra)]
        if dtype == BF:
            plan = K.PrefillPlan(args[1].cpu().numpy(), args[2].cpu().numpy(), DEV, window)
            rows.append(K.prefill_attention_tc(q.to(DEV, BF), kg, vg, args[0], plan, 1.0, window=window, **extra))
            for last in {at, at + window - 1, at + window} - set(range(400, 999)):
                one = ops.paged_attention(q[last:last + 1].to(DEV, BF), kg, vg, args[0], torch.tensor([0, 1], dtype=torch.int32, device=DEV),
                                          torch.tensor([last + 1], dtype=torch.int32, device=DEV), 1.0, window=window, max_q=1,
                                          max_kv=last + 1, decode=True, splits=3, **extra).float().cpu()
                assert (float(one[0, 1, 0]) > 4.9) == (last in seen)
        for got in rows:
            assert (got[:, 1, 0].float().cpu() > 4.9).nonzero().flatten().tolist() == seen


# ---------------------------------------------------------------------------------- engine
# (limit, cap): in 16 bits the norm of a mixer's output enlarges the rounding of a row whose mixed heads nearly cancel
LIMITS = {"float32": (2e-4, None), "bfloat16": (0.05, 0.2)}
LONG = U.config([
    U.pair(4, 2, 40, 64, 90, inner=96, state=16, rank=16, taps=4, mlp=U.moe(8, 2, 48, shared=64)),
    U.retention(2, 64, 64, base=1e4, decay=[0.9, 0.999], mlp=U.moe(4, 2, 32)),
    U.pair(6, 3, 100, 72, 200, inner=128, state=8, rank=4, taps=2),
], width=128)
CASES = {"mixed": (U.MIXED, U.SEQS), "plain": (U.PLAIN, U.SEQS), "long": (LONG, {"a": 300, "b": 65, "c": 128, "d": 190})}


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
    limit, cap = LIMITS[dtype]
    rep = make_replayer(path, dtype, 896, "cuda")
    for sizes in ([1000], [100, 1, 2, 63], [2, 65]):
        for name in seqs:
            U.play(rep, seqs, [[(name, n)] for n in U.cuts(len(seqs[name]), sizes)], want, limit, cap)
    # decoding alone (captured graphs) after most of the prompt
    n = len(seqs["c"]) - 24
    U.play(rep, seqs, [[("c", n)]] + [[("c", 1)]] * 24, want, limit, cap)
    # everyone together, then mixed portions and single tokens with slots and pages taken again
    U.play(rep, seqs, [[(n, len(s)) for n, s in seqs.items()]], want, limit, cap)
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
    U.play(rep, seqs, plan, want, limit, cap)
    assert rep.engine.graph_runner is None or rep.engine.graph_runner.replays > 0
    rep.engine.shutdown()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg", [
    U.config([U.pair(1, 1, 4, 5, 3, inner=6, state=2, rank=1, taps=2), U.retention(1, 6, 5), U.retention(2, 4, 3, rot=2)], width=40,
             vocab=7, scale=1.0, cap=30.0),
    U.config([U.pair(7, 7, 130, 150, 300, inner=200, state=70, rank=40, taps=2), U.retention(2, 70, 130, rot=64)], width=40,
             vocab=64),
    U.config([U.pair(20, 4, 48, 16, 50, inner=300, state=24, rank=20), U.pair(32, 2, 64, 64, 31, taps=6)], width=98, vocab=100),
    U.config([U.retention(4, 128, 256, base=1e6), U.retention(rot=0)], vocab=100, cap=1.0),
], ids=["small", "wide", "many-heads", "retention-only"])
def test_engine_other_sizes(cfg, dtype, tmp_path):
    w = U.weights(cfg, 2, sharp=1.0)
    path = U.save(tmp_path, cfg, w)
    seqs = {"a": U.tokens(cfg, 90, 1), "b": U.tokens(cfg, 3, 2)}
    rep = make_replayer(path, dtype, 256, "cuda")
    steps = [[("a", 70)], [("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 1)], [("a", 1)], [("a", 14)]]
    U.play(rep, seqs, steps, U.reference(cfg, w, seqs), *LIMITS[dtype])
    rep.engine.shutdown()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,at", [(64, 63), (40, 30), (128, 0)])
def test_a_planted_token_shows_exactly_where_it_is_seen(tmp_path, size, at, dtype):
    cfg, w = U.planted_token_model(size)
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
        seen = list(range(at, min(at + size, 200)))
        assert set((moved > 0).nonzero().flatten().tolist()) <= set(seen)
        assert float(moved[seen].min()) > (0 if dtype == "float32" else -1) and float(moved[seen].max()) > 0.1
    rep.engine.shutdown()


def test_long_decoding_follows_the_graphs(tmp_path):
    cfg = U.config([U.pair(size=50), U.retention(decay=[0.999, 0.9, 0.5]), U.pair(size=100)])
    w = U.weights(cfg, 4)
    rep = make_replayer(U.save(tmp_path, cfg, w), "float32", 320, "cuda")
    seqs = {"a": U.tokens(cfg, 300, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 295, U.reference(cfg, w, seqs), *LIMITS["float32"])
    rep.engine.shutdown()


def test_engine_generates_the_greedy_tokens(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cuda", dtype="fp32", page_size=16, max_running_req=4, num_page_override=128, max_extend_tokens=48)
    prompts = [seqs["a"][:59], seqs["b"], seqs["c"][:1], seqs["d"][:64]]
    n = 6 if len(seqs["a"]) < 100 else 2
    outs = llm.generate(prompts, SamplingParams(max_tokens=n, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.token_ids == U.greedy(cfg, w, p, n)
    again = seqs["d"][:64] + seqs["b"][:5]
    o = llm.generate([again], SamplingParams(max_tokens=3, ignore_eos=True))[0]
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
    """16-bit steps take the kernels made for them; nothing of the 32-bit mode (but for heads of more than 128 channels)."""
    from minisglang_rdna4_b200.ops import cuda as K

    cfg, w, path, seqs, _ = model
    K.LEDGER.clear()
    rep = make_replayer(path, "bfloat16", 512, "cuda")
    rep.step([("a", seqs["a"], [0])], [])
    rep.step([("a", [1], [0])], ["a"])
    assert {"prefill_attention", "head_mix", "talk_attention", "residual_step", "selective_scan", "selective_scan_tiles",
            "causal_conv_silu", "linear_attention", "linear_attention_chunked", "heads_rope_store"} <= set(K.LEDGER)
    assert "gemm_f32" not in K.LEDGER and ("paged_attention_f32" in K.LEDGER) == (cfg is U.MIXED)
    rep.engine.shutdown()
