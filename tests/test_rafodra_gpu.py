"""Kernels of the Rafodra design against plain fp32 restatements of the same step, and the engine on the GPU."""
import math

import pytest
import torch

import plain_rafodra as plain
import rafodra_util as U
from minisglang_rdna4_b200 import LLM, SamplingParams, ops
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.models.config import RotaryConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer
from test_mitilix_gpu import _batch, _gen

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF = torch.bfloat16


def _dev(*ts):
    out = [t.to(DEV) for t in ts]
    torch.cuda.synchronize()
    return out


@pytest.mark.parametrize("width,cols", [(320, 320), (200, 208), (97, 112), (4096, 4096), (5120, 5120), (1000, 1008), (16384, 16384)])
@pytest.mark.parametrize("rows", [3, 600])
@pytest.mark.parametrize("center", [True, False])
def test_add_norm(width, cols, rows, center):
    from minisglang_rdna4_b200.ops.cuda import SplitPartial

    g = _gen(width)
    x, d, w = torch.randn(rows, width, generator=g) * 2 + 1, torch.randn(rows, cols, generator=g), torch.randn(width, generator=g)
    planes = torch.randn(3, rows, cols, generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (BF, 1e-2)):
        for delta, added in ((d, d), (None, None), (planes, planes.sum(0))):
            want = ref.add_norm(x, added, w, 1e-5, center, dtype, cols)
            dd = None if delta is None else delta.to(DEV)
            got = ops.add_norm(x.to(DEV), SplitPartial(dd, torch.float32) if delta is planes else dd, w.to(DEV), 1e-5, center,
                               dtype, cols)
            torch.testing.assert_close(got[0].cpu(), want[0], rtol=1e-5, atol=1e-5)
            torch.testing.assert_close(got[1].float().cpu(), want[1].float(), rtol=tol, atol=tol)


@pytest.mark.parametrize("dims,rot,rank,dim,heads", [(24, 24, 72, 40, 5), (12, 14, 50, 9, 3), (16, 24, 40, 8, 5), (64, 64, 512, 96, 32), (2, 2, 33, 1, 1)])
@pytest.mark.parametrize("t", [37, 1100])
def test_latent_rope_and_store(dims, rot, rank, dim, heads, t):
    g = _gen(rank)
    width, dp = -(-(rank + rot) // 64) * 64, -(-(dim + rot) // 16) * 16
    proj, w = torch.randn(t, heads * dp + width + 16, generator=g), torch.rand(width, generator=g)
    pos = torch.randint(0, 3000, (t,), generator=g).int()
    table = get_rope_cache(RotaryConfig(rot, dims, 3000, 1e4, interleaved=True), "cpu")
    loc = torch.randperm(70 * 16, generator=g)[:t].int()
    for dtype, tol in ((torch.float32, 1e-5), (BF, 1e-2)):
        for own in (True, False):
            a, b = proj.to(dtype), proj.to(DEV, dtype)
            pools = [torch.full((70, 16, width), 3.0, dtype=dtype, device=d) for d in ("cpu", DEV)]
            for x, pool in zip((a, b), pools):
                q = x[:, :heads * dp].unflatten(1, (heads, dp))
                store = (x[:, heads * dp:heads * dp + width], w.to(x.device), rank, 1e-5, pool, loc.to(x.device), rot)
                ops.latent_rope(q, dim, dims, table.to(x.device), pos.to(x.device), store if own else None)
            torch.testing.assert_close(b.cpu(), a, rtol=tol, atol=tol)
            torch.testing.assert_close(pools[1].cpu(), pools[0], rtol=tol, atol=tol)


@pytest.mark.parametrize("t,h,n,k", [(1, 3, 64, 48), (70, 5, 80, 64), (9, 4, 128, 576)])
@pytest.mark.parametrize("dtype", [BF, torch.float32])
def test_head_gemm_gate(t, h, n, k, dtype):
    g = _gen(t)
    x, w = torch.randn(t, h, k, generator=g).to(dtype), torch.randn(h, n, k, generator=g).to(dtype)
    rows = torch.randn(t, 40, generator=g).to(dtype)
    out = torch.empty(t, h, n, dtype=dtype, device=DEV)
    ops.head_gemm(*_dev(x, w), out, gate=rows.to(DEV)[:, 16:16 + h])
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(rows[:, 16:16 + h].double())[..., None]
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    torch.testing.assert_close(out.double().cpu(), want, rtol=tol, atol=tol * k ** 0.5)


@pytest.mark.parametrize("r", [64, 128, 192, 256, 512, 576, 768])
@pytest.mark.parametrize("h,window,ps", [(7, 0, 16), (17, 70, 32), (64, 0, 64)])
def test_latent_attention_with_sinks(r, h, window, ps):
    g = _gen(r + h)
    lens, starts = [1, 70, 2, 1, 33], [300, 0, 129, 0, 90]
    cu, seq, bt = _batch(lens, starts, ps, 96 if ps == 16 else 200, g)
    pool, q = torch.randn(201, ps, r, generator=g), torch.randn(sum(lens), h, r, generator=g)
    sink = torch.randn(h, generator=g) * 4 + 2
    scale = 2.0 / r ** 0.5
    for dtype, tol in ((BF, 2e-2), (torch.float32, 1e-4)):
        qd, pd = q.to(dtype), pool.to(dtype)
        want = ref.latent_attention(qd.float(), pd.float(), bt, cu, seq, scale, window, sink)
        args = _dev(qd, pd, bt, cu, seq)
        for one_form in (False, True):
            got = ops.latent_attention(*args, scale, window, max(lens), int(seq.max()), one_form=one_form, sink=sink.to(DEV))
            torch.testing.assert_close(got.float().cpu(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("r,h,splits", [(64, 7, 2), (128, 4, 4), (512, 32, 7), (576, 16, 5), (576, 40, 16)])
def test_split_decode_counts_the_sink_once(r, h, splits):
    from minisglang_rdna4_b200.ops import cuda as K

    g = _gen(splits)
    starts = [0, 63, 64, 65, 640, 999]
    cu, seq, bt = _batch([1] * 6, starts, 16, 300, g)
    pool, q = torch.randn(301, 16, r, generator=g).to(BF), torch.randn(6, h, r, generator=g).to(BF)
    sink = torch.randn(h, generator=g) * 3
    sink[0], sink[-1] = 100.0, -100.0
    want = ref.latent_attention(q.float(), pool.float(), bt, cu, seq, 0.1, 0, sink)
    args = _dev(q, pool, bt, cu, seq)
    got = ops.latent_attention(*args, 0.1, 0, 1, 1000, splits, sink=sink.to(DEV))
    torch.testing.assert_close(got.float().cpu(), want, rtol=2e-2, atol=2e-2)
    # ranges merged by the value projection, behind the heads' gates
    w, gate = (torch.randn(h, 32, r, generator=g) * r ** -0.5).to(BF), torch.randn(6, h, generator=g).to(BF)
    out = torch.empty(6, h, 32, dtype=BF, device=DEV)
    parts = K.latent_attention(*args, 0.1, 0, 1, 1000, splits, merge=False, sink=sink.to(DEV))
    K.head_gemm_combine(parts, w.to(DEV), out, gate=gate.to(DEV))
    want = torch.einsum("thr,hvr->thv", want, w.float()) * torch.sigmoid(gate.float())[..., None]
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=3e-2)


@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 398, 399])
@pytest.mark.parametrize("rows", [1, 3, 400])
def test_a_far_key_is_seen(at, rows):
    pool, bt, q = U.loud_key(400, at, rows, 64, 16)
    args = _dev(q.to(BF), pool.to(BF), bt, torch.tensor([0, rows], dtype=torch.int32), torch.tensor([400], dtype=torch.int32))
    for splits in ((1, 3) if rows == 1 else (1,)):
        got = ops.latent_attention(*args, 1.0, 0, rows, 400, splits, sink=torch.zeros(1, device=DEV)).float().cpu()
        assert float(got[-1, 0, 0]) > 9.8
        if rows == 400 and at > 0:
            assert float(got[at - 1, 0, 0]) == 0.0


@pytest.mark.parametrize("h,dim,vdim,r", [(7, 48, 96, 64), (3, 128, 128, 192), (5, 112, 48, 576)])
def test_expanded_prefill_with_sinks_and_gates(h, dim, vdim, r):
    from minisglang_rdna4_b200.ops import cuda as K

    g = _gen(h + r)
    lens, starts = [257, 70, 300, 1, 640], [0, 200, 129, 63, 511]
    cu, seq, bt = _batch(lens, starts, 16, 200, g)
    pool, t = (torch.randn(201, 16, r, generator=g) * 0.5).to(BF), sum(lens)
    q, gate = torch.randn(t, h, dim, generator=g).to(BF), torch.randn(t, h, generator=g).to(BF)
    uk, uv = ((torch.randn(*s, generator=g) * r ** -0.5).to(BF) for s in ((h, r, dim), (h, vdim, r)))
    sink = torch.randn(h, generator=g) * 3 + 2
    sink[0] = 90.0
    scale = 2.0 * dim ** -0.5
    o = ref.latent_attention(torch.einsum("thd,hrd->thr", q.float(), uk.float()), pool.float(), bt, cu, seq, scale, 0, sink)
    want = torch.einsum("thr,hvr->thv", o, uv.float()) * torch.sigmoid(gate.float())[..., None]
    plan = K.LatentPrefillPlan(cu.numpy(), seq.numpy(), 0, DEV)
    out = torch.zeros(t, h, vdim, dtype=BF, device=DEV)
    args = _dev(q, uk.transpose(1, 2).reshape(h * dim, r).contiguous(), uv, pool)
    btd, sd, gd = _dev(bt, sink, gate)
    K.latent_prefill(*args, 0, btd, plan, scale, 0, out, sink=sd, gate=gd)
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=3e-2)


# ---------------------------------------------------------------------------------- linear attention
def _linear_case(h, dk, dv, rank, lens, dtype, seed, tau=8.0, shift=2.0, spread=2.0):
    """Packed projected rows ``[q ‖ k ‖ v ‖ low]`` and the arguments that go with them."""
    g = _gen(seed)
    t, pad = sum(lens), -(-rank // 16) * 16
    proj = torch.randn(t, 2 * h * dk + h * dv + pad, generator=g)
    if rank:
        proj[:, -pad:][:, rank:] = 0
    proj = proj.to(dtype)
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    slots = torch.randperm(len(lens) + 2, generator=g)[:len(lens)].int()
    has = (torch.arange(len(lens)) % 3 != 1).int()
    state = torch.randn(len(lens) + 2, 3 * 16 + h * dk * dv, generator=g)
    gate = None
    if rank:
        gate = ((torch.randn(h * dk, rank, generator=g) * spread * rank ** -0.5).to(dtype),
                torch.randn(h * dk, generator=g) * spread + shift)
    decay = None if rank else torch.rand(h, generator=g) ** 0.3
    return proj, cu, slots, has, state, gate, decay


def _linear_run(case, h, dk, dv, rank, dev, chunked, tau=8.0, dtype=None, **kw):
    proj, cu, slots, has, state, gate, decay = case
    p = proj.to(dev) if dtype is None else proj.to(dev).to(dtype)
    st = state.clone().to(dev)
    view = st[:, 48:].unflatten(1, (h, dk, dv))
    q, k = (p[:, i * h * dk:(i + 1) * h * dk].unflatten(1, (h, dk)) for i in range(2))
    v = p[:, 2 * h * dk:2 * h * dk + h * dv].unflatten(1, (h, dv))
    if gate is not None:
        low = p[:, 2 * h * dk + h * dv:2 * h * dk + h * dv + rank]
        kw["gate"] = (low, gate[0].to(dev).to(p.dtype), gate[1].to(dev))
    else:
        kw["decay"] = decay.to(dev)
    o = ops.linear_attention(q, k, v, view, cu.to(dev), slots.to(dev), has.to(dev), tau=tau, **kw,
                             **({"chunked": chunked} if dev == DEV else {}))
    return o.float().cpu(), st.cpu()


LENS = [1, 16, 17, 40, 2, 70, 15, 1, 33]


@pytest.mark.parametrize("h,dk,dv,rank", [(3, 16, 16, 0), (2, 32, 48, 0), (2, 80, 64, 24), (4, 64, 80, 5), (2, 128, 128, 16),
                                          (1, 112, 144, 40), (2, 256, 96, 8), (1, 256, 256, 0)])
@pytest.mark.parametrize("act", [True, False])
def test_linear_attention_forms(h, dk, dv, rank, act):
    """Recurrent form in 32 and 16 bits and chunked form against the restatement; other slots and layers stay."""
    kw = dict(q_scale=dk ** -0.5, act=act)
    for dtype, chunked in ((torch.float32, False), (BF, False), (BF, True)):
        case = _linear_case(h, dk, dv, rank, LENS, dtype, dk + dv)
        want, st_want = _linear_run(case, h, dk, dv, rank, "cpu", False, dtype=torch.float32, **kw)
        got, st = _linear_run(case, h, dk, dv, rank, DEV, chunked, **kw)
        scale = float(want.pow(2).mean().sqrt())
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        torch.testing.assert_close(got / scale, want / scale, rtol=tol, atol=tol)
        # the state keeps 32 bits whatever the rows have (values are rounded once after their activation)
        torch.testing.assert_close(st, st_want, rtol=1e-2 if chunked and act else 2e-4, atol=5e-2 if chunked and act else 2e-3)
        unused = [i for i in range(len(LENS) + 2) if i not in case[2].tolist()]
        assert torch.equal(st[unused], case[4][unused]) and torch.equal(st[:, :48], case[4][:, :48])


@pytest.mark.parametrize("tau,shift,spread", [(1.0, -8.0, 6.0), (1.0, -60.0, 1.0), (1.0, 0.0, 30.0), (16.0, -90.0, 30.0), (64.0, 12.0, 1.0)])
def test_linear_attention_with_strong_and_weak_decays(tau, shift, spread):
    """Decays far outside what a chunk of 16 tokens can factor out, beside others that hardly decay."""
    h, dk, dv, rank = 2, 64, 32, 16
    for dtype, chunked in ((torch.float32, False), (BF, False), (BF, True)):
        case = _linear_case(h, dk, dv, rank, LENS, dtype, 5, shift=shift, spread=spread)
        want, st_want = _linear_run(case, h, dk, dv, rank, "cpu", False, tau=tau, dtype=torch.float32)
        got, st = _linear_run(case, h, dk, dv, rank, DEV, chunked, tau=tau)
        assert bool(torch.isfinite(got).all()) and bool(torch.isfinite(st).all())
        scale = float(want.pow(2).mean().sqrt())
        tol = 5e-5 if dtype == torch.float32 else 1e-2
        torch.testing.assert_close(got / scale, want / scale, rtol=tol, atol=tol)
        torch.testing.assert_close(st, st_want, rtol=1e-3, atol=2e-3)


@pytest.mark.parametrize("decay", [0.0, 1e-8, 1.0])
def test_linear_attention_with_extreme_head_decays(decay):
    h, dk, dv = 2, 32, 64
    for chunked in (False, True):
        case = list(_linear_case(h, dk, dv, 0, LENS, BF, 6))
        case[6] = torch.tensor([decay, 0.5])
        want, st_want = _linear_run(case, h, dk, dv, 0, "cpu", False, dtype=torch.float32)
        got, st = _linear_run(case, h, dk, dv, 0, DEV, chunked)
        torch.testing.assert_close(got, want, rtol=1e-2, atol=1e-2 * float(want.pow(2).mean().sqrt()))
        torch.testing.assert_close(st, st_want, rtol=1e-3, atol=1e-3)


def test_wide_key_heads_take_the_recurrent_form():
    case = _linear_case(1, 320, 48, 16, [3, 20], BF, 7)
    want, _ = _linear_run(case, 1, 320, 48, 16, "cpu", False, dtype=torch.float32, q_scale=320 ** -0.5)
    got, _ = _linear_run(case, 1, 320, 48, 16, DEV, True, q_scale=320 ** -0.5)
    torch.testing.assert_close(got, want, rtol=1e-2, atol=2e-2)


@pytest.mark.parametrize("h,dv,vdim,joint", [(5, 48, 48, True), (3, 16, 10, True), (5, 80, 80, False), (2, 48, 33, False), (16, 128, 128, True)])
@pytest.mark.parametrize("act", ["sigmoid", "silu"])
def test_norm_gate(h, dv, vdim, joint, act):
    g = _gen(h)
    o, rows = torch.randn(21, h, dv, generator=g), torch.randn(21, h * dv + 48, generator=g)
    o[..., vdim:] = 0
    w = torch.rand(h * dv if joint else dv, generator=g)
    for dtype, tol in ((torch.float32, 2e-5), (BF, 2e-2)):
        a, b = o.to(dtype), rows.to(dtype)
        for total in ((None, torch.rand(21, generator=g) * 50) if joint else (None,)):
            want = ref.norm_gate(a, b[:, 48:], w, 1e-4, vdim, joint, act, h * dv, total, 2 * h)
            got = ops.norm_gate(a.to(DEV), b.to(DEV)[:, 48:], w.to(DEV), 1e-4, vdim, joint, act, h * dv,
                                None if total is None else total.to(DEV), 2 * h)
            torch.testing.assert_close(got.float().cpu(), want.float(), rtol=tol, atol=tol)


# ---------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("e,groups,keep,top", [(12, 4, 2, 5), (6, 3, 1, 2), (64, 8, 2, 6), (128, 64, 5, 8), (5, 1, 1, 3), (512, 16, 16, 16)])
def test_group_limited_routing(e, groups, keep, top):
    from minisglang_rdna4_b200.ops import moe_kernels as M

    logits = torch.randn(50, e + 8, generator=_gen(e)) * 3
    counts = torch.empty(e, dtype=torch.int32, device=DEV)
    w, ids = M.moe_route(logits.to(DEV)[:, :e], top, False, "softmax", 1.7, counts, groups=groups, keep=keep)
    ww, wi = ref.moe_route_grouped(logits[:, :e], top, False, "softmax", None, 1.7, groups, keep)
    order, worder = ids.cpu().argsort(-1), wi.argsort(-1)
    assert torch.equal(ids.cpu().gather(1, order), wi.gather(1, worder))
    torch.testing.assert_close(w.cpu().gather(1, order), ww.gather(1, worder), rtol=1e-5, atol=1e-7)
    assert torch.equal(counts.cpu(), torch.bincount(wi.flatten().long(), minlength=e).int())


@pytest.mark.parametrize("t", [1, 37, 300])
@pytest.mark.parametrize("shared", [True, False])
def test_clamped_experts(t, shared):
    g = _gen(t)
    e, k, width, wp, ff = 6, 3, 72, 80, 48
    x = torch.randn(t, wp, generator=g)
    w13, w2 = torch.randn(e, 2 * ff, wp, generator=g) * 0.3, torch.randn(e, 96, ff, generator=g) * 0.3
    tw, ids = torch.rand(t, k, generator=g), torch.stack([torch.randperm(e, generator=g)[:k] for _ in range(t)]).int()
    sh, sg = torch.randn(t, wp, generator=g), torch.randn(t, 16, generator=g)
    for dtype, tol in ((torch.float32, 1e-5), (BF, 3e-2)):
        a = [z.to(dtype) for z in (x, w13, w2)]
        extra = (sh.to(dtype), sg[:, 6]) if shared else (None, None)
        want = ref.experts_partial32(*[z.float() for z in a], tw, ids, 0.8, 1.702, None if not shared else extra[0].float(), extra[1])
        got = ops.experts_partial32(*_dev(*a), tw.to(DEV), ids.to(DEV), 0.8, 1.702, *(_dev(extra[0]) + [sg.to(DEV)[:, 6]] if shared else ()))
        torch.testing.assert_close(got.cpu(), want, rtol=tol, atol=tol)
    y = torch.randn(33, 96, generator=g) * 3
    for dtype, tol in ((torch.float32, 1e-5), (BF, 1e-2)):
        torch.testing.assert_close(ops.clamped_glu(y.to(DEV, dtype), 0.9, 1.702).float().cpu(),
                                   ref.clamped_glu(y.to(dtype), 0.9, 1.702).float(), rtol=tol, atol=tol)
    torch.testing.assert_close(ops.silu_and_mul(y.to(DEV)).cpu(), ref.silu_and_mul(y), rtol=1e-5, atol=1e-5)


# ---------------------------------------------------------------------------------- the engine on the GPU
# heads that fill neither 16, 32 nor 64 rows, wide states, experts beyond one tile
BIG = U.config([
    U.latent(5, 32, 16, 48, 112, mlp=U.dense(96)), U.gla(3, 128, 96, tau=16.0, rank=16, mlp=U.moe(16, 4, 48, groups=(4, 2))),
    U.lightning(4, 64, 128, mlp=U.dense(130)), U.latent(9, 48, 16, 128, 112, kv_from=0, mlp=U.moe(5, 5, 33, groups=None)),
    U.gla(2, 72, 80, tau=4.0, rank=33),
], width=96, vocab=131)
CASES = {"mixed": (U.MIXED, U.SEQS), "plain": (U.PLAIN, U.SEQS), "big": (BIG, {"a": 330, "b": 140, "c": 201, "d": 70})}
LIMITS = {"float32": (2e-4, None), "bfloat16": (0.03, 0.7)}


@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    cfg, lengths = CASES[request.param]
    w = U.weights(cfg, 1, sharp=1.5)
    path = U.save(tmp_path_factory.mktemp(request.param), cfg, w)
    seqs = {n: U.tokens(cfg, k, i) for i, (n, k) in enumerate(lengths.items())}
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
    # (a norm over one channel is a sign: the smallest sizes are compared in 32 bits on the CPU)
    U.config([U.latent(1, 3, 2, 5, 7), U.lightning(1, 5, 7, decay=[0.5]), U.gla(1, 7, 9, tau=1.0, rank=1),
              U.latent(1, 2, 2, 3, 7, kv_from=0, mlp=U.moe(2, 1, 3, groups=None, shared=2))], width=20, vocab=7, scale=1.0),
    U.config([U.latent(7, 130, 20, 150, 300, mlp=U.dense(33)), U.lightning(1, 130, 70), U.gla(1, 70, 130, rank=40)], width=40,
             vocab=64),
    U.config([U.latent(20, 48, 16, 48, 512, mlp=U.moe(64, 8, 40, groups=(8, 3), shared=100)), U.lightning(2, 256, 64)], width=98,
             vocab=100),
    U.config([U.lightning(mlp=U.dense(7)), U.lightning()], vocab=100),
], ids=["small", "wide", "rank512", "no-attention"])
def test_engine_other_sizes(cfg, dtype, tmp_path):
    w = U.weights(cfg, 2, sharp=1.0)
    seqs = {"a": U.tokens(cfg, 90, 1), "b": U.tokens(cfg, 3, 2)}
    rep = make_replayer(U.save(tmp_path, cfg, w), dtype, 256, "cuda")
    steps = [[("a", 70)], [("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 1)], [("a", 1)], [("a", 14)]]
    U.play(rep, seqs, steps, U.reference(cfg, w, seqs), *LIMITS[dtype])
    rep.engine.shutdown()


def test_long_decoding_follows_the_graphs(tmp_path):
    cfg = U.config([U.latent(4), U.lightning(2, decay=[0.9, 0.9999]), U.gla(tau=30.0), U.latent(4, kv_from=0)])
    w = U.weights(cfg, 4)
    rep = make_replayer(U.save(tmp_path, cfg, w), "float32", 320, "cuda")
    seqs = {"a": U.tokens(cfg, 300, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 295, U.reference(cfg, w, seqs), *LIMITS["float32"])
    rep.engine.shutdown()


def test_engine_generates_the_greedy_tokens(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cuda", dtype="fp32", page_size=16, max_running_req=4, num_page_override=128,
              max_extend_tokens=48)
    prompts = [seqs["a"][:59], seqs["b"], seqs["c"][:1], seqs["d"][:64]]
    outs = llm.generate(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.token_ids == U.greedy(cfg, w, p, 6)
    # a prefix the cache holds, with the states kept at its boundary
    again = seqs["d"][:64] + seqs["b"][:5]
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


def test_extreme_sinks_and_gates_reach_the_logits(tmp_path):
    """A sink that outweighs every key silences a head; one that weighs nothing leaves it alone."""
    cfg = U.config([U.latent(2, mlp=None)])
    rows = {}
    for sink in (-60.0, 60.0):
        w = U.weights(cfg, 5)
        w["l0.mix.sink"] = torch.tensor([sink, 0.5]).to(BF)
        seqs = {"a": U.tokens(cfg, 60, 1)}
        for dtype in LIMITS:
            rep = make_replayer(U.save(tmp_path / f"{sink}{dtype}", cfg, w), dtype, 128, "cuda")
            U.play(rep, seqs, [[("a", 40)]] + [[("a", 1)]] * 20, U.reference(cfg, w, seqs), *LIMITS[dtype])
            rep.engine.shutdown()
        rows[sink] = plain.logits(cfg, w, seqs["a"])
    assert float(U.spread(rows[60.0], rows[-60.0]).max()) > 0.2 and math.isfinite(float(rows[60.0].sum()))
