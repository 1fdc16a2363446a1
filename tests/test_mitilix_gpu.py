"""Kernels of the Mitilix design against plain fp32 restatements of the same step."""
import pytest
import torch

from minisglang_rdna4_b200 import ops
from minisglang_rdna4_b200.ops import ref

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _batch(lens, starts, ps, pages, gen):
    """cu_q, seq_lens, block table over a shuffled page pool, token slots."""
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    seq = torch.tensor([s + n for s, n in zip(starts, lens)], dtype=torch.int32)
    width = int((seq.max() + ps - 1) // ps)
    perm = torch.randperm(pages, generator=gen).to(torch.int32)
    bt = torch.zeros((len(lens), width), dtype=torch.int32)
    at = 0
    for i, s in enumerate(seq.tolist()):
        n = -(-s // ps)
        bt[i, :n] = perm[at:at + n]
        at += n
    assert at <= pages
    return cu, seq, bt


@pytest.mark.parametrize("width,taps,cols", [(320, 4, 320), (200, 3, 208), (1000, 2, 1008), (97, 5, 112), (64, 1, 64),
                                             (4096, 4, 4096), (5120, 4, 5120), (96, 12, 96), (8208, 3, 8208)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_norm_conv(width, taps, cols, dtype):
    g = _gen(width + taps)
    lens, has = [1, 2, 40, 1, 16, 17, 3], [1, 1, 0, 0, 1, 1, 0]
    t = sum(lens)
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    slots = torch.tensor([3, 0, 7, 5, 1, 2, 6], dtype=torch.int32)
    has = torch.tensor(has, dtype=torch.int32)
    x, d = torch.randn(t, width, generator=g), torch.randn(t, cols, generator=g)
    w1, w2 = (torch.randn(taps, width, generator=g) * 0.5 for _ in range(2))
    gain = torch.tensor([1.3])
    state = torch.randn(9, taps - 1, width, generator=g)
    for delta, two in ((d, True), (None, True), (d, False)):
        st_ref, st = state.clone(), state.clone().to(DEV)
        want = ref.add_scalar_norm_conv(x, delta, gain, 1e-5, w1, w2 if two else None, st_ref, cu, slots, has, dtype, cols)
        got = ops.add_scalar_norm_conv(
            x.to(DEV), None if delta is None else delta.to(DEV), gain.to(DEV), 1e-5, w1.to(DEV),
            w2.to(DEV) if two else None, st, cu.to(DEV), slots.to(DEV), has.to(DEV), max(lens), dtype, cols)
        tol = dict(rtol=1e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
        torch.testing.assert_close(got[0].cpu(), want[0], rtol=1e-6, atol=1e-6)
        torch.testing.assert_close(got[1].float().cpu(), want[1].float(), **tol)
        assert (got[2] is None) == (not two)
        if two:
            torch.testing.assert_close(got[2].float().cpu(), want[2].float(), **tol)
        torch.testing.assert_close(st.cpu(), st_ref, rtol=1e-5, atol=1e-5)
    # the norm alone, and split-K planes as the added term
    from minisglang_rdna4_b200.ops.cuda import SplitPartial

    planes = torch.randn(3, t, cols, generator=g)
    want = ref.add_scalar_norm_conv(x, planes.sum(0), gain, 1e-5, None, None, None, None, None, None, dtype, cols)
    got = ops.add_scalar_norm_conv(x.to(DEV), SplitPartial(planes.to(DEV), torch.float32), gain.to(DEV), 1e-5, None,
                                   None, None, None, None, None, 0, dtype, cols)
    torch.testing.assert_close(got[0].cpu(), want[0], rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(got[1].float().cpu(), want[1].float(), rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("m,n,k", [(1, 8, 16), (65, 70, 33), (200, 130, 257)])
def test_gemm_f32(m, n, k):
    g = _gen(m)
    a, b = torch.randn(m, k, generator=g), torch.randn(n, k, generator=g)
    got = ops.gemm(a.to(DEV), b.to(DEV)).cpu()
    torch.testing.assert_close(got, (a.double() @ b.double().T).float(), rtol=1e-5, atol=2e-5)


@pytest.mark.parametrize("t,h,n,k", [(1, 3, 64, 48), (70, 5, 80, 64), (130, 2, 512, 128), (9, 4, 128, 512), (64, 1, 16, 16)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_head_gemm(t, h, n, k, dtype):
    g = _gen(t)
    wide = torch.randn(t, h * k + 32, generator=g).to(dtype)
    w = torch.randn(h, n, k, generator=g).to(dtype)
    x = wide[:, :h * k].unflatten(1, (h, k))
    want = torch.einsum("thk,hnk->thn", x.double(), w.double())
    out = torch.zeros(t, h * n + 16, dtype=dtype, device=DEV)
    ops.head_gemm(wide.to(DEV)[:, :h * k].unflatten(1, (h, k)), w.to(DEV), out[:, :h * n].unflatten(1, (h, n)))
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    torch.testing.assert_close(out[:, :h * n].unflatten(1, (h, n)).double().cpu(), want, rtol=tol, atol=tol * k ** 0.5)
    assert float(out[:, h * n:].abs().max()) == 0.0


def test_gelu_and_embedding():
    g = _gen(4)
    x = torch.randn(33, 48, generator=g) * 3
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-2)):
        out = torch.zeros(33, 64, dtype=dtype, device=DEV)
        ops.gelu_erf(x.to(DEV, dtype), out[:, 16:])
        x[0] = torch.linspace(-6, 6, 48)
        ops.gelu_erf(x.to(DEV, dtype), out[:, 16:])
        want = torch.nn.functional.gelu(x.to(dtype).double())
        torch.testing.assert_close(out[:, 16:].double().cpu(), want, rtol=tol, atol=tol)
        emb, pos = torch.randn(50, 40, generator=g).to(dtype), torch.randn(70, 40, generator=g).to(dtype)
        ids, p = torch.randint(0, 50, (21,), generator=g), torch.randint(0, 70, (21,), generator=g)
        got = ops.embed_positions(ids.int().to(DEV), emb.to(DEV), pos.to(DEV), p.int().to(DEV))
        torch.testing.assert_close(got.cpu(), emb[ids].float() + pos[p].float())


@pytest.mark.parametrize("rank,width", [(64, 64), (40, 64), (300, 512)])
def test_latent_norm_store(rank, width):
    g = _gen(rank)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        c, w = torch.randn(13, width + 24, generator=g).to(dtype), torch.rand(width, generator=g)
        loc = torch.randperm(5 * 16, generator=g)[:13].int()
        pool = torch.zeros(5, 16, width, dtype=dtype)
        dev = pool.to(DEV)
        ref.latent_norm_store(c[:, 24:], w, rank, 1e-5, pool, loc)
        ops.latent_norm_store(c.to(DEV)[:, 24:], w.to(DEV), rank, 1e-5, dev, loc.to(DEV))
        torch.testing.assert_close(dev.cpu(), pool, rtol=tol, atol=tol)
        if dtype == torch.bfloat16:        # in the launch of the query projection
            dev2 = torch.zeros_like(dev)
            q, uk = torch.randn(13, 2, 32, generator=g).to(DEV, dtype), torch.randn(2, width, 32, generator=g).to(DEV, dtype)
            torch.cuda.synchronize()
            y = ops.head_gemm(q, uk, store=(c.to(DEV)[:, 24:], w.to(DEV), rank, 1e-5, dev2, loc.to(DEV)))
            torch.testing.assert_close(dev2, dev, rtol=0, atol=0)
            torch.testing.assert_close(y, ops.head_gemm(q, uk), rtol=0, atol=0)


@pytest.mark.parametrize("r", [64, 128, 192, 256, 512, 1024])
@pytest.mark.parametrize("h,window,ps", [(7, 70, 16), (3, 64, 16), (17, 1, 32), (64, 200, 64), (5, 0, 8)])
def test_latent_attention(r, h, window, ps):
    g = _gen(r + h)
    lens, starts = [1, 70, 2, 1, 33], [300, 0, 129, 63, 90]
    cu, seq, bt = _batch(lens, starts, ps, 96 if ps == 16 else 200, g)
    pool = torch.randn(201, ps, r, generator=g)
    q = torch.randn(sum(lens), h, r, generator=g)
    for dtype, tol in ((torch.bfloat16, 2e-2), (torch.float32, 1e-4)):
        qd, pd = q.to(dtype), pool.to(dtype)
        scale = 2.0 / r ** 0.5
        want = ref.latent_attention(qd.float(), pd.float(), bt, cu, seq, scale, window)
        got = ops.latent_attention(qd.to(DEV), pd.to(DEV), bt.to(DEV), cu.to(DEV), seq.to(DEV), scale, window, max(lens),
                                   int(seq.max()))
        torch.testing.assert_close(got.float().cpu(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("r,h,window,splits", [(64, 7, 70, 2), (128, 4, 500, 4), (512, 32, 333, 7), (512, 40, 0, 16)])
def test_latent_attention_decode_splits(r, h, window, splits):
    g = _gen(splits)
    starts = [0, 63, 64, 65, 640, 999]
    cu, seq, bt = _batch([1] * 6, starts, 16, 300, g)
    pool = torch.randn(301, 16, r, generator=g).bfloat16()
    q = torch.randn(6, h, r, generator=g).bfloat16()
    want = ref.latent_attention(q.float(), pool.float(), bt, cu, seq, 0.1, window)
    got = ops.latent_attention(q.to(DEV), pool.to(DEV), bt.to(DEV), cu.to(DEV), seq.to(DEV), 0.1, window, 1, 1000, splits)
    torch.testing.assert_close(got.float().cpu(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("t,h,n,k,splits", [(1, 4, 128, 64, 2), (70, 3, 80, 512, 5)])
def test_head_gemm_merges_splits(t, h, n, k, splits):
    from minisglang_rdna4_b200.ops import cuda as K

    g = _gen(splits)
    ws, lse = torch.randn(splits, t * h, k, generator=g), torch.randn(splits, t * h, generator=g) * 3
    lse[1, ::2] = float("-inf")
    w = torch.randn(h, n, k, generator=g).bfloat16()
    f = torch.softmax(lse * 0.6931471805599453, 0)
    want = torch.einsum("thk,hnk->thn", (ws * f[..., None]).sum(0).view(t, h, k), w.float())
    out = torch.empty(t, h, n, dtype=torch.bfloat16, device=DEV)
    wd = w.to(DEV)
    torch.cuda.synchronize()
    K.head_gemm_combine(K.LatentSplit(ws.to(DEV), lse.to(DEV), (t, h, k)), wd, out)
    torch.testing.assert_close(out.float().cpu(), want, rtol=2e-2, atol=2e-2 * k ** 0.5)


@pytest.mark.parametrize("h,dim,vdim,r,window,reach", [(7, 48, 96, 64, 70, 70), (3, 128, 128, 192, 300, 300),
                                                       (2, 16, 96, 512, 128, 500), (5, 112, 48, 128, 0, 0),
                                                       (1, 96, 16, 64, 1, 129)])
def test_latent_prefill_expanded(h, dim, vdim, r, window, reach):
    from minisglang_rdna4_b200.ops import cuda as K

    g = _gen(h + r)
    lens, starts = [257, 70, 300, 1, 640], [0, 200, 129, 63, 511]
    cu, seq, bt = _batch(lens, starts, 16, 200, g)
    pool = (torch.randn(201, 16, r, generator=g) * 0.5).bfloat16()
    t = sum(lens)
    q = torch.randn(t, h * dim + 32, generator=g).bfloat16()[:, :h * dim].unflatten(1, (h, dim))
    uk = (torch.randn(h, r, dim, generator=g) * r ** -0.5).bfloat16()
    uv = (torch.randn(h, vdim, r, generator=g) * r ** -0.5).bfloat16()
    scale = 2.0 * dim ** -0.5
    o = ref.latent_attention(torch.einsum("thd,hrd->thr", q.float(), uk.float()), pool.float(), bt, cu, seq, scale, window)
    want = torch.einsum("thr,hvr->thv", o, uv.float())
    plan = K.LatentPrefillPlan(cu.numpy(), seq.numpy(), reach, DEV)
    out = torch.zeros(t, h * vdim + 64, dtype=torch.bfloat16, device=DEV)
    qd = torch.zeros(t, h * dim + 32, dtype=torch.bfloat16, device=DEV)
    qd[:, :h * dim] = q.reshape(t, -1).to(DEV)
    ukd = uk.transpose(1, 2).reshape(h * dim, r).contiguous().to(DEV)
    args = (qd[:, :h * dim].unflatten(1, (h, dim)), ukd, uv.to(DEV), pool.to(DEV), 0, bt.to(DEV))
    torch.cuda.synchronize()
    K.latent_prefill(*args, plan, scale, window, out[:, :h * vdim].unflatten(1, (h, vdim)))
    got = out.float().cpu()
    torch.testing.assert_close(got[:, :h * vdim].unflatten(1, (h, vdim)), want, rtol=3e-2, atol=3e-2)
    assert float(got[:, h * vdim:].abs().max()) == 0.0


@pytest.mark.parametrize("r", [64, 512])
def test_latent_attention_window_edge(r):
    """The key at the window's far edge is made to dominate; one token further back must not be seen."""
    window, kv = 50, 400
    pool = torch.zeros(26, 16, r)
    flat = pool.view(-1, r)
    bt = torch.randperm(25, generator=_gen(1)).int()[None]
    slot = lambda p: int(bt[0, p // 16]) * 16 + p % 16        # noqa: E731
    for p in range(kv):
        flat[slot(p), 1] = 1.0
    for loud, seen in ((kv - window, True), (kv - window - 1, False)):
        flat2 = flat.clone()
        flat2[slot(loud), 0] = 8.0
        q = torch.zeros(1, 2, r)
        q[:, :, 0] = 8.0
        args = [t.to(DEV) for t in (bt, torch.tensor([0, 1], dtype=torch.int32), torch.tensor([kv], dtype=torch.int32))]
        for splits in (1, 3):
            got = ops.latent_attention(q.bfloat16().to(DEV), flat2.view_as(pool).bfloat16().to(DEV), *args, 1.0, window, 1,
                                       kv, splits).float().cpu()
            assert (float(got[0, 0, 0]) > 7.0) == seen


# ---------------------------------------------------------------------------------- the engine on the GPU
import mitilix_util as U  # noqa: E402
import plain_mitilix as plain  # noqa: E402
from minisglang_rdna4_b200 import LLM, SamplingParams  # noqa: E402
from minisglang_rdna4_b200.replay import make_replayer  # noqa: E402

# latents of one and two panels, heads that fill neither 16, 32 nor 64 rows, a window past a tile and one below it
BIG = U.config([U.layer(5, 32, 48, 128, 100, 96), U.layer(9, 64, 128, 64, 40, 130),
                U.layer(20, 16, 32, 128, 150, 64, kv_from=0)], width=96, vocab=131, taps=4, max_positions=400)
CASES = {"mixed": (U.MIXED, U.SEQS), "plain": (U.PLAIN, U.SEQS),
         "big": (BIG, {"a": 330, "b": 140, "c": 201, "d": 70})}


@pytest.fixture(scope="module", params=list(CASES))
def model(request, tmp_path_factory):
    cfg, lengths = CASES[request.param]
    w = U.weights(cfg, 1, sharp=1.5)
    path = U.save(tmp_path_factory.mktemp(request.param), cfg, w)
    seqs = {n: U.tokens(cfg, k, i) for i, (n, k) in enumerate(lengths.items())}
    return cfg, w, path, seqs, U.reference(cfg, w, seqs)


@pytest.mark.parametrize("dtype,limit", [("float32", 2e-4), ("bfloat16", 0.06)])
def test_engine_portions_batches_and_reuse(model, dtype, limit):
    cfg, w, path, seqs, want = model
    rep = make_replayer(path, dtype, 896, "cuda")
    for sizes in ([1000], [100, 1, 2, 63], [2, 65]):
        for name in seqs:
            U.play(rep, seqs, [[(name, n)] for n in U.cuts(len(seqs[name]), sizes)], want, limit)
    # decoding alone (captured graphs) after most of the prompt
    U.play(rep, seqs, [[("c", len(seqs["c"]) - 24)]] + [[("c", 1)]] * 24, want, limit)
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


@pytest.mark.parametrize("dtype,limit", [("float32", 2e-4), ("bfloat16", 0.06)])
@pytest.mark.parametrize("cfg", [
    # (a latent of one channel is a sign after its norm: nothing to compare in 16 bits)
    U.config([U.layer(heads=1, dim=1, vdim=1, rank=4, window=1, ff=1)], width=5, vocab=7, taps=1, max_positions=90),
    U.config([U.layer(heads=7, dim=130, vdim=150, rank=300, window=50, ff=33)], width=40, vocab=64, taps=9),
    U.config([U.layer(heads=40, rank=520, ff=0), U.layer(heads=2, window=70, ff=40)], taps=32, width=98, vocab=100),
    U.config([U.layer(heads=33, dim=64, vdim=64, rank=200, window=65), U.layer(rank=200, kv_from=0, ff=8)], width=64, taps=2),
], ids=["ones", "wide", "taps32", "rank200"])
def test_engine_other_sizes(cfg, dtype, limit, tmp_path):
    w = U.weights(cfg, 2, sharp=1.0)
    seqs = {"a": U.tokens(cfg, 90, 1), "b": U.tokens(cfg, 3, 2)}
    rep = make_replayer(U.save(tmp_path, cfg, w), dtype, 256, "cuda")
    steps = [[("a", 70)], [("a", 1), ("b", 2)], [("a", 1), ("b", 1)], [("a", 2)], [("a", 1)], [("a", 1)], [("a", 14)]]
    U.play(rep, seqs, steps, U.reference(cfg, w, seqs), limit)
    rep.engine.shutdown()


def test_engine_generates_the_greedy_tokens(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cuda", dtype="fp32", page_size=16, max_running_req=4, num_page_override=128,
              max_extend_tokens=48)
    prompts = [seqs["a"][:59], seqs["b"], seqs["c"][:1], seqs["d"][:64]]
    outs = llm.generate(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(6):
            seq.append(int(plain.logits(cfg, w, seq)[-1].argmax()))
        assert o.token_ids == seq[len(p):]
    # a prefix the cache holds, with the state kept at its boundary
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
