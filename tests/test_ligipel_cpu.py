"""The Ligipel design through the framework on the CPU (fp32) against a plain restatement of its equations."""
import json
import math
import os
import subprocess

import pytest
import torch

import ligipel_util as U
import plain_ligipel as plain
from minisglang_rdna4_b200 import LLM, SamplingParams
from minisglang_rdna4_b200.kvcache.gdn_state import GDNStateCache
from minisglang_rdna4_b200.layers.residual_norm import LayerHistory
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.models.config import LinearAttnLayer, ModelConfig, PairMixer, RotaryConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer

LIMIT = 2e-4


def _g(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("two", [False, True])
@pytest.mark.parametrize("first", [False, True])
def test_norms_around_a_sublayer_and_the_depth_average(two, first):
    g, t, w, eps = _g(0), 5, 24, 1e-2
    r = lambda *s: torch.randn(*s, generator=g) * 2
    x, d, e, pw = r(t, w), r(t, 32), r(t, 32), (r(w), r(w))
    post, norm, coef = (r(w), r(w)), (r(w), r(w)), r(3)
    hist = LayerHistory(4, t, w, "cpu")
    hist.rows[:2], hist.count = r(2, t, w), 2
    before = hist.rows[:2].clone()
    xn, y = ref.residual_step(None if first else x, (d, e) if two else d, norm, eps, torch.float32, 32, pair=pw if two else None,
                              post=post, history=hist, coef=coef)
    u = d[:, :w].double()
    if two:
        u = 0.5 * (plain.unit_rms(u, eps) * pw[0] + plain.unit_rms(e[:, :w].double(), eps) * pw[1])
    result = plain.layer_norm(u, *(p.double() for p in post), eps) + (0 if first else x.double())
    want = plain.depth_average([*before.double(), result], coef.double())
    torch.testing.assert_close(hist.rows[2].double(), result, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(xn.double(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(y[:, :w].double(), plain.layer_norm(want, *(p.double() for p in norm), eps), rtol=1e-5, atol=1e-5)
    assert hist.count == 3 and float(y[:, w:].abs().max()) == 0.0


def test_epsilon_is_inside_the_root():
    d = torch.tensor([[1e-3, -1e-3] * 4])
    one, none = torch.ones(8), torch.zeros(8)
    xn, _ = ref.residual_step(None, d, (one, none), 1e-2, torch.float32, 8, post=(one, none))
    torch.testing.assert_close(xn, d / math.sqrt(1e-6 + 1e-2))
    xn, _ = ref.residual_step(None, (d, d), (one, none), 1e-2, torch.float32, 8, pair=(one, none))
    torch.testing.assert_close(xn, 0.5 * d / math.sqrt(1e-6 + 1e-2))


def _dense_case(seed, lens, q_lens, hq, hk, d, ps):
    g = _g(seed)
    per = [-(-n // ps) for n in lens]
    ids = torch.randperm(sum(per) + 2, generator=g)[:sum(per)].to(torch.int32)
    bt = torch.zeros(len(lens), max(per), dtype=torch.int32)
    at = 0
    for b, n in enumerate(per):
        bt[b, :n] = ids[at:at + n]
        at += n
    k, v = (torch.randn(sum(per) + 2, hk, ps, d, generator=g) for _ in range(2))
    q = torch.randn(sum(q_lens), hq, d, generator=g) * 2
    cu = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32)
    return q, k, v, bt, cu, torch.tensor(lens, dtype=torch.int32)


@pytest.mark.parametrize("window", [1, 2, 16, 17, 500])
@pytest.mark.parametrize("hq,hk", [(6, 2), (3, 1), (2, 2)])
def test_attention_with_distance_bias_zero_sink_and_mixed_heads(window, hq, hk):
    lens, q_lens, d, ps, scale = [40, 33, 17, 1], [40, 1, 2, 1], 8, 16, 0.4
    q, k, v, bt, cu, seq = _dense_case(window, lens, q_lens, hq, hk, d, ps)
    g = _g(hq)
    r1, r2, talk = torch.rand(hq, generator=g) + 0.2, torch.rand(hq, generator=g) * 3, torch.randn(hq, hq, generator=g)
    bias = r1[:, None] * torch.log1p(r2[:, None] * torch.arange(window))
    got = ref.paged_attention(q, k, v, bt, cu, seq, scale, window=window, bias=bias, sink=torch.zeros(hq), talk=talk)
    for b, (n, m) in enumerate(zip(lens, q_lens)):
        pages = bt[b, :-(-n // ps)].long()
        kk, vv = (x[pages].transpose(1, 2).reshape(-1, hk, d)[:n].double() for x in (k, v))
        full = torch.zeros(n, hq, d).double()
        lo, hi = int(cu[b]), int(cu[b + 1])
        full[n - m:] = q[lo:hi].double()
        of = [h // (hq // hk) for h in range(hq)]
        w = torch.stack([plain.head_weights(full[:, h], kk[:, of[h]], r1[h].double(), r2[h].double(), scale, window)
                         for h in range(hq)])
        w = plain.mix_heads(w, talk.double())
        want = torch.stack([w[h] @ vv[:, of[h]] for h in range(hq)], 1)[n - m:]
        torch.testing.assert_close(got[lo:hi].double(), want, rtol=1e-4, atol=1e-5)


def test_the_sink_takes_its_share_and_is_not_mixed():
    """One key with score s: every head's weight is e^s / (1 + e^s); the mixture is of those weights alone."""
    q, k, v, bt = U.loud_key(1, 0, 1, 64, 16, g=2)
    talk = torch.tensor([[1.0, -0.5], [2.0, 3.0]])
    got = ref.paged_attention(q, k, v, bt, torch.tensor([0, 1]), torch.tensor([1]), 1 / 64, sink=torch.zeros(2), talk=talk)
    share = math.e / (1 + math.e)
    torch.testing.assert_close(got[0, :, 0], 5.0 * share * talk.sum(1))
    s = torch.tensor([0.5, -1.0, 3.0])
    torch.testing.assert_close(plain.softmax_off_by_one(s), torch.exp(s) / (1 + torch.exp(s).sum()))


@pytest.mark.parametrize("window", [33, 64])
@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 99])
def test_a_loud_key_is_seen_exactly_within_the_window(window, at):
    q, k, v, bt = U.loud_key(130, at, 130, 64, 16)
    bias = 0.01 * torch.log1p(torch.arange(window).float())[None]
    got = ref.paged_attention(q, k, v, bt, torch.tensor([0, 130]), torch.tensor([130]), 1.0, window=window, bias=bias,
                              sink=torch.zeros(1), talk=torch.ones(1, 1))
    assert (got[:, 0, 0] > 4.9).nonzero().flatten().tolist() == list(range(at, min(at + window, 130)))


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_convolution_with_a_carried_tail(taps):
    g, c, n = _g(taps), 10, 23
    x, w, b = torch.randn(n, c, generator=g), torch.randn(c, taps, generator=g), torch.randn(c, generator=g)
    want = plain.silu(plain.causal_filter(x.double(), w.double(), b.double()))
    state = torch.full((3, c, taps - 1), 7.0)
    at, got = 0, []
    for m in (1, 2, 9, 1, 10):
        got.append(ref.causal_conv_silu(x[at:at + m], w, b, state, torch.tensor([0, m]), torch.tensor([1]),
                                        torch.tensor([int(at > 0)])))
        at += m
    torch.testing.assert_close(torch.cat(got).double(), want, rtol=1e-5, atol=1e-5)
    assert taps == 1 or float(state[[0, 2]].min()) == 7.0


def test_selective_scan_with_a_carried_state():
    c, n, t = 16, 4, 30
    case, cu, slots, _, state = U.scan_case(c, n, [t], 1)
    dt = torch.log1p(torch.exp((case["dt"] + case["dt_bias"]).double()))
    want = plain.selective_scan(case["x"].double(), dt, case["a"].double(), case["b"].double(), case["c"].double(),
                                case["skip"].double()) * plain.silu(case["z"].double())
    view = state[:, 16:].unflatten(1, (1, c, n))
    at, got = 0, []
    for m in (1, 7, 2, 20):
        rows = {k: v[at:at + m] if k in ("x", "dt", "b", "c", "z") else v for k, v in case.items()}
        got.append(ref.selective_scan(**rows, state=view, cu_q=torch.tensor([0, m]), slots=slots,
                                      has_state=torch.tensor([int(at > 0)])))
        at += m
    torch.testing.assert_close(torch.cat(got).double(), want, rtol=1e-4, atol=1e-5)


@pytest.mark.parametrize("dim,rot", [(20, 20), (24, 10), (9, 2), (16, 0)])
def test_retention_with_neighbouring_pairs(dim, rot):
    """Channels reordered so that a pair are neighbours give the same output as half-split pairs."""
    g, t, heads, vdim = _g(dim), 40, 2, 6
    q, k, v = (torch.randn(t, heads, n, generator=g) for n in (dim, dim, vdim))
    decay = torch.tensor([0.8, 0.999])
    order = [x for j in range(rot // 2) for x in (j, j + rot // 2)] + list(range(rot, dim))
    rope = (get_rope_cache(RotaryConfig(dim, rot, 64, 90.0), "cpu"), torch.arange(t)) if rot else None
    state = torch.full((2, heads, dim, vdim), 9.0)
    got = ref.linear_attention(q[..., order], k[..., order], v, state, torch.tensor([0, t]), torch.tensor([1]),
                               torch.tensor([0]), decay=decay, q_scale=dim ** -0.5, rope=rope)
    qr, kr = (plain.rotate_halves(x.double(), rot, 90.0) for x in (q, k))
    want = torch.stack([plain.fading_memory(qr[:, h], kr[:, h] * dim ** -0.5, v[:, h].double(), float(decay[h]))
                        for h in range(heads)], 1)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-5)
    assert float(state[0].min()) == 9.0


def test_choice_by_corrected_scores_weights_by_the_scores():
    g = _g(7)
    h, router, corr = torch.randn(50, 12, generator=g), torch.randn(6, 12, generator=g), torch.randn(6, generator=g) * 0.2
    tw, ids = ref.moe_route(h @ router.T, 3, True, "softmax", corr)
    moved = 0
    for t, picks in enumerate(plain.route(h.double(), router.double(), corr.double(), 3)):
        assert sorted(int(e) for e in ids[t]) == sorted(e for e, _ in picks)
        for e, weight in picks:
            assert math.isclose(float(tw[t, ids[t].tolist().index(e)]), float(weight), rel_tol=1e-5)
        moved += sorted(e for e, _ in picks) != sorted((h[t] @ router.T).topk(3)[1].tolist())
    assert moved > 0
    torch.testing.assert_close(tw.sum(-1), torch.ones(50))


# ---------------------------------------------------------------------------------- the engine's step function
@pytest.fixture(scope="module", params=["mixed", "plain"])
def model(request, tmp_path_factory):
    cfg = U.MIXED if request.param == "mixed" else U.PLAIN
    w = U.weights(cfg, 1)
    path = U.save(tmp_path_factory.mktemp(request.param), cfg, w)
    seqs = {n: U.tokens(cfg, k, i) for i, (n, k) in enumerate(U.SEQS.items())}
    return cfg, w, path, seqs, U.reference(cfg, w, seqs)


def _rep(path, max_tokens=256, page=16):
    return make_replayer(path, "float32", max_tokens, "cpu", page)


@pytest.mark.parametrize("sizes", [[1000], [1], [2], [3], [16], [17, 2, 30, 1]])
def test_prefill_portions_and_single_tokens(model, sizes):
    cfg, w, path, seqs, want = model
    rep = _rep(path)
    for name in seqs:
        U.play(rep, seqs, [[(name, n)] for n in U.cuts(len(seqs[name]), sizes)], want, LIMIT)


@pytest.mark.parametrize("page", [8, 64])
def test_mixed_batches_and_reused_pages_and_slots(model, page):
    cfg, w, path, seqs, want = model
    U.play(_rep(path, page=page), seqs, U.mixed_schedule(), want, LIMIT)


def test_a_batch_equals_each_request_alone(model):
    cfg, w, path, seqs, want = model
    U.play(_rep(path), seqs, [[(n, len(s)) for n, s in seqs.items()]], want, LIMIT)


def test_pool_holds_exactly_the_live_tokens(model):
    cfg, w, path, seqs, want = model
    rep = _rep(path, max_tokens=80)
    for k in range(2):
        for name in seqs:
            U.play(rep, seqs, [[(f"{name}#{k}", n)] for n in U.cuts(len(seqs[name]), [25, 1])], want, LIMIT)


def test_long_decoding(tmp_path):
    cfg = U.config([U.pair(size=50), U.retention(decay=[0.999, 0.9, 0.5]), U.pair(size=100)])
    w = U.weights(cfg, 4)
    rep = _rep(U.save(tmp_path, cfg, w), 256)
    seqs = {"a": U.tokens(cfg, 200, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 195, U.reference(cfg, w, seqs), LIMIT)


@pytest.mark.parametrize("size,at", [(40, 30), (16, 16), (1, 5), (33, 0)])
@pytest.mark.parametrize("sizes", [[100], [1], [31, 2]])
def test_a_planted_token_shows_exactly_where_it_is_seen(tmp_path, size, at, sizes):
    cfg, w = U.planted_token_model(size)
    without = [3] * 100
    planted = list(without)
    planted[at] = 7
    rep = _rep(U.save(tmp_path, cfg, w))
    rows = []
    for k, seq in enumerate((without, planted)):
        lo, got = 0, []
        for n in U.cuts(100, sizes):
            got.append(rep.step([(str(k), seq[lo:lo + n], list(range(n)))], [str(k)] if lo + n == 100 else []))
            lo += n
        rows.append(torch.cat(got))
    moved = (rows[0] - rows[1]).abs().amax(-1)
    assert (moved > 0).nonzero().flatten().tolist() == list(range(at, min(at + size, 100)))
    assert float(U.spread(rows[1], plain.logits(cfg, w, planted)).max()) < LIMIT


@pytest.mark.parametrize("name,value", [("dwa", 0.0), ("mix.right.conv", 0.0), ("mix.left.r1", 0.0), ("mix.left.talk", 0.0),
                                        ("mlp.correction", 0.0), ("norm1b.b", 0.0), ("mix.right.D", 0.0)])
def test_every_tensor_reaches_the_logits(tmp_path, name, value):
    """Without it the framework and the plain model move alike."""
    cfg, w = U.PLAIN, U.weights(U.PLAIN, 1)
    seq = U.tokens(cfg, 30, 5)
    before = plain.logits(cfg, w, seq)
    w["l0." + name] = torch.full_like(w["l0." + name], value)
    after = plain.logits(cfg, w, seq)
    assert float(U.spread(before, after).max()) > 50 * LIMIT
    got = _rep(U.save(tmp_path, cfg, w)).step([("a", seq, list(range(30)))], ["a"])
    assert float(U.spread(got, after).max()) < LIMIT


@pytest.mark.parametrize("cfg", [
    U.config([U.pair(1, 1, 2, 1, 1, inner=1, state=1, rank=1, taps=1, mlp=U.moe(2, 1, 1, shared=1)),
              U.retention(1, 2, 1, mlp=U.moe(1, 1, 1))], width=6, vocab=7, scale=1.0, cap=30.0),
    U.config([U.pair(7, 7, 130, 150, 300, inner=200, state=70, rank=40, taps=2), U.retention(2, 70, 130, rot=64)], width=40,
             vocab=64),
    U.config([U.pair(mlp=U.moe(4, 4, 16)), U.pair(5, 1, taps=6)], vocab=100, eps=1e-2),
    U.config([U.retention(mlp=U.moe(7, 3, 5)), U.retention(rot=0)], vocab=100, cap=1.0),
], ids=["ones", "wide", "pairs-only", "retention-only"])
def test_other_sizes(cfg, tmp_path):
    w = U.weights(cfg, 2)
    seqs = {"a": U.tokens(cfg, 40, 1), "b": U.tokens(cfg, 2, 2)}
    rep = _rep(U.save(tmp_path, cfg, w))
    U.play(rep, seqs, [[("a", 7)], [("a", 1), ("b", 1)], [("b", 1), ("a", 32)]], U.reference(cfg, w, seqs), LIMIT)


# ---------------------------------------------------------------------------------- entry points
def test_greedy_generation_prefix_cache_and_chunks(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=3, num_page_override=64, max_extend_tokens=24)
    sp = SamplingParams(max_tokens=4, ignore_eos=True)
    prompts = [seqs["a"], seqs["b"], seqs["c"][:3], seqs["d"]]
    for o, s in zip(llm.generate(prompts, sp), prompts):
        assert o.token_ids == U.greedy(cfg, w, s, 4)
    again = seqs["d"] + seqs["a"][:9]        # a prefix whose state was kept
    o = llm.generate([again], sp)[0]
    assert o.token_ids == U.greedy(cfg, w, again, 4)
    llm.shutdown()


def test_draft_verification_keeps_the_greedy_tokens(model):
    """Rejected drafts are taken back out of the scan, the convolution tail and the retention state."""
    cfg, w, path, seqs, _ = model
    prompts = [seqs["b"] * 2, seqs["c"][:12] * 3]
    sp = SamplingParams(max_tokens=12, ignore_eos=True)
    outs = []
    for spec in ({}, dict(spec_algorithm="ngram", spec_num_draft=3)):
        llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=2, num_page_override=64, **spec)
        outs.append([o.token_ids for o in llm.generate(prompts, sp)])
        llm.shutdown()
    assert outs[0] == outs[1]


def test_trace_program(tmp_path):
    cfg, w = U.PLAIN, U.weights(U.PLAIN, 1)
    path, seqs = U.save(tmp_path / "model", cfg, w), {"a": U.tokens(cfg, 22, 0), "b": U.tokens(cfg, 2, 1)}
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": seqs["a"][:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": seqs["a"][20:21], "want": []},
                                     {"id": "q", "tokens": seqs["b"], "want": []}], "end": ["q"]},
             {"step": 5, "entries": [{"id": "p", "tokens": seqs["a"][21:], "want": [0]}], "end": ["p"]}]
    out = tmp_path / "out"
    out.mkdir()
    run = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out),
                          "--max-tokens", "128", "--device", "cpu"], input="\n".join(json.dumps(s) for s in steps),
                         capture_output=True, text=True, timeout=120)
    assert run.returncode == 0, run.stderr
    got = [torch.frombuffer(bytearray((out / f).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
           for f in ("0.f32", "5.f32")]
    assert float(U.spread(torch.cat(got), plain.logits(cfg, w, seqs["a"])[[0, 19, 21]]).max()) < LIMIT
    assert float(torch.cat(got).abs().max()) < cfg["logit_softcap"]


def test_loader_names_what_is_wrong(tmp_path):
    w = U.weights(U.PLAIN, 0)
    del w["l1.mlp.correction"]
    with pytest.raises(KeyError, match="l1.mlp.correction"):
        _rep(U.save(tmp_path, U.PLAIN, w))
    w = U.weights(U.PLAIN, 0)
    w["l1.dwa"] = torch.ones(2)
    with pytest.raises(ValueError, match="l1.dwa"):
        _rep(U.save(tmp_path, U.PLAIN, w))


def test_config():
    mc = ModelConfig.from_hf(U.MIXED)
    assert mc.architectures == ("LigipelForCausalLM",) and mc.is_recurrent and mc.has_fp32_kernels and mc.depth_average
    assert mc.num_kv_layers == 4 and mc.head_geometry() == ((2, 64), (1, 64), (2, 64), (2, 256))
    assert [mc.head_row(i) for i in (0, 2, 3, 5)] == [0, 1, 2, 3] and [mc.state_row(i) for i in range(6)] == list(range(6))
    assert mc.state_geometries()[:2] == ((1, 48, 8), (3, 32, 16)) and mc.conv_geometries()[:3] == ((48, 2), (0, 0), (64, 3))
    assert mc.output_multiplier == 0.4 and mc.final_logit_softcapping == 7.0
    first, second = mc.layer_specs[0].mixer, mc.layer_specs[1].mixer
    assert isinstance(first, PairMixer) and first.left.window == 17 and first.left.talk and first.right.taps == 3
    assert isinstance(second, LinearAttnLayer) and second.rotary.rotary_dim == 10 and not second.weighted
    for bad in (U.config([dict(U.pair(), type="other")]), U.config([U.pair(heads=3)]), U.config([U.retention(rot=7)]),
                U.config([U.retention(rot=22)]), U.config([U.retention(decay=[0.5])]),
                U.config([U.pair(mlp={"kind": "dense", "ff": 8})]), U.config([U.pair(mlp=U.moe(3, 4))])):
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)


def test_state_cache_with_a_convolution_tail_per_layer():
    st = GDNStateCache(3, 2, 0, 2, 1, 1, 1, torch.float32, "cpu", geometries=((1, 4, 2), (2, 3, 3), (1, 2, 2)),
                       conv_geometries=((4, 2), (0, 0), (2, 3)))
    assert st.conv_state(0).shape == (2, 4, 2) and st.conv_state(2).shape == (2, 2, 3) and st.conv.numel() == 2 * 14
    st.conv_state(2)[1] = 5.0
    st.ssm_state(1)[1] = 3.0
    assert float(st.conv_state(0).abs().max()) == 0 and float(st.ssm_state(2).abs().max()) == 0
    st.snapshot(1, "k")
    st.conv_state(2)[1], st.ssm_state(1)[1] = 0.0, 0.0
    assert st.restore(0, "k") and float(st.conv_state(2)[0].min()) == 5.0 and float(st.ssm_state(1)[0].min()) == 3.0


# ---------------------------------------------------------------------------------- tensor parallelism
def _rank(rank, path, prompts, port, queue):
    from minisglang_rdna4_b200 import LLM, SamplingParams

    llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=2, num_page_override=64, tp_size=2,
              tp_rank=rank, base_port=port)
    outs = llm.generate(prompts, SamplingParams(max_tokens=5, ignore_eos=True))
    if rank == 0:
        queue.put([o.token_ids for o in outs])
    llm.shutdown()


def test_two_tensor_parallel_ranks(tmp_path):
    """Scan channels, retention heads and experts are split; mixed heads are on both ranks."""
    import torch.multiprocessing as mp

    cfg = U.config([U.pair(4, 1, mlp=U.moe()), U.retention(2, decay=[0.9, 0.99]), U.pair(2, 2, inner=24)], vocab=201)
    w = U.weights(cfg, 6)
    path = U.save(tmp_path, cfg, w)
    prompts = [U.tokens(cfg, 45, 1), U.tokens(cfg, 5, 2)]
    ctx = mp.get_context("spawn")
    q = ctx.Queue()
    port = 29000 + os.getpid() % 2000
    procs = [ctx.Process(target=_rank, args=(r, path, prompts, port, q)) for r in range(2)]
    for p in procs:
        p.start()
    got = q.get(timeout=120)
    for p in procs:
        p.join(60)
    assert got == [U.greedy(cfg, w, p, 5) for p in prompts]
