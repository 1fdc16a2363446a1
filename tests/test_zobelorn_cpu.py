"""The Zobelorn design through the framework on the CPU (fp32) against a plain restatement of its equations."""
import json
import math
import os
import subprocess

import pytest
import torch

import plain_zobelorn as plain
import zobelorn_util as U
from minisglang_rdna4_b200 import LLM, SamplingParams
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.models.config import HeadLayer, ModelConfig, RotaryConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer

LIMIT = 2e-4


def _g(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("mult", [1.0, 0.35])
def test_norm_of_the_output_scaled_and_added(mult):
    g = _g(0)
    x, d = torch.randn(7, 24, generator=g) * 3, torch.randn(7, 32, generator=g) * 5
    wb, w = torch.randn(24, generator=g), torch.randn(24, generator=g)
    xn, y = ref.add_norm(x, d, w + 1, 1e-2, False, torch.float32, 32, wb + 1, mult)
    want = x.double() + mult * plain.offset_norm(d[:, :24].double(), wb.double(), 1e-2)
    torch.testing.assert_close(xn.double(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(y[:, :24].double(), plain.offset_norm(want, w.double(), 1e-2), rtol=1e-5, atol=1e-5)
    assert float(y[:, 24:].abs().max()) == 0.0


def test_epsilon_is_inside_the_root():
    d = torch.tensor([[1e-3, -1e-3] * 4])
    xn, _ = ref.add_norm(torch.zeros(1, 8), d, torch.ones(8), 1e-2, False, torch.float32, 8, torch.ones(8), 1.0)
    torch.testing.assert_close(xn, d / math.sqrt(1e-6 + 1e-2))
    x = torch.full((1, 64), 1e-3)
    q = ref.heads_rope_store(x, 1, 0, 64, 64, torch.zeros(1, dtype=torch.int32), None, False, 1e-2, unit=True)
    torch.testing.assert_close(q.flatten(), x.flatten() / math.sqrt(1e-6 + 1e-2))


@pytest.mark.parametrize("factor,low,high,original", [(4.0, 1.0, 4.0, 64), (8.0, 1.0, 2.0, 500), (3.0, 2.0, 9.0, 70)])
def test_frequency_scaling(factor, low, high, original):
    """Every class of wavelengths occurs; the table agrees with the plain frequencies."""
    rot = {"base": 700.0, "dims": 32, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}
    layer = dict(U.chunk(dim=32, rot=32, base=700.0, scaling=(factor, low, high, original)), mlp=None)
    spec = ModelConfig.from_hf(U.config([layer])).layer_specs[0].mixer
    want = torch.tensor(plain.frequencies(rot, llama=True), dtype=torch.float64)
    base = torch.tensor(plain.frequencies(dict(rot, scaling=None), llama=True), dtype=torch.float64)
    kept, cut = (want == base).sum(), torch.isclose(want, base / factor).sum()
    assert kept > 0 and cut > 0 and 0 < 16 - kept - cut
    table = get_rope_cache(spec.rotary, "cpu")[:300].double()
    p = torch.arange(300, dtype=torch.float64)[:, None]
    torch.testing.assert_close(table, torch.cat([(p * want).cos(), (p * want).sin()], 1), rtol=0, atol=1e-6)


@pytest.mark.parametrize("neighbours", [True, False])
@pytest.mark.parametrize("dim,rot", [(24, 24), (24, 10), (9, 2), (64, 32), (20, 0)])
def test_rotation_of_part_of_a_head(dim, rot, neighbours):
    g = _g(dim)
    t, heads, width = 40, 3, 64
    x = torch.zeros(t, heads, width)
    x[..., :dim] = torch.randn(t, heads, dim, generator=g)
    table = get_rope_cache(RotaryConfig(dim, rot, 64, 90.0), "cpu") if rot else None
    got = ref.heads_rope_store(x.view(t, -1), heads, 0, width, dim, torch.arange(t, dtype=torch.int32), table, neighbours, 1e-5)
    want = plain.rotate(x.double(), plain.frequencies({"dims": rot, "base": 90.0}, False), neighbours)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-5)
    assert torch.equal(got[..., rot:], x[..., rot:])


def test_the_two_pairings_differ():
    x, f = torch.randn(5, 1, 8, generator=_g(0)).double(), [1.0, 0.5, 0.2, 0.1]
    assert float((plain.rotate(x, f, True) - plain.rotate(x, f, False)).abs().max()) > 0.1


@pytest.mark.parametrize("totals", [False, True])
def test_joint_norm_ahead_of_the_rotation(totals):
    """Over all query heads at once and over all key heads at once; padding columns do not enter the mean."""
    g = _g(4)
    t, hq, hk, dim, width = 12, 4, 2, 10, 64
    x = torch.zeros(t, hq + 2 * hk, width)
    x[..., :dim] = torch.randn(t, hq + 2 * hk, dim, generator=g) * torch.arange(1, 9).view(1, -1, 1)
    qw, kw = torch.zeros(hq, width), torch.zeros(hk, width)
    qw[:, :dim], kw[:, :dim] = torch.randn(hq, dim, generator=g), torch.randn(hk, dim, generator=g)
    kc, vc = torch.full((2, hk, 8, width), 9.0), torch.full((2, hk, 8, width), 9.0)
    loc = torch.tensor([9, 2, 0, 15, 4, 5, 6, 8, 1, 3, 12, 11], dtype=torch.int32)
    table = get_rope_cache(RotaryConfig(dim, 6, 64, 50.0), "cpu")
    pos = torch.arange(t, dtype=torch.int32)
    sums = None
    if totals:
        sums = (torch.stack([x[:, :hq].pow(2).sum((1, 2)), x[:, hq:hq + hk].pow(2).sum((1, 2))], 1), hq * dim, hk * dim)
    got = ref.heads_rope_store(x.view(t, -1), hq, hk, width, dim, pos, table, False, 1e-3, qw.view(-1), kw.view(-1), sums, False,
                               (kc, vc, loc))
    f = plain.frequencies({"dims": 6, "base": 50.0}, False)
    for a, b, w, rows in ((0, hq, qw, got), (hq, hq + hk, kw, None)):
        y = x[:, a:b, :dim].double().reshape(t, -1)
        want = plain.unit_rms(y, 1e-3) * w[:, :dim].double().reshape(-1)
        want = plain.rotate(want.view(t, b - a, dim), f, False)
        if rows is None:
            rows = torch.stack([kc[loc[i] // 8, :, loc[i] % 8] for i in range(t)])
        torch.testing.assert_close(rows[..., :dim].double(), want, rtol=1e-4, atol=1e-5)
        assert float(rows[..., dim:].abs().max()) == 0.0
    stored = torch.stack([vc[loc[i] // 8, :, loc[i] % 8] for i in range(t)])
    assert torch.equal(stored, x[:, hq + hk:])
    assert float(kc.view(2, hk, 8, -1)[0, :, 7].min()) == 9.0            # a slot nobody wrote


def test_unit_norm_comes_after_the_rotation_and_counts_the_channels():
    g = _g(5)
    x = torch.zeros(6, 2, 64)
    x[..., :20] = torch.randn(6, 2, 20, generator=g) * 7
    table = get_rope_cache(RotaryConfig(20, 20, 64, 50.0), "cpu")
    got = ref.heads_rope_store(x.view(6, -1), 2, 0, 64, 20, torch.arange(6, dtype=torch.int32), table, True, 0.5, unit=True)
    r = plain.rotate(x[..., :20].double(), plain.frequencies({"dims": 20, "base": 50.0}, False), True)
    torch.testing.assert_close(got[..., :20].double(), plain.unit_rms(r, 0.5), rtol=1e-5, atol=1e-6)


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
    return q, k, v, bt, cu, torch.tensor(lens, dtype=torch.int32), torch.randn(sum(q_lens), hq * d, generator=g) * 2


@pytest.mark.parametrize("kind,size", [("window", 1), ("window", 2), ("window", 16), ("window", 17), ("window", 500),
                                       ("chunk", 1), ("chunk", 7), ("chunk", 16), ("chunk", 33), ("chunk", 500)])
@pytest.mark.parametrize("cap", [0.0, 1.5])
def test_attention_with_reach_cap_and_gate(kind, size, cap):
    lens, q_lens, hq, hk, d, ps = [40, 33, 17, 1], [40, 1, 2, 1], 6, 2, 8, 16
    q, k, v, bt, cu, seq, gate = _dense_case(size, lens, q_lens, hq, hk, d, ps)
    got = ref.paged_attention(q, k, v, bt, cu, seq, 0.4, window=size if kind == "window" else 0,
                              chunk=size if kind == "chunk" else 0, softcap=cap, gate=gate)
    first = plain.first_in_window if kind == "window" else plain.first_in_chunk
    for b, (n, m) in enumerate(zip(lens, q_lens)):
        pages = bt[b, :-(-n // ps)].long()
        kk, vv = (x[pages].transpose(1, 2).reshape(-1, hk, d)[:n].double() for x in (k, v))
        full = torch.zeros(n, hq, d).double()
        lo, hi = int(cu[b]), int(cu[b + 1])
        full[n - m:] = q[lo:hi].double()
        want = plain.attend(full, kk, vv, 0.4, lambda i: first(i, size), cap or None)[n - m:]
        want = want * torch.sigmoid(gate[lo:hi].double())
        torch.testing.assert_close(got[lo:hi].double().reshape(m, -1), want, rtol=1e-4, atol=1e-5)


@pytest.mark.parametrize("kind,size", [("window", 33), ("window", 64), ("chunk", 48), ("chunk", 50)])
@pytest.mark.parametrize("at", [0, 15, 16, 47, 48, 49, 50, 99])
def test_a_loud_key_is_seen_exactly_within_reach(kind, size, at):
    q, k, v, bt = U.loud_key(130, at, 130, 64, 16)
    got = ref.paged_attention(q, k, v, bt, torch.tensor([0, 130]), torch.tensor([130]), 1.0,
                              window=size if kind == "window" else 0, chunk=size if kind == "chunk" else 0)
    assert (got[:, 0, 0] > 4.9).nonzero().flatten().tolist() == U.seen_rows(kind, at, size, 130)


def test_soft_cap_limits_a_score():
    """Two keys, one score far above the cap: the weights are those of the capped scores."""
    q, k, v, bt = U.loud_key(2, 1, 1, 64, 16)
    got = ref.paged_attention(q, k, v, bt, torch.tensor([0, 1]), torch.tensor([2]), 1.0, softcap=2.0)
    assert math.isclose(float(got[0, 0, 0]), 5.0 / (1.0 + math.exp(-2.0)), rel_tol=1e-5)


def test_expert_weights_act_on_the_input():
    """silu is not linear: expert(w x) is not w expert(x); the weights are plain sigmoid scores."""
    g = _g(7)
    h, router = torch.randn(20, 12, generator=g), torch.randn(6, 12, generator=g)
    w = {"m.router": router.double()}
    w13, w2 = torch.randn(6, 10, 12, generator=g), torch.randn(6, 12, 5, generator=g)
    for e in range(6):
        w[f"m.e{e}.gate"], w[f"m.e{e}.up"], w[f"m.e{e}.down"] = w13[e, :5].double(), w13[e, 5:].double(), w2[e].double()
    tw, ids = ref.moe_route(h @ router.T, 3, False, "sigmoid")
    want = plain.expert_mixture(h.double(), w, "m", {"router": {"top": 3}})
    got = ref.experts_partial32(h, w13, w2, tw, ids, 0.0, 0.0, act="silu", on_input=True)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-4)
    other = ref.experts_partial32(h, w13, w2, tw, ids, 0.0, 0.0, act="silu")
    assert float((other - got).abs().max()) > 0.1
    assert float((tw.sum(-1) - 1).abs().min()) > 1e-3                  # not renormalised
    shared = torch.randn(20, 12, generator=g)
    got2 = ref.experts_partial32(h, w13, w2, tw, ids, 0.0, 0.0, shared, None, act="silu", on_input=True)
    torch.testing.assert_close(got2, got + shared, rtol=1e-5, atol=1e-5)


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


@pytest.mark.parametrize("page", [8, 16, 64])
def test_mixed_batches_and_reused_pages(model, page):
    cfg, w, path, seqs, want = model
    U.play(_rep(path, page=page), seqs, U.mixed_schedule(), want, LIMIT)


def test_a_batch_equals_each_request_alone(model):
    cfg, w, path, seqs, want = model
    U.play(_rep(path), seqs, [[(n, len(s)) for n, s in seqs.items()]], want, LIMIT)


def test_pool_holds_exactly_the_live_tokens(model):
    """The pool is as large as one request: the next can only run on the pages the last gave back."""
    cfg, w, path, seqs, want = model
    rep = _rep(path, max_tokens=80)
    for k in range(3):
        for name in seqs:
            U.play(rep, seqs, [[(f"{name}#{k}", n)] for n in U.cuts(len(seqs[name]), [25, 1])], want, LIMIT)
    with pytest.raises(RuntimeError, match="pages"):
        rep.step([("x", seqs["a"], []), ("y", seqs["d"], [])])


def test_long_decoding(tmp_path):
    cfg = U.config([U.chunk(size=64), U.window(size=50), U.chunk(size=100, kv_from=0)])
    w = U.weights(cfg, 4)
    rep = _rep(U.save(tmp_path, cfg, w), 256)
    seqs = {"a": U.tokens(cfg, 230, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 225, U.reference(cfg, w, seqs), LIMIT)


@pytest.mark.parametrize("kind,size,at", [("window", 40, 30), ("window", 16, 16), ("window", 1, 5), ("chunk", 40, 30),
                                          ("chunk", 40, 40), ("chunk", 40, 39), ("chunk", 16, 31), ("chunk", 1, 5)])
@pytest.mark.parametrize("sizes", [[100], [1], [31, 2], [60, 1]])
def test_a_planted_token_shows_exactly_where_it_is_seen(tmp_path, kind, size, at, sizes):
    cfg, w = U.planted_token_model(kind, size)
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
    assert (moved > 0).nonzero().flatten().tolist() == U.seen_rows(kind, at, size, 100)
    assert float(U.spread(rows[1], plain.logits(cfg, w, planted)).max()) < LIMIT


@pytest.mark.parametrize("cfg", [
    U.config([U.window(1, 1, 2, 1, 1), U.chunk(1, 1, 2, 1, 1), U.chunk(1, 1, 2, 1, 3, kv_from=1, mlp=U.moe(2, 1, 1, shared=1))],
             width=5, vocab=7, scale=1.0),
    U.config([U.window(7, 7, 130, 150, 300, mlp=U.dense(33)), U.chunk(6, 1, 70, 130, 8, rot=64)], width=40, vocab=64),
    U.config([U.window(mlp=U.dense(7)), U.window()], vocab=100, mult=2.0),
    U.config([U.chunk(), U.chunk(mlp=U.moe(4, 4, 16)), U.chunk(kv_from=0), U.chunk(kv_from=1)], vocab=100, eps=1e-2),
], ids=["ones", "wide", "windows-only", "chunks-only"])
def test_other_sizes(cfg, tmp_path):
    w = U.weights(cfg, 2)
    seqs = {"a": U.tokens(cfg, 40, 1), "b": U.tokens(cfg, 2, 2)}
    rep = _rep(U.save(tmp_path, cfg, w))
    U.play(rep, seqs, [[("a", 7)], [("a", 1), ("b", 1)], [("b", 1), ("a", 32)]], U.reference(cfg, w, seqs), LIMIT)


# ---------------------------------------------------------------------------------- entry points
def test_greedy_generation_prefix_cache_and_chunks(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=3, num_page_override=64, max_extend_tokens=24)
    sp = SamplingParams(max_tokens=5, ignore_eos=True)
    prompts = [seqs["a"], seqs["b"], seqs["c"][:3], seqs["d"]]
    for o, s in zip(llm.generate(prompts, sp), prompts):
        assert o.token_ids == U.greedy(cfg, w, s, 5)
    again = seqs["d"][:50] + seqs["a"][:9]        # a cached prefix
    o = llm.generate([again], sp)[0]
    assert o.cached_tokens > 0
    assert o.token_ids == U.greedy(cfg, w, again, 5)
    llm.shutdown()


def test_draft_verification_keeps_the_greedy_tokens(model):
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
    assert run.stdout.split("\n")[:3] == ["done 0", "done 1", "done 5"]
    got = [torch.frombuffer(bytearray((out / f).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
           for f in ("0.f32", "5.f32")]
    assert float(U.spread(torch.cat(got), plain.logits(cfg, w, seqs["a"])[[0, 19, 21]]).max()) < LIMIT


def test_loader_names_what_is_wrong(tmp_path):
    w = U.weights(U.PLAIN, 0)
    del w["l1.mlp.e4.up"]
    with pytest.raises(KeyError, match="l1.mlp.e4.up"):
        _rep(U.save(tmp_path, U.PLAIN, w))
    w = U.weights(U.PLAIN, 0)
    w["l0.mix.k.norm"] = torch.ones(21)
    with pytest.raises(ValueError, match="l0.mix.k.norm"):
        _rep(U.save(tmp_path, U.PLAIN, w))


def test_config():
    mc = ModelConfig.from_hf(U.MIXED)
    assert mc.architectures == ("ZobelornForCausalLM",) and not mc.is_recurrent and mc.has_fp32_kernels
    assert mc.num_kv_layers == 4 and mc.head_geometry() == ((2, 64), (1, 64), (2, 128), (1, 128))
    assert [mc.head_row(i) for i in range(6)] == [0, 1, 0, 2, 3, 3]
    assert mc.residual_multiplier == 0.6 and mc.embedding_multiplier == 5.0
    first, second = mc.layer_specs[0].mixer, mc.layer_specs[1].mixer
    assert isinstance(first, HeadLayer) and (first.window, first.chunk, first.rotary.interleaved) == (0, 23, True)
    assert (second.window, second.chunk, second.softcap, second.rotary.rotary_dim) == (17, 0, 6.0, 12)
    assert first.unit_norm and not first.joint_norm and second.joint_norm and second.gate and not first.gate
    for bad in (U.config([dict(U.chunk(), type="other")]), U.config([U.chunk(kv_from=0)]),
                U.config([U.chunk(), U.chunk(kv_from=0, kv=4)]), U.config([U.chunk(), U.chunk(kv_from=0, base=7.0)]),
                U.config([U.window(4, 2, 24, 12), U.chunk(kv_from=0)]), U.config([U.chunk(), U.chunk(kv_from=0), U.chunk(kv_from=1)]),
                U.config([U.chunk(rot=7)]), U.config([U.chunk(rot=26)]), U.config([U.chunk(heads=3)]),
                U.config([U.window(mlp={"kind": "routed", "ff": 8})]), U.config([U.chunk(mlp=U.moe(3, 4))])):
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)


def test_pool_planes_of_different_geometry():
    from minisglang_rdna4_b200.kvcache import LayeredKVCache

    pool = LayeredKVCache(5, 8, [(2, 64), (1, 128)], torch.float32, "cpu")
    assert pool.k_cache(0).shape == (6, 2, 8, 64) and pool.v_cache(1).shape == (6, 1, 8, 128) and pool.dummy_page == 5
    assert LayeredKVCache.token_bytes([(2, 64), (1, 128)], 4) * 6 * 8 == pool.nbytes
    g = _g(0)
    k, v, loc = torch.randn(3, 1, 128, generator=g), torch.randn(3, 1, 128, generator=g), torch.tensor([40, 7, 8])
    pool.store_kv(k, v, loc, 1)
    assert torch.equal(pool.k_cache(1)[5, :, 0], k[0]) and torch.equal(pool.v_cache(1)[0, :, 7], v[1])
    assert torch.equal(pool.k_cache(1)[1, :, 0], k[2]) and float(pool.k_cache(0).abs().max()) == 0.0


# ---------------------------------------------------------------------------------- tensor parallelism
def _rank(rank, path, prompts, port, queue):
    from minisglang_rdna4_b200 import LLM, SamplingParams

    llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=2, num_page_override=64, tp_size=2,
              tp_rank=rank, base_port=port)
    outs = llm.generate(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
    if rank == 0:
        queue.put([o.token_ids for o in outs])
    llm.shutdown()


def test_two_tensor_parallel_ranks(tmp_path):
    """One key / value head for two ranks is on both; the norm over all heads spans the ranks."""
    import torch.multiprocessing as mp

    cfg = U.config([U.window(4, 2, mlp=U.dense(90)), U.chunk(4, 1, mlp=U.moe()), U.window(6, 1), U.chunk(2, 1, kv_from=1)],
                   vocab=201)
    w = U.weights(cfg, 6)
    path = U.save(tmp_path, cfg, w)
    prompts = [U.tokens(cfg, 45, 1), U.tokens(cfg, 5, 2)]
    ctx = mp.get_context("spawn")
    q = ctx.Queue()
    port = 27000 + os.getpid() % 2000
    procs = [ctx.Process(target=_rank, args=(r, path, prompts, port, q)) for r in range(2)]
    for p in procs:
        p.start()
    got = q.get(timeout=120)
    for p in procs:
        p.join(60)
    assert got == [U.greedy(cfg, w, p, 6) for p in prompts]
