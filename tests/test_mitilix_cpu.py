"""The Mitilix design through the framework on the CPU (fp32) against a plain restatement of its equations."""
import json
import math
import os
import subprocess

import pytest
import torch

import mitilix_util as U
import plain_mitilix as plain
from minisglang_rdna4_b200 import LLM, SamplingParams
from minisglang_rdna4_b200.models.config import ModelConfig
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer

LIMIT = 2e-4


# ---------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("portions", [[50], [1], [2], [3, 1, 8]])
def test_norm_and_input_convolution(taps, portions):
    """The tail carries over portions of any size; both filters read the same normalised rows."""
    g = torch.Generator().manual_seed(taps)
    x, add = torch.randn(50, 24, generator=g), torch.randn(50, 32, generator=g)
    w1, w2, gain = torch.randn(24, taps, generator=g), torch.randn(24, taps, generator=g), torch.tensor([1.7])
    h = plain.scalar_rms_norm((x + add[:, :24]).double(), gain.double(), 1e-5)
    want = [plain.input_convolution(h, w.double()) for w in (w1, w2)]
    state, slots = torch.full((3, taps - 1, 24), 9.0), torch.tensor([1], dtype=torch.int32)
    lo = 0
    for n in U.cuts(50, portions):
        got = ref.add_scalar_norm_conv(x[lo:lo + n], add[lo:lo + n], gain, 1e-5, w1.t().contiguous(), w2.t().contiguous(),
                                       state, torch.tensor([0, n]), slots, torch.tensor([int(lo > 0)]), torch.float32, 32)
        torch.testing.assert_close(got[0], x[lo:lo + n] + add[lo:lo + n, :24])
        for y, wy in zip(got[1:], want):
            torch.testing.assert_close(y[:, :24].double(), wy[lo:lo + n], rtol=1e-5, atol=1e-5)
            assert float(y[:, 24:].abs().max()) == 0.0
        lo += n
    assert float(state[0].sum()) == float(state[2].sum()) == 9.0 * state[0].numel()     # other requests' tails


def test_norm_epsilon_is_inside_the_root():
    x = torch.full((1, 8), 1e-3)
    got = ref.add_scalar_norm_conv(x, None, torch.ones(1), 1e-2, None, None, None, None, None, None, torch.float32, 8)[1]
    torch.testing.assert_close(got, x / math.sqrt(1e-6 + 1e-2))


def test_gelu_is_the_exact_one():
    x = torch.linspace(-6, 6, 101)[None]
    torch.testing.assert_close(ref.gelu_erf(x, torch.empty_like(x)).double(), plain.erf_gelu(x.double()), rtol=1e-5, atol=1e-6)


def test_latent_norm():
    g = torch.Generator().manual_seed(0)
    c, w = torch.randn(5, 64, generator=g), torch.rand(64, generator=g)
    pool = torch.zeros(3, 4, 64)
    loc = torch.tensor([1, 9, 4, 3, 11], dtype=torch.int32)
    ref.latent_norm_store(c, w, 40, 1e-5, pool, loc)
    rows = pool.view(-1, 64)[loc.long()]
    torch.testing.assert_close(rows[:, :40].double(), plain.vector_rms_norm(c[:, :40].double(), w[:40].double(), 1e-5),
                               rtol=1e-5, atol=1e-6)
    assert float(rows[:, 40:].abs().max()) == 0.0


@pytest.mark.parametrize("window", [1, 2, 16, 17, 40, 100])
def test_latent_attention_window(window):
    """Absorbed attention over the paged pool equals keys and values expanded per head, in one step or in portions."""
    g = torch.Generator().manual_seed(window)
    t, heads, dim, vdim, rank, ps = 70, 2, 12, 20, 64, 16
    c = torch.randn(t, rank, generator=g)
    q, uk = torch.randn(t, heads * dim, generator=g) * 2, torch.randn(heads * dim, rank, generator=g) * 0.2
    uv = torch.randn(heads * vdim, rank, generator=g)
    p = {"q": torch.eye(heads * dim).double(), "uk": uk.double(), "uv": uv.double(), "o": torch.eye(heads * vdim).double()}
    want = plain.latent_attention(q.double(), c.double(), p, heads, dim, vdim, 0.5, window)
    bt = torch.tensor([[4, 0, 3, 1, 2]], dtype=torch.int32)
    pool = torch.randn(6, ps, rank, generator=g)
    pos = torch.arange(t)
    pool.view(-1, rank)[bt[0].long()[pos // ps] * ps + pos % ps] = c
    q_lat = ref.head_gemm(q.view(t, heads, dim), uk.view(heads, dim, rank).transpose(1, 2).contiguous())
    for sizes in ([t], [2], [1], [31, 5]):
        lo = 0
        for n in U.cuts(t, sizes):
            o = ref.latent_attention(q_lat[lo:lo + n], pool, bt, torch.tensor([0, n]), torch.tensor([lo + n]), 0.5, window)
            v = ref.head_gemm(o, uv.view(heads, vdim, rank))
            torch.testing.assert_close(v.reshape(n, -1).double(), want[lo:lo + n], rtol=1e-4, atol=1e-4)
            lo += n


@pytest.mark.parametrize("decode", [False, True])
def test_a_key_at_the_windows_edge_is_seen_and_the_next_one_is_not(decode):
    window, n, ps, r = 24, 100, 16, 64
    bt = torch.arange(7, dtype=torch.int32)[None]
    for loud, seen in ((n - window, True), (n - window - 1, False)):
        pool = torch.zeros(7, ps, r)
        flat = pool.view(-1, r)
        flat[:, 1] = 1.0
        flat[loud, 0] = 10.0
        q = torch.zeros(n, 1, r)
        q[:, :, 0] = 10.0
        rows = q[-1:] if decode else q
        got = ref.latent_attention(rows, pool, bt, torch.tensor([0, rows.shape[0]]), torch.tensor([n]), 1.0, window)
        assert (float(got[-1, 0, 0]) > 9.0) == seen


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


def planted_key_model():
    """One layer, one head; token 7's key dominates every query."""
    cfg = U.config([U.layer(heads=1, dim=16, vdim=16, rank=16, window=20, ff=0, scale=1.0)], width=16, taps=1)
    w = U.weights(cfg, 3, sharp=1.0)
    w["pos"] *= 0
    w["embed"][:, 0] = 0
    w["embed"][:, 1] = 3.0
    w["embed"][7] = torch.zeros(16).index_fill(0, torch.tensor([0]), 4.0)
    w["l0.mix.q"] = torch.zeros(16, 16).index_put((torch.tensor([0]), torch.tensor([1])), torch.tensor(40.0)).bfloat16()
    w["l0.mix.uk"] = w["l0.mix.dkv"] = torch.eye(16).bfloat16()
    w["l0.mix.dkv.norm"] = torch.ones(16).bfloat16()
    return cfg, w


@pytest.mark.parametrize("sizes", [[80], [1], [49, 1], [50, 1], [29, 2]])
def test_a_planted_key_moves_the_positions_whose_window_holds_it(tmp_path, sizes):
    """In prompts, in portions and in decoding exactly the positions that can see the key change when it is planted."""
    cfg, w = planted_key_model()
    without = [t if t != 7 else 8 for t in U.tokens(cfg, 80, 5)]
    planted = list(without)
    planted[30] = 7
    rep = _rep(U.save(tmp_path, cfg, w))
    rows = []
    for k, seq in enumerate((without, planted)):
        lo, got = 0, []
        for n in U.cuts(80, sizes):
            got.append(rep.step([(str(k), seq[lo:lo + n], list(range(n)))], [str(k)] if lo + n == 80 else []))
            lo += n
        rows.append(torch.cat(got))
    moved = (rows[0] - rows[1]).abs().amax(-1) > 1e-3
    assert moved.nonzero().flatten().tolist() == list(range(30, 50))


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


def test_long_decoding_to_the_last_position(tmp_path):
    cfg = U.config([U.layer(window=37), U.layer(window=90, kv_from=0, heads=2)], taps=2, max_positions=211)
    w = U.weights(cfg, 4)
    rep = _rep(U.save(tmp_path, cfg, w), 256)
    seqs = {"a": U.tokens(cfg, 211, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 206, U.reference(cfg, w, seqs), LIMIT)
    with pytest.raises(ValueError, match="limit"):
        rep.step([("b", U.tokens(cfg, 212, 1), [])])


@pytest.mark.parametrize("cfg", [
    U.config([U.layer(heads=1, dim=1, vdim=1, rank=1, window=1, ff=1)], width=5, vocab=7, taps=1, max_positions=40),
    U.config([U.layer(heads=7, dim=130, vdim=150, rank=300, window=300, ff=33)], width=40, vocab=64, taps=9),
    U.config([U.layer(ff=0)], taps=32, vocab=100),
], ids=["ones", "wide", "taps32"])
def test_other_sizes(cfg, tmp_path):
    w = U.weights(cfg, 2)
    seqs = {"a": U.tokens(cfg, 40, 1), "b": U.tokens(cfg, 2, 2)}
    rep = _rep(U.save(tmp_path, cfg, w))
    U.play(rep, seqs, [[("a", 7)], [("a", 1), ("b", 1)], [("b", 1), ("a", 32)]], U.reference(cfg, w, seqs), LIMIT)


# ---------------------------------------------------------------------------------- entry points
def _greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(plain.logits(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_greedy_generation_prefix_cache_and_chunks(model):
    cfg, w, path, seqs, _ = model
    llm = LLM(path, device="cpu", dtype="fp32", page_size=8, max_running_req=3, num_page_override=64, max_extend_tokens=24)
    sp = SamplingParams(max_tokens=5, ignore_eos=True)
    prompts = [seqs["a"], seqs["b"], seqs["c"][:3], seqs["d"]]
    for o, s in zip(llm.generate(prompts, sp), prompts):
        assert o.token_ids == _greedy(cfg, w, s, 5)
    again = seqs["d"][:50] + seqs["a"][:9]        # a cached prefix: its latents and the state at its boundary
    o = llm.generate([again], sp)[0]
    assert o.cached_tokens > 0
    assert o.token_ids == _greedy(cfg, w, again, 5)
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
    assert sorted(os.listdir(out)) == ["0.f32", "5.f32"]
    got = [torch.frombuffer(bytearray((out / f).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
           for f in ("0.f32", "5.f32")]
    assert float(U.spread(torch.cat(got), plain.logits(cfg, w, seqs["a"])[[0, 19, 21]]).max()) < LIMIT


def test_loader_names_what_is_wrong(tmp_path):
    w = U.weights(U.PLAIN, 0)
    del w["l1.mix.uk"]
    with pytest.raises(KeyError, match="l1.mix.uk"):
        _rep(U.save(tmp_path, U.PLAIN, w))
    w = U.weights(U.PLAIN, 0)
    w["l0.mlp.up"] = w["l0.mlp.up"][:, :-1]
    with pytest.raises(ValueError, match="l0.mlp.up"):
        _rep(U.save(tmp_path, U.PLAIN, w))


def test_config():
    mc = ModelConfig.from_hf(U.MIXED)
    assert mc.architectures == ("MitilixForCausalLM",) and mc.is_recurrent
    assert mc.num_kv_layers == 2 and mc.latent_widths == (64, 128)
    assert [mc.latent_row(i) for i in range(4)] == [0, 1, 0, 1]
    for bad in (U.config([dict(U.layer(), type="other")]), U.config([U.layer(kv_from=0)]),
                U.config([U.layer(), U.layer(kv_from=0, rank=64)]),
                U.config([dict(U.layer(), mlp={"kind": "routed", "ff": 8})])):
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)


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
    import torch.multiprocessing as mp

    cfg = U.config([U.layer(heads=4, ff=90), U.layer(heads=2, window=33, kv_from=0), U.layer(heads=2, ff=0)], vocab=201)
    w = U.weights(cfg, 6)
    path = U.save(tmp_path, cfg, w)
    prompts = [U.tokens(cfg, 45, 1), U.tokens(cfg, 5, 2)]
    ctx = mp.get_context("spawn")
    q = ctx.Queue()
    port = 23000 + os.getpid() % 2000
    procs = [ctx.Process(target=_rank, args=(r, path, prompts, port, q)) for r in range(2)]
    for p in procs:
        p.start()
    got = q.get(timeout=120)
    for p in procs:
        p.join(60)
    assert got == [_greedy(cfg, w, p, 6) for p in prompts]
