"""The Rafodra design through the framework on the CPU (fp32) against a plain restatement of its equations."""
import json
import math
import os
import subprocess

import pytest
import torch

import plain_rafodra as plain
import rafodra_util as U
from minisglang_rdna4_b200 import LLM, SamplingParams
from minisglang_rdna4_b200.models.config import LatentLayer, LinearAttnLayer, ModelConfig, RotaryConfig
from minisglang_rdna4_b200.layers.rotary import get_rope_cache
from minisglang_rdna4_b200.ops import ref
from minisglang_rdna4_b200.replay import make_replayer

LIMIT = 2e-4


def _g(seed):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------------------------- mechanisms alone
def test_layer_norm_and_rms_norm():
    g = _g(0)
    x, d, w = torch.randn(7, 24, generator=g) + 3, torch.randn(7, 32, generator=g), torch.randn(24, generator=g)
    xn, y = ref.add_norm(x, d, w, 1e-5, True, torch.float32, 32)
    torch.testing.assert_close(xn, x + d[:, :24])
    torch.testing.assert_close(y[:, :24].double(), plain.layer_norm(xn.double(), w.double(), 1e-5), rtol=1e-5, atol=1e-5)
    assert float(y[:, 24:].abs().max()) == 0.0
    y = ref.add_norm(x, None, w, 1e-5, False, torch.float32, 24)[1]
    torch.testing.assert_close(y.double(), plain.rms_norm(x.double(), w.double(), 1e-5), rtol=1e-5, atol=1e-5)


def test_norm_epsilon_is_inside_the_root():
    x = torch.tensor([[1e-3, -1e-3] * 4])
    y = ref.add_norm(x, None, torch.ones(8), 1e-2, True, torch.float32, 8)[1]
    torch.testing.assert_close(y, x / math.sqrt(1e-6 + 1e-2))


@pytest.mark.parametrize("dims,rot,rank", [(12, 12, 40), (2, 2, 7), (6, 10, 33)])
def test_rotation_and_latent_store(dims, rot, rank):
    """Neighbouring pairs turn; channels past the rotated ones and the unrotated part stay; the latent alone is normed."""
    g = _g(dims)
    t, heads, dim, width = 50, 3, 9, 64
    q, c, w = torch.randn(t, heads, 32, generator=g), torch.randn(t, width, generator=g), torch.rand(width, generator=g)
    table = get_rope_cache(RotaryConfig(rot, dims, 64, 500.0, interleaved=True), "cpu")
    want_q, want_k = plain.rotate_pairs(q[..., dim:].double(), dims, 500.0), plain.rotate_pairs(c[:, rank:rank + rot].double(), dims, 500.0)
    got, pool = q.clone(), torch.full((5, 16, width), 7.0)
    loc = torch.randperm(80, generator=g)[:t].int()
    ref.latent_rope(got, dim, dims, table, torch.arange(t, dtype=torch.int32), (c, w, rank, 1e-5, pool, loc, rot))
    torch.testing.assert_close(got[..., dim:].double(), want_q, rtol=1e-4, atol=1e-4)
    assert torch.equal(got[..., :dim], q[..., :dim])
    rows = pool.view(-1, width)[loc.long()].double()
    torch.testing.assert_close(rows[:, :rank], plain.rms_norm(c[:, :rank].double(), w[:rank].double(), 1e-5), rtol=1e-4, atol=1e-5)
    torch.testing.assert_close(rows[:, rank:rank + rot], want_k, rtol=1e-4, atol=1e-4)
    assert float(rows[:, rank + rot:].abs().max() if rank + rot < width else 0.0) == 0.0


def test_rotated_scores_depend_on_the_distance():
    q, k = torch.randn(1, 8, generator=_g(1)).expand(40, 8).double(), torch.randn(1, 8, generator=_g(2)).expand(40, 8).double()
    s = plain.rotate_pairs(q, 8, 50.0) @ plain.rotate_pairs(k, 8, 50.0).T
    torch.testing.assert_close(s[20, 13], s[37, 30], rtol=1e-9, atol=1e-9)
    assert abs(float(s[20, 13] - s[20, 12])) > 1e-3


@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 60.0])
def test_sink_takes_its_share_and_is_not_scaled(sink):
    pool, bt, _ = U.loud_key(3, 5, 1, 64, 16)          # three equal keys (no loud one)
    q = torch.zeros(1, 2, 64)
    q[..., 1] = 2.0                                     # score 2 * 0.5 = 1 for every key
    got = ref.latent_attention(q, pool, bt, torch.tensor([0, 1]), torch.tensor([3]), 0.5, 0, torch.tensor([sink, -1e9]))
    assert math.isclose(float(got[0, 0, 1]), U.sink_share([1.0] * 3, sink), rel_tol=1e-5)
    assert math.isclose(float(got[0, 1, 1]), 1.0, rel_tol=1e-6)      # another head's sink


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 199])
def test_a_far_key_is_seen(at, decode):
    pool, bt, q = U.loud_key(200, at, 1 if decode else 200, 64, 16)
    got = ref.latent_attention(q, pool, bt, torch.tensor([0, q.shape[0]]), torch.tensor([200]), 1.0, 0, torch.zeros(1))
    assert float(got[-1, 0, 0]) > 9.9
    if not decode and at > 0:
        assert float(got[at - 1, 0, 0]) == 0.0          # and not before its time


def test_gate_of_the_value_projection():
    g = _g(3)
    x, w, gate = torch.randn(5, 2, 8, generator=g), torch.randn(2, 6, 8, generator=g), torch.randn(5, 2, generator=g)
    got = ref.head_gemm(x, w, torch.empty(5, 2, 6), gate)
    want = torch.einsum("thk,hnk->thn", x, w) * torch.sigmoid(gate)[..., None]
    torch.testing.assert_close(got, want)


def _run_linear(q, k, v, sizes, slots=3, slot=1, fill=9.0, **kw):
    state = torch.full((slots, q.shape[1], q.shape[2], v.shape[2]), fill)
    out, lo = [], 0
    for n in U.cuts(q.shape[0], sizes):
        part = {key: (tuple([x[0][lo:lo + n], *x[1:]]) if key == "gate" else x) for key, x in kw.items()}
        out.append(ref.linear_attention(q[lo:lo + n], k[lo:lo + n], v[lo:lo + n], state, torch.tensor([0, n]),
                                        torch.tensor([slot]), torch.tensor([int(lo > 0)]), **part))
        lo += n
    others = [s for i, s in enumerate(state) if i != slot]
    assert all(float((s - fill).abs().max()) == 0.0 for s in others)      # other requests' states
    return torch.cat(out), state[slot]


@pytest.mark.parametrize("sizes", [[60], [1], [2], [16, 1, 3]])
@pytest.mark.parametrize("act", [True, False])
def test_linear_attention_one_decay_per_head(sizes, act):
    g = _g(4)
    q, k, v = (torch.randn(60, 3, n, generator=g) for n in (8, 8, 5))
    decay = torch.tensor([0.3, 0.97, 1.0])
    got, _ = _run_linear(q, k, v, sizes, decay=decay, q_scale=0.5, act=act)
    f = plain.silu if act else (lambda x: x)
    for n in range(3):
        want = plain.decaying_memory(f(q[:, n].double()) * 0.5, f(k[:, n].double()), f(v[:, n].double()),
                                     torch.full((60, 8), float(decay[n])).double())
        torch.testing.assert_close(got[:, n].double(), want, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("tau,shift", [(16.0, 2.0), (1.0, 0.0), (1.0, -40.0), (3.0, 90.0)])
@pytest.mark.parametrize("sizes", [[50], [1], [2], [7, 16]])
def test_linear_attention_one_decay_per_channel(tau, shift, sizes):
    g = _g(5)
    q, k, v = (torch.randn(50, 2, n, generator=g) for n in (6, 6, 9))
    low, up, bias = torch.randn(50, 4, generator=g), torch.randn(12, 4, generator=g), torch.randn(12, generator=g) + shift
    got, _ = _run_linear(q, k, v, sizes, gate=(low, up, bias), tau=tau)
    alpha = plain.channel_decay(low.double(), torch.eye(4).double(), up.double(), bias.double(), tau).view(50, 2, 6)
    for n in range(2):
        want = plain.decaying_memory(q[:, n].double(), k[:, n].double(), v[:, n].double(), alpha[:, n])
        torch.testing.assert_close(got[:, n].double(), want, rtol=1e-4, atol=1e-4)


def test_decay_acts_before_the_new_token_is_added():
    one = torch.ones(2, 1, 1)
    got, state = _run_linear(one, one, torch.tensor([4.0, 1.0]).view(2, 1, 1), [2], decay=torch.tensor([0.5]))
    assert got.flatten().tolist() == [4.0, 3.0] and float(state) == 3.0


@pytest.mark.parametrize("act", ["sigmoid", "silu"])
@pytest.mark.parametrize("joint", [True, False])
def test_norm_and_gate(joint, act):
    """Zero padding past a head's width does not enter the mean square."""
    g = _g(6)
    o, gate = torch.randn(4, 3, 16, generator=g), torch.randn(4, 48, generator=g)
    o[..., 10:] = 0
    w = torch.rand(48 if joint else 16, generator=g)
    got = ref.norm_gate(o, gate, w, 1e-3, 10, joint, act, 48).view(4, 3, 16)[..., :10].double()
    x = o[..., :10].double()
    wd = (w.view(3, 16) if joint else w.expand(3, 16))[:, :10].double()
    if joint:
        want = plain.rms_norm(x.reshape(4, 30), wd.reshape(30), 1e-3).view(4, 3, 10)
    else:
        want = torch.stack([plain.rms_norm(x[:, n], wd[n], 1e-3) for n in range(3)], 1)
    z = gate.view(4, 3, 16)[..., :10].double()
    torch.testing.assert_close(got, want * (torch.sigmoid(z) if act == "sigmoid" else plain.silu(z)), rtol=1e-5, atol=1e-6)
    if joint:                                           # the same from a sum of squares over more heads
        total = o.double().pow(2).sum((1, 2)).float() * 2
        twice = ref.norm_gate(o, gate, w, 0.0, 10, True, act, 48, total, 6)
        torch.testing.assert_close(twice, ref.norm_gate(o, gate, w, 0.0, 10, True, act, 48), rtol=1e-5, atol=1e-6)


def test_expert_clamps_and_the_missing_lower_one():
    x = torch.tensor([[9.0, -9.0, 0.3, 9.0, -9.0, 0.3]])
    got = ref.clamped_glu(x, 0.7, 1.702)[0]
    for i, (g, u) in enumerate(((0.7, 0.7), (-9.0, -0.7), (0.3, 0.3))):
        assert math.isclose(float(got[i]), g / (1 + math.exp(-1.702 * g)) * (u + 1), rel_tol=1e-4, abs_tol=1e-9)


def test_groups_bar_better_experts():
    """The second best expert of all sits in a group that is not kept."""
    scores = torch.tensor([[5.0, 0.0, 4.0, 3.0, 1.0, 2.0]]).log_softmax(-1)
    w, ids = ref.moe_route_grouped(scores, 2, False, "softmax", None, 2.0, 3, 1)
    assert ids[0].tolist() == [0, 1]
    w, ids = ref.moe_route_grouped(scores, 2, False, "softmax", None, 2.0, 3, 2)
    assert ids[0].tolist() == [0, 2]
    torch.testing.assert_close(w[0], 2.0 * torch.softmax(scores, -1)[0, [0, 2]])     # not renormalised
    h, router = torch.randn(30, 12, generator=_g(7)), torch.randn(8, 12, generator=_g(8))
    w, ids = ref.moe_route_grouped(h @ router.T, 3, False, "softmax", None, 1.3, 4, 2)
    for t, picks in enumerate(plain.route(h.double(), router.double(), {"experts": 8, "top": 3, "scale": 1.3, "groups": {"count": 4, "keep": 2}})):
        got = dict(zip(ids[t].tolist(), w[t].tolist()))
        assert set(got) == {e for e, _ in picks}
        assert all(math.isclose(got[e], float(x), rel_tol=1e-4) for e, x in picks)


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
    """The pool is as large as one request: the next can only run on the pages and the slot the last gave back."""
    cfg, w, path, seqs, want = model
    rep = _rep(path, max_tokens=80)
    for k in range(3):
        for name in seqs:
            U.play(rep, seqs, [[(f"{name}#{k}", n)] for n in U.cuts(len(seqs[name]), [25, 1])], want, LIMIT)
    with pytest.raises(RuntimeError, match="pages"):
        rep.step([("x", seqs["a"], []), ("y", seqs["d"], [])])


def test_long_decoding(tmp_path):
    cfg = U.config([U.latent(2), U.lightning(decay=[0.9, 0.99, 0.9999]), U.gla(tau=30.0), U.latent(kv_from=0)])
    w = U.weights(cfg, 4)
    rep = _rep(U.save(tmp_path, cfg, w), 256)
    seqs = {"a": U.tokens(cfg, 230, 9)}
    U.play(rep, seqs, [[("a", 5)]] + [[("a", 1)]] * 225, U.reference(cfg, w, seqs), LIMIT)


def planted_token_model(kind):
    """Every token's embedding is the same but for token 7's."""
    mixers = {"latent": U.latent(1, 14, 2, 16, 16, scale=0.02), "kept": U.lightning(1, 16, 16, decay=[1.0]),
              "forgotten": U.lightning(1, 16, 16, decay=[0.05]), "channel": U.gla(1, 16, 16, tau=1.0, rank=1)}
    cfg = U.config([mixers[kind]], width=16)
    w = U.weights(cfg, 3, sharp=1.0)
    other = w["embed"][7].clone()
    w["embed"][:] = w["embed"][0]
    w["embed"][7] = other
    if kind == "latent":
        w["l0.mix.sink"] -= 30
    if kind == "channel":
        w["l0.mix.a2"] *= 0
        w["l0.mix.a2.b"] = torch.full((16,), 12.0).bfloat16()
    return cfg, w


@pytest.mark.parametrize("kind", ["latent", "kept", "channel", "forgotten"])
@pytest.mark.parametrize("sizes", [[200], [1], [31, 2], [150, 1]])
def test_a_planted_token_is_remembered_or_forgotten(tmp_path, kind, sizes):
    cfg, w = planted_token_model(kind)
    without = [3] * 200
    planted = list(without)
    planted[30] = 7
    rep = _rep(U.save(tmp_path, cfg, w))
    rows = []
    for k, seq in enumerate((without, planted)):
        lo, got = 0, []
        for n in U.cuts(200, sizes):
            got.append(rep.step([(str(k), seq[lo:lo + n], list(range(n)))], [str(k)] if lo + n == 200 else []))
            lo += n
        rows.append(torch.cat(got))
    moved = (rows[0] - rows[1]).abs().amax(-1)
    assert float(moved[:30].max()) == 0.0 and float(moved[30]) > 0.1
    assert (float(moved[-1]) > 1e-3) == (kind != "forgotten")
    want = plain.logits(cfg, w, planted)
    assert float(U.spread(rows[1], want).max()) < LIMIT


@pytest.mark.parametrize("cfg", [
    U.config([U.latent(1, 1, 2, 1, 1), U.lightning(1, 1, 1, decay=[0.5]), U.gla(1, 1, 1, tau=1.0, rank=1),
              U.latent(1, 1, 2, 3, 1, kv_from=0, mlp=U.moe(2, 1, 1, groups=None, shared=1))], width=5, vocab=7, scale=1.0),
    U.config([U.latent(7, 130, 20, 150, 300, mlp=U.dense(33)), U.lightning(1, 130, 70), U.gla(1, 70, 130, rank=40)], width=40,
             vocab=64),
    U.config([U.lightning(mlp=U.dense(7)), U.lightning()], vocab=100),
    U.config([U.gla(tau=1.0), U.gla(tau=100.0, mlp=U.moe(4, 4, 16, groups=(2, 2)))], vocab=100, eps=1e-2),
], ids=["ones", "wide", "no-attention", "gla-only"])
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
    again = seqs["d"][:50] + seqs["a"][:9]        # a cached prefix: its latents and the states at its boundary
    o = llm.generate([again], sp)[0]
    assert o.cached_tokens > 0
    assert o.token_ids == U.greedy(cfg, w, again, 5)
    llm.shutdown()


def test_snapshots_in_the_host_arena():
    """States of layers of different sizes as one frame: kept, overwritten, put back."""
    from minisglang_rdna4_b200.kvcache.gdn_state import GDNStateCache

    st = GDNStateCache(2, 3, 0, 1, 1, 1, 2 * 16 * 32 + 16 * 16, torch.float32, "cpu", geometries=[(2, 16, 32), (1, 16, 16)])
    assert st.ssm_state(0).shape == (3, 2, 16, 32) and st.ssm_state(1).shape == (3, 1, 16, 16)
    assert st.slot_nbytes() == 4 * (2 * 16 * 32 + 16 * 16)
    assert st.attach_host_arena(1 << 20) > 0
    g = _g(0)
    for i in range(2):
        st.ssm_state(i)[1] = torch.randn(st.ssm_state(i)[1].shape, generator=g)
    kept = [st.ssm_state(i)[1].clone() for i in range(2)]
    st.snapshot(1, "k")
    saved = st.save_slots(torch.tensor([1, 2]))
    for i in range(2):
        st.ssm_state(i)[:] = -1
    assert st.restore(2, "k")
    st.load_slots(torch.tensor([1, 2]), saved, torch.tensor([0]))
    for i in range(2):
        assert torch.equal(st.ssm_state(i)[2], kept[i]) and torch.equal(st.ssm_state(i)[1], kept[i])
        assert float(st.ssm_state(i)[0].max()) == -1
    st.drop_snapshot("k")


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
    w["l2.mix.norm"] = torch.ones(21)
    with pytest.raises(ValueError, match="l2.mix.norm"):
        _rep(U.save(tmp_path, U.PLAIN, w))


def test_config(tmp_path):
    mc = ModelConfig.from_hf(U.MIXED)
    assert mc.architectures == ("RafodraForCausalLM",) and mc.is_recurrent
    assert mc.num_kv_layers == 2 and mc.latent_widths == (64, 128) and mc.num_linear_layers == 4
    assert [mc.latent_row(i) for i in (1, 3, 4)] == [0, 1, 0] and [mc.state_row(i) for i in (0, 2, 5, 6)] == [0, 1, 2, 3]
    assert mc.state_geometries() == ((2, 32, 32), (3, 32, 16), (2, 48, 48), (3, 48, 48))
    assert isinstance(mc.layer_specs[0].mixer, LinearAttnLayer) and isinstance(mc.layer_specs[1].mixer, LatentLayer)
    # the rank of the decay gate comes from the checkpoint where the configuration has none
    bare = json.loads(json.dumps(U.MIXED))
    for layer in bare["layers"]:
        layer["mixer"].pop("gate_rank", None)
    with pytest.raises(ValueError, match="rank"):
        ModelConfig.from_hf(bare)
    got = ModelConfig.from_hf(U.save(tmp_path, bare, U.weights(U.MIXED, 0)))
    assert got.layer_specs == mc.layer_specs
    for bad in (U.config([dict(U.latent(), type="other")]), U.config([U.latent(kv_from=0)]),
                U.config([U.latent(), U.latent(kv_from=0, rank=64)]), U.config([U.latent(), U.latent(kv_from=0, base=7.0)]),
                U.config([U.lightning(), U.latent(kv_from=0)]), U.config([U.lightning(2, decay=[0.5])]),
                U.config([U.latent(mlp={"kind": "routed", "ff": 8})]), U.config([U.gla(mlp=U.moe(6, 5, groups=(3, 2)))])):
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

    cfg = U.config([U.latent(4, mlp=U.dense(90)), U.lightning(4, mlp=U.moe()), U.gla(2), U.latent(2, kv_from=0)], vocab=201)
    w = U.weights(cfg, 6)
    path = U.save(tmp_path, cfg, w)
    prompts = [U.tokens(cfg, 45, 1), U.tokens(cfg, 5, 2)]
    ctx = mp.get_context("spawn")
    q = ctx.Queue()
    port = 25000 + os.getpid() % 2000
    procs = [ctx.Process(target=_rank, args=(r, path, prompts, port, q)) for r in range(2)]
    for p in procs:
        p.start()
    got = q.get(timeout=120)
    for p in procs:
        p.join(60)
    assert got == [U.greedy(cfg, w, p, 6) for p in prompts]
