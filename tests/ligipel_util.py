"""Small random Ligipel checkpoints and the models the tests share."""
import torch

import plain_ligipel as plain
from mitilix_util import SEQS, cuts, mixed_schedule, play, save, spread, tokens  # noqa: F401
from zobelorn_util import loud_key, split_planes  # noqa: F401


def pair(heads=4, kv=2, dim=20, vdim=28, size=17, scale=0.3, inner=40, state=5, rank=3, taps=3, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale},
        "right": {"inner": inner, "state": state, "dt_rank": rank, "conv": taps}}}


def retention(heads=3, dim=20, vdim=12, rot=None, base=300.0, decay=None, mlp=None):
    decay = decay or [round(1 - 2.0 ** -(1 + 2.5 * i), 5) for i in range(heads)]
    return {"type": "retention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dim if rot is None else rot}}}


def moe(experts=6, top=2, ff=24, shared=30):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=72, vocab=203, eps=1e-5, scale=0.4, cap=7.0):
    return {"architecture": "Ligipel", "layers": layers, "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": cap,
            "vocab": vocab, "width": width}


# every size differs between the layers; groups of 1, 2 and 3 heads; partial and odd rotations; one to five taps; layers
# without feed-forward; experts with and without a shared one; an odd vocabulary; sizes that are no multiples of 8
MIXED = config([
    pair(4, 2, 20, 28, 17, mlp=moe()),
    retention(3, 20, 12, rot=10, mlp=None),
    pair(3, 1, 34, 18, 30, inner=56, state=16, rank=8, taps=4, scale=0.2, mlp=moe(5, 3, 19, shared=0)),
    pair(2, 2, 9, 36, 1, inner=24, state=3, rank=1, taps=1, mlp=None),
    retention(2, 33, 48, rot=14, decay=[0.7, 0.9995], base=20.0, mlp=moe(8, 1, 8)),
    pair(6, 2, 70, 130, 64, inner=30, state=33, rank=17, taps=5, mlp=moe(4, 4, 16)),
])
PLAIN = config([pair(4, 4, 16, 16, mlp=moe()), retention(mlp=moe()), retention(mlp=None)], width=64, scale=1.0)


def weights(cfg, seed=0, sharp=2.0):
    """``sharp`` scales the attention queries: single keys stand out among their neighbours."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)

    out = {"embed": r(cfg["vocab"], w, std=1.0), "head": r(cfg["vocab"], w) * 3}

    def norm(name):
        out[name], out[name + ".b"] = 1 + 0.3 * r(w, std=1.0), r(w, std=0.2)

    norm("embed.norm")
    norm("final.norm")
    for i, spec in enumerate(cfg["layers"]):
        m, n, mlp = spec["mixer"], f"l{i}.", spec["mlp"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            norm(n + name)
        out[n + "dwa"] = r(i + 2, std=0.3)
        out[n + "dwa"][-1] += 1
        if spec["type"] == "parallel":
            a, s, p = m["left"], m["right"], n + "mix.left."
            h, c, ns = a["heads"], s["inner"], s["state"]
            out[p + "q"], out[p + "k"] = r(h * a["dim"], w) * sharp, r(a["kv_heads"] * a["dim"], w)
            out[p + "v"], out[p + "o"] = r(a["kv_heads"] * a["vdim"], w), r(w, h * a["vdim"])
            out[p + "r1"], out[p + "r2"] = r(h, std=0.5).abs() + 0.2, r(h, std=0.5).abs() + 0.1
            out[p + "talk"], out[p + "out"] = r(h, h, std=0.4) + torch.eye(h), 1 + r(w, std=0.3)
            p = n + "mix.right."
            out[p + "in"], out[p + "o"] = r(2 * c, w), r(w, c)
            out[p + "conv"], out[p + "conv.b"] = r(c, s["conv"], std=0.6), r(c, std=0.3)
            out[p + "x"], out[p + "dt"] = r(s["dt_rank"] + 2 * ns, c) * 2, r(c, s["dt_rank"])
            out[p + "dt.b"], out[p + "D"] = r(c, std=1.0) - 3, r(c, std=1.0)
            out[p + "A_log"], out[p + "out"] = r(c, ns, std=1.0), 1 + r(w, std=0.3)
        else:
            h, p = m["heads"], n + "mix."
            out[p + "q"], out[p + "k"] = r(h * m["dim"], w), r(h * m["dim"], w)
            out[p + "v"], out[p + "g"] = r(h * m["vdim"], w), r(h * m["vdim"], w)
            out[p + "o"] = r(w, h * m["vdim"])
        if mlp is None:
            continue
        n += "mlp."

        def ff(name, width):
            out[name + "gate"], out[name + "up"], out[name + "down"] = r(width, w), r(width, w), r(w, width)

        out[n + "router"], out[n + "correction"] = r(mlp["router"]["experts"], w) * 2, r(mlp["router"]["experts"], std=0.1)
        for e in range(mlp["router"]["experts"]):
            ff(f"{n}e{e}.", mlp["expert"]["ff"])
        if "shared" in mlp:
            ff(n + "shared.", mlp["shared"]["ff"])
    return {k: t.to(torch.bfloat16) for k, t in out.items()}


def clear_choices(cfg, path, seqs, margin=0.05):
    """The sequences with every token replaced whose choice of experts is a close call in some layer: in 16 bits it could fall
    the other way, and with it the rows after the token."""
    from minisglang_rdna4_b200 import ops
    from minisglang_rdna4_b200.replay import make_replayer

    if not any(layer["mlp"] for layer in cfg["layers"]):
        return seqs
    rep, route, gaps = make_replayer(path, "float32", 512, "cpu"), ops.moe_route, []

    def watch(logits, top, renorm, scoring, bias, *args):
        if top < logits.shape[1]:
            s = (torch.softmax(logits, -1) + bias).sort(-1, descending=True)[0]
            gaps.append(s[:, top - 1] - s[:, top])
        return route(logits, top, renorm, scoring, bias, *args)

    ops.moe_route, out = watch, {}
    try:
        for k, (name, seq) in enumerate(seqs.items()):
            g, seq = torch.Generator().manual_seed(77 + k), list(seq)
            for _ in range(400):
                gaps.clear()
                rep.step([(name, seq, [])], [name])
                close = (torch.stack(gaps).amin(0) < margin).nonzero().flatten().tolist() if gaps else []
                if not close:
                    break
                # a token changes what the layers choose behind it: the first of them, then again
                seq[close[0]] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
            assert not close
            out[name] = seq
    finally:
        ops.moe_route = route
        rep.engine.shutdown()
    return out


def reference(cfg, w, seqs):
    return {n: plain.logits(cfg, w, s) for n, s in seqs.items()}


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(plain.logits(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


def planted_token_model(size):
    """One layer whose scan is silent, the same embedding for every token but token 7: what a row's attention sees of it shows
    in its logits."""
    cfg = config([pair(2, 1, 16, 16, size, scale=0.05, inner=16, state=4, rank=2, taps=1)], width=16)
    w = weights(cfg, 3, sharp=1.0)
    other = w["embed"][7].clone()
    w["embed"][:] = w["embed"][0]
    w["embed"][7] = other
    for name in ("out", "o"):
        w["l0.mix.right." + name] = torch.zeros_like(w["l0.mix.right." + name])
    return cfg, w


def scan_case(c, n, lens, seed, dtype=torch.float32, extra=2):
    """Packed rows of a selective scan and the states of its slots (with a slot stride of their own)."""
    g = torch.Generator().manual_seed(seed)
    t = sum(lens)
    rows = torch.randn(t, c + 16 + 2 * n, generator=g).to(dtype)
    case = dict(
        x=torch.randn(t, c, generator=g).to(dtype), dt=torch.randn(t, c, generator=g), dt_bias=torch.randn(c, generator=g) - 2,
        a=-torch.exp(torch.randn(c, n, generator=g)), b=rows[:, c + 16:c + 16 + n], c=rows[:, c + 16 + n:],
        skip=torch.randn(c, generator=g), z=rows[:, :c])
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    slots = torch.randperm(len(lens) + extra, generator=g)[:len(lens)].int()
    has = (torch.arange(len(lens)) % 3 != 1).int()
    state = torch.randn(len(lens) + extra, 16 + c * n, generator=g)
    return case, cu, slots, has, state
