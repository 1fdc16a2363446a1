"""Small random Zobelorn checkpoints and the models the tests share."""
import torch

import plain_zobelorn as plain
from mitilix_util import SEQS, cuts, mixed_schedule, play, save, spread, tokens  # noqa: F401


def window(heads=3, kv=1, dim=20, vdim=28, size=17, rot=None, base=500.0, factor=2.5, cap=6.0, scale=0.3, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale, "softcap": cap,
        "rot": {"base": base, "dims": dim if rot is None else rot, "scaling": {"factor": factor}}}}


def chunk(heads=4, kv=2, dim=24, vdim=12, size=23, rot=None, base=300.0, scaling=(3.0, 1.0, 6.0, 40), scale=0.6, kv_from=None,
          mlp=None):
    names = ("factor", "low", "high", "original")
    mixer = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "scale": scale,
             "rot": {"base": base, "dims": dim if rot is None else rot, "scaling": dict(zip(names, scaling))}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention_2", "mixer": mixer, "mlp": mlp}


def dense(ff=60):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared=30):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=72, vocab=203, scale=5.0, eps=1e-5, mult=0.6):
    return {"architecture": "Zobelorn", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
            "residual_mult": mult, "vocab": vocab, "width": width}


# every size differs between the layers; shared keys and values read with another mask, other queries and scale; layers
# without feed-forward; experts with and without a shared one; partial rotation; groups of 1, 2, 3 and 5 heads; an odd
# vocabulary; sizes that are no multiples of 8
MIXED = config([
    chunk(4, 2, 24, 12, 23, mlp=moe()),
    window(3, 1, 20, 28, 17, rot=12, mlp=dense(50)),
    chunk(4, 2, 24, 12, 9, scale=1.1, kv_from=0, mlp=None),
    window(2, 2, 34, 70, 30, cap=3.0, mlp=moe(5, 3, 19, shared=0)),
    chunk(5, 1, 70, 18, 32, rot=6, mlp=moe(8, 1, 8)),
    chunk(5, 1, 70, 18, 50, rot=6, kv_from=4, mlp=dense(41)),
])
PLAIN = config([window(4, 2, 16, 16, mlp=dense()), chunk(4, 4, 16, 16, mlp=moe()), chunk(4, 4, 16, 16, kv_from=1, mlp=moe())],
               width=64, mult=1.0)


def weights(cfg, seed=0, sharp=2.0):
    """``sharp`` scales the query norms of windowed layers: single keys stand out among their neighbours."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)

    def around(n, centre=0.0):
        return centre + 0.3 * r(n, std=1.0)

    out = {"embed": r(cfg["vocab"], w, std=0.3), "head": r(cfg["vocab"], w), "final.norm": around(w)}
    for i, spec in enumerate(cfg["layers"]):
        m, n, mlp = spec["mixer"], f"l{i}.mix.", spec["mlp"]
        h, k = m["heads"], m["kv_heads"]
        out[f"l{i}.norm1"], out[f"l{i}.norm1b"] = around(w), around(w)
        out[n + "q"], out[n + "o"] = r(h * m["dim"], w), r(w, h * m["vdim"])
        if "kv_from" not in m:
            out[n + "k"], out[n + "v"] = r(k * m["dim"], w), r(k * m["vdim"], w)
        if spec["type"] == "attention":
            out[n + "q.norm"], out[n + "k.norm"] = around(h * m["dim"], 1.0) * sharp, around(k * m["dim"], 1.0)
            out[n + "g"] = r(h * m["vdim"], w) * 2
        if mlp is None:
            continue
        n = f"l{i}.mlp."
        out[f"l{i}.norm2"], out[f"l{i}.norm2b"] = around(w), around(w)

        def ff(name, width):
            out[name + "gate"], out[name + "up"], out[name + "down"] = r(width, w), r(width, w), r(w, width)

        if mlp["kind"] == "dense":
            ff(n, mlp["ff"])
            continue
        out[n + "router"] = r(mlp["router"]["experts"], w) * 3
        for e in range(mlp["router"]["experts"]):
            ff(f"{n}e{e}.", mlp["expert"]["ff"])
        if "shared" in mlp:
            ff(n + "shared.", mlp["shared"]["ff"])
    return {k: t.to(torch.bfloat16) for k, t in out.items()}


def clear_choices(cfg, path, seqs, margin=0.1):
    """The sequences with every token replaced whose choice of experts is a close call in some layer: in 16 bits it could fall
    the other way, and with it the rows that look back at the token."""
    from minisglang_rdna4_b200 import ops
    from minisglang_rdna4_b200.replay import make_replayer

    if not any(layer["mlp"] and layer["mlp"]["kind"] == "moe" for layer in cfg["layers"]):
        return seqs
    rep, route, gaps = make_replayer(path, "float32", 512, "cpu"), ops.moe_route, []

    def watch(logits, top, *args):
        if top < logits.shape[1]:
            s = logits.sort(-1, descending=True)[0]
            gaps.append(s[:, top - 1] - s[:, top])
        return route(logits, top, *args)

    ops.moe_route, out = watch, {}
    try:
        for k, (name, seq) in enumerate(seqs.items()):
            g, seq = torch.Generator().manual_seed(77 + k), list(seq)
            for _ in range(300):
                gaps.clear()
                rep.step([(name, seq, [])], [name])
                close = (torch.stack(gaps).amin(0) < margin).nonzero().flatten().tolist() if gaps else []
                if not close:
                    break
                for i in close:
                    seq[i] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
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


def planted_token_model(kind, size):
    """One layer, the same embedding for every token but token 7: what a row sees of it shows in its logits."""
    layer = window(2, 1, 16, 16, size, scale=0.05) if kind == "window" else chunk(2, 1, 16, 16, size, scale=0.05)
    cfg = config([layer], width=16)
    w = weights(cfg, 3, sharp=1.0)
    other = w["embed"][7].clone()
    w["embed"][:] = w["embed"][0]
    w["embed"][7] = other
    return cfg, w


def seen_rows(kind, at, size, n):
    """Rows of n that see position ``at``."""
    end = at + size if kind == "window" else at // size * size + size
    return list(range(at, min(end, n)))


def loud_key(n, at, rows, width, ps, channel=0, g=1):
    """Keys and values of one head in scattered pages: the key of token ``at`` dominates, and channel 0 of its value tells;
    queries for the last ``rows`` tokens."""
    pages = -(-n // ps)
    bt = torch.randperm(pages, generator=torch.Generator().manual_seed(n)).to(torch.int32)[None]
    k, v = torch.zeros(pages, 1, ps, width), torch.zeros(pages, 1, ps, width)
    page, off = bt[0, at // ps].long(), at % ps
    k[page, 0, off, channel] = 8.0
    v[page, 0, off, 0] = 5.0
    q = torch.zeros(rows, g, width)
    q[..., channel] = 8.0
    return q, k, v, bt


def split_planes(k, v):
    """A pool of one layer as the kernels take it: K and V planes of one buffer."""
    buf = torch.empty((2, 1, *k.shape), dtype=k.dtype, device=k.device)
    buf[0, 0], buf[1, 0] = k, v
    return buf[0, 0], buf[1, 0]
