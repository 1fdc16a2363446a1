"""Small random Rafodra checkpoints and the models the tests share."""
import math

import torch

import plain_rafodra as plain
from mitilix_util import SEQS, cuts, mixed_schedule, play, save, spread, tokens  # noqa: F401


def latent(heads=3, dim=20, rot=12, vdim=28, rank=40, scale=None, base=500.0, kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
             "rot": {"dims": rot, "base": base}, "scale": scale if scale is not None else (dim + rot) ** -0.5}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def lightning(heads=3, dim=20, vdim=12, decay=None, mlp=None):
    decay = decay or [round(1 - 2.0 ** -(1 + 2.5 * i), 5) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def gla(heads=2, dim=24, vdim=20, tau=8.0, rank=5, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "gate_rank": rank}, "mlp": mlp}


def dense(ff=60):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, limit=0.9, groups=(3, 2), scale=1.7, shared=30, shared_limit=1.3):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared, "limit": shared_limit}
    return out


def config(layers, width=72, vocab=203, scale=5.0, eps=1e-5):
    return {"architecture": "Rafodra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


# every size differs between the layers; a shared latent read with other heads and dims; layers without feed-forward;
# experts with and without groups and a shared one; an odd vocabulary; sizes that are no multiples of 8
MIXED = config([
    gla(2, 24, 20, tau=8.0, rank=5, mlp=moe()),
    latent(3, 20, 12, 28, 40, mlp=dense(50)),
    lightning(3, 20, 12, mlp=None),
    latent(2, 9, 6, 36, 72, base=10000.0, scale=0.5, mlp=moe(5, 3, 19, groups=None, shared=0)),
    latent(5, 14, 12, 10, 40, scale=0.4, kv_from=1, mlp=None),
    lightning(2, 33, 48, decay=[0.7, 0.9995], mlp=moe(8, 1, 8, groups=(2, 1), scale=1.0)),
    gla(3, 40, 33, tau=2.0, rank=19, mlp=dense(41)),
])
PLAIN = config([latent(mlp=dense()), lightning(mlp=moe()), gla(mlp=dense())], width=64)


def weights(cfg, seed=0, sharp=2.0):
    """``sharp`` scales the attention queries: single keys stand out among their neighbours."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)

    def near_one(n):
        return 1 + 0.3 * r(n, std=1.0)

    out = {"embed": r(cfg["vocab"], w, std=0.3), "head": r(cfg["vocab"], w), "final.norm": near_one(w)}
    for i, spec in enumerate(cfg["layers"]):
        m, n, kind, mlp = spec["mixer"], f"l{i}.mix.", spec["type"], spec["mlp"]
        h, v = m["heads"], m["heads"] * m["vdim"]
        out[f"l{i}.norm1"] = near_one(w)
        out[n + "o"] = r(w, v)
        if kind == "latent_attention":
            out[n + "q"] = r(h * (m["dim"] + m["rot_dim"]), w) * sharp
            out[n + "uk"], out[n + "uv"] = r(h * m["dim"], m["kv_rank"]), r(v, m["kv_rank"])
            out[n + "sink"], out[n + "g"] = r(h, std=2.0), r(h, w)
            if "kv_from" not in m:
                out[n + "dkv"], out[n + "dkv.norm"] = r(m["kv_rank"] + m["rot_dim"], w), near_one(m["kv_rank"])
        else:
            out[n + "q"], out[n + "k"] = r(h * m["dim"], w), r(h * m["dim"], w)
            out[n + "v"], out[n + "g"] = r(v, w), r(v, w)
            out[n + "norm"] = near_one(v if kind == "lightning" else m["vdim"])
            if kind == "gla":
                out[n + "a1"], out[n + "a2"] = r(m["gate_rank"], w), r(h * m["dim"], m["gate_rank"]) * 2
                out[n + "a2.b"] = r(h * m["dim"], std=2.0) + 2
        if mlp is None:
            continue
        n = f"l{i}.mlp."
        out[f"l{i}.norm2"] = near_one(w)

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
            out[n + "shared.sg"] = r(1, w)
    return {k: t.to(torch.bfloat16) for k, t in out.items()}


def reference(cfg, w, seqs):
    return {n: plain.logits(cfg, w, s) for n, s in seqs.items()}


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(plain.logits(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


def loud_key(n, at, seen_by, r, ps):
    """Pool rows, block table and a query: the key of token ``at`` dominates, channel 0 of the result tells."""
    pages = -(-n // ps)
    bt = torch.randperm(pages, generator=torch.Generator().manual_seed(n)).to(torch.int32)[None]
    pool = torch.zeros(pages, ps, r)
    for p in range(n):
        pool[bt[0, p // ps].long(), p % ps, 0 if p == at else 1] = 10.0 if p == at else 1.0
    q = torch.zeros(seen_by, 1, r)
    q[:, :, 0] = 10.0
    return pool, bt, q


def sink_share(scores, sink):
    """Softmax mass that is left for the keys."""
    e = sum(math.exp(s) for s in scores)
    return e / (e + math.exp(sink))
