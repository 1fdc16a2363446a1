"""Small random Mitilix checkpoints and a driver that compares the framework's logits with the plain restatement."""
import json
import os

import torch

import plain_mitilix as plain


def layer(heads=3, dim=24, vdim=40, rank=48, window=20, ff=96, scale=None, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
             "scale": scale if scale is not None else 2.0 * dim ** -0.5}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=203, taps=3, max_positions=300, eps=1e-5):
    return {"architecture": "Mitilix", "canon": {"taps": taps}, "layers": layers, "max_positions": max_positions,
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every size differs between the layers; a shared latent read with other heads, dims and window; a layer without
# feed-forward; an odd vocabulary; a width and feed-forwards that are no multiples of 16
MIXED = config([
    layer(3, 24, 40, 48, 20, 90),
    layer(2, 20, 12, 72, 33, 0),
    layer(5, 16, 56, 48, 1, 100, scale=0.7, kv_from=0),
    layer(1, 48, 8, 72, 64, 50, kv_from=1),
])
PLAIN = config([layer(), layer(kv_from=0)], taps=4)


def weights(cfg, seed=0, sharp=3.0):
    """``sharp`` scales the query projections: single keys stand out among their neighbours."""
    g = torch.Generator().manual_seed(seed)
    w, taps = cfg["width"], cfg["canon"]["taps"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)

    out = {"embed": r(cfg["vocab"], w, std=1.0), "pos": r(cfg["max_positions"], w, std=0.5),
           "head": r(cfg["vocab"], w), "final.norm": torch.tensor(1.3)}
    for i, spec in enumerate(cfg["layers"]):
        m, n = spec["mixer"], f"l{i}."
        out[n + "norm1"] = torch.tensor(0.7 + 0.2 * i)
        out[n + "canon1"] = r(w, taps, std=0.4)
        out[n + "mix.q"] = r(m["heads"] * m["dim"], w) * sharp
        out[n + "mix.uk"] = r(m["heads"] * m["dim"], m["kv_rank"])
        out[n + "mix.uv"] = r(m["heads"] * m["vdim"], m["kv_rank"])
        out[n + "mix.o"] = r(w, m["heads"] * m["vdim"])
        if "kv_from" not in m:
            out[n + "mix.dkv"] = r(m["kv_rank"], w)
            out[n + "mix.dkv.norm"] = 1 + 0.3 * r(m["kv_rank"], std=1.0)
        if spec["mlp"] is not None:
            out[n + "canon2"] = r(w, taps, std=0.4)
            out[n + "mlp.up"] = r(spec["mlp"]["ff"], w)
            out[n + "mlp.down"] = r(w, spec["mlp"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def save(path, cfg, w):
    from safetensors.torch import save_file

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({k: v.clone().contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def spread(got, want):
    """RMS difference of the logits of every row (their mean taken off), relative to the spread of the wanted ones."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def reference(cfg, w, seqs):
    return {n: plain.logits(cfg, w, s) for n, s in seqs.items()}


def play(rep, seqs, schedule, want, limit, cap=None):
    """``schedule``: steps of (request, count); a request ends with its last token, ``name#k`` replays ``name`` under
    another id. Every row's logits are compared. With a ``cap`` (routed experts in 16 bits, where a close choice may fall
    the other way) one row in twenty may be over the limit, none over the cap."""
    at, errs = {}, []
    for step in schedule:
        entries, end, rows = [], [], []
        for name, n in step:
            seq, lo = seqs[name.split("#")[0]], at.get(name, 0)
            entries.append((name, seq[lo:lo + n], list(range(n))))
            rows.append(want[name.split("#")[0]][lo:lo + n])
            at[name] = lo + n
            if at[name] == len(seq):
                end.append(name)
        got = rep.step(entries, end)
        err = spread(got, torch.cat(rows))
        assert float(err.max()) <= (cap or limit), (step, float(err.max()), int(err.argmax()))
        errs.append(err)
    over = torch.cat(errs) > limit
    assert float(over.float().mean()) <= 0.05 or int(over.sum()) <= 1, (int(over.sum()), over.numel())
    held = sum(-(-r.device_len // rep.page_size) for r in rep._live.values())
    assert rep.cache.free_pages == rep.cache.num_pages - held


def cuts(n, sizes):
    """Split n tokens into portions of the given sizes in turn."""
    out, i = [], 0
    while n > 0:
        out.append(min(sizes[i % len(sizes)], n))
        n -= out[-1]
        i += 1
    return out


def mixed_schedule():
    """Up to four live requests: portions beside single tokens, requests left out for a while, slots and pages of
    finished requests taken again."""
    return [
        [("a", 40)], [("a", 1), ("b", 17)], [("b", 2), ("a", 3), ("c", 9)], [("a", 1), ("b", 1), ("c", 1)],
        [("d", 30), ("a", 1)], [("d", 1), ("c", 1), ("b", 1), ("a", 1)], [("b", 19), ("c", 20)], [("a", 13), ("d", 2)],
        [("a#2", 35), ("d", 7)], [("a#2", 1), ("d", 1)], [("b#2", 5), ("a#2", 2), ("d", 1)],
        [("b#2", 2), ("a#2", 1), ("c#2", 31)], [("b#2", 33), ("a#2", 21)], [("d", 28)],
    ]


SEQS = {"a": 60, "b": 40, "c": 31, "d": 70}
