"""Plain, slow restatement of the Ligipel decoder over a whole sequence: one function per mechanism, no cache, no
batching, nothing shared with the serving code. The tests compare the framework with it."""
from __future__ import annotations

import math
from typing import Dict, List

import torch


def layer_norm(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log_distance_bias(r1: torch.Tensor, r2: torch.Tensor, distance: torch.Tensor) -> torch.Tensor:
    """What one head's score loses at a distance (in tokens)."""
    return r1 * torch.log(1.0 + r2 * distance)


def softmax_off_by_one(s: torch.Tensor) -> torch.Tensor:
    """Weights of one row of scores when the denominator has one more term, exp(0)."""
    m = torch.clamp(s.max(), min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum() + torch.exp(-m))


def head_weights(q: torch.Tensor, k: torch.Tensor, r1, r2, scale: float, window: int) -> torch.Tensor:
    """One head's weights ``[T, T]``, zero where nothing is seen. q, k [T, dim]."""
    t = q.shape[0]
    out = torch.zeros(t, t, dtype=q.dtype)
    for i in range(t):
        lo = max(0, i - window + 1)
        far = torch.arange(i - lo, -1, -1, dtype=q.dtype)
        out[i, lo:i + 1] = softmax_off_by_one(k[lo:i + 1] @ q[i] * scale - log_distance_bias(r1, r2, far))
    return out


def mix_heads(weights: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """weights [H, T, T]: head h gets the sum over g of talk[h, g] times head g's weights."""
    out = torch.zeros_like(weights)
    for h in range(talk.shape[0]):
        for g in range(talk.shape[1]):
            out[h] += talk[h, g] * weights[g]
    return out


def talking_attention(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict) -> torch.Tensor:
    t, heads, kv, dim, vdim = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = (h @ p["q"].T).view(t, heads, dim)
    k = (h @ p["k"].T).view(t, kv, dim)
    v = (h @ p["v"].T).view(t, kv, vdim)
    of = [n // (heads // kv) for n in range(heads)]
    w = torch.stack([head_weights(q[:, n], k[:, of[n]], p["r1"][n], p["r2"][n], mix["scale"], mix["mask"]["size"])
                     for n in range(heads)])
    w = mix_heads(w, p["talk"])
    return torch.cat([w[n] @ v[:, of[n]] for n in range(heads)], -1) @ p["o"].T


def causal_filter(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """One filter per channel over the current token (last tap) and the ones before; zeros ahead of the start."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            if t - j >= 0:
                out[t] += taps[:, n - 1 - j] * x[t - j]
    return out + bias


def selective_scan(x: torch.Tensor, dt: torch.Tensor, a: torch.Tensor, b: torch.Tensor, c: torch.Tensor,
                   d: torch.Tensor) -> torch.Tensor:
    """x, dt [T, channels]; a [channels, state]; b, c [T, state]: every channel has a state vector that starts at zero."""
    s = torch.zeros_like(a)
    out = []
    for t in range(x.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * x[t])[:, None] * b[t][None, :]
        out.append(s @ c[t] + d * x[t])
    return torch.stack(out)


def mamba(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict) -> torch.Tensor:
    inner, rank, state = mix["inner"], mix["dt_rank"], mix["state"]
    y = h @ p["in"].T
    x, z = y[:, :inner], y[:, inner:]
    x = silu(causal_filter(x, p["conv"], p["conv.b"]))
    y = x @ p["x"].T
    dt = y[:, :rank] @ p["dt"].T + p["dt.b"]
    dt = torch.clamp(dt, min=0.0) + torch.log1p(torch.exp(-dt.abs()))
    o = selective_scan(x, dt, -torch.exp(p["A_log"]), y[:, rank:rank + state], y[:, rank + state:], p["D"])
    return (o * silu(z)) @ p["o"].T


def parallel(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    side = {s: {k[len(s) + 1:]: v for k, v in p.items() if k.startswith(s + ".")} for s in ("left", "right")}
    left = unit_rms(talking_attention(h, side["left"], mix["left"]), eps) * side["left"]["out"]
    right = unit_rms(mamba(h, side["right"], mix["right"]), eps) * side["right"]["out"]
    return 0.5 * (left + right)


def rotate_halves(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., n] at positions 0..T-1: channel i of the first ``dims`` turns with channel i + dims / 2."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        for t in range(x.shape[0]):
            a = t * base ** (-2.0 * i / dims)
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def fading_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: float) -> torch.Tensor:
    """One head: S <- decay S + k_t v_t^T, o_t = S^T q_t, from S = 0."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        s = decay * s + k[t][:, None] * v[t][None, :]
        out.append(s.T @ q[t])
    return torch.stack(out)


def retention(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    t, heads, dim, vdim, rot = h.shape[0], mix["heads"], mix["dim"], mix["vdim"], mix["rot"]
    q = rotate_halves((h @ p["q"].T).view(t, heads, dim), rot["dims"], rot["base"])
    k = rotate_halves((h @ p["k"].T).view(t, heads, dim), rot["dims"], rot["base"]) * dim ** -0.5
    v = (h @ p["v"].T).view(t, heads, vdim)
    o = [unit_rms(fading_memory(q[:, n], k[:, n], v[:, n], mix["decay"][n]), eps) for n in range(heads)]
    return (torch.cat(o, -1) * silu(h @ p["g"].T)) @ p["o"].T


def gated_feed_forward(h: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h: torch.Tensor, w_router: torch.Tensor, correction: torch.Tensor, top: int):
    """Chosen experts and their weights per token: chosen by softmax score plus correction, weighted by score alone."""
    s = torch.softmax(h @ w_router.T, -1)
    chosen = []
    for row in s:
        best = sorted(range(row.numel()), key=lambda e: -float(row[e] + correction[e]))[:top]
        total = sum(row[e] for e in best) + 1e-20
        chosen.append([(e, row[e] / total) for e in best])
    return chosen


def expert_mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str, mlp: dict) -> torch.Tensor:
    def part(n):
        return {k: w[f"{name}.{n}.{k}"] for k in ("gate", "up", "down")}

    out = torch.zeros_like(h)
    for t, picks in enumerate(route(h, w[name + ".router"], w[name + ".correction"], mlp["router"]["top"])):
        for e, weight in picks:
            out[t] += weight * gated_feed_forward(h[t:t + 1], part(f"e{e}"))[0]
    return out + gated_feed_forward(h, part("shared")) if mlp.get("shared") else out


def depth_average(results: List[torch.Tensor], coefficients: torch.Tensor) -> torch.Tensor:
    return sum(c * x for c, x in zip(coefficients, results))


def residual_streams(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int],
                     dtype=torch.float64) -> List[torch.Tensor]:
    """What goes into the first layer and what comes out of every layer's depth average."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])

    def norm(x, n):
        return layer_norm(x, w[n], w[n + ".b"], eps)

    x = norm(w["embed"][torch.tensor(tokens)], "embed.norm")
    results, out = [x], [x]
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        p = {k[len(n) + 4:]: v for k, v in w.items() if k.startswith(n + "mix.")}
        mixer = {"parallel": parallel, "retention": retention}[layer["type"]]
        x = x + norm(mixer(norm(x, n + "norm1"), p, layer["mixer"], eps), n + "norm1b")
        if layer.get("mlp") is not None:
            x = x + norm(expert_mixture(norm(x, n + "norm2"), w, n + "mlp", layer["mlp"]), n + "norm2b")
        results.append(x)
        x = depth_average(results, w[n + "dwa"])
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64) -> torch.Tensor:
    x = residual_streams(cfg, w, tokens, dtype)[-1]
    x = layer_norm(x, w["final.norm"].to(dtype), w["final.norm.b"].to(dtype), float(cfg["norm"]["eps"]))
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(x @ w["head"].to(dtype).T * cfg["logit_scale"] / cap)
