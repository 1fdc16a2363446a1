"""Plain, slow restatement of the Rafodra decoder over a whole sequence: one function per mechanism, no cache, no
batching, nothing shared with the serving code. The tests compare the framework with it."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def layer_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """Centred, divided by the root of (mean squared deviation + eps), weighted; no bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate_pairs(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., n] at positions 0..T-1: neighbouring pairs of the first ``dims`` channels turn by position times
    base^(-2 i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        for p in range(x.shape[0]):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[p, ..., 2 * i], x[p, ..., 2 * i + 1]
            out[p, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[p, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def latents(h: torch.Tensor, w_dkv: torch.Tensor, norm: torch.Tensor, mix: dict, eps: float):
    """What a layer caches per token: the normed latent and the rotated key part all heads share."""
    y = h @ w_dkv.T
    r = mix["kv_rank"]
    return rms_norm(y[:, :r], norm, eps), rotate_pairs(y[:, r:], mix["rot"]["dims"], mix["rot"]["base"])


def softmax_with_sink(s: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights of one row of scores when the denominator also counts exp(sink), which belongs to no key."""
    m = torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + torch.exp(sink - m))


def latent_attention(h: torch.Tensor, c: torch.Tensor, k_rot: torch.Tensor, p: Dict[str, torch.Tensor],
                     mix: dict) -> torch.Tensor:
    t, heads, dim, rot, vdim = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    q = (h @ p["q"].T).view(t, heads, dim + rot)
    q_rot = rotate_pairs(q[..., dim:], mix["rot"]["dims"], mix["rot"]["base"])
    k = (c @ p["uk"].T).view(t, heads, dim)
    v = (c @ p["uv"].T).view(t, heads, vdim)
    gate = torch.sigmoid(h @ p["g"].T)
    out = torch.zeros(t, heads, vdim, dtype=h.dtype)
    for n in range(heads):
        for i in range(t):
            s = (k[:i + 1, n] @ q[i, n, :dim] + k_rot[:i + 1] @ q_rot[i, n]) * mix["scale"]
            out[i, n] = softmax_with_sink(s, p["sink"][n]) @ v[:i + 1, n] * gate[i, n]
    return out.reshape(t, heads * vdim) @ p["o"].T


def decaying_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, alpha: torch.Tensor) -> torch.Tensor:
    """One head: S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, from S = 0. q, k, alpha [T, dim], v [T, vdim]."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        s = alpha[t][:, None] * s + k[t][:, None] * v[t][None, :]
        out.append(s.T @ q[t])
    return torch.stack(out)


def lightning(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    t, heads, dim, vdim = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = silu(h @ p["q"].T).view(t, heads, dim)
    k = silu(h @ p["k"].T).view(t, heads, dim)
    v = silu(h @ p["v"].T).view(t, heads, vdim)
    o = [decaying_memory(q[:, n], k[:, n], v[:, n], torch.full_like(k[:, n], mix["decay"][n])) for n in range(heads)]
    o = rms_norm(torch.cat(o, -1), p["norm"], eps)          # all heads together
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def channel_decay(h: torch.Tensor, a1: torch.Tensor, a2: torch.Tensor, bias: torch.Tensor, tau: float) -> torch.Tensor:
    return torch.sigmoid((h @ a1.T) @ a2.T + bias) ** (1.0 / tau)


def gla(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    t, heads, dim, vdim = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q = (h @ p["q"].T).view(t, heads, dim) * dim ** -0.5
    k = (h @ p["k"].T).view(t, heads, dim)
    v = (h @ p["v"].T).view(t, heads, vdim)
    alpha = channel_decay(h, p["a1"], p["a2"], p["a2.b"], mix["tau"]).view(t, heads, dim)
    o = [rms_norm(decaying_memory(q[:, n], k[:, n], v[:, n], alpha[:, n]), p["norm"], eps) for n in range(heads)]
    return (torch.cat(o, -1) * silu(h @ p["g"].T)) @ p["o"].T


def gated_feed_forward(h: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def clamped_expert(h: torch.Tensor, p: Dict[str, torch.Tensor], limit: float) -> torch.Tensor:
    g = torch.clamp(h @ p["gate"].T, max=limit)
    u = torch.clamp(h @ p["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ p["down"].T


def route(h: torch.Tensor, w_router: torch.Tensor, router: dict):
    """Chosen experts and their weights per token: softmax scores, the best groups by their best member, then the best
    experts of those; weights are the scores times the scale."""
    s = torch.softmax(h @ w_router.T, -1)
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = router["experts"] // groups["count"]
    chosen = []
    for row in s:
        best = sorted(range(groups["count"]), key=lambda n: -float(row[n * size:(n + 1) * size].max()))[:groups["keep"]]
        open_ = [e for n in best for e in range(n * size, (n + 1) * size)]
        top = sorted(open_, key=lambda e: -float(row[e]))[:router["top"]]
        chosen.append([(e, row[e] * router.get("scale", 1.0)) for e in top])
    return chosen


def expert_mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str, mlp: dict) -> torch.Tensor:
    def part(n):
        return {k: w[f"{name}.{n}.{k}"] for k in ("gate", "up", "down")}

    out = torch.zeros_like(h)
    for t, picks in enumerate(route(h, w[name + ".router"], mlp["router"])):
        for e, weight in picks:
            out[t] += weight * clamped_expert(h[t:t + 1], part(f"e{e}"), mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        gate = torch.sigmoid(h @ w[name + ".shared.sg"].T)
        out = out + gate * clamped_expert(h, part("shared"), mlp["shared"]["limit"])
    return out


def residual_streams(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int],
                     dtype=torch.float64) -> List[torch.Tensor]:
    """The residual stream after the embedding and after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    out, cached = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        mix, n = layer["mixer"], f"l{i}."
        p = {k[len(n) + 4:]: v for k, v in w.items() if k.startswith(n + "mix.")}
        h = layer_norm(x, w[n + "norm1"], eps)
        if layer["type"] == "latent_attention":
            donor: Optional[int] = mix.get("kv_from")
            if donor is None:
                cached[i] = latents(h, p["dkv"], p["dkv.norm"], mix, eps)
            x = x + latent_attention(h, *cached[i if donor is None else donor], p, mix)
        else:
            x = x + {"lightning": lightning, "gla": gla}[layer["type"]](h, p, mix, eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = layer_norm(x, w[n + "norm2"], eps)
            if mlp["kind"] == "dense":
                x = x + gated_feed_forward(h, {k: w[f"{n}mlp.{k}"] for k in ("gate", "up", "down")})
            else:
                x = x + expert_mixture(h, w, n + "mlp", mlp)
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64) -> torch.Tensor:
    x = residual_streams(cfg, w, tokens, dtype)[-1]
    return layer_norm(x, w["final.norm"].to(dtype), float(cfg["norm"]["eps"])) @ w["head"].to(dtype).T
