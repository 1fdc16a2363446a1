"""Plain, slow restatement of the Zobelorn decoder over a whole sequence: one function per mechanism, no cache, no
batching, nothing shared with the serving code. The tests compare the framework with it."""
from __future__ import annotations

import math
from typing import Dict, List

import torch


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Each row divided by the root of (its mean square + eps)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def frequencies(rot: dict, llama: bool) -> List[float]:
    """Angle per position of every rotated pair. ``llama``: wavelengths are stretched by length class, otherwise all
    frequencies are divided by the factor."""
    out, s = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if s and not llama:
            f = f / s["factor"]
        elif s:
            turns = s["original"] * f / (2.0 * math.pi)       # original length over wavelength
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                t = (turns - s["low"]) / (s["high"] - s["low"])
                f = t * f + (1.0 - t) * f / s["factor"]
        out.append(f)
    return out


def rotate(x: torch.Tensor, freqs: List[float], neighbours: bool) -> torch.Tensor:
    """x [T, heads, n] at positions 0..T-1. Pairs: channels (2i, 2i+1) or (i, i + half of the rotated channels)."""
    out, half = x.clone(), len(freqs)
    for i, f in enumerate(freqs):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + half)
        for p in range(x.shape[0]):
            c, s = math.cos(p * f), math.sin(p * f)
            out[p, :, a] = x[p, :, a] * c - x[p, :, b] * s
            out[p, :, b] = x[p, :, b] * c + x[p, :, a] * s
    return out


def capped(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap)


def first_in_window(i: int, size: int) -> int:
    return max(0, i - size + 1)


def first_in_chunk(i: int, size: int) -> int:
    return i // size * size


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, first, cap=None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H * e]; position i sees first(i)..i."""
    t, heads, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = torch.zeros(t, heads, v.shape[2], dtype=q.dtype)
    for n in range(heads):
        for i in range(t):
            lo = first(i)
            s = (k[lo:i + 1, n // group] @ q[i, n]) * scale
            if cap is not None:
                s = capped(s, cap)
            out[i, n] = torch.softmax(s, 0) @ v[lo:i + 1, n // group]
    return out.reshape(t, -1)


def split_heads(x: torch.Tensor, n: int) -> torch.Tensor:
    return x.view(x.shape[0], n, -1)


def window_mixer(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float) -> torch.Tensor:
    """Queries and keys normed over all heads together, then rotated; capped scores in a sliding window; gated output."""
    f = frequencies(mix["rot"], llama=False)
    q = unit_rms(h @ p["q"].T, eps) * p["q.norm"]
    k = unit_rms(h @ p["k"].T, eps) * p["k.norm"]
    q = rotate(split_heads(q, mix["heads"]), f, neighbours=False)
    k = rotate(split_heads(k, mix["kv_heads"]), f, neighbours=False)
    v = split_heads(h @ p["v"].T, mix["kv_heads"])
    o = attend(q, k, v, mix["scale"], lambda i: first_in_window(i, mix["mask"]["size"]), mix["softcap"])
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def chunk_keys(h: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict, eps: float):
    """What a chunked layer caches per token: rotated, then unit-normed keys, and values."""
    k = rotate(split_heads(h @ p["k"].T, mix["kv_heads"]), frequencies(mix["rot"], llama=True), neighbours=True)
    return unit_rms(k, eps), split_heads(h @ p["v"].T, mix["kv_heads"])


def chunk_mixer(h: torch.Tensor, k: torch.Tensor, v: torch.Tensor, p: Dict[str, torch.Tensor], mix: dict,
                eps: float) -> torch.Tensor:
    q = rotate(split_heads(h @ p["q"].T, mix["heads"]), frequencies(mix["rot"], llama=True), neighbours=True)
    o = attend(unit_rms(q, eps), k, v, mix["scale"], lambda i: first_in_chunk(i, mix["mask"]["size"]))
    return o @ p["o"].T


def gated_feed_forward(h: torch.Tensor, p: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h: torch.Tensor, w_router: torch.Tensor, top: int):
    """Per token the experts with the largest sigmoid scores, with those scores."""
    s = torch.sigmoid(h @ w_router.T)
    return [[(e, row[e]) for e in sorted(range(len(row)), key=lambda e: -float(row[e]))[:top]] for row in s]


def expert_mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str, mlp: dict) -> torch.Tensor:
    """Sum of expert(score * token) over the chosen experts, and the shared expert."""
    def part(n):
        return {k: w[f"{name}.{n}.{k}"] for k in ("gate", "up", "down")}

    out = gated_feed_forward(h, part("shared")) if mlp.get("shared") else torch.zeros_like(h)
    for t, picks in enumerate(route(h, w[name + ".router"], mlp["router"]["top"])):
        for e, score in picks:
            out[t] += gated_feed_forward((score * h[t])[None], part(f"e{e}"))[0]
    return out


def residual_streams(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int],
                     dtype=torch.float64) -> List[torch.Tensor]:
    """The residual stream after the embedding and after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    out, cached = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        mix, n = layer["mixer"], f"l{i}."
        p = {k[len(n) + 4:]: v for k, v in w.items() if k.startswith(n + "mix.")}
        h = offset_norm(x, w[n + "norm1"], eps)
        if layer["type"] == "attention":
            y = window_mixer(h, p, mix, eps)
        else:
            donor = mix.get("kv_from")
            if donor is None:
                cached[i] = chunk_keys(h, p, mix, eps)
            y = chunk_mixer(h, *cached[i if donor is None else donor], p, mix, eps)
        x = x + m * offset_norm(y, w[n + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = offset_norm(x, w[n + "norm2"], eps)
            if mlp["kind"] == "dense":
                y = gated_feed_forward(h, {k: w[f"{n}mlp.{k}"] for k in ("gate", "up", "down")})
            else:
                y = expert_mixture(h, w, n + "mlp", mlp)
            x = x + m * offset_norm(y, w[n + "norm2b"], eps)
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64) -> torch.Tensor:
    x = residual_streams(cfg, w, tokens, dtype)[-1]
    return offset_norm(x, w["final.norm"].to(dtype), float(cfg["norm"]["eps"])) @ w["head"].to(dtype).T
