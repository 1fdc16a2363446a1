"""Plain, slow restatement of the Mitilix decoder over a whole sequence: one function per mechanism, no cache,
no batching, nothing shared with the serving code. The tests compare the framework with it."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def scalar_rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps), times one number for all coordinates."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain.reshape(())


def vector_rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def input_convolution(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h_t + sum_j w[:, j] h_(t - taps + 1 + j), zeros ahead of the sequence; h [T, C], w [C, taps]."""
    t, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for j in range(taps):
        back = taps - 1 - j
        for i in range(t):
            if i - back >= 0:
                out[i] += w[:, j] * h[i - back]
    return out


def latent_of(h: torch.Tensor, w_dkv: torch.Tensor, norm: torch.Tensor, eps: float) -> torch.Tensor:
    return vector_rms_norm(h @ w_dkv.T, norm, eps)


def window_visible(i: int, j: int, size: int) -> bool:
    return 0 <= i - j < size


def latent_attention(h: torch.Tensor, c: torch.Tensor, p: Dict[str, torch.Tensor], heads: int, dim: int, vdim: int,
                     scale: float, window: int) -> torch.Tensor:
    """Per head: keys and values expanded from the latents, softmax over the window, output projection."""
    t = h.shape[0]
    q = (h @ p["q"].T).view(t, heads, dim)
    k = (c @ p["uk"].T).view(t, heads, dim)
    v = (c @ p["uv"].T).view(t, heads, vdim)
    mask = torch.tensor([[window_visible(i, j, window) for j in range(t)] for i in range(t)])
    out = torch.empty(t, heads, vdim, dtype=h.dtype)
    for n in range(heads):
        s = (q[:, n] @ k[:, n].T) * scale
        s = s.masked_fill(~mask, -math.inf)
        out[:, n] = torch.softmax(s, -1) @ v[:, n]
    return out.reshape(t, heads * vdim) @ p["o"].T


def erf_gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def dense_feed_forward(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return erf_gelu(h @ up.T) @ down.T


def residual_streams(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int],
                     dtype=torch.float64) -> List[torch.Tensor]:
    """The residual stream after the embedding and after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = torch.stack([w["embed"][tok] + w["pos"][i] for i, tok in enumerate(tokens)])
    out, latents = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        mix, name = layer["mixer"], f"l{i}."
        h = scalar_rms_norm(x, w[name + "norm1"], eps)
        h1 = input_convolution(h, w[name + "canon1"])
        donor: Optional[int] = mix.get("kv_from")
        if donor is None:
            latents[i] = latent_of(h1, w[name + "mix.dkv"], w[name + "mix.dkv.norm"], eps)
        c = latents[i if donor is None else donor]
        p = {k: w[name + "mix." + k] for k in ("q", "uk", "uv", "o")}
        y = latent_attention(h1, c, p, mix["heads"], mix["dim"], mix["vdim"], float(mix["scale"]),
                             int(mix["mask"]["size"]))
        if layer.get("mlp") is not None:
            h2 = input_convolution(h, w[name + "canon2"])
            y = y + dense_feed_forward(h2, w[name + "mlp.up"], w[name + "mlp.down"])
        x = x + y
        out.append(x)
    return out


def logits(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64) -> torch.Tensor:
    x = residual_streams(cfg, w, tokens, dtype)[-1]
    return scalar_rms_norm(x, w["final.norm"].to(dtype), float(cfg["norm"]["eps"])) @ w["head"].to(dtype).T
