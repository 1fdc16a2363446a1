"""Python wrappers of the sm_100a kernels. Every function validates shapes/dtypes, allocates
the output with PyTorch's caching allocator and launches on the current stream.

``LAUNCHES`` counts kernel launches made through this module (the benchmark reports it);
``LEDGER`` remembers which kernel served which op (printed once per op when
``MSGL_DISPATCH_LEDGER=1``, the equivalent of the reference's ``[hip-engage]`` lines,
python/minisgl/_hip_engage.py:49-71).
"""
from __future__ import annotations

import ctypes
from typing import Dict, Optional, Tuple

import numpy as np
import torch

from ..env import ENV
from . import ref
from ._lib import check, lib

LAUNCHES = 0
LEDGER: Dict[str, str] = {}

_DT = {torch.bfloat16: 0, torch.float16: 1, torch.float32: 2}


def _count(op: str, kernel: str, n: int = 1) -> None:
    global LAUNCHES
    LAUNCHES += n
    if op not in LEDGER:
        LEDGER[op] = kernel
        if ENV.DISPATCH_LEDGER.value:
            print(f"[sm100-engage] {op} -> {kernel}", flush=True)


# ---- guarded workspaces and the device-side bounds report (MSGL_CHECK_BOUNDS=1) ----
_GUARD_BYTES = 256
_GUARD_BYTE = 0xA5
_GUARDED: Dict[str, Tuple[torch.Tensor, int]] = {}


def workspace(name: str, numel: int, dtype, device, zero: bool = False) -> torch.Tensor:
    """A scratch buffer the kernels write. With ``MSGL_CHECK_BOUNDS=1`` it sits between two 256-byte
    guard zones filled with a byte pattern, which :func:`verify_workspaces` re-reads: a kernel that
    wrote past either end of its scratch is named instead of corrupting a neighbour silently."""
    if not ENV.CHECK_BOUNDS.value:
        return (torch.zeros if zero else torch.empty)(numel, dtype=dtype, device=device)
    item = torch.empty((), dtype=dtype).element_size()
    g = _GUARD_BYTES // item
    full = (torch.zeros if zero else torch.empty)(numel + 2 * g, dtype=dtype, device=device)
    raw = full.view(torch.uint8)
    raw[:_GUARD_BYTES] = _GUARD_BYTE
    raw[raw.numel() - _GUARD_BYTES:] = _GUARD_BYTE
    _GUARDED[f"{name}@{device}"] = (full, g)
    return full[g:g + numel]


def verify_workspaces() -> list:
    """Names of the guarded workspaces whose guard zones no longer hold the pattern (synchronises)."""
    bad = []
    for name, (full, g) in _GUARDED.items():
        raw = full.view(torch.uint8)
        lo, hi = raw[:_GUARD_BYTES], raw[raw.numel() - _GUARD_BYTES:]
        if not (bool((lo == _GUARD_BYTE).all()) and bool((hi == _GUARD_BYTE).all())):
            bad.append(name)
    return bad


def bounds_checks_enabled() -> bool:
    """True when the loaded library is the bounds-checking build."""
    from ._lib import bind, c_i

    bind("msgl_bounds_enabled", c_i, [])
    return bool(lib().msgl_bounds_enabled())


def bounds_report(max_lines: int = 64) -> list:
    """Out-of-range indices recorded by the kernels since the last call, as text lines
    ``file.cu:LINE value V limit L`` (empty with the regular library). Synchronises the device."""
    from ._lib import bind, c_i, c_p

    bind("msgl_bounds_report", c_i, [c_p, c_i, c_i])
    width = 96
    buf = ctypes.create_string_buffer(max_lines * width)
    n = int(lib().msgl_bounds_report(buf, max_lines, width))
    raw = buf.raw
    return [raw[i * width:(i + 1) * width].split(b"\0", 1)[0].decode() for i in range(min(n, max_lines))]


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _dt(t: torch.Tensor) -> int:
    try:
        return _DT[t.dtype]
    except KeyError:
        raise TypeError(f"unsupported dtype {t.dtype} for the CUDA kernels") from None


# ------------------------------------------------------------------------------------------ elementwise
def embedding(ids, weight, vocab_start=0, vocab_len=None):
    ids = ids.to(torch.int32) if ids.dtype != torch.int32 else ids
    n = weight.shape[0] if vocab_len is None else vocab_len
    out = torch.empty((ids.numel(), weight.shape[1]), dtype=weight.dtype, device=weight.device)
    check(lib().msgl_embedding(_p(ids), _p(weight), _p(out), ids.numel(), weight.shape[1] * weight.element_size(),
                               vocab_start, n, _stream()), "embedding")
    _count("embedding", "embedding_kernel")
    return out


def _rms(x, residual, w, eps, plus_one, quant):
    assert x.is_contiguous() and x.dim() == 2
    rows, hidden = x.shape
    out = out_q = out_s = None
    if quant:
        out_q = torch.empty((rows, hidden), dtype=torch.float8_e4m3fn, device=x.device)
        out_s = torch.empty((rows,), dtype=torch.float32, device=x.device)
    else:
        out = torch.empty_like(x)
    if residual is not None:
        assert residual.is_contiguous() and residual.shape == x.shape and residual.dtype == x.dtype
    check(lib().msgl_rms_norm(_p(x), _p(residual), _p(w), _p(out), _p(out_q), _p(out_s), rows, hidden, eps,
                              int(plus_one), _dt(x), _stream()), "rms_norm")
    _count("rms_norm" + ("_add" if residual is not None else "") + ("_quant" if quant else ""), "rms_norm_kernel")
    return (out_q, out_s) if quant else out


def rms_norm_planes(part: "SplitPartial", residual, w, eps, plus_one=False, quant=False):
    """residual += (sum of the split-K planes, ascending); returns the norm of the new residual as a
    16-bit tensor or an (e4m3, scale) pair."""
    planes = part.planes
    splits, rows, hidden = planes.shape
    assert planes.is_contiguous() and residual.is_contiguous() and residual.shape == (rows, hidden)
    out = out_q = out_s = None
    if quant:
        out_q = torch.empty((rows, hidden), dtype=torch.float8_e4m3fn, device=planes.device)
        out_s = torch.empty((rows,), dtype=torch.float32, device=planes.device)
    else:
        out = torch.empty_like(residual)
    check(lib().msgl_rms_norm_planes(_p(planes), splits, _p(residual), _p(w), _p(out), _p(out_q), _p(out_s), rows,
                                     hidden, eps, int(plus_one), _dt(residual), _stream()), "rms_norm_planes")
    _count("rms_norm_add_planes" + ("_quant" if quant else ""), "rms_norm_kernel")
    return (out_q, out_s) if quant else out


def rms_norm(x, w, eps, plus_one=False):
    shape = x.shape
    return _rms(x.reshape(-1, shape[-1]), None, w, eps, plus_one, False).view(shape)


def rms_norm_add(x, residual, w, eps, plus_one=False):
    return _rms(x, residual, w, eps, plus_one, False)


def rms_norm_quant(x, w, eps, residual=None, plus_one=False):
    return _rms(x, residual, w, eps, plus_one, True)


def per_token_quant_fp8(x):
    return per_group_quant_fp8(x, 0)


def per_group_quant_fp8(x, group):
    assert x.is_contiguous() and x.dim() == 2
    rows, hidden = x.shape
    g = group or hidden
    q = torch.empty((rows, hidden), dtype=torch.float8_e4m3fn, device=x.device)
    s = torch.empty((rows, hidden // g) if group else (rows,), dtype=torch.float32, device=x.device)
    check(lib().msgl_quant_fp8(_p(x), _p(q), _p(s), rows, hidden, g, _dt(x), _stream()), "quant_fp8")
    _count("quant_fp8", "quant_group_kernel")
    return q, s


_ACT = {"silu": 0, "gelu": 1, "gelu_tanh": 2, "clamped": 3}


def act_and_mul(x, kind="silu", alpha=0.0, limit=0.0):
    """``act(gate) * up`` of rows ``[gate, up]``; ``clamped``: ``g sigmoid(alpha g) (u + 1)`` within ``limit``."""
    assert x.is_contiguous() and x.dim() == 2
    rows, two_i = x.shape
    out = torch.empty((rows, two_i // 2), dtype=x.dtype, device=x.device)
    check(lib().msgl_act_and_mul(_p(x), _p(out), None, None, rows, two_i // 2, _ACT[kind], alpha, limit, _dt(x),
                                 _stream()), "act_and_mul")
    _count("act_and_mul", "act_mul_kernel")
    return out


def silu_and_mul_quant(x):
    assert x.is_contiguous() and x.dim() == 2
    rows, two_i = x.shape
    q = torch.empty((rows, two_i // 2), dtype=torch.float8_e4m3fn, device=x.device)
    s = torch.empty((rows,), dtype=torch.float32, device=x.device)
    check(lib().msgl_act_and_mul(_p(x), None, _p(q), _p(s), rows, two_i // 2, 0, 0.0, 0.0, _dt(x), _stream()),
          "silu_and_mul_quant")
    _count("silu_and_mul_quant", "act_mul_quant_kernel")
    return q, s


# ------------------------------------------------------------------------------------------ rope / kv
def qk_norm_rope_store(qkv, q_w, k_w, positions, cos_sin, hq, hk, head_dim, rotary_dim, eps, k_cache, v_cache,
                       out_loc, k_scale=None, v_scale=None, interleaved=False):
    assert qkv.is_contiguous()
    t = qkv.shape[0]
    q_out = torch.empty((t, hq, head_dim), dtype=qkv.dtype, device=qkv.device)
    page_size = k_cache.shape[2]
    fp8 = k_cache.dtype == torch.float8_e4m3fn
    num_slots = k_cache.shape[0] * page_size
    check(lib().msgl_qk_norm_rope_store(
        _p(qkv), _p(q_w), _p(k_w), _p(positions), _p(cos_sin), _p(q_out), _p(k_cache), _p(v_cache), _p(out_loc),
        _p(k_scale), _p(v_scale), t, hq, hk, head_dim, rotary_dim, page_size, eps, int(interleaved), int(fp8),
        cos_sin.shape[0], num_slots, _dt(qkv), _stream()), "qk_norm_rope_store")
    _count("qk_norm_rope_store", "qk_norm_rope_store_kernel")
    return q_out


def heads_rope_store(x, heads, kv_heads, width, dim, positions, cos_sin, interleaved, eps, q_w=None, k_w=None,
                     totals=None, unit=False, store=None):
    assert x.dim() == 2 and x.stride(1) == 1 and positions.dtype == torch.int32
    t = x.shape[0]
    q_out = torch.empty((t, heads, width), dtype=x.dtype, device=x.device)
    k_cache = v_cache = out_loc = sums = None
    page_size = slots = 0
    q_count, k_count = heads * dim, kv_heads * dim
    if store is not None:
        k_cache, v_cache, out_loc = store
        page_size, slots = k_cache.shape[2], k_cache.shape[0] * k_cache.shape[2]
        assert k_cache.dtype == v_cache.dtype == x.dtype and k_cache.is_contiguous() and v_cache.is_contiguous()
        assert k_cache.shape[1] == kv_heads and k_cache.shape[3] == width
    if totals is not None:
        sums, q_count, k_count = totals
        assert sums.is_contiguous() and sums.dtype == torch.float32 and sums.shape == (t, 2)
    for w in (q_w, k_w):
        assert w is None or (w.dtype == torch.float32 and w.is_contiguous())
    rot, max_pos = (cos_sin.shape[1], cos_sin.shape[0]) if cos_sin is not None else (0, 0)
    check(lib().msgl_heads_rope_store(
        _p(x), x.stride(0), _p(q_w), _p(k_w), _p(sums), float(q_count), float(k_count), _p(positions), _p(cos_sin), rot,
        _p(q_out), _p(k_cache), _p(v_cache), _p(out_loc), t, heads, kv_heads, width, dim, page_size, eps, int(interleaved),
        int(unit), max_pos, slots, _dt(x), _stream()), "heads_rope_store")
    _count("heads_rope_store", "heads_rope_store_kernel")
    return q_out


def store_kv(k, v, k_cache, v_cache, out_loc, k_scale=None, v_scale=None):
    hk, page_size, d = k_cache.shape[1], k_cache.shape[2], k_cache.shape[3]
    t = out_loc.numel()
    k = k.reshape(t, hk, d).contiguous()
    v = v.reshape(t, hk, d).contiguous()
    fp8 = k_cache.dtype == torch.float8_e4m3fn
    check(lib().msgl_store_kv(_p(k), _p(v), _p(k_cache), _p(v_cache), _p(out_loc), _p(k_scale), _p(v_scale), t, hk,
                              d, page_size, int(fp8), k_cache.shape[0] * page_size, _dt(k), _stream()), "store_kv")
    _count("store_kv", "store_kv_kernel")


# ------------------------------------------------------------------------------------------ attention
_KV_MAPS: Dict[Tuple, Tuple[np.ndarray, object]] = {}


def _kv_map(k_cache: torch.Tensor):
    """TMA descriptor over the pool buffer that ``k_cache`` (one layer's K plane) is a view of.
    Returns ``(descriptor bytes, layer index, number of layers)``."""
    base = k_cache._base if k_cache._base is not None else k_cache
    pages_p1, hk, ps, d = k_cache.shape
    if base.dim() == 6:
        two, layers = base.shape[0], base.shape[1]
        plane_elems = pages_p1 * hk * ps * d
        layer = (k_cache.data_ptr() - base.data_ptr()) // (plane_elems * base.element_size())
        layer = int(layer) % layers
        root = base
    else:  # a stand-alone [pages, hk, ps, d] K tensor followed by nothing: treat as one layer
        raise ValueError("paged_attention expects k_cache / v_cache to be planes of one pool buffer")
    key = (root.data_ptr(), tuple(root.shape), root.dtype)
    hit = _KV_MAPS.get(key)
    if hit is None:
        buf = np.zeros(128, dtype=np.uint8)
        check(lib().msgl_attn_make_kv_map(buf.ctypes.data, root.data_ptr(), root.element_size(), d, ps, hk,
                                          pages_p1, 2 * layers), "attn_make_kv_map")
        if len(_KV_MAPS) > 512:            # layers with planes of their own have a map each
            _KV_MAPS.clear()
        hit = (buf, root)
        _KV_MAPS[key] = hit
    return hit[0], layer, layers


def make_pool_buffer(num_layers, pages_plus_one, hk, page_size, d, dtype, device):
    return torch.zeros((2, num_layers, pages_plus_one, hk, page_size, d), dtype=dtype, device=device)


def attention_workspace(max_rows, hq, d, device, max_splits=16):
    return workspace("attention split partials", max_splits * max_rows * hq * (d + 1), torch.float32, device)


def choose_splits(batch, hk, max_kv, decode):
    if not decode:
        return 1
    ctas = batch * hk
    want = -(-592 // ctas)
    by_len = max(1, max_kv // 256)
    return int(max(1, min(want, by_len, 16)))


def paged_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, *, causal=True, window=0, mask=None,
                    k_scale=None, v_scale=None, max_q=0, max_kv=0, decode=False, workspace=None, splits=None,
                    plan=None, tc=None, mask_window=0, chunk=0, softcap=0.0, gate=None, bias=None, sink=None, talk=None):
    """``plan`` (a ``PrefillPlan``) or ``tc=True`` sends a causal prefill / extend step to the
    tcgen05 kernel when it covers the shape (``tc=True`` without a plan builds the step tables from
    the device lengths, which synchronises). Without either the general kernel runs: decode and
    verification steps must not change kernels with the number of rows per request."""
    if talk is not None and talk_attention_ok(q, k_cache, chunk, softcap, gate):
        assert causal and mask is None
        return talk_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, talk, bias, sink, window, decode,
                              splits or 1, workspace)
    if q.dtype == torch.float32 or talk is not None:
        assert causal and mask is None
        return _paged_attention_f32(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, window, chunk, softcap, gate, bias,
                                    sink, talk)
    if bias is not None or sink is not None:
        raise NotImplementedError("16-bit attention takes a distance bias and a sink with mixed heads")
    t, hq, d = q.shape
    pages_p1, hk, ps, _ = k_cache.shape
    if max_q <= 0:
        max_q = int((cu_q[1:] - cu_q[:-1]).max())
    if tc is None:
        tc = plan is not None
    if tc and prefill_attention_tc_ok(q, k_cache, causal=causal, window=window, mask=mask, decode=decode):
        if plan is None:
            plan = PrefillPlan(cu_q.cpu().numpy(), seq_lens.cpu().numpy(), q.device)
        return prefill_attention_tc(q, k_cache, v_cache, block_table, plan, scale, k_scale=k_scale, v_scale=v_scale)
    desc, layer, layers = _kv_map(k_cache)
    b = seq_lens.numel()
    if max_q <= 0:
        max_q = int((cu_q[1:] - cu_q[:-1]).max())
    if max_kv <= 0:
        max_kv = int(seq_lens.max())
    if splits is None:
        splits = choose_splits(b, hk, max_kv, decode or max_q == 1)
    if splits > 1:
        need = int(lib().msgl_attn_workspace_floats(t, hq, d, splits))
        if workspace is None or workspace.numel() < need:
            workspace = torch.empty(need, dtype=torch.float32, device=q.device)
    out = torch.empty_like(q)
    fp8 = k_cache.dtype == torch.float8_e4m3fn
    mask_stride = 0
    if mask is not None:
        assert mask.dtype == torch.float32 and mask.stride(-1) == 1
        mask_stride = mask.stride(0)
        if mask_window:
            # windowed form: rows of exactly ``mask_window`` floats for the last ``mask_window`` KV
            # positions of each request (earlier positions are visible); passed as a negative stride
            assert mask.stride(0) == mask_window and mask.shape[-1] == mask_window
            mask_stride = -int(mask_window)
    check(lib().msgl_paged_attention(
        desc.ctypes.data, _p(q), _p(out), _p(block_table), block_table.stride(0), _p(cu_q), _p(seq_lens),
        _p(k_scale), _p(v_scale), _p(mask), mask_stride, _p(workspace) if splits > 1 else None,
        b, t, max_q, hq, hk, d, ps, pages_p1 - 1, layer, layers, int(fp8), int(causal), int(window), splits,
        float(scale), int(chunk), float(softcap), *_output_gate(gate, q), _dt(q), _stream()), "paged_attention")
    _count("paged_attention", "paged_attention_kernel", 2 if splits > 1 else 1)
    return out


def _output_gate(gate, q):
    """Pointer and row stride of the logits of a gate per output channel."""
    if gate is None:
        return None, 0
    assert gate.shape == (q.shape[0], q.shape[1] * q.shape[2]) and gate.stride(1) == 1 and gate.dtype == q.dtype
    return gate.data_ptr(), gate.stride(0)


def _distance_bias(bias, hq):
    """Pointer and length of a table of what a score loses at each distance."""
    if bias is None:
        return None, 0
    assert bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[0] == hq
    return bias.data_ptr(), bias.shape[1]


_BIAS_ROWS: Dict[Tuple, Tuple] = {}


def _bias_rows(bias):
    """The table of the prefill kernel: what a score gains at each distance, in units of log2 and in the order of the keys
    (ever nearer ones), zeros for distances that a block has and no row sees. Returns ``(table [H, entries], entry of
    distance 0)``."""
    key = (bias.data_ptr(), tuple(bias.shape), bias.device)
    hit = _BIAS_ROWS.get(key)
    if hit is None or hit[0] is not bias:
        pad = 384                                   # a tile's rows and a block's keys beyond the reach, on either side
        table = torch.nn.functional.pad((bias * -1.4426950408889634).flip(1), (pad, pad)).contiguous()
        if len(_BIAS_ROWS) > 512:
            _BIAS_ROWS.clear()
        _BIAS_ROWS[key] = hit = (bias, table, pad + bias.shape[1] - 1)
    return hit[1], hit[2]


def _paged_attention_f32(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, window, chunk, softcap, gate, bias, sink,
                         talk):
    t, hq, d = q.shape
    pages, hk, ps, _ = k_cache.shape
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.dtype == q.dtype
    out = torch.empty((t, hq, d if talk is None else hk * d), dtype=q.dtype, device=q.device)
    check(lib().msgl_paged_attention_f32(
        _p(q), _p(k_cache), _p(v_cache), _p(out), _p(block_table), block_table.stride(0), _p(cu_q), _p(seq_lens),
        seq_lens.numel(), t, hq, hk, d, ps, pages, int(window), int(chunk), float(scale), float(softcap),
        *_output_gate(gate, q), *_distance_bias(bias, hq), _p(sink), int(talk is not None), _dt(q), _stream()),
        "paged_attention_f32")
    _count("paged_attention_f32", "paged_attention_f32_kernel")
    return out if talk is None else head_mix(out, talk, hk, d)


def talk_attention_ok(q, k_cache, chunk=0, softcap=0.0, gate=None) -> bool:
    """Sizes of the decode kernel for mixed heads; others take the plain one."""
    return (q.dtype == torch.bfloat16 and q.shape[2] in (64, 128) and q.shape[1] <= 64 and k_cache.shape[2] in (8, 16, 32, 64)
            and not chunk and not softcap and gate is None)


def talk_splits(batch: int, heads: int, hk: int, d: int, reach: int) -> int:
    """Key ranges of a decode step with mixed heads: as many CTAs as fit the SMs, two blocks of 64 keys or more in a range."""
    mt = 1 if heads <= 16 else 2 if heads <= 32 else 4
    gn = 2 if hk <= 2 or (mt == 4 and d == 128) else 4
    room = 148 * (2 if mt * gn * (d // 64) <= 8 else 1)
    return int(max(1, min(room // max(batch * -(-hk // gn), 1), reach // 128, 16)))


def talk_workspace(heads, device):
    """For the largest split step of layers of ``(heads, kv heads, width)``: rows times ranges stay within two per SM."""
    need = max(int(lib().msgl_talk_workspace_floats(296, h, hk, d, 1)) for h, hk, d in heads)
    return workspace("mixed-head attention partials", need, torch.float32, device)


def talk_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, talk, bias=None, sink=None, window=0, decode=False,
                   splits=1, workspace=None):
    """Attention with mixed heads for single query rows: one pass over keys and values for all heads."""
    t, hq, d = q.shape
    pages_p1, hk, ps, _ = k_cache.shape
    assert q.is_contiguous() and talk.dtype == torch.float32 and talk.is_contiguous() and talk.shape == (hq, hq)
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.dtype == v_cache.dtype == q.dtype
    if splits > 1:
        need = int(lib().msgl_talk_workspace_floats(t, hq, hk, d, splits))
        if workspace is None or workspace.numel() < need:
            workspace = torch.empty(need, dtype=torch.float32, device=q.device)
    out = torch.empty_like(q)
    check(lib().msgl_talk_attention(
        _p(k_cache), _p(v_cache), _p(q), _p(out), _p(block_table), block_table.stride(0), _p(cu_q), _p(seq_lens),
        *_distance_bias(bias, hq), _p(sink), _p(talk), _p(workspace) if splits > 1 else None, seq_lens.numel(), t, hq, hk, d, ps,
        pages_p1 - 1, int(window), splits, int(decode), float(scale), _stream()), "talk_attention")
    _count("talk_attention", "talk_decode_kernel", 2 if splits > 1 else 1)
    return out


def head_mix(o, talk, hk, d):
    """``o [T, H, width]`` (value head c at columns ``c * d`` on) -> ``[T, H, d]``: head h gets the sum over g of
    ``talk[h, g]`` times head g's rows of h's own value head."""
    t, hq, width = o.shape
    assert o.is_contiguous() and talk.dtype == torch.float32 and talk.is_contiguous() and talk.shape == (hq, hq)
    out = torch.empty((t, hq, d), dtype=o.dtype, device=o.device)
    check(lib().msgl_head_mix(_p(o), _p(talk), _p(out), t, hq, hk, d, width, _dt(o), _stream()), "head_mix")
    _count("head_mix", "head_mix_kernel")
    return out


_PLAN_RING: Dict[torch.device, list] = {}
_PLAN_RING_POS: Dict[torch.device, int] = {}


def _upload_tables(host: np.ndarray, device) -> torch.Tensor:
    """int32 tables -> device through a small ring of pinned buffers: the copy is asynchronous, so
    building the plan of the next step does not wait for the kernels of the step in flight. A
    ring slot is reused only after the event recorded behind its copy."""
    device = torch.device(device)
    if device.type != "cuda":
        return torch.from_numpy(host.copy())
    ring = _PLAN_RING.setdefault(device, [None] * 4)
    pos = _PLAN_RING_POS.get(device, 0)
    _PLAN_RING_POS[device] = pos + 1
    slot = ring[pos % 4]
    n = int(host.size)
    if slot is not None and slot[1] is not None:
        slot[1].synchronize()
    if slot is None or slot[0].numel() < n:
        slot = [torch.empty(max(n * 2, 1 << 14), dtype=torch.int32, pin_memory=True), None]
        ring[pos % 4] = slot
    slot[0].numpy()[:n] = host
    dev = torch.empty(n, dtype=torch.int32, device=device)
    dev.copy_(slot[0][:n], non_blocking=True)
    ev = torch.cuda.Event()
    ev.record()
    slot[1] = ev
    return dev


def _first_block(pos: np.ndarray, window: int, chunk: int = 0) -> np.ndarray:
    """Start of the block of 128 positions that holds the first position a row at ``pos`` can see."""
    lo = np.zeros_like(pos)
    if window > 0:
        lo = np.maximum(lo, pos - window + 1)
    if chunk > 0:
        lo = np.maximum(lo, pos // chunk * chunk)
    return lo // 128 * 128


class PrefillPlan:
    """Per-step tables of the tensor-core prefill kernel: one item per (request, block of ``tile``
    query positions), heaviest first; the request of every 128-row scratch block; per request
    the scratch offset, KV length and first position in the scratch. Built on the host from the step's lengths, one H2D
    copy. ``window`` / ``chunk``: the reach of the layers the plan is for. ``tile`` 256: the form for query heads that do
    not come in pairs."""

    __slots__ = ("tables", "n_items", "t_pad", "n_req", "off_blk", "off_req", "tile")

    @staticmethod
    def rows_in_reach(cu_q: np.ndarray, seq_lens: np.ndarray, window: int = 0, chunk: int = 0) -> int:
        kv = np.asarray(seq_lens, dtype=np.int64)
        lo = _first_block(kv - np.diff(np.asarray(cu_q, dtype=np.int64)[:kv.size + 1]), window, chunk)
        return int(((kv - lo + 127) // 128 * 128).sum())

    def __init__(self, cu_q: np.ndarray, seq_lens: np.ndarray, device, window: int = 0, chunk: int = 0,
                 tile: int = 128) -> None:
        cu_q = np.asarray(cu_q, dtype=np.int64)
        kv = np.asarray(seq_lens, dtype=np.int64)
        b = int(kv.size)
        q_len = cu_q[1:b + 1] - cu_q[:b]
        kv_lo = _first_block(kv - q_len, window, chunk)
        kv_pad = (kv - kv_lo + 127) // 128 * 128
        kv_off = np.concatenate([[0], np.cumsum(kv_pad)[:-1]]) if b else np.zeros(0, dtype=np.int64)
        self.t_pad = int(kv_pad.sum())
        self.n_req = b
        self.tile = tile
        n_tiles = (q_len + tile - 1) // tile
        req = np.repeat(np.arange(b), n_tiles)
        first = np.concatenate([[0], np.cumsum(n_tiles)[:-1]]) if b else np.zeros(0, dtype=np.int64)
        qb = np.arange(int(n_tiles.sum())) - np.repeat(first, n_tiles)
        items = np.zeros((req.size, 8), dtype=np.int32)
        rows = np.minimum(tile, q_len[req] - qb * tile)
        pos0 = kv[req] - q_len[req] + qb * tile
        kv0 = _first_block(pos0, window, chunk)
        items[:, 0] = cu_q[req] + qb * tile
        items[:, 1] = rows
        items[:, 2] = pos0
        items[:, 3] = kv_off[req] + kv0 - kv_lo[req]
        items[:, 4] = (pos0 + rows - kv0 + 127) // 128
        items[:, 5] = req
        items[:, 6] = kv0
        items = items[np.argsort(-items[:, 4], kind="stable")]
        blk_req = np.repeat(np.arange(b), kv_pad // 128).astype(np.int32)
        req_info = np.stack([kv_off, kv, kv_lo], axis=1).astype(np.int32).reshape(-1)
        self.n_items = int(items.shape[0])
        self.off_blk = items.size
        self.off_req = self.off_blk + blk_req.size
        host = np.concatenate([items.reshape(-1), blk_req, req_info])
        self.tables = _upload_tables(host, device)


_TC_SCRATCH: Dict[Tuple[torch.device, torch.dtype, int], Tuple[torch.Tensor, torch.Tensor, int]] = {}


def _tc_scratch(device, dtype, hk: int, rows: int):
    """Dense K / V^T scratch shared by all layers of a step (each layer's gather overwrites it in
    stream order). Grows in steps of 8192 rows."""
    key = (device, dtype, hk)
    hit = _TC_SCRATCH.get(key)
    if hit is None or hit[2] < rows:
        cap = -(-rows // 8192) * 8192
        _TC_SCRATCH[key] = hit = (workspace(f"prefill K scratch {hk}", hk * cap * 128, dtype, device, zero=True),
                                   workspace(f"prefill V scratch {hk}", hk * cap * 128, dtype, device, zero=True), cap)
    return hit


def tc_prefill_pays(total_q: int, t_pad: int) -> bool:
    """The tensor-core path first copies every KV row the step can see into a dense 16-bit
    scratch. That is noise when the step has about as many query rows as KV rows (prefill, chunked
    prefill), but a short extend over a long cached prefix (a new chat turn over tens of thousands
    of tokens) would move several times the bytes the general kernel reads in place: such steps
    stay on the general kernel."""
    return t_pad <= 16 * max(int(total_q), 128)


def prefill_attention_tc_ok(q, k_cache, *, causal, window, mask, decode) -> bool:
    """The tcgen05 prefill kernel covers causal prefill / extend steps with head_dim 128 and an
    even number of query heads per KV head; everything else stays on the general kernel."""
    t, hq, d = q.shape
    hk = k_cache.shape[1]
    return (not decode and causal and not window and mask is None and d == 128 and hq % hk == 0
            and (hq // hk) % 2 == 0 and q.dtype in (torch.bfloat16, torch.float16) and q.stride(2) == 1
            and q.stride(1) == 128 and q.stride(0) % 8 == 0)


def prefill_heads_tc_ok(q, k_cache, scale) -> bool:
    """Rows of 64 or 128 channels; any head counts (``PrefillPlan.tile``), windows, chunks, soft caps and gates."""
    return (q.dtype == torch.bfloat16 and q.shape[2] in (64, 128) and q.is_contiguous() and scale > 0
            and q.shape[1] % k_cache.shape[1] == 0)


def prefill_attention_tc(q, k_cache, v_cache, block_table, plan: PrefillPlan, scale, *, k_scale=None, v_scale=None,
                         window=0, chunk=0, softcap=0.0, gate=None, bias=None, sink=None, talk=None):
    """``plan`` was made for the same window and chunk."""
    t, hq, d = q.shape
    _, hk, ps, _ = k_cache.shape
    kc, vt, cap = _tc_scratch(q.device, q.dtype, hk, plan.t_pad)
    out = torch.empty((t, hq, d if talk is None else -(-hk * d // 128) * 128), dtype=q.dtype, device=q.device)
    tb = plan.tables
    base = tb.data_ptr()
    fp8 = k_cache.dtype == torch.float8_e4m3fn
    rows, zero = (None, 0) if bias is None else _bias_rows(bias)
    check(lib().msgl_attn_prefill_tc(
        _p(q), q.stride(0), _p(out), _p(k_cache), _p(v_cache), _p(kc), _p(vt), cap, plan.t_pad,
        base, plan.n_items, base + 4 * plan.off_blk, base + 4 * plan.off_req, _p(block_table), block_table.stride(0),
        _p(k_scale), _p(v_scale), t, hq, hk, d, ps, int(fp8), float(scale), int(window), int(chunk), float(softcap),
        *_output_gate(gate, q), _p(rows), 0 if rows is None else rows.shape[1], zero, _p(sink), int(talk is not None),
        int(plan.tile == 256), _dt(q), _stream()), "attn_prefill_tc")
    _count("prefill_attention", "attn_prefill_tc_kernel", 2)
    return out if talk is None else head_mix(out, talk, hk, d)


# ------------------------------------------------------------------------------------------ GEMM
KIND_F16, KIND_BF16, KIND_F8, KIND_MXF4 = 0, 1, 2, 3


_PENDING_TP = None
SPLIT_K = ENV.GEMM_SPLIT_K.value
_SPLITK_PLANS: Dict[Tuple[int, int, int], int] = {}
_SPLITK_COUNTERS: Dict[torch.device, torch.Tensor] = {}


def _splitk_plan(kind: int, n: int, k: int) -> int:
    key = (kind, n, k)
    s = _SPLITK_PLANS.get(key)
    if s is None:
        s = _SPLITK_PLANS[key] = int(lib().msgl_gemm_splitk_plan(kind, n, k))
    return s


def _splitk_counters(device, n: int) -> torch.Tensor:
    """Per-tile arrival counters: zero between calls (the kernel resets what it used)."""
    t = _SPLITK_COUNTERS.get(device)
    if t is None or t.numel() < n:
        t = _SPLITK_COUNTERS[device] = workspace("split-K counters", max(n, 4096), torch.int32, device, zero=True)
    return t


class SplitPartial:
    """Output of a split-K GEMM whose K ranges were not reduced: fp32 planes [splits, rows, N] that
    the next fused add + norm sums in ascending order (``rms_norm_planes``)."""

    __slots__ = ("planes", "dtype")

    def __init__(self, planes: torch.Tensor, dtype: torch.dtype) -> None:
        self.planes = planes
        self.dtype = dtype

    @property
    def shape(self):
        return self.planes.shape[1:]

    def materialise(self) -> torch.Tensor:
        out = self.planes[0].clone()
        for p in self.planes[1:]:
            out += p
        return out.to(self.dtype)


# Decode-phase row-parallel projections may hand their K ranges to the following add + norm
# unreduced. Engines that need verify rows and decode rows on one GEMM code path switch it off.
SPLIT_K_DECODE = not ENV.DISABLE_SPLIT_K_DECODE.value
_PENDING_PLANES = False


def set_next_gemm_planes(on: bool = True) -> None:
    """Ask the next GEMM call of this thread (M <= 256) to return a ``SplitPartial`` when the
    split-K plan of its (N, K) has more than one range. Consumed by exactly one call."""
    global _PENDING_PLANES
    _PENDING_PLANES = on


def set_next_gemm_tp(args) -> None:
    """Tensor-parallel fusion arguments (``parallel.symm.GemmTpArgs``) for the next GEMM call of
    this thread: push the output rows to their owner ranks and / or wait for A rows that peers
    are still delivering. Consumed by exactly one call."""
    global _PENDING_TP
    _PENDING_TP = args


def take_pending_gemm_tp():
    global _PENDING_TP
    args, _PENDING_TP = _PENDING_TP, None
    return args


def _gemm(kind, a, b, n, k, out_dtype, a_scale=None, b_scale=None, bias=None, sf_atoms=None, bn=0, max_ctas=0):
    assert a.dim() == 2 and a.stride(1) == 1 and b.is_contiguous()
    m = a.shape[0]
    tp = take_pending_gemm_tp()
    if tp is not None:
        pushes = tp.rs_world > 0
        out = None if pushes else torch.empty((m, n), dtype=out_dtype, device=a.device)
        check(lib().msgl_gemm_tp(kind, _p(a), a.stride(0), _p(b), _p(out), n, m, n, k, _p(a_scale), _p(b_scale),
                                 _p(bias), _DT[bias.dtype] if bias is not None else 0, _p(sf_atoms), _DT[out_dtype],
                                 ctypes.byref(tp), _stream()), "gemm_tp")
        _count(("gemm_f16", "gemm_bf16", "gemm_w8a8", "gemm_w4a8_mxfp4")[kind] + ("_rs" if pushes else "_ag"),
               "gemm_pair_kernel")
        return out
    global _PENDING_PLANES
    want_planes, _PENDING_PLANES = _PENDING_PLANES, False
    if want_planes and 0 < m <= 256 and bn == 0:
        splits = _splitk_plan(kind, n, k)
        if splits > 1:
            planes = torch.empty((splits, m, n), dtype=torch.float32, device=a.device)
            check(lib().msgl_gemm_splitk_planes(kind, _p(a), a.stride(0), _p(b), _p(planes), m, n, k, _p(a_scale),
                                                _p(b_scale), _p(bias), _DT[bias.dtype] if bias is not None else 0,
                                                _p(sf_atoms), splits, _stream()), "gemm_splitk_planes")
            _count(("gemm_f16", "gemm_bf16", "gemm_w8a8", "gemm_w4a8_mxfp4")[kind] + "_splitk_planes",
                   "gemm_tcgen05_kernel")
            return SplitPartial(planes, out_dtype)
    out = torch.empty((m, n), dtype=out_dtype, device=a.device)
    if m == 0:
        return out
    if m <= 256 and bn == 0 and SPLIT_K:
        splits = _splitk_plan(kind, n, k)
        if splits > 1:
            # small M: K ranges of one tile run on different SMs; the plan depends on (N, K) only
            mt, nt = (m + 127) // 128, (n + 127) // 128
            ws = torch.empty((splits, mt * 128, nt * 128), dtype=torch.float32, device=a.device)
            check(lib().msgl_gemm_splitk(kind, _p(a), a.stride(0), _p(b), _p(out), n, m, n, k, _p(a_scale), _p(b_scale),
                                         _p(bias), _DT[bias.dtype] if bias is not None else 0, _p(sf_atoms),
                                         _DT[out_dtype], splits, _p(ws), _p(_splitk_counters(a.device, mt * nt)),
                                         _stream()), "gemm_splitk")
            _count(("gemm_f16", "gemm_bf16", "gemm_w8a8", "gemm_w4a8_mxfp4")[kind] + "_splitk", "gemm_tcgen05_kernel")
            return out
    check(lib().msgl_gemm(kind, _p(a), a.stride(0), _p(b), _p(out), n, m, n, k, _p(a_scale), _p(b_scale), _p(bias),
                          _DT[bias.dtype] if bias is not None else 0, _p(sf_atoms), _DT[out_dtype], bn, max_ctas,
                          _stream()), "gemm")
    _count(("gemm_f16", "gemm_bf16", "gemm_w8a8", "gemm_w4a8_mxfp4")[kind], "gemm_tcgen05_kernel")
    return out


def gemm(x, w, bias=None, out_dtype=None, bn=0, max_ctas=0):
    shape = x.shape
    x2 = x.reshape(-1, shape[-1])
    if x2.stride(1) != 1:
        x2 = x2.contiguous()
    kind = KIND_BF16 if x2.dtype == torch.bfloat16 else KIND_F16
    if x2.dtype == torch.float32 and w.dtype == torch.float32:
        if bias is not None:
            raise NotImplementedError("gemm: no bias in the fp32 form")
        return gemm_f32(x2, w).view(*shape[:-1], w.shape[0])
    if w.dtype != x2.dtype:
        raise TypeError(f"gemm: activation {x2.dtype} vs weight {w.dtype}")
    n, k = w.shape
    if n % 8:
        raise ValueError("gemm: N must be a multiple of 8")
    out = _gemm(kind, x2, w, n, k, out_dtype or x.dtype, bias=bias, bn=bn, max_ctas=max_ctas)
    if isinstance(out, SplitPartial):
        return out
    return out.view(*shape[:-1], n) if out is not None else None


def gemm_w8a8(x_q, x_scale, w_q, w_scale, out_dtype=torch.bfloat16, bias=None, bn=0):
    n, k = w_q.shape
    return _gemm(KIND_F8, x_q, w_q, n, k, out_dtype, a_scale=x_scale, b_scale=w_scale, bias=bias, bn=bn)


def gemm_w4a8_mxfp4(x_q, x_scale, w_packed, sf_atoms, out_dtype=torch.bfloat16, bias=None, bn=0):
    n, k = w_packed.shape[0], x_q.shape[-1]
    if w_packed.shape[1] * 2 != (k + 127) // 128 * 128 and w_packed.shape[1] * 2 != k:
        raise ValueError(f"gemm_w4a8_mxfp4: weights of K={w_packed.shape[1] * 2} do not match activations of K={k}")
    if w_packed.shape[1] * 2 != k and k % 128 == 0:
        raise ValueError("gemm_w4a8_mxfp4: padded weights with an unpadded K")
    if sf_atoms is None:
        raise ValueError("gemm_w4a8_mxfp4 needs the packed scale atoms (quant.mxfp4.pack_sf_atoms)")
    return _gemm(KIND_MXF4, x_q, w_packed, n, k, out_dtype, a_scale=x_scale, bias=bias, sf_atoms=sf_atoms, bn=bn)


def gemm_fp8_block(x_q, x_scale, w_q, w_scale, out_dtype=torch.bfloat16, tile_expert=None):
    """Block-scaled fp8 W8A8: ``x_q [M, K]`` e4m3 with ``x_scale [M, ceil(K/128)]`` (1 x 128 groups),
    ``w_q [N, K]`` e4m3 with ``w_scale [ceil(N/128), ceil(K/128)]`` (128 x 128 blocks). Grouped
    form: ``w_q [E, N, K]``, ``w_scale [E, N/128, ceil(K/128)]``, rows of ``x_q`` sorted by expert in
    128-row tiles and ``tile_expert [M/128]``. Every K block is accumulated on the tensor core by
    itself and promoted with its scale product (``gemm_fp8_block_kernel``)."""
    from ._lib import bind, c_i, c_ll, c_p

    if not hasattr(gemm_fp8_block, "_bound"):
        bind("msgl_gemm_fp8_block", c_i, [c_p, c_ll, c_p, c_p, c_ll, c_i, c_i, c_i, c_p, c_p, c_p, c_i, c_i, c_p])
        bind("msgl_gemm_fp8_block_status", c_i, [c_i])
        gemm_fp8_block._bound = True
    assert x_q.dtype == torch.float8_e4m3fn and w_q.dtype == torch.float8_e4m3fn
    assert x_q.dim() == 2 and x_q.stride(1) == 1 and w_q.is_contiguous()
    m, k = x_q.shape
    experts = 0
    if tile_expert is not None:
        experts, n, kw = w_q.shape
    else:
        n, kw = w_q.shape
    if kw != k:
        raise ValueError(f"gemm_fp8_block: activations of K={k} against weights of K={kw}")
    kb = (k + 127) // 128
    x_scale = x_scale.float() if x_scale.dtype != torch.float32 else x_scale
    w_scale = w_scale.float() if w_scale.dtype != torch.float32 else w_scale
    assert x_scale.is_contiguous() and x_scale.shape == (m, kb), (x_scale.shape, (m, kb))
    assert w_scale.is_contiguous() and w_scale.shape[-1] == kb and w_scale.shape[-2] == (n + 127) // 128
    out = torch.empty((m, n), dtype=out_dtype, device=x_q.device)
    check(lib().msgl_gemm_fp8_block(_p(x_q), x_q.stride(0), _p(w_q), _p(out), n, m, n, k, _p(x_scale), _p(w_scale),
                                    _p(tile_expert), experts, _DT[out_dtype], _stream()), "gemm_fp8_block")
    _count("gemm_w8a8_block" + ("_grouped" if tile_expert is not None else ""), "gemm_fp8_block_kernel")
    return out


def silu_and_mul_quant_group(x):
    """SiLU(gate) * up of ``x [rows, 2I]`` quantised to e4m3 in groups of 128 outputs:
    returns ``(q [rows, I], scales [rows, I / 128])``."""
    from ._lib import bind, c_i, c_p

    if not hasattr(silu_and_mul_quant_group, "_bound"):
        bind("msgl_silu_mul_quant_group", c_i, [c_p, c_p, c_p, c_i, c_i, c_i, c_p])
        silu_and_mul_quant_group._bound = True
    assert x.is_contiguous() and x.dim() == 2
    rows, two_i = x.shape
    inter = two_i // 2
    q = torch.empty((rows, inter), dtype=torch.float8_e4m3fn, device=x.device)
    s = torch.empty((rows, inter // 128), dtype=torch.float32, device=x.device)
    check(lib().msgl_silu_mul_quant_group(_p(x), _p(q), _p(s), rows, inter, _dt(x), _stream()), "silu_mul_quant_group")
    _count("silu_and_mul_quant_group", "silu_mul_quant_group_kernel")
    return q, s


W4_EXPAND_ROWS = 256
_W4_SCRATCH: Dict[Tuple[torch.device, torch.dtype], torch.Tensor] = {}


def _w4_scratch(device, dtype, elems: int) -> torch.Tensor:
    key = (device, dtype)
    t = _W4_SCRATCH.get(key)
    if t is None or t.numel() < elems:
        t = _W4_SCRATCH[key] = workspace("4-bit expansion scratch", elems, dtype, device)
    return t


def gemm_w4a16(x, w_packed, scales_t, zeros_t=None, channel=None, group=128, nvfp4=False, bias=None, out_dtype=None):
    """``x @ dequant(W).T`` with W kept 4-bit in HBM (``gemm_w4a16_kernel``): ``w_packed [N, K/2]`` bytes
    (low nibble = even k), ``scales_t [K/group, N]`` fp32 with ``zeros_t`` of the same shape (integer
    formats: ``w = (code - zero) * scale``), or e4m3 bytes with a per-channel fp32 factor ``channel [N]``
    (NVFP4: ``w = e2m1(code) * scale * channel``). Activations stay 16-bit."""
    from ._lib import bind, c_i, c_ll, c_p

    if not hasattr(gemm_w4a16, "_bound"):
        bind("msgl_gemm_w4a16", c_i, [c_p, c_ll, c_p, c_p, c_p, c_p, c_p, c_p, c_ll, c_i, c_i, c_i, c_i, c_i, c_i, c_i,
                                      c_p])
        bind("msgl_gemm_w4a16_status", c_i, [c_i])
        bind("msgl_w4_expand", c_i, [c_p, c_p, c_p, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_p])
        gemm_w4a16._bound = True
    shape = x.shape
    x2 = x.reshape(-1, shape[-1])
    if x2.stride(1) != 1:
        x2 = x2.contiguous()
    m, k = x2.shape
    n = w_packed.shape[0]
    assert w_packed.dtype == torch.uint8 and w_packed.is_contiguous() and w_packed.shape[1] * 2 == k
    assert scales_t.is_contiguous() and scales_t.shape == (k // group, n)
    out_dtype = out_dtype or x.dtype
    if m > W4_EXPAND_ROWS:
        # many rows (prefill): expand the matrix once into a scratch shared by all layers, then the
        # ordinary GEMM; the in-kernel expansion would repeat per 128-row tile
        scratch = _w4_scratch(x.device, x.dtype, n * k)
        check(lib().msgl_w4_expand(_p(w_packed), _p(scales_t), _p(zeros_t), _p(channel), _p(scratch), n, k, group,
                                   int(nvfp4), _dt(x2), _stream()), "w4_expand")
        _count("w4_expand", "w4_expand_kernel")
        # the scratch is written by the kernel just ahead: no weight fetch before the dependency wait
        prev = gemm_static_weights(False)
        try:
            out = _gemm(KIND_BF16 if x.dtype == torch.bfloat16 else KIND_F16, x2, scratch[: n * k].view(n, k), n, k,
                        out_dtype, bias=bias)
        finally:
            gemm_static_weights(prev)
        return out.view(*shape[:-1], n) if out is not None else None
    out = torch.empty((m, n), dtype=out_dtype, device=x.device)
    check(lib().msgl_gemm_w4a16(_p(x2), x2.stride(0), _p(w_packed), _p(scales_t), _p(zeros_t), _p(channel), _p(bias),
                                _p(out), n, m, n, k, group, int(nvfp4), _dt(x2), _DT[out_dtype], _stream()),
          "gemm_w4a16")
    _count("gemm_w4a16_nvfp4" if nvfp4 else "gemm_w4a16_int4", "gemm_w4a16_kernel")
    return out.view(*shape[:-1], n)


def gemm_w4a16_status(reset=True) -> int:
    from ._lib import bind, c_i

    bind("msgl_gemm_w4a16_status", c_i, [c_i])
    return int(lib().msgl_gemm_w4a16_status(int(reset)))


def gemm_status(reset=True) -> int:
    return int(lib().msgl_gemm_status(int(reset)))


def gemm_pair_mode(mode: int) -> int:
    """Tile policy of the GEMM family: 0 = CTA-pair kernel (256 x 256 tiles, two SMs per tile)
    above 256 rows, 1 = single-CTA kernel always, 2 = CTA-pair kernel always. Returns the
    previous setting."""
    return int(lib().msgl_gemm_pair_mode(int(mode)))


def gemm_static_weights(on) -> int:
    """Promise that the weight operands of all GEMM calls from now on are model parameters
    (written long before the kernels in flight): the decode GEMMs then fetch their first weight
    tiles while the kernel ahead of them is still running (1), and also request the rest of their
    first work item's weight stream into L2 (2). Returns the previous setting."""
    global STATIC_WEIGHTS
    STATIC_WEIGHTS = bool(on)
    return int(lib().msgl_gemm_static_weights(int(on)))


def set_pdl(on: bool) -> int:
    """Programmatic dependent launch of the library's kernels (on by default; ``MSGL_PDL=0``
    switches it off). Returns the previous setting."""
    return int(lib().msgl_set_pdl(int(on)))


def decode_attention_stages(stages: int) -> None:
    """Depth of the fp8 decode kernel's TMA ring (2-4 stages of 64 tokens)."""
    lib().msgl_attn_decode_stages(int(stages))


def force_general_decode_attention(on: bool) -> None:
    """Route single-query batches through the general attention kernel. Speculative decoding
    sets this: verification rows run on the general kernel, and greedy output is only
    bit-identical to plain decoding when the decode rows take the same code path."""
    lib().msgl_attn_force_general_decode(int(on))


def gemm_fp8_block_status(reset=True) -> int:
    from ._lib import bind, c_i

    bind("msgl_gemm_fp8_block_status", c_i, [c_i])
    return int(lib().msgl_gemm_fp8_block_status(int(reset)))


def attn_status(reset=True) -> int:
    a = int(lib().msgl_attn_status(int(reset)))
    b = int(lib().msgl_attn_tc_status(int(reset)))
    return a or b or int(lib().msgl_talk_status(int(reset)))


# ------------------------------------------------------------------------------------------ sampling
def argmax(logits):
    assert logits.dtype == torch.float32 and logits.stride(-1) == 1
    rows, vocab = logits.shape
    out = torch.empty((rows,), dtype=torch.int32, device=logits.device)
    check(lib().msgl_argmax(_p(logits), _p(out), rows, vocab, logits.stride(0), _stream()), "argmax")
    _count("argmax", "argmax_kernel")
    return out


def sample(logits, temperatures, top_k=None, top_p=None, min_p=None, generator=None, uniform=None):
    assert logits.dtype == torch.float32 and logits.stride(-1) == 1
    rows, vocab = logits.shape
    if uniform is None:
        uniform = torch.rand((rows,), dtype=torch.float32, device=logits.device, generator=generator)
    out = torch.empty((rows,), dtype=torch.int32, device=logits.device)
    check(lib().msgl_sample(_p(logits), logits.stride(0), _p(temperatures), _p(top_k), _p(top_p), _p(min_p),
                            _p(uniform), _p(out), rows, vocab, _stream()), "sample")
    _count("sample", "sample_kernel")
    return out


# ------------------------------------------------------------------------------------------ MoE (composed)
def moe_route(router_logits, top_k, renormalize, scoring="softmax", bias=None, scale=1.0, counts=None, e_start=0,
              e_local=None):
    from . import moe_kernels

    return moe_kernels.moe_route(router_logits, top_k, renormalize, scoring, scale, counts, e_start, e_local, bias)


def moe_forward(x, w13, w2, topk_w, topk_ids, expert_offset=0, counts=None):
    from . import moe_kernels

    return moe_kernels.moe_forward(x, w13, w2, topk_w, topk_ids, expert_offset, counts)


# ------------------------------------------------------------------------------------------ gated delta net
def _bind_gdn():
    from ._lib import bind, c_f, c_i, c_ll, c_p

    if getattr(_bind_gdn, "done", False):
        return
    bind("msgl_gdn_conv1d", c_i, [c_p, c_ll, c_p, c_p, c_p, c_p, c_p, c_p, c_i, c_i, c_i, c_p, c_i, c_p])
    bind("msgl_mamba2_scan", c_i, [c_p, c_p, c_ll, c_p, c_p, c_p, c_p, c_p, c_p, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_f,
                                   c_i, c_p])
    bind("msgl_rms_norm_gate_first", c_i, [c_p, c_p, c_ll, c_p, c_p, c_i, c_i, c_i, c_f, c_i, c_p])
    bind("msgl_relu2", c_i, [c_p, c_p, c_ll, c_i, c_p])
    bind("msgl_gdn_recurrent", c_i, [c_p, c_p, c_p, c_ll, c_p, c_p, c_p, c_p, c_p, c_p, c_p, c_i, c_i, c_i, c_i, c_i, c_i,
                                     c_p])
    bind("msgl_rms_norm_gated", c_i, [c_p, c_p, c_ll, c_i, c_p, c_p, c_i, c_i, c_f, c_i, c_p])
    _bind_gdn.done = True


def gdn_conv1d(x, weight, conv_state, cu_q, slots, has_state, bias=None):
    """Depthwise causal conv (4 taps, optional bias) + SiLU over packed sequences; ``x [T, C]`` may be a
    column slice of a wider projection (row stride = its leading dimension). Updates ``conv_state``."""
    _bind_gdn()
    assert x.dim() == 2 and x.stride(1) == 1 and weight.is_contiguous() and conv_state.is_contiguous()
    t, c = x.shape
    out = torch.empty((t, c), dtype=x.dtype, device=x.device)
    check(lib().msgl_gdn_conv1d(_p(x), x.stride(0), _p(weight), _p(conv_state), _p(cu_q), _p(slots), _p(has_state),
                                _p(out), cu_q.numel() - 1, c, weight.shape[1], _p(bias), _dt(x), _stream()), "gdn_conv1d")
    _count("gdn_conv1d", "gdn_conv1d_kernel")
    return out


def gdn_recurrent(qkv, a, b, a_log, dt_bias, state, cu_q, slots, has_state, hk, hv, dk, dv):
    """Gated delta rule over packed sequences. ``qkv [T, 2*hk*dk + hv*dv]`` (after the convolution),
    ``a, b [T, hv]`` raw gate projections (column slices allowed, same row stride), ``state
    [slots, hv, dk, dv]`` fp32 updated in place. Returns ``[T, hv, dv]``."""
    _bind_gdn()
    assert qkv.is_contiguous() and a.stride(1) == 1 and b.stride(1) == 1 and a.stride(0) == b.stride(0)
    assert state.dtype == torch.float32 and state.is_contiguous()
    t = qkv.shape[0]
    out = torch.empty((t, hv, dv), dtype=qkv.dtype, device=qkv.device)
    check(lib().msgl_gdn_recurrent(_p(qkv), _p(a), _p(b), a.stride(0), _p(a_log), _p(dt_bias), _p(state), _p(cu_q),
                                   _p(slots), _p(has_state), _p(out), cu_q.numel() - 1, hk, hv, dk, dv, _dt(qkv),
                                   _stream()), "gdn_recurrent")
    _count("gdn_recurrent", "gdn_recurrent_kernel")
    return out


def mamba2_scan(xbc, dt, a_log, d_skip, dt_bias, state, cu_q, slots, has_state, heads, groups, head_dim, state_size,
                dt_min=0.0):
    """Selective state-space recurrence over packed sequences. ``xbc [T, H*P + 2*G*N]`` (after the
    convolution: x heads, B groups, C groups), ``dt [T, H]`` raw step sizes (a column slice is fine),
    ``state [slots, H, P, N]`` fp32 updated in place. Returns ``[T, H, P]``."""
    _bind_gdn()
    assert xbc.is_contiguous() and dt.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    t = xbc.shape[0]
    out = torch.empty((t, heads, head_dim), dtype=xbc.dtype, device=xbc.device)
    check(lib().msgl_mamba2_scan(_p(xbc), _p(dt), dt.stride(0), _p(a_log), _p(d_skip), _p(dt_bias), _p(state), _p(cu_q),
                                 _p(slots), _p(has_state), _p(out), cu_q.numel() - 1, heads, groups, head_dim,
                                 state_size, float(dt_min), _dt(xbc), _stream()), "mamba2_scan")
    _count("mamba2_scan", "mamba2_scan_kernel")
    return out


def rms_norm_gate_first(x, z, w, eps, group):
    """``w * norm_group(x * silu(z))``: ``x [T, D]`` contiguous, ``z [T, D]`` (a column slice is fine)."""
    _bind_gdn()
    t, d = x.shape
    assert x.is_contiguous() and z.stride(1) == 1
    out = torch.empty_like(x)
    check(lib().msgl_rms_norm_gate_first(_p(x), _p(z), z.stride(0), _p(w), _p(out), t, d, group, eps, _dt(x), _stream()),
          "rms_norm_gate_first")
    _count("rms_norm_gate_first", "rms_norm_gate_first_kernel")
    return out


def relu2(x):
    _bind_gdn()
    x = x.contiguous()
    out = torch.empty_like(x)
    check(lib().msgl_relu2(_p(x), _p(out), x.numel(), _dt(x), _stream()), "relu2")
    _count("relu2", "relu2_kernel")
    return out


def rms_norm_gated(x, z, w, eps):
    """``norm(x) * w * silu(z)`` per head: ``x [T, heads, D]`` contiguous, ``z [T, heads * D]`` (a column
    slice of a wider projection is fine)."""
    _bind_gdn()
    t, heads, d = x.shape
    assert x.is_contiguous() and z.stride(1) == 1
    out = torch.empty_like(x)
    check(lib().msgl_rms_norm_gated(_p(x), _p(z), z.stride(0), heads, _p(w), _p(out), t * heads, d, eps, _dt(x),
                                    _stream()), "rms_norm_gated")
    _count("rms_norm_gated", "rms_norm_gated_kernel")
    return out


# ------------------------------------------------------------------------------------------ fp32 GEMM
def _bind_latent():
    from ._lib import bind, c_f, c_i, c_ll, c_p

    if hasattr(_bind_latent, "_done"):
        return
    bind("msgl_gemm_f32", c_i, [c_p, c_ll, c_ll, c_p, c_ll, c_ll, c_p, c_ll, c_ll, c_i, c_i, c_i, c_i, c_p, c_ll, c_p])
    bind("msgl_embed_positions", c_i, [c_p] * 5 + [c_i] * 5 + [c_f, c_i, c_p])
    bind("msgl_latent_rope", c_i, [c_p, c_ll, c_ll, c_i, c_i, c_i, c_p, c_p, c_i, c_p, c_ll, c_p, c_p, c_p] + [c_i] * 4
         + [c_f, c_ll, c_i, c_p])
    bind("msgl_norm_conv", c_i, [c_p, c_p, c_p, c_i, c_ll, c_ll, c_p, c_f] + [c_p] * 9 + [c_i] * 7 + [c_p])
    bind("msgl_gelu_erf", c_i, [c_p, c_ll, c_p, c_ll, c_i, c_i, c_i, c_p])
    bind("msgl_latent_norm_store", c_i, [c_p, c_ll, c_p, c_p, c_p, c_i, c_i, c_i, c_f, c_ll, c_i, c_p])
    bind("msgl_head_gemm", c_i, [c_p, c_ll, c_ll, c_p, c_p, c_ll, c_ll, c_i, c_i, c_i, c_i, c_i, c_p, c_p, c_i,
                                 c_p, c_ll, c_p, c_ll, c_p, c_p, c_p, c_i, c_i, c_f, c_ll, c_p])
    bind("msgl_latent_gather", c_i, [c_p] * 5 + [c_i] * 5 + [c_p])
    bind("msgl_attn_prefill_pos", c_i, [c_p, c_ll, c_ll, c_p, c_p, c_i, c_p, c_ll, c_ll, c_p, c_i, c_i, c_i, c_i, c_i, c_i,
                                        c_f, c_p, c_p, c_ll, c_i, c_p])
    bind("msgl_latent_attention", c_i, [c_p, c_p, c_p, c_p, c_i] + [c_p] * 4 + [c_i] * 9 + [c_f, c_p, c_i, c_i, c_p])
    _bind_latent._done = True


def gemm_f32(x, w):
    """``x [M, K] @ w [N, K]^T`` in fp32 on the FMA pipe (no tensor-core mode)."""
    _bind_latent()
    assert x.dim() == 2 and x.stride(1) == 1 and w.is_contiguous() and w.shape[1] == x.shape[1]
    out = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32, device=x.device)
    check(lib().msgl_gemm_f32(_p(x), x.stride(0), 0, _p(w), w.stride(0), 0, _p(out), out.stride(0), 0, x.shape[0],
                              w.shape[0], w.shape[1], 1, None, 0, _stream()), "gemm_f32")
    _count("gemm_f32", "gemm_f32_kernel")
    return out


# ------------------------------------------------------------------------------------------ fp32 residual, input convolutions
def embed_positions(ids, weight, pos, positions, vocab_start=0, vocab_len=None, scale=1.0):
    _bind_latent()
    ids = ids.to(torch.int32) if ids.dtype != torch.int32 else ids
    n = weight.shape[0] if vocab_len is None else vocab_len
    out = torch.empty((ids.numel(), weight.shape[1]), dtype=torch.float32, device=weight.device)
    check(lib().msgl_embed_positions(_p(ids), _p(weight), _p(pos), _p(positions), _p(out), ids.numel(), weight.shape[1],
                                     vocab_start, n, 0 if pos is None else pos.shape[0], scale, _dt(weight), _stream()),
          "embed_positions")
    _count("embed_positions", "embed_positions_kernel")
    return out


def add_scalar_norm_conv(x, delta, gain, eps, w1, w2, state, cu_q, slots, has_state, max_q, out_dtype, out_cols):
    _bind_latent()
    assert x.is_contiguous() and x.dtype == torch.float32
    rows, width = x.shape
    planes, plane_stride, ldd = 0, 0, 0
    if isinstance(delta, SplitPartial):
        delta = delta.planes
        planes, plane_stride, ldd = delta.shape[0], delta.stride(0), delta.stride(1)
    elif delta is not None:
        planes, plane_stride, ldd = 1, 0, delta.stride(0)
    if delta is not None:
        assert delta.dtype == torch.float32 and delta.stride(-1) == 1 and delta.shape[-2] == rows
    x_out = torch.empty_like(x) if delta is not None else x
    y1 = torch.empty((rows, out_cols), dtype=out_dtype, device=x.device)
    y2 = torch.empty_like(y1) if w2 is not None else None
    taps, b = 1, 1
    if w1 is not None:
        taps, b = w1.shape[0], cu_q.numel() - 1
        assert w1.is_contiguous() and w1.dtype == torch.float32 and state.is_contiguous()
        assert state.dtype == torch.float32 and state.shape[1:] == (taps - 1, width)
    # many rows per request: two streaming passes with the row norms in between
    scale = torch.empty(rows, dtype=torch.float32, device=x.device) if w1 is not None and max_q > 16 else None
    check(lib().msgl_norm_conv(_p(x), _p(x_out), _p(delta), planes, plane_stride, ldd, _p(gain), eps, _p(w1), _p(w2),
                               _p(y1), _p(y2), _p(state), _p(cu_q), _p(slots), _p(has_state), _p(scale), rows, width,
                               out_cols, taps, b, int(max_q), _DT[out_dtype], _stream()), "norm_conv")
    _count("add_scalar_norm_conv", "norm_conv_kernel", 1 if scale is None else 2)
    return x_out, y1, y2


def gelu_erf(x, out):
    _bind_latent()
    assert x.stride(1) == 1 and out.stride(1) == 1 and x.shape == out.shape and x.dtype == out.dtype
    check(lib().msgl_gelu_erf(_p(x), x.stride(0), _p(out), out.stride(0), x.shape[0], x.shape[1], _dt(x), _stream()),
          "gelu_erf")
    _count("gelu_erf", "gelu_erf_kernel")
    return out


# ------------------------------------------------------------------------------------------ weighted norm, linear attention
def _bind_linear():
    from ._lib import bind, c_f, c_i, c_ll, c_p

    if hasattr(_bind_linear, "_done"):
        return
    bind("msgl_add_norm", c_i, [c_p, c_p, c_p, c_i, c_ll, c_ll, c_p, c_p, c_i, c_i, c_i, c_f, c_i, c_p, c_f, c_i, c_p])
    bind("msgl_linear_attention", c_i, [c_p, c_p, c_p, c_ll, c_p, c_ll] + [c_p] * 8 + [c_i] * 7
         + [c_f, c_f, c_p, c_p, c_i, c_i, c_i, c_i, c_p])
    bind("msgl_norm_gate", c_i, [c_p, c_p, c_ll, c_p, c_p, c_p, c_ll, c_i, c_i, c_f, c_f, c_i, c_i, c_p])
    _bind_linear._done = True


def add_norm(x, delta, weight, eps, center, out_dtype, out_cols, post=None, mult=1.0):
    _bind_linear()
    assert x.is_contiguous() and x.dtype == torch.float32 and weight.dtype == torch.float32
    rows, width = x.shape
    planes, plane_stride, ldd = 0, 0, 0
    if isinstance(delta, SplitPartial):
        delta = delta.planes
        planes, plane_stride, ldd = delta.shape[0], delta.stride(0), delta.stride(1)
    elif delta is not None:
        planes, ldd = 1, delta.stride(0)
    if delta is not None:
        assert delta.dtype == torch.float32 and delta.stride(-1) == 1 and delta.shape[-2] == rows and delta.shape[-1] >= width
    x_out = torch.empty_like(x) if delta is not None else x
    y = torch.empty((rows, out_cols), dtype=out_dtype, device=x.device)
    check(lib().msgl_add_norm(_p(x), _p(x_out), _p(delta), planes, plane_stride, ldd, _p(weight), _p(y), rows, width,
                              out_cols, eps, int(center), _p(post), mult, _DT[out_dtype], _stream()), "add_norm")
    _count("add_norm", "add_norm_kernel")
    return x_out, y


def linear_attention(q, k, v, state, cu_q, slots, has_state, decay=None, gate=None, tau=1.0, q_scale=1.0, act=False,
                     chunked=False, rope=None):
    """See ``ref.linear_attention``; ``q``, ``k``, ``v`` and the low-rank input are views of the same projected rows, head
    widths multiples of 16. ``chunked``: the tensor-core form where it covers the sizes (16-bit prompts)."""
    _bind_linear()
    t, h, dk = q.shape
    dv = v.shape[2]
    ld = q.stride(0)
    low, up, bias = gate if gate is not None else (None, None, None)
    for x, n in ((q, dk), (k, dk), (v, dv)):
        assert x.stride(2) == 1 and (h == 1 or x.stride(1) == n) and (t == 1 or x.stride(0) == ld) and x.dtype == q.dtype
    assert state.dtype == torch.float32 and state.shape[1:] == (h, dk, dv) and (state.shape[0] == 1 or state[0].is_contiguous())
    if gate is not None:
        assert (t == 1 or low.stride(0) == ld) and low.stride(-1) == 1 and up.is_contiguous() and up.dtype == low.dtype == q.dtype
        assert bias.dtype == torch.float32 and up.shape == (h * dk, low.shape[1])
    cos_sin, positions = rope if rope is not None else (None, None)
    if rope is not None:
        assert cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and positions.dtype == torch.int32
        assert positions.numel() >= t
    out = torch.empty((t, h, dv), dtype=q.dtype, device=q.device)
    check(lib().msgl_linear_attention(
        _p(q), _p(k), _p(v), ld, _p(state), state.stride(0), _p(cu_q), _p(slots), _p(has_state), _p(out), _p(decay), _p(low),
        _p(up), _p(bias), cu_q.numel() - 1, h, dk, dv, 0 if low is None else low.shape[1], int(act), state.shape[0], 1.0 / tau,
        q_scale, _p(cos_sin), _p(positions), 0 if rope is None else cos_sin.shape[1], 0 if rope is None else cos_sin.shape[0],
        int(chunked), _dt(q), _stream()), "linear_attention")
    _count("linear_attention" + ("_chunked" if chunked else ""),
           "linear_attn_chunk_kernel" if chunked and q.dtype == torch.bfloat16 else "linear_attn_recurrent_kernel")
    return out


def norm_gate(o, g, weight, eps, vdim, joint, act, out_cols, total=None, total_heads=0):
    _bind_linear()
    t, h, dv = o.shape
    assert o.is_contiguous() and g.stride(1) == 1 and g.dtype == o.dtype and weight.dtype == torch.float32
    assert out_cols == h * dv and act in ("sigmoid", "silu")
    per_row, group = (1, h * dv) if joint else (h, dv)
    width = (total_heads if joint and total is not None else h if joint else 1) * vdim
    out = torch.empty((t, out_cols), dtype=o.dtype, device=o.device)
    check(lib().msgl_norm_gate(_p(o), _p(g), g.stride(0), _p(weight), _p(total), _p(out), t, per_row, group, float(width), eps,
                               int(act == "silu"), _dt(o), _stream()), "norm_gate")
    _count("norm_gate", "norm_gate_kernel")
    return out


# ------------------------------------------------------------------------------------------ selective scan, norms around a sublayer
def _bind_scan():
    from ._lib import bind, c_f, c_i, c_ll, c_p

    if hasattr(_bind_scan, "_done"):
        return
    bind("msgl_causal_conv_silu", c_i, [c_p, c_ll, c_p, c_p, c_p, c_ll] + [c_p] * 4 + [c_i] * 6 + [c_p])
    bind("msgl_selective_scan", c_i, [c_p] * 6 + [c_ll, c_p, c_p, c_ll, c_p, c_ll] + [c_p] * 4 + [c_i] * 6 + [c_p])
    _bind_scan._done = True


def causal_conv_silu(x, weight, bias, conv_state, cu_q, slots, has_state, max_q=0):
    _bind_scan()
    t, c = x.shape
    assert x.stride(1) == 1 and weight.is_contiguous() and weight.dtype == bias.dtype == torch.float32
    assert conv_state.dtype == x.dtype and conv_state.shape[1:] == (c, weight.shape[1] - 1)
    assert conv_state.shape[2] == 0 or conv_state[0].is_contiguous()
    out = torch.empty((t, c), dtype=x.dtype, device=x.device)
    check(lib().msgl_causal_conv_silu(_p(x), x.stride(0), _p(weight), _p(bias), _p(conv_state), conv_state.stride(0), _p(cu_q),
                                      _p(slots), _p(has_state), _p(out), cu_q.numel() - 1, c, weight.shape[1], max_q or t,
                                      conv_state.shape[0], _dt(x), _stream()), "causal_conv_silu")
    _count("causal_conv_silu", "causal_conv_silu_kernel")
    return out


def selective_scan(x, dt, dt_bias, a, b, c, skip, z, state, cu_q, slots, has_state, chunked=False):
    """See ``ops.selective_scan``; ``b`` and ``c`` are views of the same rows, channels a multiple of 16, states of 4."""
    _bind_scan()
    t, ch = x.shape
    n = a.shape[1]
    assert x.is_contiguous() and dt.is_contiguous() and dt.dtype == torch.float32 and a.is_contiguous() and z.stride(1) == 1
    assert b.stride(1) == c.stride(1) == 1 and b.stride(0) == c.stride(0) and b.dtype == c.dtype == z.dtype == x.dtype
    assert state.dtype == torch.float32 and state.shape[1:] == (1, ch, n) and state[0].is_contiguous()
    for w in (dt_bias, a, skip):
        assert w.dtype == torch.float32
    out = torch.empty((t, ch), dtype=x.dtype, device=x.device)
    check(lib().msgl_selective_scan(
        _p(x), _p(dt), _p(dt_bias), _p(a), _p(b), _p(c), b.stride(0), _p(skip), _p(z), z.stride(0), _p(state), state.stride(0),
        _p(cu_q), _p(slots), _p(has_state), _p(out), cu_q.numel() - 1, ch, n, state.shape[0], int(chunked), _dt(x), _stream()),
        "selective_scan")
    _count("selective_scan" + ("_tiles" if chunked else ""),
           "scan_tiles_kernel" if chunked and x.dtype != torch.float32 else "scan_rows_kernel")
    return out


def residual_step(x, delta, norm, eps, out_dtype, out_cols, pair=None, post=None, history=None, coef=None):
    """See ``ops.residual_step``."""
    from ._lib import bind, c_f, c_i, c_ll, c_p

    if not hasattr(residual_step, "_done"):
        bind("msgl_residual_step", c_i, [c_p, c_p, c_i, c_ll, c_ll, c_p, c_i, c_ll, c_ll] + [c_p] * 5 + [c_i] + [c_p] * 5
             + [c_i] * 3 + [c_f, c_i, c_p])
        residual_step._done = True
    width, rows = norm[0].shape[0], 0
    args = []
    for d in (delta if pair is not None else (delta,)):
        d = d.planes if isinstance(d, SplitPartial) else d.unsqueeze(0)
        rows = d.shape[1]
        assert d.dtype == torch.float32 and d.stride(2) == 1 and d.shape[2] >= width
        args += [_p(d), d.shape[0], d.stride(0), d.stride(1)]
    args += [None, 0, 0, 0] if pair is None else []
    for w in (*norm, *(pair or ()), *(post or ())):
        assert w.dtype == torch.float32 and w.numel() == width
    assert x is None or (x.is_contiguous() and x.dtype == torch.float32 and x.shape == (rows, width))
    n = 0
    if history is not None:
        n, history.count = history.count, history.count + 1
        assert history.rows.is_contiguous() and history.rows.shape[1:] == (rows, width) and n < history.rows.shape[0]
        assert coef is None or (coef.dtype == torch.float32 and coef.numel() == n + 1)
    own = history is None or coef is not None
    x_out = torch.empty((rows, width), dtype=torch.float32, device=norm[0].device) if own else history.rows[n]
    y = torch.empty((rows, out_cols), dtype=out_dtype, device=norm[0].device)
    w0, w1 = pair or (None, None)
    pw, pb = post or (None, None)
    check(lib().msgl_residual_step(
        _p(x), *args, _p(w0), _p(w1), _p(pw), _p(pb), None if history is None else _p(history.rows), n, _p(coef),
        _p(x_out) if own else None, _p(norm[0]), _p(norm[1]), _p(y), rows, width, out_cols, eps, _DT[out_dtype], _stream()),
        "residual_step")
    _count("residual_step", "residual_step_kernel")
    return x_out, y


# ------------------------------------------------------------------------------------------ latent attention
STATIC_WEIGHTS = False


def latent_norm_store(c, weight, rank, eps, rows, out_loc):
    _bind_latent()
    assert c.stride(1) == 1 and rows.is_contiguous() and rows.dtype == c.dtype and weight.dtype == torch.float32
    check(lib().msgl_latent_norm_store(_p(c), c.stride(0), _p(weight), _p(rows), _p(out_loc), c.shape[0], rank,
                                       rows.shape[2], eps, rows.shape[0] * rows.shape[1], _dt(c), _stream()),
          "latent_norm_store")
    _count("latent_norm_store", "latent_norm_store_kernel")


_NO_STORE = (None, 0, None, None, None, 0, 0, 0.0, 0)


def _gate(gate):
    if gate is None:
        return None, 0
    assert gate.shape[1] == 1 or gate.stride(1) == 1
    return _p(gate), gate.stride(0)


def latent_rope(q, dim, dims, cos_sin, positions, store=None):
    """Rotates channels ``dim .. dim + dims`` of the heads ``q [T, H, D]`` (a view) in place. ``store``: ``(raw latents
    [T, width], norm weight, rank, eps, pool rows, out_loc, width of the shared key part)``."""
    _bind_latent()
    assert q.stride(2) == 1 and cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.shape[1] == dims
    stored = (None, 0, None, None, None, q.shape[0], 0, 0, 0, 0.0, 0)
    if store is not None:
        c, weight, rank, eps, rows, out_loc, rot_dim = store
        assert c.stride(1) == 1 and rows.is_contiguous() and rows.dtype == c.dtype == q.dtype and weight.dtype == torch.float32
        stored = (_p(c), c.stride(0), _p(weight), _p(rows), _p(out_loc), q.shape[0], rank, rows.shape[2], rot_dim, eps,
                  rows.shape[0] * rows.shape[1])
    check(lib().msgl_latent_rope(_p(q), q.stride(0), q.stride(1), q.shape[1], dim, dims, _p(cos_sin), _p(positions),
                                 cos_sin.shape[0], *stored, _dt(q), _stream()), "latent_rope")
    _count("latent_rope", "latent_rope_kernel")


def head_gemm(x, w, out=None, store=None, gate=None):
    """``x [T, H, K]`` (any row and head stride), ``w [H, N, K]`` -> ``[T, H, N]``. ``store``: the arguments of
    ``latent_norm_store`` to run in the same launch (16-bit). ``gate [T, H]``: logits of a sigmoid on the result."""
    _bind_latent()
    t, h, k = x.shape
    n = w.shape[1]
    assert x.stride(2) == 1 and w.is_contiguous() and w.shape == (h, n, k) and w.dtype == x.dtype
    if out is None:
        out = torch.empty((t, h, n), dtype=x.dtype, device=x.device)
    assert out.stride(2) == 1 and out.shape == (t, h, n) and out.dtype == x.dtype
    if x.dtype == torch.float32:
        assert store is None
        check(lib().msgl_gemm_f32(_p(x), x.stride(0), x.stride(1), _p(w), k, n * k, _p(out), out.stride(0),
                                  out.stride(1), t, n, k, h, *_gate(gate), _stream()), "head_gemm")
        _count("head_gemm", "gemm_f32_kernel")
        return out
    stored = _NO_STORE
    if store is not None:
        c, norm, rank, eps, rows, out_loc = store
        assert c.stride(1) == 1 and c.shape[0] == t and c.dtype == x.dtype == rows.dtype and norm.dtype == torch.float32
        stored = (_p(c), c.stride(0), _p(norm), _p(rows), _p(out_loc), rank, rows.shape[2], eps,
                  rows.shape[0] * rows.shape[1])
    check(lib().msgl_head_gemm(_p(x), x.stride(0), x.stride(1), _p(w), _p(out), out.stride(0), out.stride(1), t, h, n, k,
                               int(STATIC_WEIGHTS), None, None, 1, *_gate(gate), *stored, _stream()), "head_gemm")
    _count("head_gemm", "head_gemm_kernel")
    return out


class LatentSplit:
    """Attention of a decode step whose key ranges were not merged: ``ws_o [splits, T * H, R]`` (each range's own
    normalised sum) and its log2 weights ``ws_lse [splits, T * H]``; ``head_gemm_combine`` merges them."""

    __slots__ = ("ws_o", "ws_lse", "shape")

    def __init__(self, ws_o, ws_lse, shape) -> None:
        self.ws_o, self.ws_lse, self.shape = ws_o, ws_lse, shape


def head_gemm_combine(x: LatentSplit, w, out, gate=None):
    """The value projection of a split attention: merges the key ranges while it reads them."""
    _bind_latent()
    t, h, k = x.shape
    n = w.shape[1]
    assert w.is_contiguous() and w.shape == (h, n, k) and out.stride(2) == 1 and out.shape == (t, h, n)
    check(lib().msgl_head_gemm(None, 0, 0, _p(w), _p(out), out.stride(0), out.stride(1), t, h, n, k, int(STATIC_WEIGHTS),
                               _p(x.ws_o), _p(x.ws_lse), x.ws_o.shape[0], *_gate(gate), *_NO_STORE, _stream()), "head_gemm")
    _count("head_gemm", "head_gemm_kernel")
    return out


def latent_splits(batch: int, heads: int, rank: int, up_to: int) -> int:
    """Key ranges per query tile of a decode step: one wave of CTAs on the 148 SMs (a wide latent's tiles fill an SM),
    at least two 64-token tiles each."""
    tiles = -(-up_to // 64) + 1
    ctas = batch * -(-heads // 64)
    wave = 148 if rank > 256 else 296
    return int(max(1, min(wave // max(ctas, 1), tiles // 2, 16)))


def latent_attention(q, rows, block_table, cu_q, seq_lens, scale, window, max_q, max_kv, splits=1, merge=True,
                     one_form=False, sink=None):
    """``sink [H]`` fp32: logits only the denominator counts. ``merge=False``: a split result stays a ``LatentSplit``. ``one_form``: the same kernel variant whatever the number
    of rows per request (verification rows must reproduce decode rows bit for bit)."""
    _bind_latent()
    t, h, r = q.shape
    assert q.is_contiguous() and rows.is_contiguous() and rows.shape[2] == r and rows.dtype == q.dtype
    if q.dtype == torch.float32 or r > 576:
        splits = 1
    out = torch.empty_like(q) if merge or splits == 1 else None
    ws_o = ws_l = None
    if splits > 1:
        ws_o = torch.empty((splits, t * h, r), dtype=torch.float32, device=q.device)
        ws_l = torch.empty((splits, t * h), dtype=torch.float32, device=q.device)
    check(lib().msgl_latent_attention(
        _p(q), _p(rows), _p(out), _p(block_table), block_table.stride(0), _p(cu_q), _p(seq_lens), _p(ws_o), _p(ws_l),
        seq_lens.numel(), t, int(max_q), h, r, rows.shape[1], rows.shape[0], int(window), splits, float(scale),
        _p(sink), int(one_form), _dt(q), _stream()), "latent_attention")
    _count("latent_attention", "latent_attention_kernel", 2 if splits > 1 and merge else 1)
    return out if out is not None else LatentSplit(ws_o, ws_l, (t, h, r))


class LatentPrefillPlan:
    """Per-step tables of the expanded prefill: the latents a step can see (each request from the block of 128 that
    holds the far edge of its first row's window) in one dense scratch, and one item per (request, block of 256 query
    positions), longest first. ``reach``: the widest window of the model's layers (0: everything is visible)."""

    __slots__ = ("tables", "n_items", "t_pad", "off_blk", "off_req", "dense")

    def __init__(self, cu_q: np.ndarray, seq_lens: np.ndarray, reach: int, device) -> None:
        cu_q, kv = np.asarray(cu_q, dtype=np.int64), np.asarray(seq_lens, dtype=np.int64)
        b = int(kv.size)
        q_len = cu_q[1:b + 1] - cu_q[:b]
        lo = self._first(kv - q_len, reach)
        pad = (kv - lo + 127) // 128 * 128
        off = np.concatenate([[0], np.cumsum(pad)[:-1]])
        self.t_pad = int(pad.sum())
        n_tiles = (q_len + 255) // 256
        req = np.repeat(np.arange(b), n_tiles)
        qb = np.arange(int(n_tiles.sum())) - np.repeat(np.cumsum(n_tiles) - n_tiles, n_tiles)
        rows = np.minimum(256, q_len[req] - qb * 256)
        pos0 = kv[req] - q_len[req] + qb * 256
        kv0 = self._first(pos0, reach)
        items = np.zeros((req.size, 8), dtype=np.int32)
        items[:, 0] = cu_q[req] + qb * 256
        items[:, 1] = rows
        items[:, 2] = pos0
        items[:, 3] = off[req] + kv0 - lo[req]
        items[:, 4] = (pos0 + rows - 1) // 128 - kv0 // 128 + 1
        items[:, 5] = req
        items[:, 6] = kv0
        items = items[np.argsort(-items[:, 4], kind="stable")]
        blk_req = np.repeat(np.arange(b), pad // 128).astype(np.int32)
        req_info = np.stack([off, kv, lo], axis=1).astype(np.int32).reshape(-1)
        self.n_items = int(items.shape[0])
        self.off_blk = items.size
        self.off_req = self.off_blk + blk_req.size
        self.tables = _upload_tables(np.concatenate([items.reshape(-1), blk_req, req_info]), device)
        self.dense: Optional[Tuple[int, torch.Tensor]] = None      # (pool row, its latents) of the last layer

    @staticmethod
    def _first(pos: np.ndarray, reach: int) -> np.ndarray:
        return np.maximum(pos - reach + 1, 0) // 128 * 128 if reach > 0 else np.zeros_like(pos)

    @staticmethod
    def pays(cu_q: np.ndarray, seq_lens: np.ndarray, reach: int) -> bool:
        """Expanding costs a matrix product over every latent the step can see: worth it when those rows are not many
        more than the step's own, and the step is not a handful of rows."""
        kv = np.asarray(seq_lens, dtype=np.int64)
        q_len = np.diff(np.asarray(cu_q, dtype=np.int64)[:kv.size + 1])
        total = int(q_len.sum())
        lo = LatentPrefillPlan._first(kv - q_len, reach)
        return total >= 64 and int(((kv - lo + 127) // 128 * 128).sum()) <= 4 * total


def latent_prefill_ok(dim: int, vdim: int, scale: float) -> bool:
    return dim <= 128 and vdim <= 128 and dim % 8 == 0 and vdim % 8 == 0 and scale > 0


def latent_prefill(q, expand_k, up_v, rows, row_id, block_table, plan: LatentPrefillPlan, scale, window, out, sink=None,
                   gate=None):
    """Prefill with per-head keys and values expanded from the latents: ``q [T, H, dim]``, ``expand_k [H * dim, R]``,
    ``up_v [H, vdim, R]``, one layer of the latent pool ``rows`` -> ``out [T, H, vdim]``. The values come out of their
    matrix product transposed (``[H * vdim, tokens]``), the layout the tensor core reads them in."""
    _bind_latent()
    t, h, dim = q.shape
    vdim, r = up_v.shape[1], up_v.shape[2]
    assert q.dtype == torch.bfloat16 and rows.is_contiguous() and rows.shape[2] == r
    base = plan.tables.data_ptr()
    if plan.dense is None or plan.dense[0] != row_id:
        dense = torch.empty((plan.t_pad, r), dtype=q.dtype, device=q.device)
        check(lib().msgl_latent_gather(_p(rows), _p(dense), base + 4 * plan.off_blk, base + 4 * plan.off_req,
                                       _p(block_table), block_table.stride(0), rows.shape[1], rows.shape[0], r,
                                       plan.t_pad, _stream()), "latent_gather")
        _count("latent_gather", "latent_gather_kernel")
        plan.dense = (row_id, dense)
    dense = plan.dense[1]
    k = _gemm(KIND_BF16, dense, expand_k, h * dim, r, q.dtype)
    # the latents are the second operand here: no fetch of it ahead of the kernel that gathers them
    static = gemm_static_weights(0)
    try:
        vt = _gemm(KIND_BF16, up_v.view(h * vdim, r), dense, plan.t_pad, r, q.dtype)
    finally:
        gemm_static_weights(static)
    check(lib().msgl_attn_prefill_pos(_p(q), q.stride(0), q.stride(1), _p(k), _p(vt), plan.t_pad, _p(out), out.stride(0),
                                      out.stride(1), base, plan.n_items, t, h, dim, vdim, int(window), float(scale),
                                      _p(sink), *_gate(gate), _dt(q), _stream()), "attn_prefill_pos")
    _count("latent_prefill", "attn_prefill_tc_kernel")
    return out
