"""Op entry points used by layers.

A CUDA tensor is served by the hand-written sm_100a kernels in ``ops.cuda`` (which raise if
the native library is missing: there is no silent eager fallback on a GPU). A CPU tensor is
served by the fp32 PyTorch restatements in ``ops.ref``: that path is the numerics oracle and
runs the CPU plumbing configuration.
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from . import ref


def _cuda():
    from . import cuda

    return cuda


# ---------------------------------------------------------------------------- elementwise
def embedding(ids, weight, vocab_start: int = 0, vocab_len: Optional[int] = None):
    if weight.is_cuda:
        return _cuda().embedding(ids, weight, vocab_start, vocab_len)
    return ref.embedding(ids, weight, vocab_start, vocab_len)


def rms_norm(x, w, eps: float, plus_one: bool = False):
    if x.is_cuda:
        return _cuda().rms_norm(x, w, eps, plus_one)
    return ref.rms_norm(x, w, eps, plus_one)


def rms_norm_add(x, residual, w, eps: float, plus_one: bool = False):
    """``residual += x`` in place; returns ``norm(residual) * w``."""
    if x.is_cuda:
        return _cuda().rms_norm_add(x, residual, w, eps, plus_one)
    return ref.rms_norm_add(x, residual, w, eps, plus_one)


def rms_norm_quant(x, w, eps: float, residual=None, plus_one: bool = False):
    """Norm (optionally after ``residual += x``) with a per-token e4m3 producer:
    returns ``(q, scale)`` (python/minisgl/layers/norm.py:134-168)."""
    if x.is_cuda:
        return _cuda().rms_norm_quant(x, w, eps, residual, plus_one)
    y = ref.rms_norm(x, w, eps, plus_one) if residual is None else ref.rms_norm_add(x, residual, w, eps, plus_one)
    return ref.per_token_quant_fp8(y)


def per_token_quant_fp8(x):
    if x.is_cuda:
        return _cuda().per_token_quant_fp8(x)
    return ref.per_token_quant_fp8(x)


def per_group_quant_fp8(x, group: int = 128):
    if x.is_cuda:
        return _cuda().per_group_quant_fp8(x, group)
    return ref.per_group_quant_fp8(x, group)


def silu_and_mul(x):
    if x.is_cuda:
        return _cuda().act_and_mul(x, "silu")
    return ref.silu_and_mul(x)


def gelu_and_mul(x, tanh: bool = False):
    if x.is_cuda:
        return _cuda().act_and_mul(x, "gelu_tanh" if tanh else "gelu")
    return ref.gelu_and_mul(x, tanh)


def silu_and_mul_quant(x):
    """SiLU(gate)·up followed by per-token e4m3 quantisation: ``(q, scale)``."""
    if x.is_cuda:
        return _cuda().silu_and_mul_quant(x)
    return ref.per_token_quant_fp8(ref.silu_and_mul(x))


# ---------------------------------------------------------------------------- attention side
def qk_norm_rope_store(qkv, q_w, k_w, positions, cos_sin, num_q_heads: int, num_kv_heads: int,
                       head_dim: int, rotary_dim: int, eps: float, k_cache, v_cache, out_loc,
                       k_scale=None, v_scale=None, interleaved: bool = False):
    """Fused per-head QK RMSNorm + rotary embedding + KV scatter.

    ``qkv`` ``[T, (Hq + 2 Hk) * D]``. Returns the rotated queries ``[T, Hq, D]``; K and V are
    written to the paged pool at ``out_loc`` (cast or scaled to e4m3 when scales are given).
    Replaces the reference's ``qk_norm_rope`` + ``store_kv`` pair
    (python/minisgl/layers/attention.py:137-141, python/minisgl/kvcache/mha_pool.py:189-192).
    """
    if qkv.is_cuda:
        return _cuda().qk_norm_rope_store(qkv, q_w, k_w, positions, cos_sin, num_q_heads, num_kv_heads,
                                          head_dim, rotary_dim, eps, k_cache, v_cache, out_loc,
                                          k_scale, v_scale, interleaved)
    qs, ks = num_q_heads * head_dim, num_kv_heads * head_dim
    q, k, v = qkv.split([qs, ks, ks], dim=-1)
    q, k = ref.qk_norm_rope(q, k, q_w, k_w, positions, cos_sin, head_dim, rotary_dim, eps, interleaved)
    ref.store_kv(k, v, k_cache, v_cache, out_loc, k_scale, v_scale)
    return q.reshape(-1, num_q_heads, head_dim)


def heads_rope_store(x, heads: int, kv_heads: int, width: int, dim: int, positions, cos_sin, interleaved: bool,
                     eps: float, q_w=None, k_w=None, totals=None, unit: bool = False, store=None):
    """Norms and rotation of projected query and key heads, and the store of keys and values, in one pass.

    ``x [T, ld]``: ``heads`` queries and, with ``store = (k_cache, v_cache, out_loc)``, ``kv_heads`` keys and as many
    values, each ``width`` columns of which ``dim`` count (values may use more). ``q_w`` / ``k_w`` (fp32, as wide as the
    columns): RMS norm over all heads together first; ``totals = (sums [T, 2], q count, k count)`` where other ranks hold
    some of them. Then the rotation (``cos_sin`` None: none), then, with ``unit``, every head divided by its root mean
    square. Returns the queries ``[T, heads, width]``."""
    fn = _cuda().heads_rope_store if x.is_cuda else ref.heads_rope_store
    return fn(x, heads, kv_heads, width, dim, positions, cos_sin, interleaved, eps, q_w, k_w, totals, unit, store)


def q_norm_rope(q, q_w, positions, cos_sin, num_q_heads: int, head_dim: int, rotary_dim: int, eps: float,
                interleaved: bool = False):
    """Per-head RMSNorm + rotary embedding of the queries alone ``[T, Hq * D]`` → ``[T, Hq, D]``: the form a
    layer takes that reads another layer's K/V (Gemma-4's shared layers) and so has nothing to store."""
    if q.is_cuda:
        raise NotImplementedError("no kernel for the query-only norm + rotary step of a layer that shares K/V")
    dummy_k = q[:, :head_dim]
    out, _ = ref.qk_norm_rope(q, dummy_k, q_w, q_w, positions, cos_sin, head_dim, rotary_dim, eps, interleaved)
    return out.reshape(-1, num_q_heads, head_dim)


def store_kv(k, v, k_cache, v_cache, out_loc, k_scale=None, v_scale=None):
    if k.is_cuda:
        return _cuda().store_kv(k, v, k_cache, v_cache, out_loc, k_scale, v_scale)
    return ref.store_kv(k, v, k_cache, v_cache, out_loc, k_scale, v_scale)


def paged_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale: float, *, causal: bool = True,
                    window: int = 0, mask=None, k_scale=None, v_scale=None, max_q: int = 0,
                    max_kv: int = 0, decode: bool = False, workspace=None, splits=None, mask_window: int = 0,
                    chunk: int = 0, softcap: float = 0.0, gate=None, bias=None, sink=None, talk=None):
    if q.is_cuda:
        return _cuda().paged_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale,
                                       causal=causal, window=window, mask=mask, k_scale=k_scale,
                                       v_scale=v_scale, max_q=max_q, max_kv=max_kv, decode=decode,
                                       workspace=workspace, splits=splits, mask_window=mask_window, chunk=chunk,
                                       softcap=softcap, gate=gate, bias=bias, sink=sink, talk=talk)
    return ref.paged_attention(q, k_cache, v_cache, block_table, cu_q, seq_lens, scale, causal, window,
                               mask, k_scale, v_scale, mask_window, chunk, softcap, gate, bias, sink, talk)


# ---------------------------------------------------------------------------- GEMMs
def gemm(x, w, bias=None, out_dtype: Optional[torch.dtype] = None):
    """``x @ w.T (+ bias)`` with 16-bit operands and fp32 accumulation."""
    if x.is_cuda:
        return _cuda().gemm(x, w, bias, out_dtype)
    return ref.gemm(x, w, bias, out_dtype)


def gemm_w8a8(x_q, x_scale, w_q, w_scale, out_dtype=torch.bfloat16, bias=None):
    if x_q.is_cuda:
        return _cuda().gemm_w8a8(x_q, x_scale, w_q, w_scale, out_dtype, bias)
    return ref.gemm_w8a8(x_q, x_scale, w_q, w_scale, out_dtype, bias)


def gemm_w4a8_mxfp4(x_q, x_scale, w_packed, w_sf, sf_atoms=None, out_dtype=torch.bfloat16, bias=None):
    if x_q.is_cuda:
        return _cuda().gemm_w4a8_mxfp4(x_q, x_scale, w_packed, sf_atoms, out_dtype, bias)
    return ref.gemm_w4a8_mxfp4(x_q, x_scale, w_packed, w_sf, out_dtype, bias)


def gemm_fp8_block(x_q, x_scale, w_q, w_scale, out_dtype=torch.bfloat16):
    if x_q.is_cuda:
        return _cuda().gemm_fp8_block(x_q, x_scale, w_q, w_scale, out_dtype)
    return ref.gemm_fp8_block(x_q, x_scale, w_q, w_scale, 128, out_dtype)


# ---------------------------------------------------------------------------- gated delta net
def gdn_conv1d(x, weight, conv_state, cu_q, slots, has_state, bias=None):
    if x.is_cuda:
        return _cuda().gdn_conv1d(x, weight, conv_state, cu_q, slots, has_state, bias)
    return ref.causal_conv1d(x, weight, conv_state, cu_q, slots, has_state, bias)


def mamba2_scan(xbc, dt, a_log, d_skip, dt_bias, state, cu_q, slots, has_state, heads: int, groups: int,
                head_dim: int, state_size: int, dt_min: float = 0.0):
    """Selective state-space recurrence on the rows ``xbc = [x heads ‖ B groups ‖ C groups]`` left by the
    convolution (python/minisgl/mamba2/)."""
    if xbc.is_cuda:
        return _cuda().mamba2_scan(xbc, dt, a_log, d_skip, dt_bias, state, cu_q, slots, has_state, heads, groups,
                                   head_dim, state_size, dt_min)
    t = xbc.shape[0]
    x, b, c = xbc.split([heads * head_dim, groups * state_size, groups * state_size], dim=-1)
    return ref.mamba2_scan(x.reshape(t, heads, head_dim), dt, b.reshape(t, groups, state_size),
                           c.reshape(t, groups, state_size), a_log, d_skip, dt_bias, state, cu_q, slots, has_state,
                           dt_min)


def rms_norm_gate_first(x, z, w, eps: float, group: int):
    if x.is_cuda:
        return _cuda().rms_norm_gate_first(x, z, w, eps, group)
    return ref.rms_norm_gate_first(x, z, w, eps, group)


def relu2(x):
    if x.is_cuda:
        return _cuda().relu2(x)
    return ref.relu2(x)


def gdn_recurrent(qkv, a, b, a_log, dt_bias, state, cu_q, slots, has_state, hk: int, hv: int, dk: int, dv: int):
    """Gated delta rule on the rows ``qkv = [q heads ‖ k heads ‖ v heads]`` left by the convolution."""
    if qkv.is_cuda:
        return _cuda().gdn_recurrent(qkv, a, b, a_log, dt_bias, state, cu_q, slots, has_state, hk, hv, dk, dv)
    t = qkv.shape[0]
    q, k, v = qkv.split([hk * dk, hk * dk, hv * dv], dim=-1)
    g, beta = ref.gdn_gates(a, b, a_log, dt_bias)
    return ref.gdn_recurrent(q.reshape(t, hk, dk), k.reshape(t, hk, dk), v.reshape(t, hv, dv), g, beta, state,
                             cu_q, slots, has_state)


def rms_norm_gated(x, z, w, eps: float):
    if x.is_cuda:
        return _cuda().rms_norm_gated(x, z, w, eps)
    return ref.rms_norm_gated(x, z.reshape(x.shape), w, eps)


# ---------------------------------------------------------------------------- fp32 residual, latent attention
def embed_positions(ids, weight, pos, positions, vocab_start: int = 0, vocab_len: Optional[int] = None,
                    scale: float = 1.0):
    if weight.is_cuda:
        return _cuda().embed_positions(ids, weight, pos, positions, vocab_start, vocab_len, scale)
    return ref.embed_positions(ids, weight, pos, positions, vocab_start, vocab_len, scale)


def add_scalar_norm_conv(x, delta, gain, eps: float, w1, w2, state, cu_q, slots, has_state, max_q: int, out_dtype,
                         out_cols: int):
    """Residual add, scalar-gain RMS norm and one or two short causal convolutions in one pass:
    ``(new residual, y1, y2)``. ``delta`` may be the unreduced K ranges of a GEMM (``SplitPartial``)."""
    if x.is_cuda:
        return _cuda().add_scalar_norm_conv(x, delta, gain, eps, w1, w2, state, cu_q, slots, has_state, max_q,
                                            out_dtype, out_cols)
    return ref.add_scalar_norm_conv(x, delta, gain, eps, w1, w2, state, cu_q, slots, has_state, out_dtype, out_cols)


def gelu_erf(x, out):
    """Exact gelu of ``x [T, N]`` into ``out [T, N]`` (any row stride)."""
    if x.is_cuda:
        return _cuda().gelu_erf(x, out)
    return ref.gelu_erf(x, out)


def latent_norm_store(c, weight, rank: int, eps: float, rows, out_loc):
    if c.is_cuda:
        return _cuda().latent_norm_store(c, weight, rank, eps, rows, out_loc)
    return ref.latent_norm_store(c, weight, rank, eps, rows, out_loc)


def latent_rope(q, dim: int, dims: int, cos_sin, positions, store=None):
    """Rotates the rotary channels of the query heads in place and, with ``store``, norms, rotates and stores the step's
    latents in the same launch."""
    if q.is_cuda:
        return _cuda().latent_rope(q, dim, dims, cos_sin, positions, store)
    return ref.latent_rope(q, dim, dims, cos_sin, positions, store)


def head_gemm(x, w, out=None, store=None, gate=None):
    if x.is_cuda:
        return _cuda().head_gemm(x, w, out, store, gate)
    assert store is None
    return ref.head_gemm(x, w, out, gate)


def latent_attention(q, rows, block_table, cu_q, seq_lens, scale: float, window: int, max_q: int, max_kv: int,
                     splits: int = 1, one_form: bool = False, sink=None):
    if q.is_cuda:
        return _cuda().latent_attention(q, rows, block_table, cu_q, seq_lens, scale, window, max_q, max_kv, splits,
                                        one_form=one_form, sink=sink)
    return ref.latent_attention(q, rows, block_table, cu_q, seq_lens, scale, window, sink)


# ---------------------------------------------------------------------------- weighted norm, decaying linear attention
def add_norm(x, delta, weight, eps: float, center: bool, out_dtype, out_cols: int, post=None, mult: float = 1.0):
    """Residual add and norm (layer norm without a bias, or RMS) in one pass: ``(new residual, y)``. ``delta`` may be
    the unreduced K ranges of a GEMM (``SplitPartial``). ``post``: weight of an RMS norm that ``delta`` takes before it
    is multiplied by ``mult`` and added."""
    if x.is_cuda:
        return _cuda().add_norm(x, delta, weight, eps, center, out_dtype, out_cols, post, mult)
    return ref.add_norm(x, delta, weight, eps, center, out_dtype, out_cols, post, mult)


def linear_attention(q, k, v, state, cu_q, slots, has_state, decay=None, gate=None, tau: float = 1.0,
                     q_scale: float = 1.0, act: bool = False, chunked: bool = False, rope=None):
    """``chunked``: the step may take the tensor-core form (prompts); otherwise every row takes the recurrent one.
    ``rope = (cos_sin, positions)``: q and k are rotated first, neighbouring channels as pairs, in fp32."""
    if q.is_cuda:
        return _cuda().linear_attention(q, k, v, state, cu_q, slots, has_state, decay, gate, tau, q_scale, act, chunked,
                                        rope)
    return ref.linear_attention(q, k, v, state, cu_q, slots, has_state, decay, gate, tau, q_scale, act, rope)


def norm_gate(o, g, weight, eps: float, vdim: int, joint: bool, act: str, out_cols: int, total=None,
              total_heads: int = 0):
    if o.is_cuda:
        return _cuda().norm_gate(o, g, weight, eps, vdim, joint, act, out_cols, total, total_heads)
    return ref.norm_gate(o, g, weight, eps, vdim, joint, act, out_cols, total, total_heads)


# ---------------------------------------------------------------------------- selective scan, norms around a sublayer
def causal_conv_silu(x, weight, bias, conv_state, cu_q, slots, has_state, max_q: int = 0):
    """A filter per channel over the current and earlier rows of a sequence (last tap: the current one), bias, silu.
    ``x [T, C]``, ``weight [C, taps]`` and ``bias [C]`` fp32, ``conv_state [slots, C, taps - 1]``, updated in place."""
    if x.is_cuda:
        return _cuda().causal_conv_silu(x, weight, bias, conv_state, cu_q, slots, has_state, max_q)
    return ref.causal_conv_silu(x, weight, bias, conv_state, cu_q, slots, has_state)


def selective_scan(x, dt, dt_bias, a, b, c, skip, z, state, cu_q, slots, has_state, chunked: bool = False):
    """``S <- exp(dt a) S + dt x B``, ``y = S C + skip x`` per channel with ``dt`` the softplus of ``dt + dt_bias``; returns
    ``y silu(z)``. ``chunked``: the step may take the form for prompts."""
    fn = _cuda().selective_scan if x.is_cuda else ref.selective_scan
    return fn(x, dt, dt_bias, a, b, c, skip, z, state, cu_q, slots, has_state, chunked)


def residual_step(x, delta, norm, eps: float, out_dtype, out_cols: int, pair=None, post=None, history=None, coef=None):
    """The end of a sublayer and the norm of the next, in one pass: ``(new residual, y [T, out_cols])``.

    ``delta`` (fp32 rows, possibly unreduced K ranges; with ``pair = (w, w')`` two of them): the sublayer's output, or half
    the sum of two RMS-normed and weighted ones. It takes the layer norm ``post`` (weight, bias) and is added to ``x`` (None:
    zero). ``history`` (``layers.residual_norm.LayerHistory``): the sum is a layer's result and joins it; with ``coef``
    the residual that goes on is the sum of ``coef[j]`` times result j. ``y``: the layer norm ``norm`` of it."""
    fn = _cuda().residual_step if norm[0].is_cuda else ref.residual_step
    return fn(x, delta, norm, eps, out_dtype, out_cols, pair, post, history, coef)


def clamped_glu(x, limit: float, alpha: float):
    if x.is_cuda:
        return _cuda().act_and_mul(x, "clamped", alpha, limit)
    return ref.clamped_glu(x, limit, alpha)


# ---------------------------------------------------------------------------- sampling
def argmax(logits):
    if logits.is_cuda:
        return _cuda().argmax(logits)
    return logits.float().argmax(-1).to(torch.int32)


def sample(logits, temperatures, top_k=None, top_p=None, min_p=None, generator=None, uniform=None):
    if logits.is_cuda:
        return _cuda().sample(logits, temperatures, top_k, top_p, min_p, generator, uniform)
    return ref.sample(logits, temperatures, top_k, top_p, min_p, generator, uniform)


# ---------------------------------------------------------------------------- MoE
def moe_route(router_logits, top_k: int, renormalize: bool, scoring: str = "softmax", bias=None,
              scale: float = 1.0):
    if router_logits.is_cuda:
        return _cuda().moe_route(router_logits, top_k, renormalize, scoring, bias, scale)
    return ref.moe_route(router_logits, top_k, renormalize, scoring, bias, scale)


def experts_partial32(x, w13, w2, topk_w, topk_ids, limit: float, alpha: float, shared=None, shared_gate=None,
                      counts=None, act: str = "clamped", on_input: bool = False):
    """fp32 sum of the routed experts and a shared one (behind the sigmoid of ``shared_gate`` where given), for an fp32
    residual stream. ``on_input``: the weights multiply the experts' inputs."""
    if x.is_cuda:
        from . import moe_kernels

        return moe_kernels.experts_partial32(x, w13, w2, topk_w, topk_ids, limit, alpha, shared, shared_gate, counts, act,
                                             on_input)
    return ref.experts_partial32(x, w13, w2, topk_w, topk_ids, limit, alpha, shared, shared_gate, act, on_input)


def moe_forward(x, w13, w2, topk_w, topk_ids, expert_offset: int = 0):
    if x.is_cuda:
        return _cuda().moe_forward(x, w13, w2, topk_w, topk_ids, expert_offset)
    return ref.moe_forward(x, w13, w2, topk_w, topk_ids, expert_offset)


def moe_forward_plain(x, w1, w2, topk_w, topk_ids, expert_offset: int = 0, counts=None, act: str = "relu2"):
    if x.is_cuda:
        from . import moe_kernels

        return moe_kernels.moe_forward_plain(x, w1, w2, topk_w, topk_ids, expert_offset, counts, act)
    return ref.moe_forward_plain(x, w1, w2, topk_w, topk_ids, expert_offset, act)


__all__ = [n for n in dir() if not n.startswith("_")]
