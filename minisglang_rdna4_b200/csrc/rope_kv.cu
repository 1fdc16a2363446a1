// Fused per-head QK-RMSNorm + rotary embedding + paged KV store, and a stand-alone KV store.
//
// Replaces the reference's tail_hip.qk_norm_rope / rope / store_kv
// (python/minisgl/layers/attention.py:137-141, python/minisgl/layers/rotary.py:104-129,
// python/minisgl/kvcache/mha_pool.py:189-192) and the upstream store kernel
// (python/minisgl/kernel/csrc/jit/store.cu:25-53) with one pass over the QKV projection:
// q heads are normed, rotated and written to a packed [T, Hq, D] buffer; k heads are normed,
// rotated and scattered into the paged pool; v heads are scattered. The pool layout is
// [pages, Hk, page_size, D]; with fp8 storage a row is divided by its per-head descale and
// saturated to e4m3.
#include "common.cuh"

using namespace msgl;

// One warp per (token, head). The head row is staged in shared memory as fp32.
template <typename T, int D>
__global__ void __launch_bounds__(128) qk_norm_rope_store_kernel(
    const T* __restrict__ qkv, const T* __restrict__ q_w, const T* __restrict__ k_w,
    const int32_t* __restrict__ positions, const float* __restrict__ cos_sin, T* __restrict__ q_out,
    void* __restrict__ k_cache, void* __restrict__ v_cache, const int32_t* __restrict__ out_loc,
    const float* __restrict__ k_scale, const float* __restrict__ v_scale, int hq, int hk, int rot,
    int page_size, float eps, int interleaved, int cache_fp8, int max_pos, int num_slots) {
  pdl_enter();
  __shared__ float rows[4][D];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int token = blockIdx.x;
  const int head = blockIdx.y * 4 + warp;
  const int heads_total = hq + 2 * hk;
  if (head >= heads_total) return;
  constexpr int PER = D / 32;
  float* row = rows[warp];
  const T* src = qkv + (size_t)token * heads_total * D + (size_t)head * D;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    float v = to_float(src[lane * PER + i]);
    row[lane * PER + i] = v;
    ss += v * v;
  }
  const bool is_q = head < hq, is_k = !is_q && head < hq + hk;
  const T* w = is_q ? q_w : k_w;
  if (!(is_q || is_k)) {
    // V head: straight scatter
  } else {
    if (w != nullptr) {
      ss = warp_sum(ss);
      const float rstd = rsqrtf(ss / (float)D + eps);
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        int d = lane * PER + i;
        // the normed value is rounded to T before the rotation, as the unfused ops would
        row[d] = to_float(from_float<T>(row[d] * rstd * to_float(w[d])));
      }
    }
    __syncwarp();
    int pos = positions[token];
    (void)MSGL_OOB(pos, max_pos);
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    const float* cs = cos_sin + (size_t)pos * rot;
    const int half = rot >> 1;
    // each lane rotates pairs p = lane, lane + 32, ...
    for (int p = lane; p < half; p += 32) {
      const float c = cs[p], s = cs[half + p];
      const int i0 = interleaved ? 2 * p : p, i1 = interleaved ? 2 * p + 1 : p + half;
      const float a = row[i0], b = row[i1];
      row[i0] = a * c - b * s;
      row[i1] = b * c + a * s;
    }
  }
  __syncwarp();
  if (is_q) {
    T* dst = q_out + ((size_t)token * hq + head) * D;
#pragma unroll
    for (int i = 0; i < PER; ++i) dst[lane * PER + i] = from_float<T>(row[lane * PER + i]);
    return;
  }
  const int kvh = is_k ? head - hq : head - hq - hk;
  int slot = out_loc[token];
  if (slot >= 0) (void)MSGL_OOB(slot, num_slots);
  if (slot < 0 || slot >= num_slots) return;  // padded row: nothing to store
  const int page = slot / page_size, off = slot % page_size;
  const size_t base = (((size_t)page * hk + kvh) * page_size + off) * D;
  void* cache = is_k ? k_cache : v_cache;
  if (cache_fp8) {
    const float sc = is_k ? k_scale[kvh] : v_scale[kvh];
    uint8_t* dst = (uint8_t*)cache + base;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      dst[lane * PER + i] = float_to_e4m3(to_float(from_float<T>(row[lane * PER + i])) / sc);
  } else {
    T* dst = (T*)cache + base;
#pragma unroll
    for (int i = 0; i < PER; ++i) dst[lane * PER + i] = from_float<T>(row[lane * PER + i]);
  }
}

// E consecutive 16-bit elements as one access (E = 1, 2 or 4)
template <typename T, int E> __device__ __forceinline__ void load_run(const T* p, float (&out)[E]) {
  if constexpr (E == 1) {
    out[0] = to_float(p[0]);
  } else if constexpr (E == 2) {
    typename Pack2<T>::type v = *reinterpret_cast<const typename Pack2<T>::type*>(p);
    float2 f = to_float2(v);
    out[0] = f.x; out[1] = f.y;
  } else {
    uint2 raw = *reinterpret_cast<const uint2*>(p);
    float2 f0 = to_float2(*reinterpret_cast<typename Pack2<T>::type*>(&raw.x));
    float2 f1 = to_float2(*reinterpret_cast<typename Pack2<T>::type*>(&raw.y));
    out[0] = f0.x; out[1] = f0.y; out[2] = f1.x; out[3] = f1.y;
  }
}
template <typename T, int E> __device__ __forceinline__ void store_run(T* p, const float (&in)[E]) {
  if constexpr (E == 1) {
    p[0] = from_float<T>(in[0]);
  } else if constexpr (E == 2) {
    *reinterpret_cast<typename Pack2<T>::type*>(p) = Pack2<T>::make(in[0], in[1]);
  } else {
    typename Pack2<T>::type lo = Pack2<T>::make(in[0], in[1]), hi = Pack2<T>::make(in[2], in[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
}

// Fast path for full rotary (rot == D): no shared memory. A lane owns E = D/64 elements of each
// half of the head (NeoX pairing i <-> i + D/2) or 2E consecutive elements (interleaved pairing),
// so both members of every rotation pair live in the same lane; the per-head RMS statistic is a
// warp reduction.
template <typename T, int D>
__global__ void __launch_bounds__(128) qk_norm_rope_store_fast_kernel(
    const T* __restrict__ qkv, const T* __restrict__ q_w, const T* __restrict__ k_w,
    const int32_t* __restrict__ positions, const float* __restrict__ cos_sin, T* __restrict__ q_out,
    void* __restrict__ k_cache, void* __restrict__ v_cache, const int32_t* __restrict__ out_loc,
    const float* __restrict__ k_scale, const float* __restrict__ v_scale, int hq, int hk, int page_size, float eps,
    int interleaved, int cache_fp8, int max_pos, int num_slots) {
  pdl_enter();
  constexpr int E = D / 64, H2 = D / 2;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int token = blockIdx.x;
  const int head = blockIdx.y * 4 + warp;
  const int heads_total = hq + 2 * hk;
  if (head >= heads_total) return;
  const T* src = qkv + (size_t)token * heads_total * D + (size_t)head * D;
  // element indices owned by this lane: lo[t], hi[t]
  int idx_lo[E], idx_hi[E];
#pragma unroll
  for (int t = 0; t < E; ++t) {
    if (interleaved) { idx_lo[t] = 2 * (E * lane + t); idx_hi[t] = idx_lo[t] + 1; }
    else { idx_lo[t] = E * lane + t; idx_hi[t] = idx_lo[t] + H2; }
  }
  float a[E], b[E];
  float ss = 0.f;
  if (interleaved) {
#pragma unroll
    for (int t = 0; t < E; ++t) {
      a[t] = to_float(src[idx_lo[t]]);
      b[t] = to_float(src[idx_hi[t]]);
    }
  } else {
    load_run<T, E>(src + E * lane, a);
    load_run<T, E>(src + H2 + E * lane, b);
  }
#pragma unroll
  for (int t = 0; t < E; ++t) ss += a[t] * a[t] + b[t] * b[t];
  const bool is_q = head < hq, is_k = !is_q && head < hq + hk;
  if (is_q || is_k) {
    const T* w = is_q ? q_w : k_w;
    if (w != nullptr) {
      ss = warp_sum(ss);
      const float rstd = rsqrtf(ss / (float)D + eps);
#pragma unroll
      for (int t = 0; t < E; ++t) {
        a[t] = to_float(from_float<T>(a[t] * rstd * to_float(w[idx_lo[t]])));
        b[t] = to_float(from_float<T>(b[t] * rstd * to_float(w[idx_hi[t]])));
      }
    }
    int pos = positions[token];
    (void)MSGL_OOB(pos, max_pos);
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    const float* cs = cos_sin + (size_t)pos * D;
#pragma unroll
    for (int t = 0; t < E; ++t) {
      const int p = E * lane + t;
      const float c = cs[p], sn = cs[H2 + p];
      const float x0 = a[t], x1 = b[t];
      a[t] = x0 * c - x1 * sn;
      b[t] = x1 * c + x0 * sn;
    }
  }
  if (is_q) {
    T* dst = q_out + ((size_t)token * hq + head) * D;
    if (interleaved) {
#pragma unroll
      for (int t = 0; t < E; ++t) {
        dst[idx_lo[t]] = from_float<T>(a[t]);
        dst[idx_hi[t]] = from_float<T>(b[t]);
      }
    } else {
      store_run<T, E>(dst + E * lane, a);
      store_run<T, E>(dst + H2 + E * lane, b);
    }
    return;
  }
  const int kvh = is_k ? head - hq : head - hq - hk;
  const int slot = out_loc[token];
  if (slot >= 0) (void)MSGL_OOB(slot, num_slots);
  if (slot < 0 || slot >= num_slots) return;
  const int page = slot / page_size, off = slot % page_size;
  const size_t base = (((size_t)page * hk + kvh) * page_size + off) * D;
  void* cache = is_k ? k_cache : v_cache;
  if (cache_fp8) {
    const float sc = is_k ? k_scale[kvh] : v_scale[kvh];
    uint8_t* dst = (uint8_t*)cache + base;
#pragma unroll
    for (int t = 0; t < E; ++t) {
      dst[idx_lo[t]] = float_to_e4m3(to_float(from_float<T>(a[t])) / sc);
      dst[idx_hi[t]] = float_to_e4m3(to_float(from_float<T>(b[t])) / sc);
    }
  } else {
    T* dst = (T*)cache + base;
#pragma unroll
    for (int t = 0; t < E; ++t) {
      dst[idx_lo[t]] = from_float<T>(a[t]);
      dst[idx_hi[t]] = from_float<T>(b[t]);
    }
  }
}

// Vectorised variant for the common case (head_dim 128, full NeoX rotation): eight lanes own one
// head, each lane holding eight consecutive elements of the low half and the matching eight of
// the high half (one 16-byte load each), so a warp covers four heads; the per-head RMS is a
// reduction over the eight lanes; q leaves as 16-byte stores and fp8 K/V as 8-byte stores.
template <typename T>
__global__ void __launch_bounds__(128) qk_norm_rope_store_vec128_kernel(
    const T* __restrict__ qkv, const T* __restrict__ q_w, const T* __restrict__ k_w,
    const int32_t* __restrict__ positions, const float* __restrict__ cos_sin, T* __restrict__ q_out,
    void* __restrict__ k_cache, void* __restrict__ v_cache, const int32_t* __restrict__ out_loc,
    const float* __restrict__ k_scale, const float* __restrict__ v_scale, int hq, int hk, int page_size, float eps,
    int cache_fp8, int max_pos, int num_slots) {
  pdl_enter();
  constexpr int D = 128, H2 = 64;
  const int token = blockIdx.x;
  const int sub = threadIdx.x & 7;                       // lane within the head's group of eight
  const int head = blockIdx.y * 16 + (threadIdx.x >> 3);
  const int heads_total = hq + 2 * hk;
  const bool live = head < heads_total;
  const int hd = live ? head : heads_total - 1;          // idle groups shadow the last head (no stores)
  const T* src = qkv + (size_t)token * heads_total * D + (size_t)hd * D;
  float a[8], b[8];
  load8(src + sub * 8, a);
  load8(src + H2 + sub * 8, b);
  float ss = 0.f;
#pragma unroll
  for (int t = 0; t < 8; ++t) ss += a[t] * a[t] + b[t] * b[t];
  ss += __shfl_xor_sync(0xffffffffu, ss, 1);
  ss += __shfl_xor_sync(0xffffffffu, ss, 2);
  ss += __shfl_xor_sync(0xffffffffu, ss, 4);
  if (!live) return;
  const bool is_q = head < hq, is_k = !is_q && head < hq + hk;
  if (is_q || is_k) {
    const T* w = is_q ? q_w : k_w;
    if (w != nullptr) {
      const float rstd = rsqrtf(ss / (float)D + eps);
      float wl[8], wh[8];
      load8(w + sub * 8, wl);
      load8(w + H2 + sub * 8, wh);
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        a[t] = to_float(from_float<T>(a[t] * rstd * wl[t]));
        b[t] = to_float(from_float<T>(b[t] * rstd * wh[t]));
      }
    }
    int pos = positions[token];
    (void)MSGL_OOB(pos, max_pos);
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
    const float4* cs = reinterpret_cast<const float4*>(cos_sin + (size_t)pos * D + sub * 8);
    const float4* sn = reinterpret_cast<const float4*>(cos_sin + (size_t)pos * D + H2 + sub * 8);
    const float4 c0 = cs[0], c1 = cs[1], s0 = sn[0], s1 = sn[1];
    const float c[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
    const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const float x0 = a[t], x1 = b[t];
      a[t] = x0 * c[t] - x1 * sv[t];
      b[t] = x1 * c[t] + x0 * sv[t];
    }
  }
  if (is_q) {
    T* dst = q_out + ((size_t)token * hq + head) * D;
    store8(dst + sub * 8, a);
    store8(dst + H2 + sub * 8, b);
    return;
  }
  const int kvh = is_k ? head - hq : head - hq - hk;
  const int slot = out_loc[token];
  if (slot >= 0) (void)MSGL_OOB(slot, num_slots);
  if (slot < 0 || slot >= num_slots) return;
  const int page = slot / page_size, off = slot % page_size;
  const size_t base = (((size_t)page * hk + kvh) * page_size + off) * D;
  void* cache = is_k ? k_cache : v_cache;
  if (cache_fp8) {
    const float sc = is_k ? k_scale[kvh] : v_scale[kvh];
    uint8_t* dst = (uint8_t*)cache + base;
    float ra[8], rb[8];
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      ra[t] = to_float(from_float<T>(a[t])) / sc;   // same rounding and division as the scalar kernel
      rb[t] = to_float(from_float<T>(b[t])) / sc;
    }
    uint2 pa, pb;
    pa.x = (uint32_t)float_to_e4m3(ra[0]) | ((uint32_t)float_to_e4m3(ra[1]) << 8) | ((uint32_t)float_to_e4m3(ra[2]) << 16) |
           ((uint32_t)float_to_e4m3(ra[3]) << 24);
    pa.y = (uint32_t)float_to_e4m3(ra[4]) | ((uint32_t)float_to_e4m3(ra[5]) << 8) | ((uint32_t)float_to_e4m3(ra[6]) << 16) |
           ((uint32_t)float_to_e4m3(ra[7]) << 24);
    pb.x = (uint32_t)float_to_e4m3(rb[0]) | ((uint32_t)float_to_e4m3(rb[1]) << 8) | ((uint32_t)float_to_e4m3(rb[2]) << 16) |
           ((uint32_t)float_to_e4m3(rb[3]) << 24);
    pb.y = (uint32_t)float_to_e4m3(rb[4]) | ((uint32_t)float_to_e4m3(rb[5]) << 8) | ((uint32_t)float_to_e4m3(rb[6]) << 16) |
           ((uint32_t)float_to_e4m3(rb[7]) << 24);
    *reinterpret_cast<uint2*>(dst + sub * 8) = pa;
    *reinterpret_cast<uint2*>(dst + H2 + sub * 8) = pb;
  } else {
    T* dst = (T*)cache + base;
    store8(dst + sub * 8, a);
    store8(dst + H2 + sub * 8, b);
  }
}

MSGL_API int msgl_qk_norm_rope_store(const void* qkv, const void* q_w, const void* k_w, const void* positions,
                                     const void* cos_sin, void* q_out, void* k_cache, void* v_cache,
                                     const void* out_loc, const void* k_scale, const void* v_scale, int tokens,
                                     int hq, int hk, int head_dim, int rot, int page_size, float eps,
                                     int interleaved, int cache_fp8, int max_pos, int num_slots, int dtype,
                                     cudaStream_t stream) {
  if (tokens == 0) return MSGL_OK;
  if (rot > head_dim || rot % 2) return MSGL_BAD_ARG;
 dim3 grid(tokens, (hq + 2 * hk + 3) / 4);
#define LAUNCH(T, D)                                                                                        \
  do {                                                                                                      \
  if (rot == head_dim && D == 128 && !interleaved)                                                          \
    msgl_launch(qk_norm_rope_store_vec128_kernel<T>, dim3(dim3(tokens, (hq + 2 * hk + 15) / 16)), dim3(128), 0, stream, \
        (const T*)qkv, (const T*)q_w, (const T*)k_w, (const int32_t*)positions, (const float*)cos_sin,      \
        (T*)q_out, k_cache, v_cache, (const int32_t*)out_loc, (const float*)k_scale, (const float*)v_scale, \
        hq, hk, page_size, eps, cache_fp8, max_pos, num_slots);                                             \
  else if (rot == head_dim)                                                                                 \
    msgl_launch(qk_norm_rope_store_fast_kernel<T, D>, dim3(grid), dim3(128), 0, stream, \
        (const T*)qkv, (const T*)q_w, (const T*)k_w, (const int32_t*)positions, (const float*)cos_sin,      \
        (T*)q_out, k_cache, v_cache, (const int32_t*)out_loc, (const float*)k_scale, (const float*)v_scale, \
        hq, hk, page_size, eps, interleaved, cache_fp8, max_pos, num_slots);                                \
  else                                                                                                      \
                                                                                        \
  msgl_launch(qk_norm_rope_store_kernel<T, D>, dim3(grid), dim3(128), 0, stream, \
      (const T*)qkv, (const T*)q_w, (const T*)k_w, (const int32_t*)positions, (const float*)cos_sin,        \
      (T*)q_out, k_cache, v_cache, (const int32_t*)out_loc, (const float*)k_scale, (const float*)v_scale,   \
      hq, hk, rot, page_size, eps, interleaved, cache_fp8, max_pos, num_slots);                            \
  } while (0)
  if (dtype == MSGL_BF16) {
    if (head_dim == 128) LAUNCH(__nv_bfloat16, 128);
    else if (head_dim == 64) LAUNCH(__nv_bfloat16, 64);
    else if (head_dim == 256) LAUNCH(__nv_bfloat16, 256);
    else return MSGL_BAD_ARG;
  } else if (dtype == MSGL_F16) {
    if (head_dim == 128) LAUNCH(__half, 128);
    else if (head_dim == 64) LAUNCH(__half, 64);
    else if (head_dim == 256) LAUNCH(__half, 256);
    else return MSGL_BAD_ARG;
  } else {
    return MSGL_BAD_ARG;
  }
#undef LAUNCH
  MSGL_CHECK_LAUNCH("qk_norm_rope_store");
  return MSGL_OK;
}

// ------------------------------------------------------------------------------------------
// stand-alone store: k, v [T, Hk, D] -> paged pool
// ------------------------------------------------------------------------------------------
template <typename T>
__global__ void store_kv_kernel(const T* __restrict__ k, const T* __restrict__ v, void* __restrict__ k_cache,
                                void* __restrict__ v_cache, const int32_t* __restrict__ out_loc,
                                const float* __restrict__ k_scale, const float* __restrict__ v_scale, int hk,
                                int d, int page_size, int cache_fp8, int num_slots) {
  pdl_enter();
  const int token = blockIdx.x;
  const int slot = out_loc[token];
  if (slot >= 0) (void)MSGL_OOB(slot, num_slots);
  if (slot < 0 || slot >= num_slots) return;
  const int page = slot / page_size, off = slot % page_size;
  for (int i = threadIdx.x; i < hk * d; i += blockDim.x) {
    const int h = i / d, e = i % d;
    const size_t dst = (((size_t)page * hk + h) * page_size + off) * d + e;
    const float kv = to_float(k[(size_t)token * hk * d + i]), vv = to_float(v[(size_t)token * hk * d + i]);
    if (cache_fp8) {
      ((uint8_t*)k_cache)[dst] = float_to_e4m3(kv / k_scale[h]);
      ((uint8_t*)v_cache)[dst] = float_to_e4m3(vv / v_scale[h]);
    } else {
      ((T*)k_cache)[dst] = from_float<T>(kv);
      ((T*)v_cache)[dst] = from_float<T>(vv);
    }
  }
}

MSGL_API int msgl_store_kv(const void* k, const void* v, void* k_cache, void* v_cache, const void* out_loc,
                           const void* k_scale, const void* v_scale, int tokens, int hk, int head_dim,
                           int page_size, int cache_fp8, int num_slots, int dtype, cudaStream_t stream) {
  if (tokens == 0) return MSGL_OK;
  if (dtype == MSGL_BF16)
    msgl_launch(store_kv_kernel<__nv_bfloat16>, dim3(tokens), dim3(256), 0, stream, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, k_cache, v_cache, (const int32_t*)out_loc,
        (const float*)k_scale, (const float*)v_scale, hk, head_dim, page_size, cache_fp8, num_slots);
  else if (dtype == MSGL_F16)
    msgl_launch(store_kv_kernel<__half>, dim3(tokens), dim3(256), 0, stream, (const __half*)k, (const __half*)v, k_cache, v_cache, (const int32_t*)out_loc, (const float*)k_scale,
        (const float*)v_scale, hk, head_dim, page_size, cache_fp8, num_slots);
  else
    return MSGL_BAD_ARG;
  MSGL_CHECK_LAUNCH("store_kv");
  return MSGL_OK;
}

// ------------------------------------------------------------------------------------------
// Heads of a layer with a geometry of its own: RMS norm over all query (key) heads together or none, rotation of the
// first `rot` channels in either pairing, division of every query and key head by its root mean square or none, store of
// keys and values. fp32 throughout, rounded once at the end. One CTA per token; rows of a multiple of 64 columns of which
// `dim` count (the others are zero). Two forms: sixteen columns per lane and every head in registers at once (rotated
// channels a multiple of 16), and a warp per head with the rotation through shared memory (any sizes).
// ------------------------------------------------------------------------------------------
namespace {

struct HeadsRopeArgs {
  const void* x;          // [tokens, ld]: hq query heads, then hk keys and hk values when there is a store
  long long ld;
  const float* q_w;       // [hq * D] / [hk * D] weights of the norm over all heads, or null
  const float* k_w;
  const float* totals;    // [tokens, 2] sums of squares over the heads of all ranks, or null
  float q_count, k_count; // channels behind those sums
  const int32_t* positions;
  const float* cos_sin;   // [max_pos, rot], or null
  void* q_out;            // [tokens, hq, D]
  void* k_cache;          // [pages, hk, page_size, D], or null: queries alone
  void* v_cache;
  const int32_t* out_loc;
  int hq, hk, dim, rot, page_size, interleaved, unit, max_pos, num_slots;
  float eps;
};

template <typename T> __device__ __forceinline__ float2 load_pair(const T* p) {
  if constexpr (sizeof(T) == 4) return *reinterpret_cast<const float2*>(p);
  else return to_float2(*reinterpret_cast<const typename Pack2<T>::type*>(p));
}
template <typename T> __device__ __forceinline__ void store_pair(T* p, float a, float b) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float2*>(p) = make_float2(a, b);
  else *reinterpret_cast<typename Pack2<T>::type*>(p) = Pack2<T>::make(a, b);
}

template <typename T, int NP>
__global__ void __launch_bounds__(512) heads_rope_store_kernel(const HeadsRopeArgs a) {
  pdl_enter();
  constexpr int D = 64 * NP;
  extern __shared__ __align__(16) float rows[];       // a rotated row per warp
  __shared__ float part[2][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int token = blockIdx.x;
  const int hk = a.k_cache != nullptr ? a.hk : 0;
  const T* x = reinterpret_cast<const T*>(a.x) + token * a.ld;
  float rq = 1.f, rk = 1.f;
  if (a.q_w != nullptr) {
    float sq = 0.f, sk = 0.f;
    if (a.totals != nullptr) {
      sq = a.totals[2 * token];
      sk = a.totals[2 * token + 1];
    } else {
      for (int h = warp; h < a.hq + hk; h += nw) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const float2 v = load_pair(x + h * D + 64 * i + 2 * lane);
          s = fmaf(v.x, v.x, fmaf(v.y, v.y, s));
        }
        if (h < a.hq) sq += s; else sk += s;
      }
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      if (lane == 0) { part[0][warp] = sq; part[1][warp] = sk; }
      __syncthreads();
      sq = warp_sum(lane < nw ? part[0][lane] : 0.f);
      sk = warp_sum(lane < nw ? part[1][lane] : 0.f);
    }
    rq = 1.f / sqrtf(sq / a.q_count + a.eps);
    if (hk > 0) rk = 1.f / sqrtf(sk / a.k_count + a.eps);
  }
  int pos = a.positions[token];
  if (a.rot > 0) {
    (void)MSGL_OOB(pos, a.max_pos);
    pos = pos < 0 ? 0 : (pos >= a.max_pos ? a.max_pos - 1 : pos);
  }
  const int half = a.rot >> 1;
  const float* cs = a.cos_sin + (size_t)pos * a.rot;
  int slot = -1;
  if (hk > 0) {
    slot = a.out_loc[token];
    if (slot >= 0) (void)MSGL_OOB(slot, a.num_slots);
    if (slot >= a.num_slots) slot = -1;
  }
  float* row = rows + warp * a.rot;
  for (int h = warp; h < a.hq + 2 * hk; h += nw) {
    const bool is_q = h < a.hq, is_v = h >= a.hq + hk;
    if (!is_q && slot < 0) break;            // a padding row: nothing to store
    float v[NP][2];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const float2 p = load_pair(x + h * D + 64 * i + 2 * lane);
      v[i][0] = p.x;
      v[i][1] = p.y;
    }
    if (!is_v) {
      if (a.q_w != nullptr) {
        const float r = is_q ? rq : rk;
        const float* w = is_q ? a.q_w + h * D : a.k_w + (h - a.hq) * D;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const float2 p = load_pair(w + 64 * i + 2 * lane);
          v[i][0] *= r * p.x;
          v[i][1] *= r * p.y;
        }
      }
      if (a.rot > 0 && a.interleaved) {
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int p = 32 * i + lane;
          if (p < half) {
            const float c = cs[p], s = cs[half + p], v0 = v[i][0], v1 = v[i][1];
            v[i][0] = v0 * c - v1 * s;
            v[i][1] = v1 * c + v0 * s;
          }
        }
      } else if (a.rot > 0) {
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int e = 64 * i + 2 * lane;
          if (e < a.rot) *reinterpret_cast<float2*>(row + e) = make_float2(v[i][0], v[i][1]);
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NP; ++i) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int e = 64 * i + 2 * lane + j;
            if (e < a.rot) {
              const bool first = e < half;
              const int p = first ? e : e - half;
              const float c = cs[p], s = cs[half + p];
              v[i][j] = first ? v[i][j] * c - row[e + half] * s : v[i][j] * c + row[p] * s;
            }
          }
        }
      }
      if (a.unit) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) s = fmaf(v[i][0], v[i][0], fmaf(v[i][1], v[i][1], s));
        const float r = 1.f / sqrtf(warp_sum(s) / (float)a.dim + a.eps);
#pragma unroll
        for (int i = 0; i < NP; ++i) { v[i][0] *= r; v[i][1] *= r; }
      }
    }
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(a.q_out) + ((size_t)token * a.hq + h) * D;
    } else {
      const int kvh = is_v ? h - a.hq - hk : h - a.hq;
      dst = reinterpret_cast<T*>(is_v ? a.v_cache : a.k_cache) +
            (((size_t)(slot / a.page_size) * hk + kvh) * a.page_size + slot % a.page_size) * D;
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) store_pair(dst + 64 * i + 2 * lane, v[i][0], v[i][1]);
  }
}

// LPH lanes per head (D = 16 * LPH), NI heads per lane group. A lane has two runs of eight columns, both members of every
// pair among them. A CTA takes tokens in turn; the next one's row is on its way while one is worked on.
template <typename T, int LPH, int NI>
__global__ void __launch_bounds__(384) heads_rope_store_vec_kernel(const HeadsRopeArgs a, int tokens) {
  pdl_enter();
  constexpr int D = 16 * LPH, HPW = 32 / LPH, Q = sizeof(T) / 2;
  __shared__ float part[2][2][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int sub = lane % LPH;
  const int hk = a.k_cache != nullptr ? a.hk : 0, total = a.hq + 2 * hk;
  const int half = a.rot >> 1;
  int col[2], angle;                       // first columns of the runs, first angle
  bool turns;
  if (a.interleaved) {
    col[0] = 16 * sub;
    col[1] = col[0] + 8;
    turns = col[0] < a.rot;
    angle = 8 * sub;
  } else {
    turns = 8 * sub < half;
    col[0] = turns ? 8 * sub : a.rot + 16 * (sub - (half >> 3));
    col[1] = turns ? half + 8 * sub : col[0] + 8;
    angle = 8 * sub;
  }
  uint4 raw[NI][2][Q];
  int pos = 0, slot = -1;
  auto fetch = [&](int token) {
    pos = a.positions[token];
    if (hk > 0) slot = a.out_loc[token];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int h = (i * nw + warp) * HPW + lane / LPH;
      const T* src = reinterpret_cast<const T*>(a.x) + token * a.ld + h * D;
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int j = 0; j < Q; ++j)
          raw[i][r][j] = h < total ? reinterpret_cast<const uint4*>(src + col[r])[j] : make_uint4(0, 0, 0, 0);
    }
  };
  if ((int)blockIdx.x < tokens) fetch(blockIdx.x);
  int buf = 0;
  for (int token = blockIdx.x; token < tokens; token += gridDim.x, buf ^= 1) {
    float cs[8], sn[8];
    if (turns) {
      (void)MSGL_OOB(pos, a.max_pos);
      pos = pos < 0 ? 0 : (pos >= a.max_pos ? a.max_pos - 1 : pos);
      load8(a.cos_sin + (size_t)pos * a.rot + angle, cs);
      load8(a.cos_sin + (size_t)pos * a.rot + half + angle, sn);
    }
    float v[NI][2][8];
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) load8(reinterpret_cast<const T*>(raw[i][r]), v[i][r]);
    int to = slot;
    if (to >= 0) (void)MSGL_OOB(to, a.num_slots);
    if (to >= a.num_slots) to = -1;
    if (token + (int)gridDim.x < tokens) fetch(token + gridDim.x);
    float rq = 1.f, rk = 1.f;
    if (a.q_w != nullptr) {
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int h = (i * nw + warp) * HPW + lane / LPH;
        float s = 0.f;
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
          for (int e = 0; e < 8; ++e) s = fmaf(v[i][r][e], v[i][r][e], s);
        if (h < a.hq) sq += s;
        else if (h < a.hq + hk) sk += s;
        if (h < a.hq + hk) {
          const float* src = h < a.hq ? a.q_w + h * D : a.k_w + (h - a.hq) * D;
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            float w[8];
            load8(src + col[r], w);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[i][r][e] *= w[e];
          }
        }
      }
      if (a.totals != nullptr) {
        sq = a.totals[2 * token];
        sk = a.totals[2 * token + 1];
      } else {
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) { part[buf][0][warp] = sq; part[buf][1][warp] = sk; }
        __syncthreads();
        sq = sk = 0.f;
        for (int w = 0; w < nw; ++w) { sq += part[buf][0][w]; sk += part[buf][1][w]; }
      }
      rq = 1.f / sqrtf(sq / a.q_count + a.eps);
      if (hk > 0) rk = 1.f / sqrtf(sk / a.k_count + a.eps);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int h = (i * nw + warp) * HPW + lane / LPH;
      const bool is_q = h < a.hq, is_v = h >= a.hq + hk;
      if (turns && !is_v) {
        if (a.interleaved) {
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float& v0 = v[i][e >> 2][2 * (e & 3)];
            float& v1 = v[i][e >> 2][2 * (e & 3) + 1];
            const float t = v0;
            v0 = t * cs[e] - v1 * sn[e];
            v1 = v1 * cs[e] + t * sn[e];
          }
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float t = v[i][0][e];
            v[i][0][e] = t * cs[e] - v[i][1][e] * sn[e];
            v[i][1][e] = v[i][1][e] * cs[e] + t * sn[e];
          }
        }
      }
      float scale = is_v ? 1.f : is_q ? rq : rk;
      if (a.unit) {
        float s = 0.f;
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
          for (int e = 0; e < 8; ++e) s = fmaf(v[i][r][e], v[i][r][e], s);
#pragma unroll
        for (int o = 1; o < LPH; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (!is_v) scale /= sqrtf(scale * scale * s / (float)a.dim + a.eps);
      }
      if (h >= total || (!is_q && to < 0)) continue;
      T* dst;
      if (is_q) {
        dst = reinterpret_cast<T*>(a.q_out) + ((size_t)token * a.hq + h) * D;
      } else {
        const int kvh = is_v ? h - a.hq - hk : h - a.hq;
        dst = reinterpret_cast<T*>(is_v ? a.v_cache : a.k_cache) +
              (((size_t)(to / a.page_size) * hk + kvh) * a.page_size + to % a.page_size) * D;
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        if (!is_v && (a.unit || a.q_w != nullptr)) {
#pragma unroll
          for (int e = 0; e < 8; ++e) v[i][r][e] *= scale;
        }
        store8(dst + col[r], v[i][r]);
      }
    }
    __syncwarp();
  }
}

template <typename T, int LPH>
bool launch_heads_rope_vec(const HeadsRopeArgs& a, int tokens, int heads, cudaStream_t stream) {
  const int groups = (heads + 32 / LPH - 1) / (32 / LPH);        // warps' worth of heads
  const int ni = groups <= 12 ? 1 : 2;
  const int warps = (groups + ni - 1) / ni;
  if (warps > 12) return false;
  const dim3 grid(tokens < 148 * 8 ? tokens : 148 * (24 / warps > 1 ? 24 / warps : 1));
  if (ni == 1) msgl_launch(heads_rope_store_vec_kernel<T, LPH, 1>, grid, dim3(32 * warps), 0, stream, a, tokens);
  else msgl_launch(heads_rope_store_vec_kernel<T, LPH, 2>, grid, dim3(32 * warps), 0, stream, a, tokens);
  return true;
}

}  // namespace

MSGL_API int msgl_heads_rope_store(const void* x, long long ld, const void* q_w, const void* k_w, const void* totals,
                                   float q_count, float k_count, const void* positions, const void* cos_sin, int rot,
                                   void* q_out, void* k_cache, void* v_cache, const void* out_loc, int tokens, int hq,
                                   int hk, int width, int dim, int page_size, float eps, int interleaved, int unit,
                                   int max_pos, int num_slots, int dtype, cudaStream_t stream) {
  if (tokens == 0) return MSGL_OK;
  if (rot < 0 || rot % 2 || rot > dim || dim > width || hq <= 0 || ld % 2 || (rot > 0 && cos_sin == nullptr) ||
      (k_cache != nullptr && (hk <= 0 || page_size <= 0 || (q_w != nullptr && k_w == nullptr))))
    return MSGL_BAD_ARG;
  HeadsRopeArgs a{x, ld, (const float*)q_w, (const float*)k_w, (const float*)totals, q_count, k_count,
                  (const int32_t*)positions, (const float*)cos_sin, q_out, k_cache, v_cache, (const int32_t*)out_loc, hq, hk,
                  dim, rot, page_size, interleaved, unit, max_pos, num_slots, eps};
  const int heads = hq + (k_cache != nullptr ? 2 * hk : 0);
  if (rot % 16 == 0 && ld % 8 == 0 && (uintptr_t)x % 16 == 0 && width <= 256) {
    bool done = false;
#define HEADS_ROPE_VEC(T)                                                              \
  done = width == 64    ? launch_heads_rope_vec<T, 4>(a, tokens, heads, stream)         \
         : width == 128 ? launch_heads_rope_vec<T, 8>(a, tokens, heads, stream)        \
         : width == 256 ? launch_heads_rope_vec<T, 16>(a, tokens, heads, stream) : false
    if (dtype == MSGL_BF16) HEADS_ROPE_VEC(__nv_bfloat16);
    else if (dtype == MSGL_F32) HEADS_ROPE_VEC(float);
#undef HEADS_ROPE_VEC
    if (done) {
      MSGL_CHECK_LAUNCH("heads_rope_store");
      return MSGL_OK;
    }
  }
  const int warps = heads < 16 ? heads : 16;
  const size_t smem = interleaved ? 0 : (size_t)warps * rot * sizeof(float);
#define HEADS_ROPE(T, NP) msgl_launch(heads_rope_store_kernel<T, NP>, dim3(tokens), dim3(32 * warps), smem, stream, a)
#define HEADS_ROPE_WIDTHS(T)              \
  do {                                    \
    if (width == 64) HEADS_ROPE(T, 1);    \
    else if (width == 128) HEADS_ROPE(T, 2); \
    else if (width == 256) HEADS_ROPE(T, 4); \
    else if (width == 512) HEADS_ROPE(T, 8); \
    else return MSGL_BAD_ARG;             \
  } while (0)
  if (dtype == MSGL_BF16) HEADS_ROPE_WIDTHS(__nv_bfloat16);
  else if (dtype == MSGL_F32) HEADS_ROPE_WIDTHS(float);
  else return MSGL_BAD_ARG;
#undef HEADS_ROPE_WIDTHS
#undef HEADS_ROPE
  MSGL_CHECK_LAUNCH("heads_rope_store");
  return MSGL_OK;
}
