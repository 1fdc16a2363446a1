// Paged attention in true fp32 (the 32-bit serving mode): grouped-query heads over an fp32 pool, causal, with a sliding
// window or chunks, a soft cap or a distance bias on the scores, a sink in the softmax denominator and a sigmoid gate on the
// output. One CTA per (query row, head), blocks of 128 keys: a thread scores a key, then sums channels. Plain FMA arithmetic,
// blocks counted from the first visible key, so that a row's result depends on nothing but its own keys.
//
// Heads that mix their weights: every head's weights meet the values of every key / value head (a CTA per value head), and
// head_mix_kernel adds them up, out[h] = sum_g talk[h, g] o[g, value head of h]. The attention kernel also has a 16-bit form
// for such layers with sizes that the tensor-core kernels do not take.
#include "common.cuh"

using namespace msgl;

namespace {

constexpr int kKeys = 128, kMaxD = 512;

struct F32AttnArgs {
  const void* q;         // [rows, Hq, D]
  const void* k;         // [pages, Hk, page_size, D]
  const void* v;
  void* out;             // [rows, Hq, D], or [rows, Hq, Hk, D] with every head on all values
  const int32_t* block_table;
  const int32_t* cu_q;
  const int32_t* seq_lens;
  const float* gate;     // [rows, Hq * D] (row stride ldg), or null
  long long ldg;
  int bt_stride, B, Hq, Hk, D, page_size, pages, window, chunk;
  float scale, softcap;
  const float* bias;     // [Hq, reach]: what a score loses at each distance, or null
  int reach;
  const float* sink;     // [Hq] scores that only the denominator counts, or null
};

__device__ __forceinline__ float4 load4f(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4f(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(u.x, u.y, v.x, v.y);
}

// ALL: grid.z value heads
template <typename T, bool ALL>
__global__ void __launch_bounds__(kKeys) paged_attention_f32_kernel(const F32AttnArgs a) {
  pdl_enter();
  __shared__ float q[kMaxD], p[kKeys], scratch[32];
  __shared__ long long at[kKeys];
  const int row = blockIdx.x, head = blockIdx.y, t = threadIdx.x;
  const int hk = head / (a.Hq / a.Hk), hv = ALL ? (int)blockIdx.z : hk;
  T* out = reinterpret_cast<T*>(a.out) + (((size_t)row * a.Hq + head) * (ALL ? a.Hk : 1) + (ALL ? hv : 0)) * a.D;
  int b = 0, hi = a.B;                   // the request of this row
  while (hi - b > 1) {
    const int mid = (b + hi) >> 1;
    if (a.cu_q[mid] <= row) b = mid; else hi = mid;
  }
  if (row < a.cu_q[b] || row >= a.cu_q[b + 1]) {          // padding of a captured batch
    for (int c = t; c < a.D; c += kKeys) out[c] = from_float<T>(0.f);
    return;
  }
  const int pos = a.seq_lens[b] - (a.cu_q[b + 1] - row);
  int lo = 0;
  if (a.window > 0) lo = max(lo, pos - a.window + 1);
  if (a.chunk > 0) lo = max(lo, pos - pos % a.chunk);
  for (int c = t; c < a.D; c += kKeys) q[c] = to_float(reinterpret_cast<const T*>(a.q)[((size_t)row * a.Hq + head) * a.D + c]);
  float acc[kMaxD / kKeys] = {}, m = -INFINITY, l = 0.f;
  for (int k0 = lo; k0 <= pos; k0 += kKeys) {
    const int tok = k0 + t;
    float s = -INFINITY;
    __syncthreads();
    if (tok <= pos) {
      int page = a.block_table[(size_t)b * a.bt_stride + min(tok / a.page_size, a.bt_stride - 1)];
      (void)MSGL_OOB(page, a.pages);
      page = page < 0 ? 0 : (page >= a.pages ? a.pages - 1 : page);
      const long long first = (long long)page * a.Hk * a.page_size + tok % a.page_size;
      at[t] = (first + (long long)hv * a.page_size) * a.D;
      const T* k = reinterpret_cast<const T*>(a.k) + (first + (long long)hk * a.page_size) * a.D;
      float dot = 0.f;
      for (int c = 0; c < a.D; c += 4) {
        const float4 x = load4f(k + c);
        dot = fmaf(q[c], x.x, fmaf(q[c + 1], x.y, fmaf(q[c + 2], x.z, fmaf(q[c + 3], x.w, dot))));
      }
      s = dot * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      if (a.bias != nullptr) s -= a.bias[(size_t)head * a.reach + min(pos - tok, a.reach - 1)];
    }
    const float mn = fmaxf(m, block_max(s, scratch)), alpha = expf(m - mn), e = tok <= pos ? expf(s - mn) : 0.f;
    p[t] = e;
    l = l * alpha + block_sum(e, scratch);               // its barriers also publish p and at
    m = mn;
    const int n = min(kKeys, pos - k0 + 1);
    for (int i = 0; i < kMaxD / kKeys; ++i) {
      const int c = t + i * kKeys;
      if (c >= a.D) break;
      float o = acc[i] * alpha;
      for (int j = 0; j < n; ++j) o = fmaf(p[j], to_float(reinterpret_cast<const T*>(a.v)[at[j] + c]), o);
      acc[i] = o;
    }
  }
  float num = 1.f;
  if (a.sink != nullptr) {
    const float mn = fmaxf(m, a.sink[head]);
    num = expf(m - mn);
    l = l * num + expf(a.sink[head] - mn);
  }
  for (int i = 0; i < kMaxD / kKeys; ++i) {
    const int c = t + i * kKeys;
    if (c >= a.D) break;
    float o = acc[i] * num / l;
    if (a.gate != nullptr) o *= 1.f / (1.f + expf(-a.gate[row * a.ldg + head * a.D + c]));
    out[c] = from_float<T>(o);
  }
}

__device__ __forceinline__ void store4(float* p, const float (&x)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&x)[4]) {
  uint2 q;
  *reinterpret_cast<__nv_bfloat162*>(&q.x) = __floats2bfloat162_rn(x[0], x[1]);
  *reinterpret_cast<__nv_bfloat162*>(&q.y) = __floats2bfloat162_rn(x[2], x[3]);
  *reinterpret_cast<uint2*>(p) = q;
}

// o [rows, H, width] with value head c at columns c * D on; out [rows, H, D]. A thread sums four channels for up to eight
// heads of one value head, so that the rows are read once per eight heads: grid (rows * Hk * D / 4 / 128, parts of a group).
template <typename T>
__global__ void __launch_bounds__(128) head_mix_kernel(const T* __restrict__ o, const float* __restrict__ talk,
                                                       T* __restrict__ out, int rows, int H, int Hk, int D, int width) {
  pdl_enter();
  extern __shared__ float mix[];               // [Hk][H][8]: weights of this part's heads, zero past the group
  const int group = H / Hk, h0 = blockIdx.y * 8, n = min(8, group - h0);
  for (int i = threadIdx.x; i < Hk * H * 8; i += 128) {
    const int k = i & 7, g = (i >> 3) % H, c = (i >> 3) / H;
    mix[i] = k < n ? talk[(size_t)(c * group + h0 + k) * H + g] : 0.f;
  }
  __syncthreads();
  const int per_row = Hk * D / 4;
  const long long id = (long long)blockIdx.x * 128 + threadIdx.x;
  const int row = (int)(id / per_row), col = (int)(id - (long long)row * per_row) * 4, c = col / D;
  if (row >= rows) return;
  const T* src = o + (size_t)row * H * width + col;
  const float* w = mix + (size_t)c * H * 8;
  float acc[8][4] = {};
#pragma unroll 8
  for (int g = 0; g < H; ++g) {
    const float4 x = load4f(src + (size_t)g * width);
    const float4 f0 = *reinterpret_cast<const float4*>(w + g * 8), f1 = *reinterpret_cast<const float4*>(w + g * 8 + 4);
    const float f[8] = {f0.x, f0.y, f0.z, f0.w, f1.x, f1.y, f1.z, f1.w};
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      acc[k][0] = fmaf(f[k], x.x, acc[k][0]);
      acc[k][1] = fmaf(f[k], x.y, acc[k][1]);
      acc[k][2] = fmaf(f[k], x.z, acc[k][2]);
      acc[k][3] = fmaf(f[k], x.w, acc[k][3]);
    }
  }
  T* dst = out + ((size_t)row * H + c * group + h0) * D + col % D;
#pragma unroll
  for (int k = 0; k < 8; ++k)
    if (k < n) store4(dst + (size_t)k * D, acc[k]);
}

}  // namespace

MSGL_API int msgl_paged_attention_f32(const void* q, const void* k, const void* v, void* out, const void* block_table,
                                      int bt_stride, const void* cu_q, const void* seq_lens, int B, int rows, int hq, int hk,
                                      int d, int page_size, int pages, int window, int chunk, float scale, float softcap,
                                      const void* gate, long long ldg, const void* bias, int reach, const void* sink,
                                      int all_values, int dtype, cudaStream_t stream) {
  if (B == 0 || rows == 0) return MSGL_OK;
  if (hk <= 0 || hq % hk || d <= 0 || d % 4 || d > kMaxD || page_size <= 0 || bt_stride < 1) {
    msgl_set_error_text("fp32 attention: heads of up to 512 channels");
    return MSGL_BAD_ARG;
  }
  if ((bias != nullptr && reach <= 0) || (all_values && (gate != nullptr || hk > 65535)) ||
      (dtype != MSGL_F32 && !(dtype == MSGL_BF16 && all_values)))
    return MSGL_BAD_ARG;
  F32AttnArgs a{q, k, v, out, (const int32_t*)block_table, (const int32_t*)cu_q, (const int32_t*)seq_lens, (const float*)gate,
                ldg, bt_stride, B, hq, hk, d, page_size, pages, window, chunk, scale, softcap, (const float*)bias, reach,
                (const float*)sink};
  const dim3 grid(rows, hq, all_values ? hk : 1);
  if (dtype == MSGL_BF16) msgl_launch(paged_attention_f32_kernel<__nv_bfloat16, true>, dim3(grid), dim3(kKeys), 0, stream, a);
  else if (all_values) msgl_launch(paged_attention_f32_kernel<float, true>, dim3(grid), dim3(kKeys), 0, stream, a);
  else msgl_launch(paged_attention_f32_kernel<float, false>, dim3(grid), dim3(kKeys), 0, stream, a);
  MSGL_CHECK_LAUNCH("paged_attention_f32");
  return MSGL_OK;
}

// o [rows, H, width] (value head c at columns c * d on), talk [H, H] fp32 -> out [rows, H, d]
MSGL_API int msgl_head_mix(const void* o, const void* talk, void* out, int rows, int h, int hk, int d, int width, int dtype,
                           cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  const size_t smem = (size_t)h * hk * 32;
  if (hk <= 0 || h % hk || d <= 0 || d % 8 || width % 8 || width < hk * d || smem > 200 * 1024 || (uintptr_t)o % 16 ||
      (uintptr_t)out % 16) {
    msgl_set_error_text("head_mix: widths in eights, up to 6400 pairs of a query and a key / value head");
    return MSGL_BAD_ARG;
  }
  const long long threads = (long long)rows * hk * d / 4;
  const dim3 grid((unsigned)((threads + 127) / 128), (h / hk + 7) / 8);
#define HEAD_MIX(T)                                                                                                     \
  do {                                                                                                                  \
    if (smem > 48 * 1024 &&                                                                                             \
        cudaFuncSetAttribute(head_mix_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) \
      return MSGL_CUDA_ERROR;                                                                                           \
    msgl_launch(head_mix_kernel<T>, dim3(grid), dim3(128), smem, stream, (const T*)o, (const float*)talk, (T*)out, rows, \
                h, hk, d, width);                                                                                       \
  } while (0)
  if (dtype == MSGL_BF16) HEAD_MIX(__nv_bfloat16);
  else if (dtype == MSGL_F32) HEAD_MIX(float);
  else return MSGL_BAD_ARG;
#undef HEAD_MIX
  MSGL_CHECK_LAUNCH("head_mix");
  return MSGL_OK;
}
