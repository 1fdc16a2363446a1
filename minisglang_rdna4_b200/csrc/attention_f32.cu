// Paged attention in true fp32 (the 32-bit serving mode): grouped-query heads over an fp32 pool, causal, with a sliding
// window or chunks, a soft cap on the scores and a sigmoid gate on the output. One CTA per (query row, head), blocks of 128
// keys: a thread scores a key, then sums channels. Plain FMA arithmetic, blocks counted from the first visible key, so
// that a row's result depends on nothing but its own keys.
#include "common.cuh"

using namespace msgl;

namespace {

constexpr int kKeys = 128, kMaxD = 512;

struct F32AttnArgs {
  const float* q;        // [rows, Hq, D]
  const float* k;        // [pages, Hk, page_size, D]
  const float* v;
  float* out;            // [rows, Hq, D]
  const int32_t* block_table;
  const int32_t* cu_q;
  const int32_t* seq_lens;
  const float* gate;     // [rows, Hq * D] (row stride ldg), or null
  long long ldg;
  int bt_stride, B, Hq, Hk, D, page_size, pages, window, chunk;
  float scale, softcap;
};

__global__ void __launch_bounds__(kKeys) paged_attention_f32_kernel(const F32AttnArgs a) {
  pdl_enter();
  __shared__ float q[kMaxD], p[kKeys], scratch[32];
  __shared__ long long at[kKeys];
  const int row = blockIdx.x, head = blockIdx.y, t = threadIdx.x;
  const int hk = head / (a.Hq / a.Hk);
  float* out = a.out + ((size_t)row * a.Hq + head) * a.D;
  int b = 0, hi = a.B;                   // the request of this row
  while (hi - b > 1) {
    const int mid = (b + hi) >> 1;
    if (a.cu_q[mid] <= row) b = mid; else hi = mid;
  }
  if (row < a.cu_q[b] || row >= a.cu_q[b + 1]) {          // padding of a captured batch
    for (int c = t; c < a.D; c += kKeys) out[c] = 0.f;
    return;
  }
  const int pos = a.seq_lens[b] - (a.cu_q[b + 1] - row);
  int lo = 0;
  if (a.window > 0) lo = max(lo, pos - a.window + 1);
  if (a.chunk > 0) lo = max(lo, pos - pos % a.chunk);
  for (int c = t; c < a.D; c += kKeys) q[c] = a.q[((size_t)row * a.Hq + head) * a.D + c];
  float acc[kMaxD / kKeys] = {}, m = -INFINITY, l = 0.f;
  for (int k0 = lo; k0 <= pos; k0 += kKeys) {
    const int tok = k0 + t;
    float s = -INFINITY;
    __syncthreads();
    if (tok <= pos) {
      int page = a.block_table[(size_t)b * a.bt_stride + min(tok / a.page_size, a.bt_stride - 1)];
      (void)MSGL_OOB(page, a.pages);
      page = page < 0 ? 0 : (page >= a.pages ? a.pages - 1 : page);
      at[t] = (((long long)page * a.Hk + hk) * a.page_size + tok % a.page_size) * a.D;
      const float* k = a.k + at[t];
      float dot = 0.f;
      for (int c = 0; c < a.D; c += 4) {
        const float4 x = *reinterpret_cast<const float4*>(k + c);
        dot = fmaf(q[c], x.x, fmaf(q[c + 1], x.y, fmaf(q[c + 2], x.z, fmaf(q[c + 3], x.w, dot))));
      }
      s = dot * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
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
      for (int j = 0; j < n; ++j) o = fmaf(p[j], a.v[at[j] + c], o);
      acc[i] = o;
    }
  }
  for (int i = 0; i < kMaxD / kKeys; ++i) {
    const int c = t + i * kKeys;
    if (c >= a.D) break;
    float o = acc[i] / l;
    if (a.gate != nullptr) o *= 1.f / (1.f + expf(-a.gate[row * a.ldg + head * a.D + c]));
    out[c] = o;
  }
}

}  // namespace

MSGL_API int msgl_paged_attention_f32(const void* q, const void* k, const void* v, void* out, const void* block_table,
                                      int bt_stride, const void* cu_q, const void* seq_lens, int B, int rows, int hq, int hk,
                                      int d, int page_size, int pages, int window, int chunk, float scale, float softcap,
                                      const void* gate, long long ldg, cudaStream_t stream) {
  if (B == 0 || rows == 0) return MSGL_OK;
  if (hk <= 0 || hq % hk || d <= 0 || d % 4 || d > kMaxD || page_size <= 0 || bt_stride < 1) {
    msgl_set_error_text("fp32 attention: heads of up to 512 channels");
    return MSGL_BAD_ARG;
  }
  F32AttnArgs a{(const float*)q, (const float*)k, (const float*)v, (float*)out, (const int32_t*)block_table,
                (const int32_t*)cu_q, (const int32_t*)seq_lens, (const float*)gate, ldg, bt_stride, B, hq, hk, d, page_size,
                pages, window, chunk, scale, softcap};
  msgl_launch(paged_attention_f32_kernel, dim3(rows, hq), dim3(kKeys), 0, stream, a);
  MSGL_CHECK_LAUNCH("paged_attention_f32");
  return MSGL_OK;
}
