// fp32 residual stream of models whose layers read one scalar-gain RMS norm through short causal
// depthwise convolutions: embedding + learned position, residual add + norm + convolutions, exact
// gelu. The convolution of a row needs the normalised rows ahead of it. Steps of few rows per request
// take one kernel, in which a CTA recomputes the rows ahead of its block from the residual instead of
// reading another CTA's output; steps of many rows take a pass for the residual and the row norms and
// a pass for the convolutions. The new residual goes to a second buffer.
#include "common.cuh"

using namespace msgl;

namespace {

template <typename T>
__global__ void __launch_bounds__(256) embed_positions_kernel(const int32_t* __restrict__ ids, const T* __restrict__ w,
                                                              const T* __restrict__ pos,
                                                              const int32_t* __restrict__ positions,
                                                              float* __restrict__ out, int width, int start, int len,
                                                              int n_pos, float scale) {
  pdl_enter();
  const int t = blockIdx.x;
  const int id = ids[t] - start;
  const bool in = id >= 0 && id < len;
  int p = pos != nullptr ? positions[t] : 0;
  const bool has_pos = pos != nullptr && !MSGL_OOB(p, n_pos) && p >= 0 && p < n_pos;
  for (int c = threadIdx.x; c < width; c += 256) {
    float v = in ? to_float(w[(size_t)id * width + c]) * scale : 0.f;
    if (has_pos) v += to_float(pos[(size_t)p * width + c]);
    out[(size_t)t * width + c] = v;
  }
}

struct NormConvArgs {
  const float* x;         // [rows, width] residual
  float* x_out;           // residual + delta (may equal x when there is no delta)
  const float* delta;     // [planes][rows][ldd], summed in ascending order
  int planes;
  long long plane_stride, ldd;
  const float* gain;
  float eps;
  const float* w1;        // [taps, width] or null
  const float* w2;
  void* y1;               // [rows, cols]
  void* y2;
  float* state;           // [slots, taps - 1, width]
  const int32_t* cu_q;
  const int32_t* slots;
  const int32_t* has_state;
  int rows, width, cols, taps, block_rows;
};

// V consecutive floats, zeros unless ``ok``
template <int V> __device__ __forceinline__ void load_vec(const float* p, size_t off, bool ok, float (&q)[V]) {
#pragma unroll
  for (int v = 0; v < V; ++v) q[v] = 0.f;
  if (!ok) return;
  if constexpr (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p + off);
    q[0] = x.x; q[1] = x.y; q[2] = x.z; q[3] = x.w;
  } else {
#pragma unroll
    for (int v = 0; v < V; ++v) q[v] = p[off + v];
  }
}

// V consecutive channels per thread, NC such groups; MT >= taps: the filter is right-aligned in MT taps.
template <typename T, int V, int NC, int MT>
__global__ void __launch_bounds__(1024) norm_conv_kernel(const NormConvArgs a) {
  pdl_enter();
  __shared__ float red[2][32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const bool conv = a.w1 != nullptr;
  const int b = blockIdx.y;
  const int lo = conv ? a.cu_q[b] : 0;
  const int n = (conv ? a.cu_q[b + 1] : a.rows) - lo;
  const int r0 = blockIdx.x * a.block_rows;
  if (r0 >= n) return;
  const int r1 = min(r0 + a.block_rows, n);
  const int hist_n = a.taps - 1;
  const float gain = a.gain[0];

  float hist[NC][V][MT > 1 ? MT - 1 : 1];
  float f1[NC][V][MT], f2[NC][V][MT];
  int ch[NC];
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    ch[g] = (g * blockDim.x + tid) * V;
#pragma unroll
    for (int j = 0; j < MT; ++j) {
      const int src = j - (MT - a.taps);
      float q1[V], q2[V];
      load_vec<V>(a.w1, (size_t)src * a.width + ch[g], conv && src >= 0 && ch[g] < a.width, q1);
      load_vec<V>(a.w2, (size_t)src * a.width + ch[g], a.w2 != nullptr && src >= 0 && ch[g] < a.width, q2);
#pragma unroll
      for (int v = 0; v < V; ++v) { f1[g][v][j] = q1[v]; f2[g][v][j] = q2[v]; }
    }
  }
  float* st = nullptr;
  bool keep = false;
  if (conv && hist_n > 0 && r0 == 0) {
    st = a.state + (size_t)a.slots[b] * a.width * hist_n;
    keep = a.has_state[b] != 0;
  }
#pragma unroll
  for (int g = 0; g < NC; ++g)
#pragma unroll
    for (int j = 0; j < MT - 1; ++j) {
      const int src = j - (MT - 1 - hist_n);
      float q[V];
      load_vec<V>(st, (size_t)src * a.width + ch[g], keep && src >= 0 && ch[g] < a.width, q);
#pragma unroll
      for (int v = 0; v < V; ++v) hist[g][v][j] = q[v];
    }

  auto load_row = [&](int r, float (&x)[NC][V]) {
    const size_t row = (size_t)(lo + r);
#pragma unroll
    for (int g = 0; g < NC; ++g) {
#pragma unroll
      for (int v = 0; v < V; ++v) x[g][v] = 0.f;
      if (ch[g] < a.width) {
        if constexpr (V == 4) {
          const float4 q = *reinterpret_cast<const float4*>(a.x + row * a.width + ch[g]);
          x[g][0] = q.x; x[g][1] = q.y; x[g][2] = q.z; x[g][3] = q.w;
          for (int p = 0; p < a.planes; ++p) {
            const float4 d = *reinterpret_cast<const float4*>(a.delta + p * a.plane_stride + row * a.ldd + ch[g]);
            x[g][0] += d.x; x[g][1] += d.y; x[g][2] += d.z; x[g][3] += d.w;
          }
        } else {
#pragma unroll
          for (int v = 0; v < V; ++v) {
            x[g][v] = a.x[row * a.width + ch[g] + v];
            for (int p = 0; p < a.planes; ++p) x[g][v] += a.delta[p * a.plane_stride + row * a.ldd + ch[g] + v];
          }
        }
      }
    }
  };
  int flip = 0;
  auto rms_scale = [&](const float (&x)[NC][V]) {   // gain / rms of the row; one barrier (alternating scratch)
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < NC; ++g)
#pragma unroll
      for (int v = 0; v < V; ++v) s = fmaf(x[g][v], x[g][v], s);
    s = warp_sum(s);
    if (lane == 0) red[flip][warp] = s;
    __syncthreads();
    s = lane < n_warps ? red[flip][lane] : 0.f;
    s = warp_sum(s);
    flip ^= 1;
    return gain / sqrtf(s / (float)a.width + a.eps);
  };
  auto push = [&](const float (&h)[NC][V]) {
#pragma unroll
    for (int g = 0; g < NC; ++g)
#pragma unroll
      for (int v = 0; v < V; ++v) {
#pragma unroll
        for (int j = 0; j + 1 < MT - 1; ++j) hist[g][v][j] = hist[g][v][j + 1];
        if (MT > 1) hist[g][v][MT - 2 > 0 ? MT - 2 : 0] = h[g][v];
      }
  };
  T* y1 = reinterpret_cast<T*>(a.y1);
  T* y2 = reinterpret_cast<T*>(a.y2);

  float x[NC][V], nx[NC][V];
  const int first = conv ? max(r0 - hist_n, 0) : r0;
  load_row(first, x);
  for (int r = first; r < r1; ++r) {
    if (r + 1 < r1) load_row(r + 1, nx);
    const float sc = rms_scale(x);
    const size_t row = (size_t)(lo + r);
    if (r >= r0) {
#pragma unroll
      for (int g = 0; g < NC; ++g) {
        if (ch[g] < a.width) {
          if (a.x_out != a.x) {
            if constexpr (V == 4)
              *reinterpret_cast<float4*>(a.x_out + row * a.width + ch[g]) =
                  make_float4(x[g][0], x[g][1], x[g][2], x[g][3]);
            else
#pragma unroll
              for (int v = 0; v < V; ++v) a.x_out[row * a.width + ch[g] + v] = x[g][v];
          }
        }
        if (ch[g] < a.cols) {
          float o1[V], o2[V];
#pragma unroll
          for (int v = 0; v < V; ++v) {
            const float h = x[g][v] * sc;
            o1[v] = fmaf(f1[g][v][MT - 1], h, h);
            o2[v] = fmaf(f2[g][v][MT - 1], h, h);
#pragma unroll
            for (int j = 0; j < MT - 1; ++j) {
              o1[v] = fmaf(f1[g][v][j], hist[g][v][j], o1[v]);
              o2[v] = fmaf(f2[g][v][j], hist[g][v][j], o2[v]);
            }
          }
          const size_t off = row * a.cols + ch[g];
          if constexpr (V == 4 && sizeof(T) == 2) {
            uint2 q;
            *reinterpret_cast<typename Pack2<T>::type*>(&q.x) = Pack2<T>::make(o1[0], o1[1]);
            *reinterpret_cast<typename Pack2<T>::type*>(&q.y) = Pack2<T>::make(o1[2], o1[3]);
            *reinterpret_cast<uint2*>(y1 + off) = q;
            if (y2 != nullptr) {
              *reinterpret_cast<typename Pack2<T>::type*>(&q.x) = Pack2<T>::make(o2[0], o2[1]);
              *reinterpret_cast<typename Pack2<T>::type*>(&q.y) = Pack2<T>::make(o2[2], o2[3]);
              *reinterpret_cast<uint2*>(y2 + off) = q;
            }
          } else {
#pragma unroll
            for (int v = 0; v < V; ++v) {
              y1[off + v] = from_float<T>(o1[v]);
              if (y2 != nullptr) y2[off + v] = from_float<T>(o2[v]);
            }
          }
        }
      }
    }
#pragma unroll
    for (int g = 0; g < NC; ++g)
#pragma unroll
      for (int v = 0; v < V; ++v) x[g][v] *= sc;
    push(x);
#pragma unroll
    for (int g = 0; g < NC; ++g)
#pragma unroll
      for (int v = 0; v < V; ++v) x[g][v] = nx[g][v];
  }
  if (st == nullptr) return;
  // The CTA that read the request's tail also writes the new one (recomputing the last rows when they
  // are another CTA's), so no CTA reads a tail that another one is replacing.
  if (r1 < n) {
    for (int r = n - hist_n; r < n; ++r) {
      load_row(r, x);
      const float sc = rms_scale(x);
#pragma unroll
      for (int g = 0; g < NC; ++g)
#pragma unroll
        for (int v = 0; v < V; ++v) x[g][v] *= sc;
      push(x);
    }
  }
#pragma unroll
  for (int g = 0; g < NC; ++g)
#pragma unroll
    for (int j = 0; j < MT - 1; ++j) {
      const int dst = j - (MT - 1 - hist_n);
      if (dst < 0 || ch[g] >= a.width) continue;
      float* p = st + (size_t)dst * a.width + ch[g];
      if constexpr (V == 4)
        *reinterpret_cast<float4*>(p) = make_float4(hist[g][0][j], hist[g][1][j], hist[g][2][j], hist[g][3][j]);
      else
#pragma unroll
        for (int v = 0; v < V; ++v) p[v] = hist[g][v][j];
    }
}

// Prefill form, two streaming passes. First a warp per row: residual add and gain / rms (one float per row). Then a
// thread per four channels walks down kRows rows; the rows ahead of its block are read back from the new residual, so
// no CTA waits for another. width and cols multiples of 4.
constexpr int kRows = 16;

__global__ void __launch_bounds__(256) residual_rms_kernel(const NormConvArgs a, float* __restrict__ scale) {
  pdl_enter();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= a.rows) return;
  const float* src = a.x + (size_t)row * a.width;
  const float* add = a.delta + (size_t)row * a.ldd;
  float* dst = a.x_out + (size_t)row * a.width;
  float s = 0.f;
#pragma unroll 4
  for (int c = lane * 4; c < a.width; c += 128) {
    float4 x = *reinterpret_cast<const float4*>(src + c);
    if (a.planes > 0) {
      for (int p = 0; p < a.planes; ++p) {
        const float4 d = *reinterpret_cast<const float4*>(add + p * a.plane_stride + c);
        x.x += d.x; x.y += d.y; x.z += d.z; x.w += d.w;
      }
      *reinterpret_cast<float4*>(dst + c) = x;
    }
    s = fmaf(x.x, x.x, s);
    s = fmaf(x.y, x.y, s);
    s = fmaf(x.z, x.z, s);
    s = fmaf(x.w, x.w, s);
  }
  s = warp_sum(s);
  if (lane == 0) scale[row] = a.gain[0] / sqrtf(s / (float)a.width + a.eps);
}

// x_out holds the residual; grid (cols / 1024, row blocks, requests).
template <typename T, int MT>
__global__ void __launch_bounds__(256) conv_rows_kernel(const NormConvArgs a, const float* __restrict__ scale) {
  pdl_enter();
  const int b = blockIdx.z;
  const int lo = a.cu_q[b], n = a.cu_q[b + 1] - lo;
  const int r0 = blockIdx.y * kRows, c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (r0 >= n || c >= a.cols) return;
  const int r1 = min(r0 + kRows, n), hist_n = a.taps - 1;
  const bool in = c < a.width;
  float* st = r0 == 0 && hist_n > 0 ? a.state + (size_t)a.slots[b] * a.width * hist_n : nullptr;
  const bool keep = st != nullptr && a.has_state[b] != 0;
  T* y1 = reinterpret_cast<T*>(a.y1) + c;
  T* y2 = a.y2 != nullptr ? reinterpret_cast<T*>(a.y2) + c : nullptr;
  auto row_h = [&](int r, float (&h)[4]) {
    const float4 x = in ? *reinterpret_cast<const float4*>(a.x_out + (size_t)(lo + r) * a.width + c)
                        : make_float4(0.f, 0.f, 0.f, 0.f);
    const float sc = scale[lo + r];
    h[0] = x.x * sc; h[1] = x.y * sc; h[2] = x.z * sc; h[3] = x.w * sc;
  };
  // hist[MT - taps .. MT - 2]: the rows ahead; hist[MT - 1]: the row itself
  float f1[MT][4], f2[MT][4], hist[MT][4];
#pragma unroll
  for (int j = 0; j < MT; ++j) {
    const int src = j - (MT - a.taps);
    float4 q1 = make_float4(0.f, 0.f, 0.f, 0.f), q2 = q1, q3 = q1;
    if (in && src >= 0) {
      q1 = *reinterpret_cast<const float4*>(a.w1 + (size_t)src * a.width + c);
      if (y2 != nullptr) q2 = *reinterpret_cast<const float4*>(a.w2 + (size_t)src * a.width + c);
      if (keep && src < hist_n) q3 = *reinterpret_cast<const float4*>(st + (size_t)src * a.width + c);
    }
    f1[j][0] = q1.x; f1[j][1] = q1.y; f1[j][2] = q1.z; f1[j][3] = q1.w;
    f2[j][0] = q2.x; f2[j][1] = q2.y; f2[j][2] = q2.z; f2[j][3] = q2.w;
    hist[j][0] = q3.x; hist[j][1] = q3.y; hist[j][2] = q3.z; hist[j][3] = q3.w;
    if (r0 > 0 && src >= 0 && src < hist_n) row_h(r0 - hist_n + src, hist[j]);
  }
#pragma unroll 4
  for (int r = r0; r < r1; ++r) {
    row_h(r, hist[MT - 1]);
    float o1[4], o2[4];
#pragma unroll
    for (int v = 0; v < 4; ++v) {
      o1[v] = o2[v] = hist[MT - 1][v];
#pragma unroll
      for (int j = 0; j < MT; ++j) {
        o1[v] = fmaf(f1[j][v], hist[j][v], o1[v]);
        o2[v] = fmaf(f2[j][v], hist[j][v], o2[v]);
      }
    }
    const size_t off = (size_t)(lo + r) * a.cols;
    if constexpr (sizeof(T) == 2) {
      uint2 q;
      *reinterpret_cast<typename Pack2<T>::type*>(&q.x) = Pack2<T>::make(o1[0], o1[1]);
      *reinterpret_cast<typename Pack2<T>::type*>(&q.y) = Pack2<T>::make(o1[2], o1[3]);
      *reinterpret_cast<uint2*>(y1 + off) = q;
      if (y2 != nullptr) {
        *reinterpret_cast<typename Pack2<T>::type*>(&q.x) = Pack2<T>::make(o2[0], o2[1]);
        *reinterpret_cast<typename Pack2<T>::type*>(&q.y) = Pack2<T>::make(o2[2], o2[3]);
        *reinterpret_cast<uint2*>(y2 + off) = q;
      }
    } else {
      *reinterpret_cast<float4*>(y1 + off) = make_float4(o1[0], o1[1], o1[2], o1[3]);
      if (y2 != nullptr) *reinterpret_cast<float4*>(y2 + off) = make_float4(o2[0], o2[1], o2[2], o2[3]);
    }
#pragma unroll
    for (int j = 0; j + 1 < MT; ++j)
#pragma unroll
      for (int v = 0; v < 4; ++v) hist[j][v] = hist[j + 1][v];
  }
  if (st == nullptr || !in) return;
  // the thread that read this part of the tail also writes the new one, whichever block the last rows are in
#pragma unroll
  for (int j = 0; j + 1 < MT; ++j) {
    const int dst = j - (MT - a.taps);
    if (dst < 0) continue;
    if (r1 < n) row_h(n - hist_n + dst, hist[j]);
    *reinterpret_cast<float4*>(st + (size_t)dst * a.width + c) =
        make_float4(hist[j][0], hist[j][1], hist[j][2], hist[j][3]);
  }
}

template <typename T, int V, int NC>
void launch_norm_conv(const NormConvArgs& a, dim3 grid, int threads, cudaStream_t s) {
  if (a.taps <= 1)
    msgl_launch(norm_conv_kernel<T, V, NC, 1>, grid, dim3(threads), 0, s, a);
  else if (a.taps <= 4)
    msgl_launch(norm_conv_kernel<T, V, NC, 4>, grid, dim3(threads), 0, s, a);
  else if (a.taps <= 8)
    msgl_launch(norm_conv_kernel<T, V, NC, 8>, grid, dim3(threads), 0, s, a);
  else
    msgl_launch(norm_conv_kernel<T, V, NC, 32>, grid, dim3(threads), 0, s, a);
}

template <typename T>
int norm_conv_typed(NormConvArgs a, float* scale, int B, int max_q, cudaStream_t s) {
  const bool conv = a.w1 != nullptr;
  // enough rows per CTA to make the recomputed rows cheap (and at least taps - 1 of them)
  a.block_rows = conv ? (a.taps > 8 ? 32 : 16) : 1;
  const int n = conv ? max_q : a.rows;
  dim3 grid((n + a.block_rows - 1) / a.block_rows, conv ? B : 1);
  const bool vec = a.width % 4 == 0 && a.cols % 4 == 0 && a.ldd % 4 == 0 && (uintptr_t)a.delta % 16 == 0;
  const int per = vec ? 4 : 1;
  const int groups = (a.cols + per - 1) / per;
  if (vec && conv && scale != nullptr && a.taps <= 8 && n <= 65535 * kRows) {
    msgl_launch(residual_rms_kernel, dim3((a.rows + 7) / 8), dim3(256), 0, s, a, scale);
    const dim3 conv_grid((a.cols + 1023) / 1024, (n + kRows - 1) / kRows, B);
    if (a.taps <= 4)
      msgl_launch(conv_rows_kernel<T, 4>, conv_grid, dim3(256), 0, s, a, scale);
    else
      msgl_launch(conv_rows_kernel<T, 8>, conv_grid, dim3(256), 0, s, a, scale);
    MSGL_CHECK_LAUNCH("norm_conv_rows");
    return MSGL_OK;
  }
  const int nc = (groups + 1023) / 1024;
  const int threads = ((groups + nc - 1) / nc + 31) / 32 * 32;
  if (vec) {
    if (nc == 1) launch_norm_conv<T, 4, 1>(a, grid, threads, s);
    else if (nc == 2) launch_norm_conv<T, 4, 2>(a, grid, threads, s);
    else if (nc <= 4) launch_norm_conv<T, 4, 4>(a, grid, threads, s);
    else return MSGL_BAD_ARG;
  } else {
    if (nc == 1) launch_norm_conv<T, 1, 1>(a, grid, threads, s);
    else if (nc <= 4) launch_norm_conv<T, 1, 4>(a, grid, threads, s);
    else return MSGL_BAD_ARG;
  }
  MSGL_CHECK_LAUNCH("norm_conv");
  return MSGL_OK;
}

// erf by formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions (absolute error at
// most 1.5e-7): far below what a 16-bit result keeps. The fp32 form calls erff.
__device__ __forceinline__ float erf_as(float x) {
  const float ax = fabsf(x);
  const float t = __fdividef(1.f, fmaf(0.3275911f, ax, 1.f));
  float p = fmaf(1.061405429f, t, -1.453152027f);
  p = fmaf(p, t, 1.421413741f);
  p = fmaf(p, t, -0.284496736f);
  p = fmaf(p, t, 0.254829592f);
  return copysignf(1.f - p * t * __expf(-ax * ax), x);
}

// Exact gelu of [rows, n] with row strides; n a multiple of the vector width.
template <typename T>
__global__ void __launch_bounds__(256) gelu_erf_kernel(const T* __restrict__ x, long long ldx, T* __restrict__ out,
                                                       long long ldo, int n) {
  pdl_enter();
  constexpr int V = 16 / sizeof(T);
  const int c = (blockIdx.y * 256 + threadIdx.x) * V;
  if (c >= n) return;
  const long long r = blockIdx.x;
  float v[V];
  if constexpr (sizeof(T) == 2) {
    load8(x + r * ldx + c, v);
  } else {
    const float4 q = *reinterpret_cast<const float4*>(x + r * ldx + c);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
#pragma unroll
  for (int e = 0; e < V; ++e) {
    const float z = v[e] * 0.70710678118654752f;
    v[e] = 0.5f * v[e] * (1.f + (sizeof(T) == 2 ? erf_as(z) : erff(z)));
  }
  if constexpr (sizeof(T) == 2)
    store8(out + r * ldo + c, v);
  else
    *reinterpret_cast<float4*>(out + r * ldo + c) = make_float4(v[0], v[1], v[2], v[3]);
}

}  // namespace

MSGL_API int msgl_embed_positions(const void* ids, const void* w, const void* pos, const void* positions, void* out,
                                  int rows, int width, int start, int len, int n_pos, float scale, int dtype,
                                  cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
#define EMB(T)                                                                                                      \
  msgl_launch(embed_positions_kernel<T>, dim3(rows), dim3(256), 0, stream, (const int32_t*)ids, (const T*)w,        \
              (const T*)pos, (const int32_t*)positions, (float*)out, width, start, len, n_pos, scale)
  if (dtype == MSGL_BF16) EMB(__nv_bfloat16);
  else if (dtype == MSGL_F32) EMB(float);
  else return MSGL_BAD_ARG;
#undef EMB
  MSGL_CHECK_LAUNCH("embed_positions");
  return MSGL_OK;
}

MSGL_API int msgl_norm_conv(const void* x, void* x_out, const void* delta, int planes, long long plane_stride,
                            long long ldd, const void* gain, float eps, const void* w1, const void* w2, void* y1,
                            void* y2, void* state, const void* cu_q, const void* slots, const void* has_state, void* scale,
                            int rows, int width, int cols, int taps, int B, int max_q, int dtype, cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (taps < 1 || taps > 32 || cols < width || (planes > 0 && x == x_out)) return MSGL_BAD_ARG;
  if (w1 != nullptr && (B <= 0 || max_q <= 0)) return MSGL_BAD_ARG;
  NormConvArgs a{(const float*)x, (float*)x_out, (const float*)delta, planes, plane_stride, ldd, (const float*)gain, eps,
                 (const float*)w1, (const float*)w2, y1, y2, (float*)state, (const int32_t*)cu_q,
                 (const int32_t*)slots, (const int32_t*)has_state, rows, width, cols, taps, 0};
  if (dtype == MSGL_BF16) return norm_conv_typed<__nv_bfloat16>(a, (float*)scale, B, max_q, stream);
  if (dtype == MSGL_F32) return norm_conv_typed<float>(a, (float*)scale, B, max_q, stream);
  return MSGL_BAD_ARG;
}

MSGL_API int msgl_gelu_erf(const void* x, long long ldx, void* out, long long ldo, int rows, int n, int dtype,
                           cudaStream_t stream) {
  if (rows <= 0 || n <= 0) return rows == 0 || n == 0 ? MSGL_OK : MSGL_BAD_ARG;
  const int v = dtype == MSGL_BF16 ? 8 : 4;
  if (n % v || ldx % v || ldo % v || (uintptr_t)x % 16 || (uintptr_t)out % 16) return MSGL_BAD_ARG;
  dim3 grid(rows, (n / v + 255) / 256);
  if (dtype == MSGL_BF16)
    msgl_launch(gelu_erf_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)x, ldx,
                (__nv_bfloat16*)out, ldo, n);
  else if (dtype == MSGL_F32)
    msgl_launch(gelu_erf_kernel<float>, grid, dim3(256), 0, stream, (const float*)x, ldx, (float*)out, ldo, n);
  else
    return MSGL_BAD_ARG;
  MSGL_CHECK_LAUNCH("gelu_erf");
  return MSGL_OK;
}
