// Norm of an fp32 residual stream with a weight per channel: residual += delta, then layer norm without a bias (the
// variance is the mean of the squared deviations, taken in a second pass over registers) or RMS norm. delta may be the
// unreduced K ranges of a split GEMM. With a post weight, what is added is mult times the RMS norm of delta. One CTA
// per row.
#include "common.cuh"

using namespace msgl;

namespace {

struct AddNormArgs {
  const float* x;         // [rows, width]
  float* x_out;           // residual + delta (x itself when there is no delta)
  const float* delta;     // [planes][rows][ldd], summed in ascending order
  int planes;
  long long plane_stride, ldd;
  const float* w;
  void* y;                // [rows, cols], zero past the width
  int width, cols;
  float eps;
  const float* post_w;    // POST: weight of the norm of delta
  float mult;
};

// V consecutive channels per thread, NC such groups.
template <typename T, int V, int NC, bool CENTER, bool POST>
__global__ void __launch_bounds__(1024) add_norm_kernel(const AddNormArgs a) {
  pdl_enter();
  __shared__ float scratch[32];
  const size_t row = blockIdx.x;
  float x[NC][V];
  float s = 0.f;
  float d[POST ? NC : 1][V];
  if constexpr (POST) {
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const int c = (g * blockDim.x + threadIdx.x) * V;
#pragma unroll
      for (int v = 0; v < V; ++v) d[g][v] = 0.f;
      if (c < a.width) {
        for (int p = 0; p < a.planes; ++p) {
          const float* src = a.delta + p * a.plane_stride + row * a.ldd + c;
          if constexpr (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(src);
            d[g][0] += q.x; d[g][1] += q.y; d[g][2] += q.z; d[g][3] += q.w;
          } else {
            d[g][0] += *src;
          }
        }
      }
#pragma unroll
      for (int v = 0; v < V; ++v) s = fmaf(d[g][v], d[g][v], s);
    }
    const float r = a.mult / sqrtf(block_sum(s, scratch) / (float)a.width + a.eps);
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const int c = (g * blockDim.x + threadIdx.x) * V;
#pragma unroll
      for (int v = 0; v < V; ++v) d[g][v] *= c < a.width ? r * a.post_w[c + v] : 0.f;
    }
    s = 0.f;
  }
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * blockDim.x + threadIdx.x) * V;
    const bool in = c < a.width;
#pragma unroll
    for (int v = 0; v < V; ++v) x[g][v] = 0.f;
    if (in) {
      if constexpr (V == 4) {
        float4 q = *reinterpret_cast<const float4*>(a.x + row * a.width + c);
        if constexpr (POST) {
          q.x += d[g][0]; q.y += d[g][1]; q.z += d[g][2]; q.w += d[g][3];
        } else {
          for (int p = 0; p < a.planes; ++p) {
            const float4 d = *reinterpret_cast<const float4*>(a.delta + p * a.plane_stride + row * a.ldd + c);
            q.x += d.x; q.y += d.y; q.z += d.z; q.w += d.w;
          }
        }
        if (a.planes > 0) *reinterpret_cast<float4*>(a.x_out + row * a.width + c) = q;
        x[g][0] = q.x; x[g][1] = q.y; x[g][2] = q.z; x[g][3] = q.w;
      } else {
        float q = a.x[row * a.width + c];
        if constexpr (POST) q += d[g][0];
        else
          for (int p = 0; p < a.planes; ++p) q += a.delta[p * a.plane_stride + row * a.ldd + c];
        if (a.planes > 0) a.x_out[row * a.width + c] = q;
        x[g][0] = q;
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) s += CENTER ? x[g][v] : x[g][v] * x[g][v];
  }
  s = block_sum(s, scratch);
  float mean = 0.f;
  if constexpr (CENTER) {
    mean = s / (float)a.width;
    s = 0.f;
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const bool in = (g * blockDim.x + threadIdx.x) * V < a.width;
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const float d = in ? x[g][v] - mean : 0.f;
        s = fmaf(d, d, s);
      }
    }
    s = block_sum(s, scratch);
  }
  const float rs = 1.f / sqrtf(s / (float)a.width + a.eps);
  T* y = reinterpret_cast<T*>(a.y) + row * a.cols;
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * blockDim.x + threadIdx.x) * V;
    if (c >= a.cols) continue;
    float o[V];
#pragma unroll
    for (int v = 0; v < V; ++v) o[v] = c < a.width ? (x[g][v] - mean) * rs * a.w[c + v] : 0.f;
    if constexpr (V == 4 && sizeof(T) == 2) {
      uint2 q;
      *reinterpret_cast<typename Pack2<T>::type*>(&q.x) = Pack2<T>::make(o[0], o[1]);
      *reinterpret_cast<typename Pack2<T>::type*>(&q.y) = Pack2<T>::make(o[2], o[3]);
      *reinterpret_cast<uint2*>(y + c) = q;
    } else if constexpr (V == 4) {
      *reinterpret_cast<float4*>(y + c) = make_float4(o[0], o[1], o[2], o[3]);
    } else {
      y[c] = from_float<T>(o[0]);
    }
  }
}

template <typename T, bool CENTER, bool POST> int add_norm_typed(const AddNormArgs& a, int rows, cudaStream_t s) {
  const bool vec = a.width % 4 == 0 && a.cols % 4 == 0 && a.ldd % 4 == 0 && a.plane_stride % 4 == 0 &&
                   (uintptr_t)a.delta % 16 == 0;
  const int groups = (a.cols + (vec ? 3 : 0)) / (vec ? 4 : 1);
  // few rows: as many threads per row as there are vectors; many rows: fewer, the rows in flight come from the grid
  const int want = rows <= 512 ? 1024 : 256;
  int nc = (groups + want - 1) / want;
  nc = nc <= 1 ? 1 : nc <= 2 ? 2 : nc <= 4 ? 4 : 8;
  const int threads = ((groups + nc - 1) / nc + 31) / 32 * 32;
  if (threads > 1024) {
    msgl_set_error_text("add_norm: row too wide");
    return MSGL_BAD_ARG;
  }
#define ADD_NORM(V, N) msgl_launch(add_norm_kernel<T, V, N, CENTER, POST>, dim3(rows), dim3(threads), 0, s, a)
  if (vec) {
    if (nc == 1) ADD_NORM(4, 1);
    else if (nc == 2) ADD_NORM(4, 2);
    else if (nc == 4) ADD_NORM(4, 4);
    else ADD_NORM(4, 8);
  } else {
    if (nc == 1) ADD_NORM(1, 1);
    else if (nc == 2) ADD_NORM(1, 2);
    else if (nc == 4) ADD_NORM(1, 4);
    else ADD_NORM(1, 8);
  }
#undef ADD_NORM
  MSGL_CHECK_LAUNCH("add_norm");
  return MSGL_OK;
}

}  // namespace

MSGL_API int msgl_add_norm(const void* x, void* x_out, const void* delta, int planes, long long plane_stride, long long ldd,
                           const void* w, void* y, int rows, int width, int cols, float eps, int center,
                           const void* post_w, float mult, int dtype, cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (width <= 0 || cols < width || (post_w != nullptr && (planes <= 0 || center)) || (planes > 0 && (x == x_out || delta == nullptr))) return MSGL_BAD_ARG;
  AddNormArgs a{(const float*)x, (float*)x_out, (const float*)delta, planes, plane_stride, ldd, (const float*)w, y, width,
                cols, eps, (const float*)post_w, mult};
#define ADD_NORM_TYPED(T)                                              \
  (center             ? add_norm_typed<T, true, false>(a, rows, stream) \
   : post_w != nullptr ? add_norm_typed<T, false, true>(a, rows, stream) \
                       : add_norm_typed<T, false, false>(a, rows, stream))
  if (dtype == MSGL_BF16) return ADD_NORM_TYPED(__nv_bfloat16);
  if (dtype == MSGL_F32) return ADD_NORM_TYPED(float);
#undef ADD_NORM_TYPED
  return MSGL_BAD_ARG;
}
