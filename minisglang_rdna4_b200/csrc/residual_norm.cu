// Norm of an fp32 residual stream with a weight per channel: residual += delta, then layer norm without a bias (the
// variance is the mean of the squared deviations, taken in a second pass over registers) or RMS norm. delta may be the
// unreduced K ranges of a split GEMM. With a post weight, what is added is mult times the RMS norm of delta. One CTA
// per row.
//
// residual_step: the same for sublayers with a layer norm (weight and bias) on both sides. The sublayer's output may be half
// the sum of two RMS-normed rows; the result may join the results of the layers so far, whose weighted sum goes on.
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

struct StepArgs {
  const float* x;              // [rows, width], or null: zero
  const float* d[2];           // [planes][rows][ldd]; the second one with PAIR
  int planes[2];
  long long plane_stride[2], ldd[2];
  const float* pair_w[2];      // PAIR: weights of the two RMS norms
  const float *post_w, *post_b;     // layer norm of the sublayer's output, or null
  float* hist;                 // [n + 1][rows][width]: the sum becomes row n; or null
  int n;
  const float* coef;           // [n + 1]: what goes on is the sum of coef[j] hist[j]; or null: the sum itself
  float* x_out;                // what goes on (not written where it is row n of hist)
  const float *w, *b;
  void* y;                     // [rows, cols], zero past the width
  int rows, width, cols;
  float eps;
};

template <int V> __device__ __forceinline__ void load_v(const float* p, float (&x)[V]) {
  if constexpr (V == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    x[0] = q.x; x[1] = q.y; x[2] = q.z; x[3] = q.w;
  } else {
    x[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void store_v(float* p, const float (&x)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  else *p = x[0];
}

template <int V, int NC>
__device__ __forceinline__ void load_planes(const float* d, int planes, long long stride, long long at, int width, int first,
                                            int step, float (&u)[NC][V]) {
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * step + first) * V;
#pragma unroll
    for (int v = 0; v < V; ++v) u[g][v] = 0.f;
    if (c >= width) continue;
    for (int p = 0; p < planes; ++p) {
      float q[V];
      load_v<V>(d + p * stride + at + c, q);
#pragma unroll
      for (int v = 0; v < V; ++v) u[g][v] += q[v];
    }
  }
}

// mean and 1 / root of (mean squared deviation + eps); entries past the width are zero
template <int V, int NC>
__device__ __forceinline__ float2 centre(const float (&u)[NC][V], int width, float eps, float* scratch) {
  float s = 0.f;
#pragma unroll
  for (int g = 0; g < NC; ++g)
#pragma unroll
    for (int v = 0; v < V; ++v) s += u[g][v];
  const float mean = block_sum(s, scratch) / (float)width;
  s = 0.f;
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const bool in = (int)(g * blockDim.x + threadIdx.x) * V < width;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const float d = in ? u[g][v] - mean : 0.f;
      s = fmaf(d, d, s);
    }
  }
  return make_float2(mean, 1.f / sqrtf(block_sum(s, scratch) / (float)width + eps));
}

// two block sums at once; scratch holds 64 floats
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) {
    scratch[warp] = a;
    scratch[32 + warp] = b;
  }
  __syncthreads();
  return make_float2(warp_sum(lane < nw ? scratch[lane] : 0.f), warp_sum(lane < nw ? scratch[32 + lane] : 0.f));
}

template <typename T, int V, int NC, bool PAIR>
__global__ void __launch_bounds__(1024) residual_step_kernel(const StepArgs a) {
  pdl_enter();
  __shared__ float scratch[64];
  const size_t row = blockIdx.x;
  const int first = threadIdx.x, step = blockDim.x;
  const size_t plane = (size_t)a.rows * a.width, at = row * a.width;
  float u[NC][V], x[NC][V];
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * step + first) * V;
#pragma unroll
    for (int v = 0; v < V; ++v) x[g][v] = 0.f;
    if (a.x != nullptr && c < a.width) load_v<V>(a.x + at + c, x[g]);
  }
  load_planes<V, NC>(a.d[0], a.planes[0], a.plane_stride[0], row * a.ldd[0], a.width, first, step, u);
  if constexpr (PAIR) {
    float e[NC][V];
    load_planes<V, NC>(a.d[1], a.planes[1], a.plane_stride[1], row * a.ldd[1], a.width, first, step, e);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int g = 0; g < NC; ++g)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        s0 = fmaf(u[g][v], u[g][v], s0);
        s1 = fmaf(e[g][v], e[g][v], s1);
      }
    const float2 ss = block_sum2(s0, s1, scratch);
    const float r0 = 0.5f / sqrtf(ss.x / (float)a.width + a.eps), r1 = 0.5f / sqrtf(ss.y / (float)a.width + a.eps);
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const int c = (g * step + first) * V;
      if (c >= a.width) continue;
#pragma unroll
      for (int v = 0; v < V; ++v) u[g][v] = u[g][v] * r0 * a.pair_w[0][c + v] + e[g][v] * r1 * a.pair_w[1][c + v];
    }
  }
  if (a.post_w != nullptr) {
    const float2 m = centre<V, NC>(u, a.width, a.eps, scratch);
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const int c = (g * step + first) * V;
      if (c >= a.width) continue;
#pragma unroll
      for (int v = 0; v < V; ++v) u[g][v] = (u[g][v] - m.x) * m.y * a.post_w[c + v] + a.post_b[c + v];
    }
  }
  const float own = a.coef != nullptr ? a.coef[a.n] : 1.f;
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * step + first) * V;
    if (c >= a.width) continue;
#pragma unroll
    for (int v = 0; v < V; ++v) u[g][v] += x[g][v];
    if (a.hist != nullptr) store_v<V>(a.hist + a.n * plane + at + c, u[g]);
#pragma unroll
    for (int v = 0; v < V; ++v) u[g][v] *= own;
  }
  if (a.coef != nullptr) {
    for (int j0 = 0; j0 < a.n; j0 += 4) {        // four results in flight
#pragma unroll
      for (int g = 0; g < NC; ++g) {
        const int c = (g * step + first) * V;
        if (c >= a.width) continue;
        float q[4][V], f[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const bool in = j0 + k < a.n;
          f[k] = in ? a.coef[j0 + k] : 0.f;
          load_v<V>(a.hist + (in ? j0 + k : j0) * plane + at + c, q[k]);
        }
#pragma unroll
        for (int k = 0; k < 4; ++k)
#pragma unroll
          for (int v = 0; v < V; ++v) u[g][v] = j0 + k < a.n ? fmaf(f[k], q[k][v], u[g][v]) : u[g][v];
      }
    }
  }
  if (a.x_out != nullptr) {
#pragma unroll
    for (int g = 0; g < NC; ++g) {
      const int c = (g * step + first) * V;
      if (c < a.width) store_v<V>(a.x_out + at + c, u[g]);
    }
  }
  const float2 m = centre<V, NC>(u, a.width, a.eps, scratch);
  T* y = reinterpret_cast<T*>(a.y) + row * a.cols;
#pragma unroll
  for (int g = 0; g < NC; ++g) {
    const int c = (g * step + first) * V;
    if (c >= a.cols) continue;
    float o[V];
#pragma unroll
    for (int v = 0; v < V; ++v) o[v] = c < a.width ? (u[g][v] - m.x) * m.y * a.w[c + v] + a.b[c + v] : 0.f;
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

template <typename T, bool PAIR> int residual_step_typed(const StepArgs& a, cudaStream_t s) {
  bool vec = a.width % 4 == 0 && a.cols % 4 == 0;
  for (int i = 0; i < (PAIR ? 2 : 1); ++i)
    vec = vec && a.ldd[i] % 4 == 0 && a.plane_stride[i] % 4 == 0 && (uintptr_t)a.d[i] % 16 == 0;
  const int groups = (a.cols + (vec ? 3 : 0)) / (vec ? 4 : 1);
  const int want = a.rows <= 512 ? 512 : 128;
  int nc = (groups + want - 1) / want;
  nc = nc <= 1 ? 1 : nc <= 2 ? 2 : nc <= 4 ? 4 : 8;
  const int threads = ((groups + nc - 1) / nc + 31) / 32 * 32;
  if (threads > 1024) {
    msgl_set_error_text("residual_step: row too wide");
    return MSGL_BAD_ARG;
  }
#define STEP(V, N) msgl_launch(residual_step_kernel<T, V, N, PAIR>, dim3(a.rows), dim3(threads), 0, s, a)
  if (vec) {
    if (nc == 1) STEP(4, 1);
    else if (nc == 2) STEP(4, 2);
    else if (nc == 4) STEP(4, 4);
    else STEP(4, 8);
  } else {
    if (nc == 1) STEP(1, 1);
    else if (nc == 2) STEP(1, 2);
    else if (nc == 4) STEP(1, 4);
    else STEP(1, 8);
  }
#undef STEP
  MSGL_CHECK_LAUNCH("residual_step");
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

// d1 null: one sublayer output. hist null: no results of layers are kept; coef null: the sum itself goes on.
MSGL_API int msgl_residual_step(const void* x, const void* d0, int planes0, long long plane_stride0, long long ldd0,
                                const void* d1, int planes1, long long plane_stride1, long long ldd1, const void* w0,
                                const void* w1, const void* post_w, const void* post_b, void* hist, int n, const void* coef,
                                void* x_out, const void* w, const void* b, void* y, int rows, int width, int cols, float eps,
                                int dtype, cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (width <= 0 || cols < width || planes0 <= 0 || d0 == nullptr || w == nullptr || b == nullptr ||
      (d1 != nullptr && (planes1 <= 0 || w0 == nullptr || w1 == nullptr)) || (post_w == nullptr) != (post_b == nullptr) ||
      (coef != nullptr && hist == nullptr) || n < 0 || (x_out != nullptr && x == x_out))
    return MSGL_BAD_ARG;
  StepArgs a{(const float*)x, {(const float*)d0, (const float*)d1}, {planes0, planes1}, {plane_stride0, plane_stride1},
             {ldd0, ldd1}, {(const float*)w0, (const float*)w1}, (const float*)post_w, (const float*)post_b, (float*)hist, n,
             (const float*)coef, (float*)x_out, (const float*)w, (const float*)b, y, rows, width, cols, eps};
#define STEP_TYPED(T) (d1 != nullptr ? residual_step_typed<T, true>(a, stream) : residual_step_typed<T, false>(a, stream))
  if (dtype == MSGL_BF16) return STEP_TYPED(__nv_bfloat16);
  if (dtype == MSGL_F32) return STEP_TYPED(float);
#undef STEP_TYPED
  return MSGL_BAD_ARG;
}
