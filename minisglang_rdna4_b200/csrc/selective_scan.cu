// Selective scan (Mamba): per request and channel c a state vector, S_n <- exp(dt_c a_cn) S_n + dt_c x_c B_n,
// y_c = sum_n S_n C_n + skip_c x_c, with dt the softplus of a projection; and the causal convolution with silu ahead of it.
//
//   causal_conv_silu_kernel   a filter per channel; the last taps - 1 inputs are a request's state
//   scan_rows_kernel          token by token, operands straight from global memory: decode, draft verification, 32 bits
//   scan_tiles_kernel         prompts: tiles of tokens staged through shared memory, two deep
//
// State, decays, step sizes and everything that enters the recurrence are fp32. A group of LN lanes owns a channel, four
// states each and every LN * 4 further ones. Sequences are packed rows described by cu_q; a sequence without a state
// (has_state == 0) starts from zeros.
#include "common.cuh"

#include <type_traits>

using namespace msgl;

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2a(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// 32 bits take the library's functions, 16 bits the approximate instructions
template <typename T> __device__ __forceinline__ float softplus(float x) {
  if constexpr (sizeof(T) == 4) return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
  const float e = __expf(-fabsf(x));
  // log(1 + e): a short series where 1 + e would lose e's digits
  return fmaxf(x, 0.f) + (e < 0.03125f ? e * (1.f - e * (0.5f - e * (0.33333333f - 0.25f * e))) : __logf(1.f + e));
}
template <typename T> __device__ __forceinline__ float silu(float x) {
  if constexpr (sizeof(T) == 4) return x / (1.f + expf(-x));
  return __fdividef(x, 1.f + __expf(-x));
}
// a is negative and, in 16 bits, in units of log2
template <typename T> __device__ __forceinline__ float decay(float dta) {
  if constexpr (sizeof(T) == 4) return expf(dta);
  return ex2a(dta);
}
template <typename T> constexpr float kAUnit = sizeof(T) == 4 ? 1.f : kLog2e;

// ------------------------------------------------------------------------------------------ convolution
struct ConvArgs {
  const void* x;               // [T, C] with row stride ldx
  long long ldx;
  const float* w;              // [C, taps]
  const float* bias;           // [C]
  void* state;                 // [slots, C, taps - 1] with slot stride
  long long slot_stride;
  const int32_t* cu_q;
  const int32_t* slots;
  const int32_t* has_state;
  void* out;                   // [T, C]
  int channels, taps, num_slots;
};

// grid (channels / 256, stretches of tokens, B), a channel pair per thread. A stretch reads the taps - 1 rows ahead of it
// again. Only the first one touches the tail: it reads the old one and, when its rows are done, writes the new one.
constexpr int kStretch = 64;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_silu_kernel(const ConvArgs a) {
  pdl_enter();
  using P2 = typename std::conditional<sizeof(T) == 2, uint32_t, float2>::type;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 2, b = blockIdx.z;
  if (c >= a.channels) return;
  const int lo = a.cu_q[b], len = a.cu_q[b + 1] - lo;
  const int t0 = blockIdx.y * kStretch, t1 = min(t0 + kStretch, len);
  if (t0 >= t1) return;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  T* st = reinterpret_cast<T*>(a.state) + slot * a.slot_stride + (size_t)c * (TAPS - 1);
  const T* x = reinterpret_cast<const T*>(a.x) + lo * a.ldx + c;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)lo * a.channels + c;
  const bool keep = a.has_state[b] != 0;
  auto load2 = [&](const T* p, float& u, float& v) {
    union { P2 w; T e[2]; } q;
    q.w = *reinterpret_cast<const P2*>(p);
    u = to_float(q.e[0]);
    v = to_float(q.e[1]);
  };
  float w[2][TAPS], h[2][TAPS];           // h[.][TAPS - 1]: the current input
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    w[0][j] = a.w[(size_t)c * TAPS + j];
    w[1][j] = a.w[(size_t)(c + 1) * TAPS + j];
  }
  const float b0 = a.bias[c], b1 = a.bias[c + 1];
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = t0 - (TAPS - 1) + j;    // the input that h[.][j + 1] is ahead of the first step's shift
    h[0][j + 1] = h[1][j + 1] = 0.f;
    if (t >= 0) load2(x + t * a.ldx, h[0][j + 1], h[1][j + 1]);
    else if (keep) {
      h[0][j + 1] = to_float(st[t + TAPS - 1]);
      h[1][j + 1] = to_float(st[TAPS - 1 + t + TAPS - 1]);
    }
  }
#pragma unroll 8
  for (int t = t0; t < t1; ++t) {
    float acc0 = b0, acc1 = b1;
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) { h[0][j] = h[0][j + 1]; h[1][j] = h[1][j + 1]; }
    load2(x + t * a.ldx, h[0][TAPS - 1], h[1][TAPS - 1]);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      acc0 = fmaf(w[0][j], h[0][j], acc0);
      acc1 = fmaf(w[1][j], h[1][j], acc1);
    }
    union { P2 w; T e[2]; } q;
    q.e[0] = from_float<T>(silu<T>(acc0));
    q.e[1] = from_float<T>(silu<T>(acc1));
    *reinterpret_cast<P2*>(out + (size_t)t * a.channels) = q.w;
  }
  if (t0 == 0) {
    if (t1 < len) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) load2(x + (len - (TAPS - 1) + j) * a.ldx, h[0][j + 1], h[1][j + 1]);
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      st[j] = from_float<T>(h[0][j + 1]);
      st[TAPS - 1 + j] = from_float<T>(h[1][j + 1]);
    }
  }
}

// any number of taps, one stretch per request
template <typename T>
__global__ void __launch_bounds__(128) causal_conv_silu_any_kernel(const ConvArgs a) {
  pdl_enter();
  const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y, taps = a.taps;
  if (c >= a.channels) return;
  const int lo = a.cu_q[b], len = a.cu_q[b + 1] - lo;
  if (len <= 0) return;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  T* st = reinterpret_cast<T*>(a.state) + slot * a.slot_stride + (size_t)c * (taps - 1);
  const T* x = reinterpret_cast<const T*>(a.x) + lo * a.ldx + c;
  const bool keep = a.has_state[b] != 0;
  auto input = [&](int t) { return t >= 0 ? to_float(x[t * a.ldx]) : keep ? to_float(st[t + taps - 1]) : 0.f; };
  for (int t = 0; t < len; ++t) {
    float acc = a.bias[c];
    for (int j = 0; j < taps; ++j) acc = fmaf(a.w[(size_t)c * taps + j], input(t - taps + 1 + j), acc);
    reinterpret_cast<T*>(a.out)[(size_t)(lo + t) * a.channels + c] = from_float<T>(silu<T>(acc));
  }
  // in ascending order: what is read lies ahead of what has been written
  for (int j = 0; j < taps - 1; ++j) st[j] = from_float<T>(input(len - taps + 1 + j));
}

// ------------------------------------------------------------------------------------------ scan
struct ScanArgs {
  const void* x;               // [T, C]
  const float* dt;             // [T, C] ahead of bias and softplus
  const float* dt_bias;        // [C]
  const float* A;              // [C, N], negative
  const void* B;               // [T, N] with row stride ldb (C: the same rows)
  const void* Cm;
  const float* skip;           // [C]
  const void* z;               // [T, C] with row stride ldz
  float* state;                // [slots, C, N] with slot stride
  long long ldb, ldz, slot_stride;
  const int32_t* cu_q;
  const int32_t* slots;
  const int32_t* has_state;
  void* out;                   // [T, C]
  int channels, N, num_slots;
};

template <typename T> __device__ __forceinline__ float4 load4f(const T* p);
template <> __device__ __forceinline__ float4 load4f<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4f<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(u.x, u.y, v.x, v.y);
}

// One step of the states a lane owns (4 G of them): returns its part of y.
template <typename T, int G>
__device__ __forceinline__ float advance(float4 (&s)[G], const float4 (&A)[G], const float4 (&B)[G], const float4 (&C)[G],
                                         float dt, float dtx) {
  float y = 0.f;
#pragma unroll
  for (int g = 0; g < G; ++g) {
    s[g].x = fmaf(s[g].x, decay<T>(dt * A[g].x), dtx * B[g].x);
    s[g].y = fmaf(s[g].y, decay<T>(dt * A[g].y), dtx * B[g].y);
    s[g].z = fmaf(s[g].z, decay<T>(dt * A[g].z), dtx * B[g].z);
    s[g].w = fmaf(s[g].w, decay<T>(dt * A[g].w), dtx * B[g].w);
    y = fmaf(s[g].x, C[g].x, fmaf(s[g].y, C[g].y, fmaf(s[g].z, C[g].z, fmaf(s[g].w, C[g].w, y))));
  }
  return y;
}

// grid (channels * LN / 128, B)
template <typename T, int LN, int G>
__global__ void __launch_bounds__(128) scan_rows_kernel(const ScanArgs a) {
  pdl_enter();
  const int b = blockIdx.y, id = blockIdx.x * 128 + threadIdx.x, c = id / LN, ln = id % LN;
  const int lo = a.cu_q[b], hi = a.cu_q[b + 1];
  if (hi <= lo) return;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  const bool live = c < a.channels;
  const int ch = live ? c : 0;
  float* S = a.state + slot * a.slot_stride + (size_t)ch * a.N;
  const bool keep = a.has_state[b] != 0;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 s[G], A[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    s[g] = keep && n < a.N ? *reinterpret_cast<const float4*>(S + n) : zero;
    A[g] = n < a.N ? *reinterpret_cast<const float4*>(a.A + (size_t)ch * a.N + n) : zero;
    A[g].x *= kAUnit<T>; A[g].y *= kAUnit<T>; A[g].z *= kAUnit<T>; A[g].w *= kAUnit<T>;
  }
  const float bias = a.dt_bias[ch], skip = a.skip[ch];
  for (int t = lo; t < hi; ++t) {
    float4 B[G], C[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const int n = (g * LN + ln) * 4;
      B[g] = n < a.N ? load4f(reinterpret_cast<const T*>(a.B) + t * a.ldb + n) : zero;
      C[g] = n < a.N ? load4f(reinterpret_cast<const T*>(a.Cm) + t * a.ldb + n) : zero;
    }
    const size_t at = (size_t)t * a.channels + ch;
    const float x = to_float(reinterpret_cast<const T*>(a.x)[at]);
    const float dt = softplus<T>(a.dt[at] + bias);
    float y = advance<T, G>(s, A, B, C, dt, dt * x);
#pragma unroll
    for (int m = 1; m < LN; m <<= 1) y += __shfl_xor_sync(0xffffffffu, y, m);
    if (live && ln == 0)
      reinterpret_cast<T*>(a.out)[at] = from_float<T>(
          fmaf(skip, x, y) * silu<T>(to_float(reinterpret_cast<const T*>(a.z)[t * a.ldz + ch])));
  }
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    if (live && n < a.N) *reinterpret_cast<float4*>(S + n) = s[g];
  }
}

template <typename T> int launch_rows(const ScanArgs& a, int B, cudaStream_t s) {
#define ROWS(LN, G) \
  msgl_launch(scan_rows_kernel<T, LN, G>, dim3((a.channels * LN + 127) / 128, B), dim3(128), 0, s, a)
  if (a.N <= 4) ROWS(1, 1);
  else if (a.N <= 8) ROWS(2, 1);
  else if (a.N <= 16) ROWS(4, 1);
  else if (a.N <= 32) ROWS(8, 1);
  else if (a.N <= 64) ROWS(16, 1);
  else if (a.N <= 128) ROWS(32, 1);
  else if (a.N <= 256) ROWS(32, 2);
  else if (a.N <= 512) ROWS(32, 4);
  else {
    msgl_set_error_text("selective_scan: states of up to 512");
    return MSGL_BAD_ARG;
  }
#undef ROWS
  MSGL_CHECK_LAUNCH("selective_scan");
  return MSGL_OK;
}

// ------------------------------------------------------------------------------------------ prompts
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp8(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 8 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

constexpr int kTile = 32;      // tokens
template <int LN, int G> struct TileSmem {
  static constexpr int CH = 128 / LN, NP = LN * G * 4;      // channels of a CTA, states
  // raw rows, two deep: x, z, B ‖ C in 16 bits, dt
  static constexpr int off_z = kTile * CH * 2, off_dt = 2 * off_z, off_bc = off_dt + kTile * CH * 4;
  static constexpr int raw = off_bc + kTile * 2 * NP * 2;
  static constexpr int off_step = 2 * raw;                    // (dt, dt x) [tile][CH]
  static constexpr int off_b = off_step + kTile * CH * 8;     // B and C in fp32 [tile][2][NP]
  static constexpr int off_y = off_b + kTile * 2 * NP * 4;    // [tile][CH]
  static constexpr int bytes = off_y + kTile * CH * 4;
};

// grid (channels / CH, B), 128 threads. Per tile: softplus and products of all (token, channel) pairs; the recurrence, LN
// lanes per channel; skip, gate and store of all pairs. The next tile's rows arrive meanwhile.
template <int LN, int G>
__global__ void __launch_bounds__(128) scan_tiles_kernel(const ScanArgs a) {
  pdl_enter();
  using bf = __nv_bfloat16;
  using L = TileSmem<LN, G>;
  constexpr int CH = L::CH, NP = L::NP;
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
  const int tid = threadIdx.x, b = blockIdx.y, cl = tid / LN, ln = tid % LN, c_first = blockIdx.x * CH, c = c_first + cl;
  const int lo = a.cu_q[b], len = a.cu_q[b + 1] - lo;
  if (len <= 0) return;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  const bf* x = reinterpret_cast<const bf*>(a.x) + (size_t)lo * a.channels + c_first;
  const bf* z = reinterpret_cast<const bf*>(a.z) + (size_t)lo * a.ldz + c_first;
  const float* dt = a.dt + (size_t)lo * a.channels + c_first;
  const bf* B = reinterpret_cast<const bf*>(a.B) + (size_t)lo * a.ldb;
  const bf* C = reinterpret_cast<const bf*>(a.Cm) + (size_t)lo * a.ldb;
  const int left = min(CH, a.channels - c_first);
  auto fetch = [&](int t0, int buf) {
    if (t0 < len) {
      const uint32_t dst = base + buf * L::raw;
      for (int i = tid; i < kTile * CH / 8; i += 128) {
        const int t = i / (CH / 8), k = i % (CH / 8) * 8;
        const bool ok = t0 + t < len && k < left;
        cp16(dst + i * 16, x + (ok ? (size_t)(t0 + t) * a.channels + k : 0), ok);
        cp16(dst + L::off_z + i * 16, z + (ok ? (size_t)(t0 + t) * a.ldz + k : 0), ok);
      }
      for (int i = tid; i < kTile * CH / 4; i += 128) {
        const int t = i / (CH / 4), k = i % (CH / 4) * 4;
        const bool ok = t0 + t < len && k < left;
        cp16(dst + L::off_dt + i * 16, dt + (ok ? (size_t)(t0 + t) * a.channels + k : 0), ok);
      }
      for (int i = tid; i < kTile * 2 * NP / 4; i += 128) {
        const int t = i / (2 * NP / 4), k = i % (2 * NP / 4) * 4, n = k < NP ? k : k - NP;
        const bool ok = t0 + t < len && n < a.N;
        cp8(dst + L::off_bc + i * 8, (k < NP ? B : C) + (ok ? (size_t)(t0 + t) * a.ldb + n : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);

  const bool live = c < a.channels, keep = a.has_state[b] != 0;
  float* S = a.state + slot * a.slot_stride + (size_t)(live ? c : 0) * a.N;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 s[G], A[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    s[g] = keep && live && n < a.N ? *reinterpret_cast<const float4*>(S + n) : zero;
    A[g] = live && n < a.N ? *reinterpret_cast<const float4*>(a.A + (size_t)c * a.N + n) : zero;
    A[g].x *= kLog2e; A[g].y *= kLog2e; A[g].z *= kLog2e; A[g].w *= kLog2e;
  }
  // the channel that this thread takes ahead of and behind the recurrence
  constexpr int ROWS = 128 / CH;             // tokens side by side
  const int pc = tid % CH, pt = tid / CH;
  const bool plive = pc < left;
  const float bias = plive ? a.dt_bias[c_first + pc] : 0.f, skip = plive ? a.skip[c_first + pc] : 0.f;
  float2* step = reinterpret_cast<float2*>(smem + L::off_step);
  float* bc = reinterpret_cast<float*>(smem + L::off_b);
  float* ys = reinterpret_cast<float*>(smem + L::off_y);
  for (int t0 = 0, buf = 0; t0 < len; t0 += kTile, buf ^= 1) {
    const int n = min(kTile, len - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                         // the tile is there, and the one before is done with its buffers
    fetch(t0 + kTile, buf ^ 1);
    const uint8_t* raw = smem + buf * L::raw;
    const bf* xs = reinterpret_cast<const bf*>(raw);
    const bf* zs = reinterpret_cast<const bf*>(raw + L::off_z);
    const float* ds = reinterpret_cast<const float*>(raw + L::off_dt);
#pragma unroll
    for (int t = pt; t < kTile; t += ROWS) {
      const float d = t < n ? softplus<bf>(ds[t * CH + pc] + bias) : 0.f;       // past the end: the state stays
      step[t * CH + pc] = make_float2(d, d * to_float(xs[t * CH + pc]));
    }
    for (int i = tid; i < kTile * 2 * NP / 4; i += 128)
      *reinterpret_cast<float4*>(bc + i * 4) = load4f(reinterpret_cast<const bf*>(raw + L::off_bc) + i * 4);
    __syncthreads();
    for (int t = 0; t < n; t += 4) {
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 d = step[(t + k) * CH + cl];
        const float* row = bc + (t + k) * 2 * NP + ln * 4;
        float4 Bv[G], Cv[G];
#pragma unroll
        for (int g = 0; g < G; ++g) {
          Bv[g] = *reinterpret_cast<const float4*>(row + g * LN * 4);
          Cv[g] = *reinterpret_cast<const float4*>(row + NP + g * LN * 4);
        }
        y[k] = advance<bf, G>(s, A, Bv, Cv, d.x, d.y);
      }
      // sums over the lanes of a channel; every exchange halves the tokens a lane is left with
      if constexpr (LN == 1) {
#pragma unroll
        for (int k = 0; k < 4; ++k) ys[(t + k) * CH + cl] = y[k];
      } else {
        const bool up = ln & 1;
        const float v0 = (up ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, up ? y[0] : y[2], 1);
        const float v1 = (up ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, up ? y[1] : y[3], 1);
        if constexpr (LN == 2) {
          ys[(t + 2 * up) * CH + cl] = v0;
          ys[(t + 2 * up + 1) * CH + cl] = v1;
        } else {
          const bool up2 = ln & 2;
          float w = (up2 ? v1 : v0) + __shfl_xor_sync(0xffffffffu, up2 ? v0 : v1, 2);
#pragma unroll
          for (int m = 4; m < LN; m <<= 1) w += __shfl_xor_sync(0xffffffffu, w, m);
          if (ln < 4) ys[(t + 2 * up + up2) * CH + cl] = w;
        }
      }
    }
    __syncthreads();
    if (plive) {
      bf* out = reinterpret_cast<bf*>(a.out) + (size_t)(lo + t0) * a.channels + c_first + pc;
#pragma unroll 4
      for (int t = pt; t < n; t += ROWS)
        out[(size_t)t * a.channels] = __float2bfloat16(fmaf(skip, to_float(xs[t * CH + pc]), ys[t * CH + pc]) *
                                                       silu<bf>(to_float(zs[t * CH + pc])));
    }
  }
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    if (live && n < a.N) *reinterpret_cast<float4*>(S + n) = s[g];
  }
}

template <int LN, int G> int launch_tiles_form(const ScanArgs& a, int B, cudaStream_t s) {
  using L = TileSmem<LN, G>;
  static bool set = false;
  if (!set) {
    const cudaError_t e = cudaFuncSetAttribute(scan_tiles_kernel<LN, G>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::bytes);
    if (e != cudaSuccess) { msgl_set_error("selective_scan smem", e); return MSGL_CUDA_ERROR; }
    set = true;
  }
  msgl_launch(scan_tiles_kernel<LN, G>, dim3((a.channels + L::CH - 1) / L::CH, B), dim3(128), L::bytes, s, a);
  MSGL_CHECK_LAUNCH("selective_scan");
  return MSGL_OK;
}
int launch_tiles(const ScanArgs& a, int B, cudaStream_t s) {
  if (a.N <= 4) return launch_tiles_form<1, 1>(a, B, s);
  if (a.N <= 8) return launch_tiles_form<2, 1>(a, B, s);
  if (a.N <= 16) return launch_tiles_form<4, 1>(a, B, s);
  if (a.N <= 32) return launch_tiles_form<4, 2>(a, B, s);
  if (a.N <= 64) return launch_tiles_form<8, 2>(a, B, s);
  if (a.N <= 128) return launch_tiles_form<8, 4>(a, B, s);
  if (a.N <= 256) return launch_tiles_form<16, 4>(a, B, s);
  return launch_rows<__nv_bfloat16>(a, B, s);
}

}  // namespace

// x [T, channels] with row stride ldx (channels even); out [T, channels]
MSGL_API int msgl_causal_conv_silu(const void* x, long long ldx, const void* w, const void* bias, void* state,
                                   long long slot_stride, const void* cu_q, const void* slots, const void* has_state,
                                   void* out, int B, int channels, int taps, int max_q, int num_slots, int dtype,
                                   cudaStream_t stream) {
  if (B <= 0) return B == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (channels <= 0 || channels % 2 || taps <= 0 || max_q <= 0 || B > 65535 || ldx % 2 || (uintptr_t)x % 8 ||
      (uintptr_t)out % 8)
    return MSGL_BAD_ARG;
  const ConvArgs a{x, ldx, (const float*)w, (const float*)bias, state, slot_stride, (const int32_t*)cu_q,
                   (const int32_t*)slots, (const int32_t*)has_state, out, channels, taps, num_slots};
  const dim3 grid((channels + 255) / 256, (max_q + kStretch - 1) / kStretch, B);
#define CONV(T)                                                                                          \
  do {                                                                                                   \
    if (taps == 1) msgl_launch(causal_conv_silu_kernel<T, 1>, grid, dim3(128), 0, stream, a);            \
    else if (taps == 2) msgl_launch(causal_conv_silu_kernel<T, 2>, grid, dim3(128), 0, stream, a);       \
    else if (taps == 3) msgl_launch(causal_conv_silu_kernel<T, 3>, grid, dim3(128), 0, stream, a);       \
    else if (taps == 4) msgl_launch(causal_conv_silu_kernel<T, 4>, grid, dim3(128), 0, stream, a);       \
    else msgl_launch(causal_conv_silu_any_kernel<T>, dim3((channels + 127) / 128, B), dim3(128), 0, stream, a); \
  } while (0)
  if (dtype == MSGL_BF16) CONV(__nv_bfloat16);
  else if (dtype == MSGL_F32) CONV(float);
  else return MSGL_BAD_ARG;
#undef CONV
  MSGL_CHECK_LAUNCH("causal_conv_silu");
  return MSGL_OK;
}

// tiles: prompts may take the tiled form (16 bits)
MSGL_API int msgl_selective_scan(const void* x, const void* dt, const void* dt_bias, const void* A, const void* B,
                                 const void* C, long long ldb, const void* skip, const void* z, long long ldz, void* state,
                                 long long slot_stride, const void* cu_q, const void* slots, const void* has_state,
                                 void* out, int batch, int channels, int N, int num_slots, int tiles, int dtype,
                                 cudaStream_t stream) {
  if (batch <= 0) return batch == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (channels <= 0 || channels % 16 || N <= 0 || N % 4 || batch > 65535 || ldb % 4 || ldz % 8 || slot_stride % 4 ||
      (uintptr_t)state % 16 || (uintptr_t)A % 16 || (uintptr_t)B % 16 || (uintptr_t)C % 8 || (uintptr_t)x % 16 ||
      (uintptr_t)dt % 16 || (uintptr_t)z % 16 || (uintptr_t)out % 16)
    return MSGL_BAD_ARG;
  const ScanArgs a{x, (const float*)dt, (const float*)dt_bias, (const float*)A, B, C, (const float*)skip, z, (float*)state,
                   ldb, ldz, slot_stride, (const int32_t*)cu_q, (const int32_t*)slots, (const int32_t*)has_state, out,
                   channels, N, num_slots};
  if (dtype == MSGL_F32) return launch_rows<float>(a, batch, stream);
  if (dtype != MSGL_BF16) return MSGL_BAD_ARG;
  return tiles ? launch_tiles(a, batch, stream) : launch_rows<__nv_bfloat16>(a, batch, stream);
}
