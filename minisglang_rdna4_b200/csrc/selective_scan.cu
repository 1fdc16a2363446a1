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

// grid (channels / 512, stretches of tokens, B), four channels per thread. A stretch reads the taps - 1 rows ahead of it
// again. Only the first one touches the tail: it reads the old one and, when its rows are done, writes the new one.
constexpr int kStretch = 32;
__device__ __forceinline__ float4 load4f(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4f(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(u.x, u.y, v.x, v.y);
}
__device__ __forceinline__ void store4f(float* p, float4 x) { *reinterpret_cast<float4*>(p) = x; }
__device__ __forceinline__ void store4f(__nv_bfloat16* p, float4 x) {
  uint2 q;
  *reinterpret_cast<__nv_bfloat162*>(&q.x) = __floats2bfloat162_rn(x.x, x.y);
  *reinterpret_cast<__nv_bfloat162*>(&q.y) = __floats2bfloat162_rn(x.z, x.w);
  *reinterpret_cast<uint2*>(p) = q;
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_silu_kernel(const ConvArgs a) {
  pdl_enter();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4, b = blockIdx.z;
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
  float w[TAPS][4];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) w[j][e] = a.w[(size_t)(c + e) * TAPS + j];
  const float4 bias = load4f(a.bias + c);
  float4 h[TAPS];                         // h[TAPS - 1]: the current input
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = t0 - (TAPS - 1) + j;    // the input that h[j + 1] is ahead of the first step's shift
    h[j + 1] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t >= 0) h[j + 1] = load4f(x + t * a.ldx);
    else if (keep) {
      const T* s = st + t + TAPS - 1;
      h[j + 1] = make_float4(to_float(s[0]), to_float(s[TAPS - 1]), to_float(s[2 * (TAPS - 1)]), to_float(s[3 * (TAPS - 1)]));
    }
  }
#pragma unroll 8
  for (int t = t0; t < t1; ++t) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) h[j] = h[j + 1];
    h[TAPS - 1] = load4f(x + t * a.ldx);
    float4 acc = bias;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      acc.x = fmaf(w[j][0], h[j].x, acc.x);
      acc.y = fmaf(w[j][1], h[j].y, acc.y);
      acc.z = fmaf(w[j][2], h[j].z, acc.z);
      acc.w = fmaf(w[j][3], h[j].w, acc.w);
    }
    store4f(out + (size_t)t * a.channels, make_float4(silu<T>(acc.x), silu<T>(acc.y), silu<T>(acc.z), silu<T>(acc.w)));
  }
  if (t0 == 0) {
    if (t1 < len) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) h[j + 1] = load4f(x + (len - (TAPS - 1) + j) * a.ldx);
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      st[j] = from_float<T>(h[j + 1].x);
      st[TAPS - 1 + j] = from_float<T>(h[j + 1].y);
      st[2 * (TAPS - 1) + j] = from_float<T>(h[j + 1].z);
      st[3 * (TAPS - 1) + j] = from_float<T>(h[j + 1].w);
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

// two fp32 operations per instruction
__device__ __forceinline__ uint64_t f2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unf2(uint64_t x) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(x));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
struct Four { uint64_t lo, hi; };
__device__ __forceinline__ Four four(float4 x) { return {f2(x.x, x.y), f2(x.z, x.w)}; }
__device__ __forceinline__ float4 unfour(Four x) {
  const float2 a = unf2(x.lo), b = unf2(x.hi);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ uint64_t decay2(uint64_t dta) {
  const float2 x = unf2(dta);
  return f2(decay<T>(x.x), decay<T>(x.y));
}

// One step of the states a lane owns (4 G of them): returns its part of y.
template <typename T, int G>
__device__ __forceinline__ float advance(Four (&s)[G], const Four (&A)[G], const float4 (&B)[G], const float4 (&C)[G],
                                         float dt, float dtx) {
  const uint64_t dt2 = f2(dt, dt), dtx2 = f2(dtx, dtx);
  uint64_t y = 0;
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const Four b = four(B[g]), c = four(C[g]);
    s[g].lo = fma2(s[g].lo, decay2<T>(mul2(dt2, A[g].lo)), mul2(dtx2, b.lo));
    s[g].hi = fma2(s[g].hi, decay2<T>(mul2(dt2, A[g].hi)), mul2(dtx2, b.hi));
    y = g == 0 ? mul2(s[g].lo, c.lo) : fma2(s[g].lo, c.lo, y);
    y = fma2(s[g].hi, c.hi, y);
  }
  const float2 r = unf2(y);
  return r.x + r.y;
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
  Four s[G], A[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    s[g] = four(keep && n < a.N ? *reinterpret_cast<const float4*>(S + n) : zero);
    float4 x = n < a.N ? *reinterpret_cast<const float4*>(a.A + (size_t)ch * a.N + n) : zero;
    x.x *= kAUnit<T>; x.y *= kAUnit<T>; x.z *= kAUnit<T>; x.w *= kAUnit<T>;
    A[g] = four(x);
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
    if (live && n < a.N) *reinterpret_cast<float4*>(S + n) = unfour(s[g]);
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
  // [tile][CH], rows apart so that the tokens that a warp stores at once lie on different banks
  static constexpr int LDY = CH + 32 / LN;
  static constexpr int off_y = off_b + kTile * 2 * NP * 4;
  static constexpr int bytes = off_y + kTile * LDY * 4;
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
  Four s[G], A[G];
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    s[g] = four(keep && live && n < a.N ? *reinterpret_cast<const float4*>(S + n) : zero);
    float4 x = live && n < a.N ? *reinterpret_cast<const float4*>(a.A + (size_t)c * a.N + n) : zero;
    x.x *= kLog2e; x.y *= kLog2e; x.z *= kLog2e; x.w *= kLog2e;
    A[g] = four(x);
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
        for (int k = 0; k < 4; ++k) ys[(t + k) * L::LDY + cl] = y[k];
      } else {
        const bool up = ln & 1;
        const float v0 = (up ? y[2] : y[0]) + __shfl_xor_sync(0xffffffffu, up ? y[0] : y[2], 1);
        const float v1 = (up ? y[3] : y[1]) + __shfl_xor_sync(0xffffffffu, up ? y[1] : y[3], 1);
        if constexpr (LN == 2) {
          ys[(t + 2 * up) * L::LDY + cl] = v0;
          ys[(t + 2 * up + 1) * L::LDY + cl] = v1;
        } else {
          const bool up2 = ln & 2;
          float w = (up2 ? v1 : v0) + __shfl_xor_sync(0xffffffffu, up2 ? v0 : v1, 2);
#pragma unroll
          for (int m = 4; m < LN; m <<= 1) w += __shfl_xor_sync(0xffffffffu, w, m);
          if (ln < 4) ys[(t + 2 * up + up2) * L::LDY + cl] = w;
        }
      }
    }
    __syncthreads();
    if (plive) {
      bf* out = reinterpret_cast<bf*>(a.out) + (size_t)(lo + t0) * a.channels + c_first + pc;
#pragma unroll 4
      for (int t = pt; t < n; t += ROWS)
        out[(size_t)t * a.channels] = __float2bfloat16(fmaf(skip, to_float(xs[t * CH + pc]), ys[t * L::LDY + pc]) *
                                                       silu<bf>(to_float(zs[t * CH + pc])));
    }
  }
#pragma unroll
  for (int g = 0; g < G; ++g) {
    const int n = (g * LN + ln) * 4;
    if (live && n < a.N) *reinterpret_cast<float4*>(S + n) = unfour(s[g]);
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

// x [T, channels] with row stride ldx (channels a multiple of 4); out [T, channels]
MSGL_API int msgl_causal_conv_silu(const void* x, long long ldx, const void* w, const void* bias, void* state,
                                   long long slot_stride, const void* cu_q, const void* slots, const void* has_state,
                                   void* out, int B, int channels, int taps, int max_q, int num_slots, int dtype,
                                   cudaStream_t stream) {
  if (B <= 0) return B == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (channels <= 0 || channels % 4 || taps <= 0 || max_q <= 0 || B > 65535 || ldx % 4 || (uintptr_t)x % 16 ||
      (uintptr_t)out % 16 || (uintptr_t)bias % 16)
    return MSGL_BAD_ARG;
  const ConvArgs a{x, ldx, (const float*)w, (const float*)bias, state, slot_stride, (const int32_t*)cu_q,
                   (const int32_t*)slots, (const int32_t*)has_state, out, channels, taps, num_slots};
  const dim3 grid((channels + 511) / 512, (max_q + kStretch - 1) / kStretch, B);
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
