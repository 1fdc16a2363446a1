// Causal prefill / extend attention on the tcgen05 tensor cores: head_dim 128 and an even GQA group, and extended forms
// (rows of 64, any group, windows, chunks, capped scores, a gate on the output, a distance bias, every head on the values of
// all key / value heads).
//
// The reference's prefill kernels (flash_prefill, flash_prefill_paged[_fp8];
// python/minisgl/attention/hip.py:670-792, python/minisgl/attention/rdna4.py:419-503) walk the
// page table inside the attention loop. Here a step is two launches:
//
//   1. kv_gather_kernel copies the K and V rows that this step's requests can see out of the
//      paged pool into a dense 16-bit scratch: K as [Hk][T][128], V transposed as [Hk][128][T],
//      every request starting on a multiple of 128 tokens, rows past a request's length zeroed.
//      fp8 pools are widened here (e4m3 -> 16 bit is exact; the per-head descales are applied
//      to the fp32 scores / output, not to the data). The copy moves a few bytes per token while
//      attention does ~hundreds of FLOP per byte, so it is noise next to the main kernel, and it
//      leaves the main kernel with plain 2-D tensor maps and K-major operands only.
//   2. attn_prefill_tc_kernel: one CTA per (128 query positions of one request, two query heads
//      of one KV head). S = Q K^T and O += P_j V_j are tcgen05.mma (kind::f16, M = N = 128) with
//      S and the output accumulator in tensor memory (2 x 128 + 2 x 128 columns); warp 0 is the
//      TMA producer (Q once, then a 3-slot ring of K_j / V_j tiles), warp 1 issues the MMAs, and
//      two groups of four warps (warps 4-7, 8-11) own one head each: they pull a block of S into
//      registers with tcgen05.ld (which frees S for the next QK^T at once), keep the online-
//      softmax state, rescale O in tensor memory when the running maximum has to move
//      (tcgen05.ld / st, rare), and hand P_j to the MMA through shared memory in the swizzled
//      K-major layout it reads. The two heads alternate on the tensor pipe, so one group's
//      softmax overlaps the other's MMAs. setmaxnreg moves the idle warps' registers to the
//      softmax groups.
//
// A row's result does not depend on which other rows share its tile or on how a prompt was
// chunked: KV blocks are absolute (0, 128, ...), visited in ascending order, and a block that
// is fully masked for a row changes nothing (alpha = 1, P = 0).
#include "common.cuh"
#include "ptx.cuh"

#include <string>

using namespace msgl;
using namespace msgl::ptx;

namespace {

constexpr int kD = 128;            // head dim
constexpr int kTile = 128;         // query rows per head tile, KV rows per block
constexpr int kPanel = 16384;      // 128 rows x 128 bytes (64 16-bit columns), 128B-swizzled
constexpr int kTcThreads = 384;   // warps 0-3: TMA / MMA / two idle; warps 4-7, 8-11: one head each
constexpr float kLog2eTc = 1.4426950408889634f;
constexpr float kFixedCap = 80.f;  // capped scores (in units of log2) up to this need no running maximum: 2^score, summed
                                   // over any number of keys, stays far from both ends of the fp32 and bf16 ranges

struct TcItem {        // one per (request, block of 128 query positions); eight int32
  int q_row0;          // first row of the tile in the packed q / out tensors
  int q_rows;          // valid rows (<= 128)
  int q_pos0;          // absolute position of the first row
  int kv_off;          // first scratch row of the request (multiple of 128)
  int n_blocks;        // KV blocks of 128 the tile can see
  int req;
  int kv_pos0;         // absolute position of the first of those blocks (a multiple of 128; 0 without a window)
  int pad1;
};

struct TcArgs {
  const TcItem* items;
  int n_items, pairs;  // pairs = Hq / 2
  int Hq, Hk;
  long long t_cap;     // scratch rows per KV head
  void* out;
  const float* k_scale;
  const float* v_scale;
  float scale;
  int* status;
  int window;          // > 0: a row sees the last ``window`` positions, its own included
  int chunk;           // > 0: a row sees its own block of this many positions only
  float softcap;       // c > 0: scores go through c tanh(s / c)
  int cgate;           // a sigmoid gate per output channel: its logits come through tma_g, in the layout of q
  long long ldo, ho;   // element strides of a row and a head of out
  int v_chunks;        // 16-byte chunks of a value head
  const float* sink;   // [Hq] logits that only the softmax denominator counts, or null
  const void* gate;    // [rows, ...] logits of a sigmoid gate per row and head (row stride ldg), or null
  long long ldg;
};

__device__ int g_attn_tc_status = 0;

struct TcSmem {
  static constexpr int off_q = 0;                       // [2 heads][2 panels]
  static constexpr int off_p = 4 * kPanel;              // [2 heads][2 panels]
  static constexpr int off_kv = 8 * kPanel;             // [3 slots][2 panels]
  static constexpr int off_bar = 14 * kPanel;
  static constexpr int n_bars = 1 + 3 + 3 + 2 * 5 + 2;
  static constexpr int bytes = off_bar + 256 + 1024;    // + slack to align the base to 1024
};

__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two fp32 operations per instruction
__device__ __forceinline__ uint64_t f2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unf2(uint64_t x, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(x)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// 2^(cap_out tanh(x)) of four scores with cap_in s = 2 x log2(e): tanh(x) = 1 - 2 / (1 + e^(2x)), one reciprocal for the
// four (exponents held at 30, where tanh is 1 in fp32, so that the product stays finite)
__device__ __forceinline__ void capped_exp2(uint32_t* s, uint64_t cap_in, float m2cap, uint64_t cap_out, float (&p)[4]) {
  const uint64_t one = f2(1.f, 1.f);
  float a0, a1, b0, b1, t0, t1;
  unf2(mul2(f2(__uint_as_float(s[0]), __uint_as_float(s[1])), cap_in), a0, a1);
  unf2(mul2(f2(__uint_as_float(s[2]), __uint_as_float(s[3])), cap_in), b0, b1);
  const uint64_t a = add2(f2(ex2f(fminf(a0, 30.f)), ex2f(fminf(a1, 30.f))), one);
  const uint64_t b = add2(f2(ex2f(fminf(b0, 30.f)), ex2f(fminf(b1, 30.f))), one);
  unf2(mul2(a, b), t0, t1);
  const float r = __fdividef(m2cap, t0 * t1);
  const uint64_t rr = f2(r * t1, r * t0);
  unf2(fma2(rr, b, cap_out), a0, a1);
  unf2(fma2(rr, a, cap_out), b0, b1);
  p[0] = ex2f(a0); p[1] = ex2f(a1); p[2] = ex2f(b0); p[3] = ex2f(b1);
}

template <typename T> __device__ __forceinline__ uint32_t pack2_tc(float a, float b);
template <> __device__ __forceinline__ uint32_t pack2_tc<__nv_bfloat16>(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
template <> __device__ __forceinline__ uint32_t pack2_tc<__half>(float a, float b) {
  __half2 h = __floats2half2_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
template <typename T> struct TcFmt;
template <> struct TcFmt<__half> { static constexpr uint32_t fmt = 0; };
template <> struct TcFmt<__nv_bfloat16> { static constexpr uint32_t fmt = 1; };

// ------------------------------------------------------------------------------------------
// 1. Pool -> dense scratch. grid (scratch rows / 64, Hk), 256 threads.
// ------------------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t e4m3x2_to_h2(uint32_t x) {
  uint32_t r;
  asm("{\n\t.reg .b16 t;\n\tcvt.u16.u32 t, %1;\n\tcvt.rn.f16x2.e4m3x2 %0, t;\n\t}" : "=r"(r) : "r"(x));
  return r;
}
template <typename T> __device__ __forceinline__ uint32_t widen2(uint32_t two_bytes) {
  const uint32_t h = e4m3x2_to_h2(two_bytes);
  if constexpr (sizeof(T) == 2 && TcFmt<T>::fmt == 0) {
    return h;
  } else {
    const float2 f = __half22float2(*reinterpret_cast<const __half2*>(&h));
    return pack2_tc<__nv_bfloat16>(f.x, f.y);
  }
}
template <typename T> __device__ __forceinline__ uint4 widen8(uint2 b) {
  uint4 o;
  o.x = widen2<T>(b.x & 0xFFFFu);
  o.y = widen2<T>(b.x >> 16);
  o.z = widen2<T>(b.y & 0xFFFFu);
  o.w = widen2<T>(b.y >> 16);
  return o;
}

template <typename T, bool KV8, int ROW>
__global__ void __launch_bounds__(256)
kv_gather_kernel(const void* __restrict__ k_pool, const void* __restrict__ v_pool, T* __restrict__ kc,
                 T* __restrict__ vt, const int* __restrict__ blk_req, const int* __restrict__ req_info,
                 const int* __restrict__ block_table, int bt_stride, int Hk, int page_size, long long t_cap, int v_rows) {
  pdl_enter();
  __shared__ __align__(16) T vs[64][kD + 8];
  const int t0 = blockIdx.x * 64, h = blockIdx.y;
  const int req = blk_req[t0 >> 7];
  const int kv_off = req_info[3 * req], kv_len = req_info[3 * req + 1], kv_lo = req_info[3 * req + 2];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int id = threadIdx.x + i * 256;
    const int tt = id >> 4, c = id & 15;
    const int tok = t0 + tt - kv_off + kv_lo;
    uint4 kq = make_uint4(0, 0, 0, 0), vq = make_uint4(0, 0, 0, 0);
    if (tok >= kv_lo && tok < kv_len && c * 8 < ROW) {
      const int page = block_table[(long long)req * bt_stride + tok / page_size];
      const long long src = (((long long)page * Hk + h) * page_size + tok % page_size) * ROW + c * 8;
      if constexpr (KV8) {
        kq = widen8<T>(*reinterpret_cast<const uint2*>(reinterpret_cast<const uint8_t*>(k_pool) + src));
        vq = widen8<T>(*reinterpret_cast<const uint2*>(reinterpret_cast<const uint8_t*>(v_pool) + src));
      } else {
        kq = *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(k_pool) + src);
        vq = *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(v_pool) + src);
      }
    }
    *reinterpret_cast<uint4*>(kc + ((long long)h * t_cap + t0 + tt) * kD + c * 8) = kq;
    *reinterpret_cast<uint4*>(&vs[tt][c * 8]) = vq;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int id = threadIdx.x + i * 256;
    const int d = id >> 3, ch = id & 7;
    const uint16_t* col = reinterpret_cast<const uint16_t*>(&vs[ch * 8][d]);
    constexpr int rs = kD + 8;
    uint4 o;
    o.x = (uint32_t)col[0 * rs] | ((uint32_t)col[1 * rs] << 16);
    o.y = (uint32_t)col[2 * rs] | ((uint32_t)col[3 * rs] << 16);
    o.z = (uint32_t)col[4 * rs] | ((uint32_t)col[5 * rs] << 16);
    o.w = (uint32_t)col[6 * rs] | ((uint32_t)col[7 * rs] << 16);
    if (d < v_rows) *reinterpret_cast<uint4*>(vt + ((long long)h * v_rows + d) * t_cap + t0 + ch * 8) = o;
  }
}

// ------------------------------------------------------------------------------------------
// 2. The attention kernel. grid = items x head pairs (heaviest items first), 320 threads.
// ------------------------------------------------------------------------------------------
// POS: the two tiles of a CTA are consecutive blocks of 128 positions of one head (where query heads that share keys
// and values do not come in pairs, K / V tiles can only be shared along the positions) instead of two heads.
// MODE: plain (for two heads: no reach, rows of 128), extended (reach, soft cap, gate, narrower rows), or extended with
// scores that are capped within kFixedCap.
enum { TC_PLAIN = 0, TC_EXTENDED = 1, TC_FIXED_CAP = 2 };
template <typename T, bool POS, int MODE>
__global__ void __launch_bounds__(kTcThreads, 1)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                       const __grid_constant__ CUtensorMap tma_v, const __grid_constant__ CUtensorMap tma_g,
                       const TcArgs args) {
  pdl_enter();
  constexpr bool EXT = MODE != TC_PLAIN, FIXCAP = MODE == TC_FIXED_CAP, REACH = POS || EXT;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t s_base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (s_base - raw);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  const int item_idx = blockIdx.x / args.pairs, pair = blockIdx.x - item_idx * args.pairs;
  const TcItem it = args.items[item_idx];
  const int head0 = POS ? pair : pair * 2;
  const int hk = head0 / (args.Hq / args.Hk);
  const int nb = it.n_blocks;

  const uint32_t q_s = s_base + TcSmem::off_q, p_s = s_base + TcSmem::off_p, kv_s = s_base + TcSmem::off_kv;
  const uint32_t bars = s_base + TcSmem::off_bar;
  auto bar = [&](int i) { return bars + 8u * (uint32_t)i; };
  auto q_full = [&]() { return bar(0); };
  auto kv_full = [&](int s) { return bar(1 + s); };
  auto kv_empty = [&](int s) { return bar(4 + s); };
  auto s_full = [&](int t) { return bar(7 + 5 * t); };
  auto s_free = [&](int t) { return bar(8 + 5 * t); };
  auto p_full = [&](int t) { return bar(9 + 5 * t); };
  auto o_full = [&](int t) { return bar(10 + 5 * t); };
  auto g_full = [&](int t) { return bar(17 + t); };
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + TcSmem::off_bar + 8 * TcSmem::n_bars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + TcSmem::off_bar + 8 * TcSmem::n_bars + 8);

  if (threadIdx.x == 0) {
    mbar_init(q_full(), 1);
    for (int s = 0; s < 3; ++s) { mbar_init(kv_full(s), 1); mbar_init(kv_empty(s), 1); }
    for (int t = 0; t < 2; ++t) {
      mbar_init(s_full(t), 1);
      mbar_init(s_free(t), 128);
      mbar_init(p_full(t), 128);
      mbar_init(o_full(t), 1);
      mbar_init(g_full(t), 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&tma_q);
    prefetch_tensormap(&tma_k);
    prefetch_tensormap(&tma_v);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(const_cast<uint32_t*>(tmem_slot)), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  // The two softmax groups keep a 128-float output row per thread; the first warpgroup gives
  // them its registers (3 warps per scheduler: 56 + 2 x 224 registers x 32 lanes fit 16384).
  if (warp < 4) {
  asm volatile("setmaxnreg.dec.sync.aligned.u32 56;");
  if (warp == 0) {
    // ---------------------------------------------------------------- TMA producer
    if (lane == 0) {
      mbar_expect_tx(q_full(), 4 * kPanel);
      for (int t = 0; t < 2; ++t)
        for (int p = 0; p < 2; ++p)
          tma_load_3d(q_s + (t * 2 + p) * kPanel, &tma_q, q_full(), 64 * p, head0 + (POS ? 0 : t),
                      it.q_row0 + (POS ? t * kTile : 0));
      const int k_row0 = (int)((long long)hk * args.t_cap) + it.kv_off;
      for (int i = 0; i < 2 * nb && !*abort_flag; ++i) {
        const int slot = i % 3, n = i / 3, j = i >> 1;
        if (!mbar_wait(kv_empty(slot), (uint32_t)((n & 1) ^ 1), abort_flag, args.status, 201)) break;
        mbar_expect_tx(kv_full(slot), 2 * kPanel);
        const uint32_t dst = kv_s + slot * 2 * kPanel;
        if constexpr (POS) {
          for (int p = 0; p < 2; ++p) {
            if ((i & 1) == 0) tma_load_3d(dst + p * kPanel, &tma_k, kv_full(slot), 64 * p, hk, it.kv_off + j * kTile);
            else tma_load_3d(dst + p * kPanel, &tma_v, kv_full(slot), it.kv_off + j * kTile + 64 * p, 0, hk);
          }
        } else if ((i & 1) == 0) {
          tma_load_2d(dst, &tma_k, kv_full(slot), 0, k_row0 + j * kTile);
          tma_load_2d(dst + kPanel, &tma_k, kv_full(slot), 64, k_row0 + j * kTile);
        } else {
          tma_load_2d(dst, &tma_v, kv_full(slot), it.kv_off + j * kTile, hk * kD);
          tma_load_2d(dst + kPanel, &tma_v, kv_full(slot), it.kv_off + j * kTile + 64, hk * kD);
        }
      }
      if (*abort_flag) {  // let copies that are still in flight land before the CTA exits
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc = idesc_dense(TcFmt<T>::fmt, TcFmt<T>::fmt, 128, 128);
      auto issue_s = [&](int t, uint32_t k_tile) {
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          mma_f16(tmem_base + t * 128, smem_desc_sw128(q_s + (t * 2 + (kk >> 2)) * kPanel + (kk & 3) * 32),
                  smem_desc_sw128(k_tile + (kk >> 2) * kPanel + (kk & 3) * 32), idesc, kk > 0 ? 1u : 0u);
      };
      auto issue_pv = [&](int t, uint32_t v_tile, bool first) {
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          mma_f16(tmem_base + 256 + t * 128, smem_desc_sw128(p_s + (t * 2 + (kk >> 2)) * kPanel + (kk & 3) * 32),
                  smem_desc_sw128(v_tile + (kk >> 2) * kPanel + (kk & 3) * 32), idesc, (kk > 0 || !first) ? 1u : 0u);
      };
      bool ok = mbar_wait(q_full(), 0, abort_flag, args.status, 202) &&
                mbar_wait(kv_full(0), 0, abort_flag, args.status, 203);
      if (ok) {
        tc_fence_after();
        issue_s(0, kv_s);
        tc_commit(s_full(0));
        issue_s(1, kv_s);
        tc_commit(s_full(1));
        tc_commit(kv_empty(0));
      }
      for (int j = 0; ok && j < nb; ++j) {
        const bool next = j + 1 < nb;
        const int iv = 2 * j + 1, ik = 2 * j + 2;
        if (next && !mbar_wait(kv_full(ik % 3), (uint32_t)((ik / 3) & 1), abort_flag, args.status, 204)) break;
        if (!mbar_wait(kv_full(iv % 3), (uint32_t)((iv / 3) & 1), abort_flag, args.status, 205)) break;
        for (int t = 0; t < 2; ++t) {
          if (next) {
            if (!mbar_wait(s_free(t), (uint32_t)(j & 1), abort_flag, args.status, 206)) { ok = false; break; }
            tc_fence_after();
            issue_s(t, kv_s + (ik % 3) * 2 * kPanel);
            tc_commit(s_full(t));
          }
          if (!mbar_wait(p_full(t), (uint32_t)(j & 1), abort_flag, args.status, 207)) { ok = false; break; }
          tc_fence_after();
          issue_pv(t, kv_s + (iv % 3) * 2 * kPanel, j == 0);
          tc_commit(o_full(t));
        }
        if (!ok) break;
        if (next) tc_commit(kv_empty(ik % 3));
        tc_commit(kv_empty(iv % 3));
      }
    }
  }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 224;");
    // ---------------------------------------------------------------- softmax / output groups
    const int t = (warp - 4) >> 2;               // head of the pair
    const int quarter = warp & 3;                // tensor-memory lanes this warp may read
    const int row = quarter * 32 + lane;
    const int head = head0 + (POS ? 0 : t);
    const int tile_pos0 = it.q_pos0 + (POS ? t * kTile : 0);
    const int q_pos = tile_pos0 + row;
    const uint32_t lane_base = tmem_base + ((uint32_t)(quarter * 32) << 16);
    const uint32_t s_addr = lane_base + t * 128, o_addr = lane_base + 256 + t * 128;
    const uint32_t p_row = p_s + t * 2 * kPanel + row * 128;
    const uint32_t swz = (uint32_t)(row & 7);
    const float raw_scale = args.scale * kLog2eTc * (args.k_scale != nullptr ? args.k_scale[hk] : 1.f);
    // capped scores come out in units of log2: tanh(x) = 1 - 2 / (1 + e^(2x))
    const bool capped = EXT && !FIXCAP && args.softcap > 0.f, gated = EXT && args.cgate;
    const float sl2 = capped ? 1.f : raw_scale;
    const float cap_in = FIXCAP || capped ? 2.f * raw_scale / args.softcap : 0.f, cap_out = args.softcap * kLog2eTc;
    auto below = [&](int pos) {                        // last position ahead of what a row at pos sees
      int lo = -1;
      if (REACH && args.window > 0) lo = pos - args.window;
      if (EXT && args.chunk > 0) lo = max(lo, pos - pos % args.chunk - 1);
      return lo;
    };
    const int lo = below(q_pos), lo_last = below(tile_pos0 + kTile - 1);

    // The output row accumulates in tensor memory across KV blocks. The running maximum is only
    // raised when a block exceeds it by more than 2^8 (probabilities then stay below 256, exact
    // enough in 16 bits and harmless in the fp32 row sum), so rescaling the accumulator - read,
    // multiply, write back - is rare after the first blocks. The decision depends on the row's
    // own history over absolute KV blocks only.
    float m = -INFINITY, l = 0.f;
    uint32_t s[4][32];
    bool ok = true;
    for (int j = 0; j < nb; ++j) {
      const int kv0 = (REACH ? it.kv_pos0 : 0) + j * kTile;
      // the block reaches past some row's position, or starts below some row's window or chunk
      const bool masked = kv0 + kTile - 1 > tile_pos0 || (REACH && kv0 <= lo_last);
      if (!mbar_wait(s_full(t), (uint32_t)(j & 1), abort_flag, args.status, 209)) { ok = false; break; }
      tc_fence_after();
      if (gated && j == nb - 1 && row == 0) {
        // the last product with the query tile is done: the gate's tile takes its place while this block is worked on
        mbar_expect_tx(g_full(t), 2 * kPanel);
        for (int p = 0; p < 2; ++p)
          tma_load_3d(q_s + (t * 2 + p) * kPanel, &tma_g, g_full(t), 64 * p, head, it.q_row0 + (POS ? t * kTile : 0));
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32b_x32(s_addr + c * 32, s[c]);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(s_free(t));                             // S is in registers: the next QK^T may start
      if constexpr (FIXCAP) {
        uint64_t sum = 0;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            float p[4];
            capped_exp2(&s[c][i], f2(cap_in, cap_in), -2.f * cap_out, f2(cap_out, cap_out), p);
            if (masked) {
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const int tok = kv0 + c * 32 + i + e;
                p[e] = tok > q_pos || tok <= lo ? 0.f : p[e];
              }
            }
            sum = add2(sum, add2(f2(p[0], p[1]), f2(p[2], p[3])));
            s[c][i >> 1] = pack2_tc<T>(p[0], p[1]);
            s[c][(i >> 1) + 1] = pack2_tc<T>(p[2], p[3]);
          }
        }
        float s0, s1;
        unf2(sum, s0, s1);
        l += s0 + s1;
        // P V of the previous block is complete: the P buffer is free
        if (j > 0 && !mbar_wait(o_full(t), (uint32_t)((j - 1) & 1), abort_flag, args.status, 210)) { ok = false; break; }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const uint32_t panel = p_row + (uint32_t)(c >> 1) * kPanel;
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            const uint32_t u = (uint32_t)((c & 1) * 4 + g);
            asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(panel + ((u ^ swz) << 4)), "r"(s[c][g * 4]),
                         "r"(s[c][g * 4 + 1]), "r"(s[c][g * 4 + 2]), "r"(s[c][g * 4 + 3])
                         : "memory");
          }
        }
        tc_fence_before();
        fence_proxy_async();
        mbar_arrive(p_full(t));
        continue;
      }
      float mx = -INFINITY;
      if (capped) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            // one reciprocal for four: exponents held at 30 (tanh is 1 there in fp32), so that the product stays finite
            float d[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) d[e] = 1.f + ex2f(fminf(__uint_as_float(s[c][i + e]) * cap_in, 30.f));
            const float p01 = d[0] * d[1], p23 = d[2] * d[3], r = __fdividef(-2.f * cap_out, p01 * p23);
            const float r01 = r * p23, r23 = r * p01;
            s[c][i] = __float_as_uint(fmaf(r01, d[1], cap_out));
            s[c][i + 1] = __float_as_uint(fmaf(r01, d[0], cap_out));
            s[c][i + 2] = __float_as_uint(fmaf(r23, d[3], cap_out));
            s[c][i + 3] = __float_as_uint(fmaf(r23, d[2], cap_out));
          }
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          if (masked && (kv0 + c * 32 + i > q_pos || (REACH && kv0 + c * 32 + i <= lo))) s[c][i] = 0xFF800000u;   // -inf
          mx = fmaxf(mx, __uint_as_float(s[c][i]));
        }
      }
      const bool grow = (mx - m) * sl2 > 8.f;             // false when both are -inf (NaN compares false)
      float alpha = 1.f;
      if (grow) {
        alpha = ex2f((m - mx) * sl2);                     // m = -inf on the first block: 0
        m = mx;
        l *= alpha;
      }
      if (j > 0) {
        // P V of the previous block is complete: the P buffer is free and O may be rescaled
        if (!mbar_wait(o_full(t), (uint32_t)((j - 1) & 1), abort_flag, args.status, 210)) { ok = false; break; }
        tc_fence_after();
        if (__any_sync(0xFFFFFFFFu, grow)) {
          uint32_t r[32];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            tmem_ld_32x32b_x32(o_addr + c * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_32x32b_x32(o_addr + c * 32, r);
          }
          tmem_st_wait();
        }
      }
      // probabilities -> shared memory (K-major, 128-byte swizzle), row sum
      const float mb = (m == -INFINITY ? 0.f : m) * sl2;
      float l_blk = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const uint32_t panel = p_row + (uint32_t)(c >> 1) * kPanel;
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint32_t pk[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = g * 8 + e * 2;
            const float p0 = ex2f(fmaf(__uint_as_float(s[c][i]), sl2, -mb));
            const float p1 = ex2f(fmaf(__uint_as_float(s[c][i + 1]), sl2, -mb));
            l_blk += p0 + p1;
            pk[e] = pack2_tc<T>(p0, p1);
          }
          const uint32_t u = (uint32_t)((c & 1) * 4 + g);
          asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(panel + ((u ^ swz) << 4)), "r"(pk[0]),
                       "r"(pk[1]), "r"(pk[2]), "r"(pk[3])
                       : "memory");
        }
      }
      l += l_blk;
      tc_fence_before();
      fence_proxy_async();
      mbar_arrive(p_full(t));
    }
    if (ok && nb > 0 && mbar_wait(o_full(t), (uint32_t)((nb - 1) & 1), abort_flag, args.status, 211) &&
        (!gated || mbar_wait(g_full(t), 0, abort_flag, args.status, 212))) {
      tc_fence_after();
      const int out_row = row + (POS ? t * kTile : 0);
      float num = args.v_scale != nullptr ? args.v_scale[hk] : 1.f;
      if (POS && args.sink != nullptr) {
        // m is in units of raw scores; the sink is not scaled
        const float sk = args.sink[head] * kLog2eTc, ms = (m == -INFINITY ? 0.f : m) * sl2, mn = fmaxf(ms, sk);
        num *= ex2f(ms - mn);
        l = fmaf(l, ex2f(ms - mn), ex2f(sk - mn));
      }
      if (POS && args.gate != nullptr && out_row < it.q_rows)
        num *= 1.f / (1.f + __expf(-to_float(reinterpret_cast<const T*>(args.gate)[(it.q_row0 + out_row) * args.ldg + head])));
      const float inv = l > 0.f ? num / l : 0.f;
      T* dst = reinterpret_cast<T*>(args.out) +
               (REACH ? (long long)(it.q_row0 + out_row) * args.ldo + head * args.ho
                      : ((long long)(it.q_row0 + row) * args.Hq + head) * kD);
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32b_x32(o_addr + c * 32, s[c]);
      tmem_ld_wait();
      if (out_row < it.q_rows) {
#pragma unroll
        for (int c = 0; c < 16; ++c) {
          if (REACH && c >= args.v_chunks) break;
          uint32_t* o = &s[c >> 2][(c & 3) * 8];
          if (gated) {
            float g[8];
            load8(reinterpret_cast<const T*>(smem + TcSmem::off_q + (t * 2 + (c >> 3)) * kPanel + row * 128 +
                                             (((c & 7) ^ (row & 7)) << 4)),
                  g);
#pragma unroll
            for (int e = 0; e < 8; ++e)
              o[e] = __float_as_uint(__uint_as_float(o[e]) * __fdividef(1.f, 1.f + ex2f(-kLog2eTc * g[e])));
          }
          uint4 v;
          v.x = pack2_tc<T>(__uint_as_float(o[0]) * inv, __uint_as_float(o[1]) * inv);
          v.y = pack2_tc<T>(__uint_as_float(o[2]) * inv, __uint_as_float(o[3]) * inv);
          v.z = pack2_tc<T>(__uint_as_float(o[4]) * inv, __uint_as_float(o[5]) * inv);
          v.w = pack2_tc<T>(__uint_as_float(o[6]) * inv, __uint_as_float(o[7]) * inv);
          *reinterpret_cast<uint4*>(dst + 8 * c) = v;
        }
      }
    } else if (gated && row == 0) {       // gave up: let the gate's copies land before the CTA exits
      const uint64_t t0 = globaltimer_ns();
      while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

// ------------------------------------------------------------------------------------------
// 3. The form with a distance bias and a sink, whose heads may meet the values of all key / value heads. A unit of work is
// (128 query positions, query head, up to two blocks of 128 value columns); one CTA per SM takes units in turn, heaviest
// first, and loads and multiplies for the next one while the last blocks and the output of this one are worked on. S is
// double-buffered in tensor memory (2 x 128 columns) ahead of the output (256 columns). Two teams of eight warps take the
// KV blocks in turn, a thread per query row and half of the block's keys; the running maximum passes from one team to the
// other through shared memory, so that the output has one scale: as above it moves by more than 2^8 only, and then the
// warps that moved it rescale their rows once the block before is in. Two more warps lay out the bias of a block ahead of
// its team: its 255 distances in the order of the keys, in four copies shifted by one float each, so that a row reads its
// own 128 of them as aligned 16-byte words without conflicts.
// ------------------------------------------------------------------------------------------
struct BiasedArgs {
  const TcItem* items;
  int n_units, heads, group, v_blocks, v_groups, all_values;   // v_groups: pairs of value blocks, a unit each
  long long t_cap;
  __nv_bfloat16* out;        // row stride ldo, head stride ho
  long long ldo, ho;
  int v_chunks;              // 16-byte chunks of a value block
  float scale;               // in units of log2
  const float* table;        // [heads][entries]: entry i is minus the bias (in units of log2) at distance zero - i
  int entries, zero;
  const float* sink;         // [heads], or null
  int window;
  int* status;
};

__device__ __forceinline__ void tmem_ld_32x32b_x16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}

struct BiasedSmem {
  static constexpr int slots = 3;
  static constexpr int off_q = 0;                       // 2 panels
  static constexpr int off_p = 2 * kPanel;              // [2 blocks][2 panels]; at a unit's end its output rows
  static constexpr int off_ring = 6 * kPanel;           // [slots][2 panels]
  static constexpr int off_bar = off_ring + slots * 2 * kPanel;
  static constexpr int n_bars = 3 + 2 * slots + 2 * 6;
  // running maxima after a block of either parity [2][128]; maxima of a block's halves [2 teams][2][128]; row sums of the
  // four parts at a unit's end
  static constexpr int off_row = off_bar + 256, off_top = off_row + 1024, off_sum = off_top + 2048;
  static constexpr int copy = 264;                      // floats from one copy of a block's bias to the next: 8 banks on
  static constexpr int off_bias = off_sum + 2048;       // [2 blocks][4 copies]
  static constexpr int bytes = off_bias + 2 * 4 * copy * 4 + 1024;    // + slack to align the base to 1024
};
constexpr int kBiasedThreads = 640;     // warps 0-3: TMA / MMA / bias; warps 4-11, 12-19: the teams

struct BiasedUnit {
  TcItem it;
  int head, hk, vb0, nv;
  __device__ __forceinline__ BiasedUnit(const BiasedArgs& a, int u) {
    const int per_item = a.heads * a.v_groups, i = u / per_item, in_item = u - i * per_item;
    it = a.items[i];
    head = in_item / a.v_groups;
    hk = head / a.group;
    vb0 = a.all_values ? (in_item - head * a.v_groups) * 2 : hk;
    nv = a.all_values ? min(2, a.v_blocks - vb0) : 1;
  }
};

__global__ void __launch_bounds__(kBiasedThreads, 1)
attn_prefill_biased_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                           const __grid_constant__ CUtensorMap tma_v, const BiasedArgs args) {
  pdl_enter();
  using T = __nv_bfloat16;
  using L = BiasedSmem;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t s_base = (raw + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (s_base - raw);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  const uint32_t q_s = s_base + L::off_q, p_s = s_base + L::off_p, ring = s_base + L::off_ring;
  auto bar = [&](int i) { return s_base + L::off_bar + 8u * (uint32_t)i; };
  const uint32_t q_full = bar(0), q_free = bar(1), o_free = bar(2);
  auto kv_full = [&](int s) { return bar(3 + s); };
  auto kv_empty = [&](int s) { return bar(3 + L::slots + s); };
  auto of_block = [&](int kind, int b) { return bar(3 + 2 * L::slots + 2 * kind + b); };
  auto s_full = [&](int b) { return of_block(0, b); };
  auto s_free = [&](int b) { return of_block(1, b); };
  auto p_full = [&](int b) { return of_block(2, b); };
  auto o_done = [&](int b) { return of_block(3, b); };
  auto bias_full = [&](int b) { return of_block(4, b); };
  auto bias_free = [&](int b) { return of_block(5, b); };
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + L::off_bar + 8 * L::n_bars);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::off_bar + 8 * L::n_bars + 8);
  float* row_m = reinterpret_cast<float*>(smem + L::off_row);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(q_free, 1);
    mbar_init(o_free, 512);
    for (int s = 0; s < L::slots; ++s) { mbar_init(kv_full(s), 1); mbar_init(kv_empty(s), 1); }
    for (int b = 0; b < 2; ++b) {
      mbar_init(s_full(b), 1);
      mbar_init(s_free(b), 256);
      mbar_init(p_full(b), 256);
      mbar_init(o_done(b), 1);
      mbar_init(bias_full(b), 64);
      mbar_init(bias_free(b), 256);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&tma_q);
    prefetch_tensormap(&tma_k);
    prefetch_tensormap(&tma_v);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(const_cast<uint32_t*>(tmem_slot)), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  // Blocks are counted through all units of the CTA: block g has the parity g & 1 in every double buffer and is the
  // (g >> 1)-th user of it.
  auto turn = [](int g) { return (uint32_t)((g >> 1) & 1); };

  if (warp < 4) {
    if (warp == 0 && lane == 0) {
      // -------------------------------------------------------------- TMA producer, per unit: Q K0 K1 | K2 V0 | K3 V1 | ...
      int n = 0, k = 0;
      bool ok = true;
      auto take_slot = [&]() {
        const int slot = n % L::slots;
        ok = ok && mbar_wait(kv_empty(slot), (uint32_t)((n / L::slots & 1) ^ 1), abort_flag, args.status, 231);
        if (ok) mbar_expect_tx(kv_full(slot), 2 * kPanel);
        ++n;
        return slot;
      };
      for (int u = blockIdx.x; u < args.n_units && ok; u += gridDim.x, ++k) {
        const BiasedUnit w(args, u);
        const int nb = w.it.n_blocks, k_row0 = (int)((long long)w.hk * args.t_cap) + w.it.kv_off;
        if (k > 0) ok = mbar_wait(q_free, (uint32_t)((k - 1) & 1), abort_flag, args.status, 230);
        if (!ok) break;
        mbar_expect_tx(q_full, 2 * kPanel);
        for (int p = 0; p < 2; ++p) tma_load_3d(q_s + p * kPanel, &tma_q, q_full, 64 * p, w.head, w.it.q_row0);
        auto load_k = [&](int j) {
          const int slot = take_slot();
          for (int p = 0; p < 2 && ok; ++p)
            tma_load_2d(ring + (slot * 2 + p) * kPanel, &tma_k, kv_full(slot), 64 * p, k_row0 + j * kTile);
        };
        for (int j = 0; j < 2 && j < nb && ok; ++j) load_k(j);
        for (int j = 0; j < nb && ok; ++j) {
          if (j + 2 < nb) load_k(j + 2);
          // two value blocks: a slot has 64 keys of both, one operand of 256 rows; one block: its 128 keys
          for (int v = 0; v < w.nv && ok; ++v) {
            const int slot = take_slot();
            for (int p = 0; p < 2 && ok; ++p)
              tma_load_2d(ring + (slot * 2 + p) * kPanel, &tma_v, kv_full(slot),
                          w.it.kv_off + j * kTile + 64 * (w.nv == 2 ? v : p), (w.vb0 + (w.nv == 2 ? p : 0)) * kD);
          }
        }
      }
      if (*abort_flag) {  // let copies that are still in flight land before the CTA exits
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
      }
    } else if (warp == 1 && lane == 0) {
      // -------------------------------------------------------------- MMA issuer
      constexpr uint32_t idesc = idesc_dense(TcFmt<T>::fmt, TcFmt<T>::fmt, 128, 128);
      constexpr uint32_t idesc2 = idesc_dense(TcFmt<T>::fmt, TcFmt<T>::fmt, 128, 256);
      int n = 0, k = 0, g0 = 0;
      bool ok = true;
      auto next_full = [&](int code) {
        ok = ok && mbar_wait(kv_full(n % L::slots), (uint32_t)(n / L::slots & 1), abort_flag, args.status, code);
        return ring + (n % L::slots) * 2 * kPanel;
      };
      for (int u = blockIdx.x; u < args.n_units && ok; u += gridDim.x, ++k) {
        const BiasedUnit w(args, u);
        const int nb = w.it.n_blocks;
        ok = mbar_wait(q_full, (uint32_t)(k & 1), abort_flag, args.status, 232);
        auto issue_s = [&](int j) {
          const int g = g0 + j;
          if (g > 1) ok = ok && mbar_wait(s_free(g & 1), turn(g - 2), abort_flag, args.status, 234);
          const uint32_t k_tile = next_full(233);
          if (!ok) return;
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            mma_f16(tmem_base + (g & 1) * 128, smem_desc_sw128(q_s + (kk >> 2) * kPanel + (kk & 3) * 32),
                    smem_desc_sw128(k_tile + (kk >> 2) * kPanel + (kk & 3) * 32), idesc, kk > 0 ? 1u : 0u);
          tc_commit(s_full(g & 1));
          tc_commit(kv_empty(n % L::slots));
          if (j == nb - 1) tc_commit(q_free);
          ++n;
        };
        for (int j = 0; j < 2 && j < nb && ok; ++j) issue_s(j);
        for (int j = 0; ok && j < nb; ++j) {
          const int g = g0 + j;
          if (j + 2 < nb) issue_s(j + 2);
          // the unit before has read its output
          if (j == 0 && k > 0) ok = ok && mbar_wait(o_free, (uint32_t)((k - 1) & 1), abort_flag, args.status, 229);
          ok = ok && mbar_wait(p_full(g & 1), turn(g), abort_flag, args.status, 235);
          for (int v = 0; v < w.nv && ok; ++v) {
            const uint32_t v_tile = next_full(236);
            if (!ok) break;
            tc_fence_after();
            const uint32_t p_tile = p_s + (g & 1) * 2 * kPanel;
            if (w.nv == 2) {
#pragma unroll
              for (int kk = 0; kk < 4; ++kk)
                mma_f16(tmem_base + 256, smem_desc_sw128(p_tile + v * kPanel + kk * 32), smem_desc_sw128(v_tile + kk * 32),
                        idesc2, (v > 0 || kk > 0 || j > 0) ? 1u : 0u);
            } else {
#pragma unroll
              for (int kk = 0; kk < 8; ++kk)
                mma_f16(tmem_base + 256, smem_desc_sw128(p_tile + (kk >> 2) * kPanel + (kk & 3) * 32),
                        smem_desc_sw128(v_tile + (kk >> 2) * kPanel + (kk & 3) * 32), idesc, (kk > 0 || j > 0) ? 1u : 0u);
            }
            if (v == w.nv - 1) tc_commit(o_done(g & 1));
            tc_commit(kv_empty(n % L::slots));
            ++n;
          }
        }
        g0 += nb;
      }
    } else if (warp >= 2) {
      // -------------------------------------------------------------- bias: entry i of a block is the distance of row r and
      // key k with i = k - r + 127
      const int i0 = (threadIdx.x - 64) * 4;
      int g = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < args.n_units; u += gridDim.x) {
        const BiasedUnit w(args, u);
        const float* line = args.table + (size_t)w.head * args.entries + args.zero - w.it.q_pos0 - 127 + w.it.kv_pos0 + i0;
        for (int j = 0; j < w.it.n_blocks; ++j, ++g) {
          float x[7];
#pragma unroll
          for (int i = 0; i < 7; ++i) x[i] = __ldg(line + j * kTile + i);
          if (g > 1) ok = ok && mbar_wait(bias_free(g & 1), turn(g - 2), abort_flag, args.status, 241);
          float* dst = reinterpret_cast<float*>(smem + L::off_bias) + (g & 1) * 4 * L::copy + i0;
#pragma unroll
          for (int c = 0; c < 4; ++c)
            *reinterpret_cast<float4*>(dst + c * L::copy) = make_float4(x[c], x[c + 1], x[c + 2], x[c + 3]);
          mbar_arrive(bias_full(g & 1));
        }
      }
    }
  } else {
    // ---------------------------------------------------------------- softmax / output teams
    const int part = (warp - 4) >> 2, t = part >> 1, half = part & 1, quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t lane_base = tmem_base + ((uint32_t)(quarter * 32) << 16);
    const uint32_t s_addr = lane_base + t * 128 + half * 64, o_addr = lane_base + 256;
    const uint32_t p_row = p_s + (t * 2 + half) * kPanel + row * 128;
    const uint32_t swz = (uint32_t)(row & 7);
    const int first = 127 - row + half * 64;             // the bias entry of this row and half's first key
    const float4* bias = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(smem + L::off_bias) +
                                                         (t * 4 + (first & 3)) * L::copy + (first & ~3));
    const uint64_t scale2 = f2(args.scale, args.scale);
    float* sums = reinterpret_cast<float*>(smem + L::off_sum);
    float* top_of = reinterpret_cast<float*>(smem + L::off_top) + t * 256;      // [half][128]
    uint32_t s[2][32];
    bool ok = true;
    int g0 = 0;
    for (int u = blockIdx.x; u < args.n_units; u += gridDim.x) {
      const BiasedUnit w(args, u);
      const int nb = w.it.n_blocks, q_pos = w.it.q_pos0 + row;
      const int lo = args.window > 0 ? q_pos - args.window : -1;                // last position ahead of the window
      const int lo_last = args.window > 0 ? w.it.q_pos0 + kTile - 1 - args.window : -1;
      float m = -INFINITY, l = 0.f;
      for (int j = (t ^ g0) & 1; j < nb; j += 2) {
        const int g = g0 + j, kv0 = w.it.kv_pos0 + j * kTile + half * 64;
        ok = ok && mbar_wait(s_full(t), turn(g), abort_flag, args.status, 237);
        tc_fence_after();
        tmem_ld_32x32b_x32(s_addr, s[0]);
        tmem_ld_32x32b_x32(s_addr + 32, s[1]);
        tmem_ld_wait();
        tc_fence_before();
        mbar_arrive(s_free(t));
        ok = ok && mbar_wait(bias_full(t), turn(g), abort_flag, args.status, 242);
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        const bool cut = kv0 + 63 > w.it.q_pos0 || kv0 <= lo_last;   // the half crosses some row's diagonal or window
#pragma unroll
        for (int c = 0; c < 2; ++c) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 x = bias[c * 8 + (i >> 2)];
            float x0, x1, x2, x3;
            unf2(fma2(f2(__uint_as_float(s[c][i]), __uint_as_float(s[c][i + 1])), scale2, f2(x.x, x.y)), x0, x1);
            unf2(fma2(f2(__uint_as_float(s[c][i + 2]), __uint_as_float(s[c][i + 3])), scale2, f2(x.z, x.w)), x2, x3);
            s[c][i] = __float_as_uint(x0);
            s[c][i + 1] = __float_as_uint(x1);
            s[c][i + 2] = __float_as_uint(x2);
            s[c][i + 3] = __float_as_uint(x3);
          }
          if (cut) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const int tok = kv0 + c * 32 + i;
              if (tok > q_pos || tok <= lo) s[c][i] = 0xFF800000u;   // -inf
            }
          }
#pragma unroll
          for (int i = 0; i < 32; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(s[c][i]));
        }
        mbar_arrive(bias_free(t));
        top_of[half * 128 + row] = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
        // both halves of the block; then the other team's decision on the block before, and this one
        asm volatile("bar.sync %0, 256;" ::"r"(4 + t) : "memory");
        const float top = fmaxf(top_of[row], top_of[128 + row]);
        if (j > 0) asm volatile("bar.sync %0, 512;" ::"r"(3 - t) : "memory");
        else asm volatile("bar.sync %0, 256;" ::"r"(4 + t) : "memory");        // the maxima have been read, here too
        const float before = j > 0 ? row_m[(t ^ 1) * 128 + row] : -INFINITY;
        const bool grow = top - before > 8.f;              // false when both are -inf (NaN compares false)
        const float now = grow ? top : before;
        if (half == 0) row_m[t * 128 + row] = now;
        if (j + 1 < nb) asm volatile("bar.arrive %0, 512;" ::"r"(2 + t) : "memory");
        if (now != m) {
          l *= ex2f(m - now);                                // m = -inf: 0
          m = now;
        }
        // (rows that have seen nothing yet have nothing to rescale)
        if (j > 0 && half < w.nv && __any_sync(0xFFFFFFFFu, grow && before != -INFINITY)) {
          // O may be rescaled when the product of the block before is in; a half takes one value block
          ok = ok && mbar_wait(o_done(t ^ 1), turn(g - 1), abort_flag, args.status, 238);
          tc_fence_after();
          const float alpha = grow && before != -INFINITY ? ex2f(before - now) : 1.f;
          uint32_t r[16];
#pragma unroll 1
          for (int c = 0; c < 8; ++c) {
            tmem_ld_32x32b_x16(o_addr + half * 128 + c * 16, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_32x32b_x16(o_addr + half * 128 + c * 16, r);
          }
          tmem_st_wait();
        }
        // the product two blocks ago is in: this team's P buffer is free
        if (g > 1) ok = ok && mbar_wait(o_done(t), turn(g - 2), abort_flag, args.status, 239);
        const float mb = m == -INFINITY ? 0.f : m;
        const uint64_t mb2 = f2(-mb, -mb);
        uint64_t sum[2] = {0, 0};
#pragma unroll
        for (int c = 0; c < 2; ++c) {
#pragma unroll
          for (int gg = 0; gg < 4; ++gg) {
            uint32_t pk[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int i = gg * 8 + e * 2;
              float x0, x1;
              unf2(add2(f2(__uint_as_float(s[c][i]), __uint_as_float(s[c][i + 1])), mb2), x0, x1);
              x0 = ex2f(x0);
              x1 = ex2f(x1);
              sum[e & 1] = add2(sum[e & 1], f2(x0, x1));
              pk[e] = pack2_tc<T>(x0, x1);
            }
            const uint32_t c16 = (uint32_t)(c * 4 + gg);
            asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + ((c16 ^ swz) << 4)), "r"(pk[0]),
                         "r"(pk[1]), "r"(pk[2]), "r"(pk[3])
                         : "memory");
          }
        }
        float l0, l1;
        unf2(add2(sum[0], sum[1]), l0, l1);
        l += l0 + l1;
        tc_fence_before();
        fence_proxy_async();
        mbar_arrive(p_full(t));
      }
      // ---- sums of all parts on the last scale, the sink, the output: a quarter of the value columns each
      const int g_last = g0 + nb - 1;
      asm volatile("bar.sync 1, 512;" ::: "memory");
      const float last = row_m[(g_last & 1) * 128 + row];
      sums[part * 128 + row] = l > 0.f ? l * ex2f(m - last) : 0.f;
      asm volatile("bar.sync 1, 512;" ::: "memory");
      float sum = sums[row] + sums[128 + row] + sums[256 + row] + sums[384 + row];
      ok = ok && mbar_wait(o_done(g_last & 1), turn(g_last), abort_flag, args.status, 240);
      tc_fence_after();
      if (t < w.nv) {
#pragma unroll
        for (int c = 0; c < 2; ++c) tmem_ld_32x32b_x32(o_addr + part * 64 + c * 32, s[c]);
        tmem_ld_wait();
      }
      tc_fence_before();
      mbar_arrive(o_free);
      if (ok && t < w.nv) {
        float num = 1.f;
        if (args.sink != nullptr) {
          const float sk = args.sink[w.head] * kLog2eTc, ms = last == -INFINITY ? sk : last, mn = fmaxf(ms, sk);
          num = ex2f(ms - mn);
          sum = fmaf(sum, num, ex2f(sk - mn));
        }
        const float inv = sum > 0.f ? num / sum : 0.f;
        // through this warp's own rows of P (all products have read them), so that whole lines leave
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const uint32_t* o = &s[c >> 2][(c & 3) * 8];
          asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + (((uint32_t)c ^ swz) << 4)),
                       "r"(pack2_tc<T>(__uint_as_float(o[0]) * inv, __uint_as_float(o[1]) * inv)),
                       "r"(pack2_tc<T>(__uint_as_float(o[2]) * inv, __uint_as_float(o[3]) * inv)),
                       "r"(pack2_tc<T>(__uint_as_float(o[4]) * inv, __uint_as_float(o[5]) * inv)),
                       "r"(pack2_tc<T>(__uint_as_float(o[6]) * inv, __uint_as_float(o[7]) * inv))
                       : "memory");
        }
        __syncwarp();
        const int c = lane & 7;
        T* dst = args.out + w.head * args.ho + (args.all_values ? (w.vb0 + t) * kD : 0) + half * 64 + c * 8;
        if (half * 8 + c < args.v_chunks) {
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int r = quarter * 32 + i * 4 + (lane >> 3);
            if (r < w.it.q_rows)
              *reinterpret_cast<uint4*>(dst + (long long)(w.it.q_row0 + r) * args.ldo) = *reinterpret_cast<const uint4*>(
                  smem + L::off_p + (t * 2 + half) * kPanel + r * 128 + ((c ^ (r & 7)) << 4));
          }
        }
        __syncwarp();
      }
      g0 += nb;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

bool encode_map(CUtensorMap* map, const void* base, int rank, const cuuint64_t* dims, const cuuint64_t* strides,
                const cuuint32_t* box, const char* what) {
  msgl_encode_tiled_fn enc = msgl_get_encode_tiled();
  if (enc == nullptr) return false;
  cuuint32_t estr[5] = {1, 1, 1, 1, 1};
  CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_UINT16, (cuuint32_t)rank, const_cast<void*>(base), dims, strides, box,
                   estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                   CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    msgl_set_error_text((std::string("prefill attention: cuTensorMapEncodeTiled(") + what + ") failed with code " +
                         std::to_string((int)r)).c_str());
    return false;
  }
  return true;
}

template <typename T, bool POS, int MODE>
int launch_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mg, const TcArgs& a,
              cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_prefill_tc_kernel<T, POS, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         TcSmem::bytes);
    if (e != cudaSuccess) { msgl_set_error("prefill attention smem attribute", e); return MSGL_CUDA_ERROR; }
    configured = true;
  }
  msgl_launch(attn_prefill_tc_kernel<T, POS, MODE>, dim3(a.n_items * a.pairs), dim3(kTcThreads), TcSmem::bytes, stream, mq, mk, mv, mg, a);
  MSGL_CHECK_LAUNCH("attn_prefill_tc");
  return MSGL_OK;
}

// Rows of a latent pool ([pages, page_size, R]) a step can see -> dense [t_pad, R]; rows past a request's length are
// zero. req_info: per request (scratch offset, KV length, absolute position of the first scratch row). One warp per row.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pool, uint4* __restrict__ out, const int* __restrict__ blk_req,
                     const int* __restrict__ req_info, const int* __restrict__ block_table, int bt_stride,
                     int page_size, int num_pages, int chunks, int t_pad) {
  pdl_enter();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= t_pad) return;
  const int req = blk_req[row >> 7];
  const int tok = row - req_info[3 * req] + req_info[3 * req + 2];
  const bool in = tok >= 0 && tok < req_info[3 * req + 1];
  long long src = 0;
  if (in) {
    int page = block_table[(long long)req * bt_stride + min(tok / page_size, bt_stride - 1)];
    (void)MSGL_OOB(page, num_pages);
    page = page < 0 ? 0 : (page >= num_pages ? num_pages - 1 : page);
    src = ((long long)page * page_size + tok % page_size) * chunks;
  }
  for (int c = lane; c < chunks; c += 32)
    out[(long long)row * chunks + c] = in ? pool[src + c] : make_uint4(0, 0, 0, 0);
}

}  // namespace

MSGL_API int msgl_latent_gather(const void* pool, void* out, const void* blk_req, const void* req_info,
                                const void* block_table, int bt_stride, int page_size, int num_pages, int R, int t_pad,
                                cudaStream_t stream) {
  if (t_pad <= 0 || t_pad % 128 || R % 8 || (uintptr_t)pool % 16 || (uintptr_t)out % 16 || page_size <= 0 || bt_stride < 1)
    return MSGL_BAD_ARG;
  msgl_launch(latent_gather_kernel, dim3(t_pad / 8), dim3(256), 0, stream, (const uint4*)pool, (uint4*)out,
              (const int*)blk_req, (const int*)req_info, (const int*)block_table, bt_stride, page_size, num_pages, R / 8,
              t_pad);
  MSGL_CHECK_LAUNCH("latent_gather");
  return MSGL_OK;
}

// Windowed causal prefill over keys and values of a step in dense scratch, every head with its own: q [total_q, h]
// heads of dk channels (element strides ldq, hq_stride), k [t_pad, h * dk] row-major, vt [h * dv, t_pad]; out rows of
// h heads of dv channels (strides ldo, ho). dk and dv up to 128, multiples of 8 (channels up to 128 read as zero).
MSGL_API int msgl_attn_prefill_pos(const void* q, long long ldq, long long hq_stride, const void* k, const void* vt,
                                   int t_pad, void* out, long long ldo, long long ho, const void* items, int n_items,
                                   int total_q, int h, int dk, int dv, int window, float scale, const void* sink,
                                   const void* gate, long long ldg, int dtype, cudaStream_t stream) {
  if (n_items == 0 || total_q == 0) return MSGL_OK;
  if (h <= 0 || t_pad % 128 || dk % 8 || dv % 8 || dk > kD || dv > kD || ldq % 8 || hq_stride % 8 || ldo % 8 || ho % 8 ||
      (uintptr_t)q % 16 || (uintptr_t)out % 16 || scale <= 0.f || dtype != MSGL_BF16) {
    msgl_set_error_text("prefill attention: needs bf16 heads of up to 128 channels and a positive scale");
    return MSGL_BAD_ARG;
  }
  CUtensorMap mq, mk, mv;
  cuuint32_t box[3] = {64, 1, 128};
  {
    cuuint64_t dims[3] = {(cuuint64_t)dk, (cuuint64_t)h, (cuuint64_t)total_q};
    cuuint64_t strides[2] = {(cuuint64_t)hq_stride * 2, (cuuint64_t)ldq * 2};
    if (!encode_map(&mq, q, 3, dims, strides, box, "q")) return MSGL_CUDA_ERROR;
  }
  {
    cuuint64_t dims[3] = {(cuuint64_t)dk, (cuuint64_t)h, (cuuint64_t)t_pad};
    cuuint64_t strides[2] = {(cuuint64_t)dk * 2, (cuuint64_t)h * dk * 2};
    if (!encode_map(&mk, k, 3, dims, strides, box, "k")) return MSGL_CUDA_ERROR;
  }
  {
    cuuint64_t dims[3] = {(cuuint64_t)t_pad, (cuuint64_t)dv, (cuuint64_t)h};
    cuuint64_t strides[2] = {(cuuint64_t)t_pad * 2, (cuuint64_t)dv * t_pad * 2};
    cuuint32_t vbox[3] = {64, 128, 1};
    if (!encode_map(&mv, vt, 3, dims, strides, vbox, "v")) return MSGL_CUDA_ERROR;
  }
  TcArgs a = {};
  int* status = nullptr;
  cudaGetSymbolAddress((void**)&status, g_attn_tc_status);
  a.items = (const TcItem*)items; a.n_items = n_items; a.pairs = h; a.Hq = h; a.Hk = h; a.t_cap = t_pad;
  a.out = out; a.scale = scale; a.status = status; a.window = window; a.ldo = ldo; a.ho = ho; a.v_chunks = dv / 8;
  a.sink = (const float*)sink; a.gate = gate; a.ldg = ldg;
  return launch_tc<__nv_bfloat16, true, TC_PLAIN>(mq, mk, mv, mq, a, stream);
}

// Causal prefill / extend attention for one layer. `kc` / `vt` are scratch buffers of
// hk * t_cap * 128 16-bit elements each; `items` (n_items x 8 int32), `blk_req` (t_pad / 128
// int32) and `req_info` (B x 3 int32: scratch offset, KV length, absolute position of the first
// scratch row) describe the step (and the layer's window or chunk) and are built once per step by the caller. q and out
// are [total_q, hq, d] with rows `q_row_stride` / hq * d elements apart, d 64 or 128; items of 128 positions pair
// two query heads of a key / value head, items of 256 (`pos_form`) two blocks of one.
MSGL_API int msgl_attn_prefill_tc(const void* q, long long q_row_stride, void* out, const void* k_pool,
                                  const void* v_pool, void* kc, void* vt, long long t_cap, int t_pad,
                                  const void* items, int n_items, const void* blk_req, const void* req_info,
                                  const void* block_table, int bt_stride, const void* k_scale, const void* v_scale,
                                  int total_q, int hq, int hk, int d, int page_size, int kv_fp8, float scale,
                                  int window, int chunk, float softcap, const void* gate, long long ldg, const void* bias,
                                  int entries, int zero, const void* sink, int all_values, int pos_form, int dtype,
                                  cudaStream_t stream) {
  if (n_items == 0 || total_q == 0) return MSGL_OK;
  if (bias == nullptr ? (all_values || sink != nullptr)
                      : (entries <= 0 || zero < 0 || softcap > 0.f || chunk > 0 || pos_form ||
                         gate != nullptr || dtype != MSGL_BF16 || kv_fp8)) {
    msgl_set_error_text("prefill attention: a distance bias stands without soft cap, chunks, gate and fp8; sinks and mixed heads with one");
    return MSGL_BAD_ARG;
  }
  const bool ext = d != kD || window > 0 || chunk > 0 || softcap > 0.f || gate != nullptr;
  if ((ext || pos_form) && (dtype != MSGL_BF16 || kv_fp8)) {
    msgl_set_error_text("prefill attention: reaches, soft caps, gates, rows of 64 and unpaired query heads need bf16");
    return MSGL_BAD_ARG;
  }
  if (hq % hk || (!pos_form && bias == nullptr && (hq / hk) % 2) || (d != 64 && d != 128) || scale <= 0.f || (gate != nullptr && ldg % 8) ||
      (uintptr_t)gate % 16 || t_cap % 128 || t_pad % 128 || t_pad > t_cap || (q_row_stride % 8) ||
      (dtype != MSGL_BF16 && dtype != MSGL_F16)) {
    msgl_set_error_text("prefill attention: needs rows of 64 or 128, pairs of heads or of blocks, 16-bit q, a positive scale "
                        "and a scratch of whole blocks");
    return MSGL_BAD_ARG;
  }
  const int v_rows = all_values && d == 64 ? 64 : kD;      // value channels of a head in the scratch
  const int v_blocks = all_values ? (hk * d + kD - 1) / kD : hk;
  CUtensorMap mq, mk, mv, mg;
  {
    cuuint64_t dims[3] = {(cuuint64_t)d, (cuuint64_t)hq, (cuuint64_t)total_q};
    cuuint64_t strides[2] = {(cuuint64_t)d * 2, (cuuint64_t)q_row_stride * 2};
    cuuint32_t box[3] = {64, 1, 128};
    if (!encode_map(&mq, q, 3, dims, strides, box, "q")) return MSGL_CUDA_ERROR;
    mg = mq;
    strides[1] = (cuuint64_t)ldg * 2;
    if (gate != nullptr && !encode_map(&mg, gate, 3, dims, strides, box, "gate")) return MSGL_CUDA_ERROR;
  }
  if (pos_form) {
    cuuint64_t kdims[3] = {(cuuint64_t)kD, (cuuint64_t)hk, (cuuint64_t)t_cap};
    cuuint64_t kstr[2] = {(cuuint64_t)t_cap * kD * 2, (cuuint64_t)kD * 2};
    cuuint32_t kbox[3] = {64, 1, 128};
    if (!encode_map(&mk, kc, 3, kdims, kstr, kbox, "k")) return MSGL_CUDA_ERROR;
    cuuint64_t vdims[3] = {(cuuint64_t)t_cap, (cuuint64_t)kD, (cuuint64_t)v_blocks};
    cuuint64_t vstr[2] = {(cuuint64_t)t_cap * 2, (cuuint64_t)t_cap * kD * 2};
    cuuint32_t vbox[3] = {64, 128, 1};
    if (!encode_map(&mv, vt, 3, vdims, vstr, vbox, "v")) return MSGL_CUDA_ERROR;
  } else {
    cuuint64_t dims[2] = {(cuuint64_t)kD, (cuuint64_t)hk * (cuuint64_t)t_cap};
    cuuint64_t strides[1] = {(cuuint64_t)kD * 2};
    cuuint32_t box[2] = {64, 128};
    if (!encode_map(&mk, kc, 2, dims, strides, box, "k")) return MSGL_CUDA_ERROR;
    cuuint64_t vdims[2] = {(cuuint64_t)t_cap, (cuuint64_t)v_blocks * kD};
    cuuint64_t vstr[1] = {(cuuint64_t)t_cap * 2};
    if (!encode_map(&mv, vt, 2, vdims, vstr, box, "v")) return MSGL_CUDA_ERROR;
  }
  int* status = nullptr;
  cudaGetSymbolAddress((void**)&status, g_attn_tc_status);
  const dim3 ggrid(t_pad / 64, hk);
#define GATHER(T, F8, ROW)                                                                                              \
  msgl_launch(kv_gather_kernel<T, F8, ROW>, dim3(ggrid), dim3(256), 0, stream, k_pool, v_pool, (T*)kc, (T*)vt, (const int*)blk_req,          \
                                                     (const int*)req_info, (const int*)block_table, bt_stride, hk, \
                                                     page_size, t_cap, v_rows)
  if (d == 64) GATHER(__nv_bfloat16, false, 64);
  else if (dtype == MSGL_BF16) { if (kv_fp8) GATHER(__nv_bfloat16, true, 128); else GATHER(__nv_bfloat16, false, 128); }
  else { if (kv_fp8) GATHER(__half, true, 128); else GATHER(__half, false, 128); }
#undef GATHER
  MSGL_CHECK_LAUNCH("kv_gather");
  TcArgs a = {};
  a.items = (const TcItem*)items; a.n_items = n_items; a.pairs = pos_form ? hq : hq / 2; a.Hq = hq; a.Hk = hk;
  a.t_cap = t_cap; a.out = out; a.k_scale = (const float*)k_scale; a.v_scale = (const float*)v_scale; a.scale = scale;
  a.status = status; a.window = window; a.chunk = chunk; a.softcap = softcap; a.cgate = gate != nullptr;
  a.ho = all_values ? v_blocks * kD : d; a.ldo = a.ho * hq; a.v_chunks = all_values ? 16 : d / 8;
  if (bias != nullptr) {
    static bool configured = false;
    if (!configured) {
      cudaError_t e = cudaFuncSetAttribute(attn_prefill_biased_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                           BiasedSmem::bytes);
      if (e != cudaSuccess) { msgl_set_error("prefill attention smem attribute", e); return MSGL_CUDA_ERROR; }
      configured = true;
    }
    const int v_groups = all_values ? (v_blocks + 1) / 2 : 1, units = n_items * hq * v_groups;
    static int sms = 0;
    if (sms == 0) {
      int dev = 0;
      cudaGetDevice(&dev);
      cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    }
    BiasedArgs ba{a.items, units, hq, hq / hk, v_blocks, v_groups, all_values, t_cap, (__nv_bfloat16*)out, a.ldo, a.ho,
                  a.v_chunks, scale * kLog2eTc, (const float*)bias, entries, zero, (const float*)sink, window, status};
    msgl_launch(attn_prefill_biased_kernel, dim3(units < sms ? units : sms), dim3(kBiasedThreads), BiasedSmem::bytes, stream, mq,
                mk, mv, ba);
    MSGL_CHECK_LAUNCH("attn_prefill_biased");
    return MSGL_OK;
  }
  const bool fixcap = softcap > 0.f && softcap * kLog2eTc <= kFixedCap && dtype == MSGL_BF16;
  if (pos_form) {
    return fixcap ? launch_tc<__nv_bfloat16, true, TC_FIXED_CAP>(mq, mk, mv, mg, a, stream)
                  : launch_tc<__nv_bfloat16, true, TC_EXTENDED>(mq, mk, mv, mg, a, stream);
  }
  if (fixcap) return launch_tc<__nv_bfloat16, false, TC_FIXED_CAP>(mq, mk, mv, mg, a, stream);
  if (ext) return launch_tc<__nv_bfloat16, false, TC_EXTENDED>(mq, mk, mv, mg, a, stream);
  if (dtype == MSGL_BF16) return launch_tc<__nv_bfloat16, false, TC_PLAIN>(mq, mk, mv, mg, a, stream);
  return launch_tc<__half, false, TC_PLAIN>(mq, mk, mv, mg, a, stream);
}

MSGL_API int msgl_attn_tc_status(int reset) {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_attn_tc_status, sizeof(int));
  if (reset && v != 0) {
    int z = 0;
    cudaMemcpyToSymbol(g_attn_tc_status, &z, sizeof(int));
  }
  return v;
}
