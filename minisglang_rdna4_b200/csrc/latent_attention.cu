// Latent attention: every query head attends to one latent row per position that is key and value
// at once ([pages, page_size, R] of one layer of the latent pool), causal, with a sliding window. A row may end in
// a rotary key that all heads share (the values' projection has zeros there); a head may have a sink, a logit that
// only the softmax denominator counts.
//
//   latent_rope_kernel         rotary channels of the query heads, in place, and in the same launch norm, rotation and
//                              store of this step's latents
//   latent_norm_store_kernel   RMS norm of this step's latents, into their pool slots (in a decode step extra CTAs
//                              of the query projection do it)
//   head_gemm_kernel           per-head projections into and out of the latent space (merging a split's ranges)
//   latent_attention_kernel    bf16: 16 / 32 / 64 (position, head) rows per CTA against 64-token tiles
//                              that are fetched once (cp.async, two or three stages, through the block table)
//                              and serve QK^T and PV; warp-level tensor products, fp32 scores,
//                              softmax and accumulation; optional split of the key range
//   latent_combine_kernel      merges the ranges of a split
//   latent_attention_simt_kernel   fp32 pools (and latents wider than the tensor kernel holds)
//
// Tiles are absolute (0, 64, ...), so what a row adds up does not depend on how its prompt was cut.
#include "common.cuh"
#include "ptx.cuh"

using namespace msgl;
using namespace msgl::ptx;

namespace {

constexpr float kLog2eL = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ------------------------------------------------------------------------------------------ store
template <typename T> struct StoreArgs {
  const T* c;             // [rows, width] with row stride ldc
  long long ldc;
  const float* weight;
  T* pool;
  const int32_t* out_loc;
  int rows, rank, width;
  float eps;
  long long num_slots;
  // a shared key behind the latent: rot_dim channels, the first rot_dims of which are rotated (0: none)
  int rot_dim, rot_dims;
  const float* cos_sin;   // [table_rows, rot_dims]: cosines, then sines
  const int32_t* positions;
  int table_rows;
};

__device__ __forceinline__ void rotate(float& u, float& v, float c, float s) {
  const float a = u * c - v * s;
  v = v * c + u * s;
  u = a;
}
__device__ __forceinline__ int table_row(const int32_t* positions, int t, int rows) {
  int p = positions[t];
  (void)MSGL_OOB(p, rows);
  return p < 0 ? 0 : (p >= rows ? rows - 1 : p);
}

// One warp per row, eight channels per lane and step (width a multiple of 64, up to 1024).
template <typename T> __device__ __forceinline__ void store_latent(const StoreArgs<T>& a, int t, int lane) {
  const T* src = a.c + (size_t)t * a.ldc;
  const long long slot = a.out_loc[t];
  float v[4][8];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int c = (lane + 32 * i) * 8;
    if (c < a.width) {
      if constexpr (sizeof(T) == 2) {
        load8(src + c, v[i]);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = src[c + e];
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      if (c + e >= a.rank) v[i][e] = 0.f;
      s = fmaf(v[i][e], v[i][e], s);
    }
  }
  s = warp_sum(s);
  const float sc = 1.f / sqrtf(s / (float)a.rank + a.eps);
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  T* dst = a.pool + slot * a.width;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int c = (lane + 32 * i) * 8;
    if (c >= a.width) break;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[i][e] *= c + e < a.rank ? sc * a.weight[c + e] : 0.f;
    if constexpr (sizeof(T) == 2) {
      store8(dst + c, v[i]);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) dst[c + e] = v[i][e];
    }
  }
  if (a.rot_dim > 0) {
    __syncwarp();                          // over the zeros just written
    const float* cs = a.rot_dims > 0 ? a.cos_sin + (size_t)table_row(a.positions, t, a.table_rows) * a.rot_dims : nullptr;
    const int half = a.rot_dims / 2;
    for (int i = lane; 2 * i < a.rot_dim; i += 32) {
      float x = to_float(src[a.rank + 2 * i]), y = 2 * i + 1 < a.rot_dim ? to_float(src[a.rank + 2 * i + 1]) : 0.f;
      if (i < half) rotate(x, y, cs[i], cs[half + i]);
      dst[a.rank + 2 * i] = from_float<T>(x);
      if (2 * i + 1 < a.rot_dim) dst[a.rank + 2 * i + 1] = from_float<T>(y);
    }
  }
}

template <typename T> __global__ void __launch_bounds__(128) latent_norm_store_kernel(const StoreArgs<T> a) {
  pdl_enter();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (t < a.rows) store_latent(a, t, threadIdx.x & 31);
}

// `per_row` warps (1 or 4) per row rotate the query heads' pairs; the last of them stores the row's latent after that
// (store.c != null). vec: four pairs are one aligned 16-byte piece (the fp32 form takes them as two).
template <typename T>
__global__ void __launch_bounds__(128) latent_rope_kernel(T* __restrict__ q, long long ldq, long long hq, int H, int first,
                                                          int dims, int per_row, int vec, const StoreArgs<T> a) {
  pdl_enter();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * (4 / per_row) + warp / per_row, part = warp % per_row;
  if (t >= a.rows) return;
  const float* cs = a.cos_sin + (size_t)table_row(a.positions, t, a.table_rows) * dims;
  const int half = dims / 2;
  T* row = q + t * ldq + first;
  if (vec) {
    const int pieces = dims / 8;
#pragma unroll 2
    for (int id = part * 32 + lane; id < H * pieces; id += per_row * 32) {
      const int h = id / pieces, i = (id - h * pieces) * 4;
      T* p = row + h * hq + 2 * i;
      float x[8];
      load8(p, x);
      const float4 c = *reinterpret_cast<const float4*>(cs + i), n = *reinterpret_cast<const float4*>(cs + half + i);
      rotate(x[0], x[1], c.x, n.x);
      rotate(x[2], x[3], c.y, n.y);
      rotate(x[4], x[5], c.z, n.z);
      rotate(x[6], x[7], c.w, n.w);
      store8(p, x);
    }
  } else {
    for (int id = part * 32 + lane; id < H * half; id += per_row * 32) {
      const int h = id / half, i = id - h * half;
      T* p = row + h * hq + 2 * i;
      float x = to_float(p[0]), y = to_float(p[1]);
      rotate(x, y, cs[i], cs[half + i]);
      p[0] = from_float<T>(x);
      p[1] = from_float<T>(y);
    }
  }
  if (a.c != nullptr && part == per_row - 1) store_latent(a, t, lane);
}

// ------------------------------------------------------------------------------------------ attention args
struct LatArgs {
  const void* q;          // [T, H, R]
  const void* pool;       // [pages + 1, page_size, R]
  void* out;              // [T, H, R]
  const int32_t* block_table;
  int bt_stride;
  const int32_t* cu_q;
  const int32_t* seq_lens;
  float* ws_o;            // [splits, T * H, R]
  float* ws_lse;          // [splits, T * H]
  int H, page_size, page_shift, num_pages, window, splits, total_rows;   // num_pages includes the scratch page
  float scale;
  const float* sink;      // [H] or null
};

__device__ __forceinline__ long long token_slot(const LatArgs& a, const int32_t* bt, int tok) {
  // page_shift >= 0: the page size is a power of two
  int col = a.page_shift >= 0 ? tok >> a.page_shift : tok / a.page_size;
  const int in = tok - col * a.page_size;
  col = col < a.bt_stride ? col : a.bt_stride - 1;
  int page = bt[col];
  (void)MSGL_OOB(page, a.num_pages);
  page = page < 0 ? 0 : (page >= a.num_pages ? a.num_pages - 1 : page);
  return (long long)page * a.page_size + in;
}

// One warp per (query row, head); lane i holds the latent channels i, i + 32, ...
template <typename T, int NR>
__global__ void __launch_bounds__(128) latent_attention_simt_kernel(const LatArgs a, int R) {
  pdl_enter();
  const int lane = threadIdx.x & 31;
  const int b = blockIdx.y;
  const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0;
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (row >= q_len * a.H) return;
  const int kv_len = a.seq_lens[b];
  const int pos = kv_len - q_len + row / a.H;
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const size_t off = ((size_t)q0 * a.H + row) * R;
  const T* q = reinterpret_cast<const T*>(a.q) + off;
  const T* pool = reinterpret_cast<const T*>(a.pool);
  const int32_t* bt = a.block_table + (size_t)b * a.bt_stride;
  float qr[NR], o[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    qr[i] = c < R ? to_float(q[c]) * a.scale : 0.f;
    o[i] = 0.f;
  }
  float m = a.sink != nullptr ? a.sink[row % a.H] : -INFINITY, l = a.sink != nullptr ? 1.f : 0.f;
  for (int tok = lo; tok <= pos; ++tok) {
    const T* k = pool + token_slot(a, bt, tok) * R;
    float kr[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = lane + 32 * i;
      kr[i] = c < R ? to_float(k[c]) : 0.f;
      s = fmaf(qr[i], kr[i], s);
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float al = expf(m - mn), p = expf(s - mn);
    m = mn;
    l = fmaf(l, al, p);
#pragma unroll
    for (int i = 0; i < NR; ++i) o[i] = fmaf(o[i], al, p * kr[i]);
  }
  T* out = reinterpret_cast<T*>(a.out) + off;
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    if (c < R) out[c] = from_float<T>(o[i] * inv);
  }
}

// ------------------------------------------------------------------------------------------ tensor-core pieces
__device__ __forceinline__ void ldm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes global -> shared; bytes past ``valid`` (0 or 16) are zero-filled without being read
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t pack_bf(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
// byte offset of 16-byte chunk c of row r in a tile of `chunks` chunks per row (chunks a multiple of 8)
__device__ __forceinline__ uint32_t swz(int r, int c, int chunks) {
  return (uint32_t)(r * chunks + (c ^ (r & 7))) * 16u;
}

// ------------------------------------------------------------------------------------------ per-head GEMM
// out[t, h, n] = sum_k x[t, h, k] w[h, n, k]. 64 rows x 64 columns per CTA, K in panels of 64, two stages;
// four warps, each 16 rows x 64 columns.
struct HeadGemmArgs {
  const __nv_bfloat16* x;
  long long ldx, hx;      // element strides of t and h
  const __nv_bfloat16* w; // [H, N, K]
  __nv_bfloat16* out;
  long long ldo, ho;
  int T, N, K, static_weights;
  // COMBINE: the rows are the ranges of a split attention, merged while they are read
  const float* ws_o;      // [splits, T * H, K]
  const float* ws_lse;    // [splits, T * H]
  int splits, H;
  const __nv_bfloat16* gate;        // [T, ...] logits of the heads' output gates with row stride ldg, or null
  long long ldg;
  StoreArgs<__nv_bfloat16> store;   // store.c != null: the CTAs at blockIdx.y >= H store the step's latents
};

constexpr int kMaxSplits = 16;

template <bool COMBINE>
__global__ void __launch_bounds__(128) head_gemm_kernel(const HeadGemmArgs a) {
  __shared__ __align__(128) uint8_t smem[2][2][64 * 128];
  __shared__ float part[COMBINE ? kMaxSplits : 1][64];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * 64, h = blockIdx.y, t0 = blockIdx.z * 64;
  if (h >= a.H) {                          // a warp per row of this block of 64
    pdl_enter();
    const int r = ((h - a.H) * gridDim.x + blockIdx.x) * 4 + warp;
    if (r < 64 && t0 + r < a.T) store_latent(a.store, t0 + r, lane);
    return;
  }
  const int panels = (a.K + 63) / 64;
  const __nv_bfloat16* xh = a.x + (long long)h * a.hx;
  const __nv_bfloat16* wh = a.w + (long long)h * a.N * a.K;
  auto load = [&](int p, int s, bool weights) {
    const uint32_t dst = smem_u32(smem[s][weights]);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int id = tid + i * 128, r = id >> 3, c = id & 7, k = p * 64 + c * 8;
      if (weights) {
        const bool ok = n0 + r < a.N && k < a.K;
        cp16(dst + swz(r, c, 8), ok ? wh + (long long)(n0 + r) * a.K + k : wh, ok);
      } else if constexpr (COMBINE) {
        float v[8] = {};
        if (t0 + r < a.T && k < a.K) {
          const long long rows = (long long)a.T * a.H;
          const float* src = a.ws_o + ((long long)(t0 + r) * a.H + h) * a.K + k;
#pragma unroll 4
          for (int sp = 0; sp < a.splits; ++sp) {
            const float f = part[sp][r];
            const float4 x = *reinterpret_cast<const float4*>(src + sp * rows * a.K);
            const float4 y = *reinterpret_cast<const float4*>(src + sp * rows * a.K + 4);
            v[0] = fmaf(f, x.x, v[0]); v[1] = fmaf(f, x.y, v[1]); v[2] = fmaf(f, x.z, v[2]); v[3] = fmaf(f, x.w, v[3]);
            v[4] = fmaf(f, y.x, v[4]); v[5] = fmaf(f, y.y, v[5]); v[6] = fmaf(f, y.z, v[6]); v[7] = fmaf(f, y.w, v[7]);
          }
        }
        *reinterpret_cast<uint4*>(smem[s][0] + swz(r, c, 8)) =
            make_uint4(pack_bf(v[0], v[1]), pack_bf(v[2], v[3]), pack_bf(v[4], v[5]), pack_bf(v[6], v[7]));
      } else {
        const bool ok = t0 + r < a.T && k < a.K;
        cp16(dst + swz(r, c, 8), ok ? xh + (long long)(t0 + r) * a.ldx + k : xh, ok);
      }
    }
  };
  if (a.static_weights) load(0, 0, true);   // weights no earlier kernel writes: fetched ahead of the dependency
  pdl_enter();
  if (!a.static_weights) load(0, 0, true);
  if constexpr (COMBINE) {
    if (tid < 64 && t0 + tid < a.T) {
      const long long rows = (long long)a.T * a.H;
      const float* lse = a.ws_lse + (long long)(t0 + tid) * a.H + h;
      float m = -INFINITY, total = 0.f;
      for (int sp = 0; sp < a.splits; ++sp) m = fmaxf(m, lse[sp * rows]);
      for (int sp = 0; sp < a.splits; ++sp) {
        const float f = m == -INFINITY ? 0.f : ex2(lse[sp * rows] - m);
        part[sp][tid] = f;
        total += f;
      }
      const float inv = total > 0.f ? 1.f / total : 0.f;
      for (int sp = 0; sp < a.splits; ++sp) part[sp][tid] *= inv;
    }
    __syncthreads();
  }
  load(0, 0, false);
  cp_commit();
  float acc[8][4] = {};
  for (int p = 0; p < panels; ++p) {
    if (p + 1 < panels) {
      load(p + 1, (p + 1) & 1, true);
      load(p + 1, (p + 1) & 1, false);
    }
    cp_commit();
    cp_wait<1>();
    __syncthreads();
    const uint32_t as = smem_u32(smem[p & 1][0]), bs = smem_u32(smem[p & 1][1]);
    uint32_t af[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ldm_x4(as + swz(warp * 16 + (lane & 15), kk * 2 + (lane >> 4), 8), af[kk]);
#pragma unroll
    for (int nb = 0; nb < 8; ++nb) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t bf[4];
        ldm_x4(bs + swz(nb * 8 + (lane & 7), half * 4 + (lane >> 3), 8), bf);
        mma_bf16(acc[nb], af[half * 2], bf[0], bf[1]);
        mma_bf16(acc[nb], af[half * 2 + 1], bf[2], bf[3]);
      }
    }
    __syncthreads();
  }
  const int r = t0 + warp * 16 + (lane >> 2), col = n0 + (lane & 3) * 2;
  __nv_bfloat16* o = a.out + (long long)h * a.ho;
  if (a.gate != nullptr) {
    const float g0 = r < a.T ? 1.f / (1.f + __expf(-to_float(a.gate[(long long)r * a.ldg + h]))) : 0.f;
    const float g1 = r + 8 < a.T ? 1.f / (1.f + __expf(-to_float(a.gate[(long long)(r + 8) * a.ldg + h]))) : 0.f;
#pragma unroll
    for (int nb = 0; nb < 8; ++nb) {
      acc[nb][0] *= g0; acc[nb][1] *= g0;
      acc[nb][2] *= g1; acc[nb][3] *= g1;
    }
  }
#pragma unroll
  for (int nb = 0; nb < 8; ++nb) {
    const int n = col + nb * 8;
    if (n >= a.N) break;
    if (r < a.T) *reinterpret_cast<uint32_t*>(o + (long long)r * a.ldo + n) = pack_bf(acc[nb][0], acc[nb][1]);
    if (r + 8 < a.T) *reinterpret_cast<uint32_t*>(o + (long long)(r + 8) * a.ldo + n) = pack_bf(acc[nb][2], acc[nb][3]);
  }
}

// ------------------------------------------------------------------------------------------ attention
template <int NP> struct LatentStages { static constexpr int value = NP <= 4 ? 3 : 2; };

// NP: latent panels of 64 channels (R = 64 NP). WM row groups of 16 x WN column groups: a warp owns 16 rows x
// (64 / WN) keys of S and 16 rows x (R / WN) channels of O. KS = 2: the two warps of a pair of column groups
// compute their keys' scores together, half of the channels each (so that the queries are read from shared memory
// half as often, or fit in registers), and exchange the halves.
template <int NP, int WM, int WN, int KS>
__global__ void __launch_bounds__(32 * WM * WN) latent_attention_kernel(const LatArgs a) {
  pdl_enter();
  constexpr int R = NP * 64, MT = 16 * WM, TK = 64, NT = 32 * WM * WN;
  constexpr int CH = R / 8;                      // 16-byte chunks per row
  constexpr int NS = TK / WN / 8;                // key blocks of 8 per warp
  constexpr int NX = NS * KS;                    // ... whose scores it computes over R / KS channels
  constexpr int NO = R / WN / 8;                 // channel blocks of 8 per warp
  constexpr int Q_BYTES = MT * R * 2, C_BYTES = TK * R * 2, ST = LatentStages<NP>::value;
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem) + 127) & ~uintptr_t(127));
  const uint32_t q_s = smem_u32(base), c_s = q_s + Q_BYTES, p_s = c_s + ST * C_BYTES;
  float* red = reinterpret_cast<float*>(base + Q_BYTES + ST * C_BYTES + MT * 128);   // [WN][MT]
  float4* swap = reinterpret_cast<float4*>(red + WN * MT);                            // [warps][NS][32], KS = 2

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp / WN, wn = warp % WN;
  const int b = blockIdx.y, split = blockIdx.z;
  const int q0 = a.cu_q[b], q_len = a.cu_q[b + 1] - q0;
  const int n_rows = q_len * a.H;
  const int row0 = (int)(gridDim.x - 1 - blockIdx.x) * MT;      // late (long) tiles first
  if (row0 >= n_rows) return;
  const int row1 = min(row0 + MT, n_rows);
  const int kv_len = a.seq_lens[b];
  const int pos_first = kv_len - q_len + row0 / a.H, pos_last = kv_len - q_len + (row1 - 1) / a.H;
  const int kv_lo = a.window > 0 ? max(0, pos_first - a.window + 1) : 0;
  const int tile_lo = kv_lo / TK, tiles_all = pos_last / TK + 1 - tile_lo;
  const int per = (tiles_all + a.splits - 1) / a.splits;
  const int t_begin = tile_lo + split * per;
  const int n_tiles = max(0, min(tile_lo + tiles_all, t_begin + per) - t_begin);
  const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(a.pool);
  const int32_t* bt = a.block_table + (size_t)b * a.bt_stride;

  // Pool slots of the tile that is fetched next: lane i knows those of its rows i and i + 32 (-1 past the end), looked
  // up one tile ahead so that the block table's latency is not in front of the copies.
  int next_slot[2];
  auto look_up = [&](int t) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int tok = (t_begin + t) * TK + i * 32 + lane;
      next_slot[i] = t < n_tiles && tok < kv_len ? (int)token_slot(a, bt, tok) : -1;
    }
  };
  auto load_tile = [&](int t) {
    const uint32_t dst = c_s + (t % ST) * C_BYTES;
    const int slot[2] = {next_slot[0], next_slot[1]};
    look_up(t + 1);
#pragma unroll
    for (int i = 0; i < TK * CH / NT; ++i) {
      const int id = tid + i * NT, r = id / CH, c = id % CH;
      const int s0 = __shfl_sync(0xffffffffu, slot[0], r & 31), s1 = __shfl_sync(0xffffffffu, slot[1], r & 31);
      const int sl = r < 32 ? s0 : s1;
      cp16(dst + swz(r, c, CH), pool + (long long)(sl < 0 ? 0 : sl) * R + c * 8, sl >= 0);
    }
  };
  look_up(0);
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q) + ((size_t)q0 * a.H + row0) * R;
    for (int id = tid; id < MT * CH; id += NT) {
      const int r = id / CH, c = id % CH;
      const bool ok = row0 + r < row1;
      cp16(q_s + swz(r, c, CH), ok ? q + (size_t)r * R + c * 8 : q, ok);
    }
  }
#pragma unroll
  for (int t = 0; t < ST - 1; ++t) {             // (the queries belong to the first group)
    if (t < n_tiles) load_tile(t);
    cp_commit();
  }

  // this thread's two rows of the 16-row group
  const int ra = wm * 16 + (lane >> 2), rb = ra + 8;
  const int pa = kv_len - q_len + min(row0 + ra, row1 - 1) / a.H, pb = kv_len - q_len + min(row0 + rb, row1 - 1) / a.H;
  const int lo_a = a.window > 0 ? pa - a.window + 1 : 0, lo_b = a.window > 0 ? pb - a.window + 1 : 0;
  const float sc = a.scale * kLog2eL;
  constexpr int KK = R / 32 / KS;                // steps of 32 channels
  constexpr bool QREG = WM <= KS && KK <= 8;     // few rows: the queries fit in registers
  const int kk0 = KS == 2 ? (wn & 1) * KK : 0, key0 = (KS == 2 ? wn & ~1 : wn) * NS * 8;
  uint32_t qf[QREG ? 2 * KK : 1][4];
  float o[NO][4];
#pragma unroll
  for (int i = 0; i < NO; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;

  for (int t = 0; t < n_tiles; ++t) {
    cp_wait<ST - 2>();
    __syncthreads();                              // tile t has landed; everyone is done with tile t - 1
    if (t + ST - 1 < n_tiles) load_tile(t + ST - 1);
    cp_commit();
    const uint32_t cb = c_s + (t % ST) * C_BYTES;
    float x[NX][4], x2[NX][4];                    // two accumulators: half as long a chain of dependent products
#pragma unroll
    for (int i = 0; i < NX; ++i) {
      x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.f;
      x2[i][0] = x2[i][1] = x2[i][2] = x2[i][3] = 0.f;
    }
    if constexpr (QREG) {
      if (t == 0) {
#pragma unroll
        for (int kk = 0; kk < 2 * KK; ++kk)
          ldm_x4(q_s + swz(wm * 16 + (lane & 15), (kk0 * 2 + kk) * 2 + (lane >> 4), CH), qf[kk]);
      }
    }
#pragma unroll (QREG ? KK : 4)
    for (int kk = 0; kk < KK; ++kk) {
      uint32_t a0[4], a1[4];
      if constexpr (QREG) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          a0[i] = qf[2 * kk][i];
          a1[i] = qf[2 * kk + 1][i];
        }
      } else {
        ldm_x4(q_s + swz(wm * 16 + (lane & 15), (kk0 + kk) * 4 + (lane >> 4), CH), a0);
        ldm_x4(q_s + swz(wm * 16 + (lane & 15), (kk0 + kk) * 4 + 2 + (lane >> 4), CH), a1);
      }
#pragma unroll
      for (int nb = 0; nb < NX; ++nb) {
        uint32_t bf[4];
        ldm_x4(cb + swz(key0 + nb * 8 + (lane & 7), (kk0 + kk) * 4 + (lane >> 3), CH), bf);
        mma_bf16(x[nb], a0, bf[0], bf[1]);
        mma_bf16(KS == 1 ? x2[nb] : x[nb], a1, bf[2], bf[3]);
      }
    }
    float s[NS][4];
    if constexpr (KS == 2) {
      // the partner's key blocks out, this warp's other half of the channels in
      const bool hi = wn & 1;
#pragma unroll
      for (int nb = 0; nb < NS; ++nb) {
        float out_[4];                            // (selected by value: the accumulators stay in registers)
#pragma unroll
        for (int e = 0; e < 4; ++e) out_[e] = hi ? x[nb][e] : x[NS + nb][e];
        swap[((warp ^ 1) * NS + nb) * 32 + lane] = make_float4(out_[0], out_[1], out_[2], out_[3]);
      }
      asm volatile("bar.sync %0, 64;" ::"r"(1 + (warp >> 1)) : "memory");
#pragma unroll
      for (int nb = 0; nb < NS; ++nb) {
        const float4 v = swap[(warp * NS + nb) * 32 + lane];
        const float in[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nb][e] = (hi ? x[NS + nb][e] : x[nb][e]) + in[e];
      }
    } else {
#pragma unroll
      for (int nb = 0; nb < NS; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nb][e] = x[nb][e] + x2[nb][e];
    }
    const int tok0 = (t_begin + t) * TK + wn * (TK / WN) + (lane & 3) * 2;
    float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
    for (int nb = 0; nb < NS; ++nb)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int tok = tok0 + nb * 8 + e;
        const float va = tok <= pa && tok >= lo_a ? s[nb][e] * sc : -INFINITY;
        const float vb = tok <= pb && tok >= lo_b ? s[nb][2 + e] * sc : -INFINITY;
        s[nb][e] = va;
        s[nb][2 + e] = vb;
        mx_a = fmaxf(mx_a, va);
        mx_b = fmaxf(mx_b, vb);
      }
    mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1));
    mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
    mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1));
    mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
    if ((lane & 3) == 0) {
      red[wn * MT + ra] = mx_a;
      red[wn * MT + rb] = mx_b;
    }
    __syncthreads();
#pragma unroll
    for (int w = 0; w < WN; ++w) {
      mx_a = fmaxf(mx_a, red[w * MT + ra]);
      mx_b = fmaxf(mx_b, red[w * MT + rb]);
    }
    const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
    const float ms_a = mn_a == -INFINITY ? 0.f : mn_a, ms_b = mn_b == -INFINITY ? 0.f : mn_b;
    const float al_a = ex2(m_a - ms_a), al_b = ex2(m_b - ms_b);
    m_a = mn_a;
    m_b = mn_b;
    float sum_a = 0.f, sum_b = 0.f;
#pragma unroll
    for (int nb = 0; nb < NS; ++nb) {
      const float p0 = ex2(s[nb][0] - ms_a), p1 = ex2(s[nb][1] - ms_a);
      const float p2 = ex2(s[nb][2] - ms_b), p3 = ex2(s[nb][3] - ms_b);
      sum_a += p0 + p1;
      sum_b += p2 + p3;
      const int chunk = wn * NS + nb, in = (lane & 3) * 4;
      *reinterpret_cast<uint32_t*>(base + (p_s - q_s) + swz(ra, chunk, 8) + in) = pack_bf(p0, p1);
      *reinterpret_cast<uint32_t*>(base + (p_s - q_s) + swz(rb, chunk, 8) + in) = pack_bf(p2, p3);
    }
    l_a = fmaf(l_a, al_a, sum_a);
    l_b = fmaf(l_b, al_b, sum_b);
    if (__any_sync(0xffffffffu, al_a != 1.f || al_b != 1.f)) {
#pragma unroll
      for (int i = 0; i < NO; ++i) {
        o[i][0] *= al_a; o[i][1] *= al_a;
        o[i][2] *= al_b; o[i][3] *= al_b;
      }
    }
    __syncthreads();
    uint32_t pf[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ldm_x4(p_s + swz(wm * 16 + (lane & 15), kk * 2 + (lane >> 4), 8), pf[kk]);
#pragma unroll
    for (int nb = 0; nb < NO; ++nb) {
      const int chunk = wn * NO + nb;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t bf[4];
        ldm_x4_trans(cb + swz(half * 32 + lane, chunk, CH), bf);
        mma_bf16(o[nb], pf[half * 2], bf[0], bf[1]);
        mma_bf16(o[nb], pf[half * 2 + 1], bf[2], bf[3]);
      }
    }
  }
  cp_wait<0>();

  // row sums: quads, then the column groups (every warp kept the sum of its own keys)
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 1);
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 1);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
  __syncthreads();
  if ((lane & 3) == 0) {
    red[wn * MT + ra] = l_a;
    red[wn * MT + rb] = l_b;
  }
  __syncthreads();
  l_a = l_b = 0.f;
#pragma unroll
  for (int w = 0; w < WN; ++w) {
    l_a += red[w * MT + ra];
    l_b += red[w * MT + rb];
  }
  float num_a = 1.f, num_b = 1.f;
  if (a.sink != nullptr && split == 0) {         // counted once, by the first key range
    auto add_sink = [&](int r, float& m, float& l, float& num) {
      const float sk = a.sink[min(row0 + r, row1 - 1) % a.H] * kLog2eL, mn = fmaxf(m, sk);
      num = ex2(m - mn);                         // m = -inf: no key in this range
      l = fmaf(l, num, ex2(sk - mn));
      m = mn;
    };
    add_sink(ra, m_a, l_a, num_a);
    add_sink(rb, m_b, l_b, num_b);
  }
  const float inv_a = l_a > 0.f ? num_a / l_a : 0.f, inv_b = l_b > 0.f ? num_b / l_b : 0.f;
  const size_t row_base = (size_t)q0 * a.H + row0;
  const bool ok_a = row0 + ra < row1, ok_b = row0 + rb < row1;
  const int col = wn * (R / WN) + (lane & 3) * 2;
  if (a.splits == 1) {
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + row_base * R;
#pragma unroll
    for (int nb = 0; nb < NO; ++nb) {
      if (ok_a) *reinterpret_cast<uint32_t*>(out + (size_t)ra * R + col + nb * 8) = pack_bf(o[nb][0] * inv_a, o[nb][1] * inv_a);
      if (ok_b) *reinterpret_cast<uint32_t*>(out + (size_t)rb * R + col + nb * 8) = pack_bf(o[nb][2] * inv_b, o[nb][3] * inv_b);
    }
    return;
  }
  float* wo = a.ws_o + ((size_t)split * a.total_rows + row_base) * R;
#pragma unroll
  for (int nb = 0; nb < NO; ++nb) {
    if (ok_a) *reinterpret_cast<float2*>(wo + (size_t)ra * R + col + nb * 8) = make_float2(o[nb][0] * inv_a, o[nb][1] * inv_a);
    if (ok_b) *reinterpret_cast<float2*>(wo + (size_t)rb * R + col + nb * 8) = make_float2(o[nb][2] * inv_b, o[nb][3] * inv_b);
  }
  if (wn == 0 && (lane & 3) == 0) {
    float* lse = a.ws_lse + (size_t)split * a.total_rows + row_base;
    if (ok_a) lse[ra] = l_a > 0.f ? m_a + log2f(l_a) : -INFINITY;
    if (ok_b) lse[rb] = l_b > 0.f ? m_b + log2f(l_b) : -INFINITY;
  }
}

// One warp per (row, head); R a multiple of 64, up to 640 (five float4 per lane).
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ ws_o,
                                                             const float* __restrict__ ws_lse,
                                                             __nv_bfloat16* __restrict__ out, int rows, int R,
                                                             int splits) {
  pdl_enter();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const float lse = lane < splits ? ws_lse[(size_t)lane * rows + row] : -INFINITY;    // splits <= 16
  float acc[5][4] = {};
  float4 v[5];
  auto fetch = [&](int s) {
#pragma unroll
    for (int i = 0; i < 5; ++i) {
      const int c = lane * 4 + i * 128;
      v[i] = c < R ? *reinterpret_cast<const float4*>(ws_o + ((size_t)s * rows + row) * R + c)
                   : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  const float m = warp_max(lse);
  float w = m == -INFINITY ? 0.f : ex2(lse - m);
  const float total = warp_sum(w);
  w = total > 0.f ? w / total : 0.f;
#pragma unroll 4
  for (int s = 0; s < splits; ++s) {
    fetch(s);
    const float f = __shfl_sync(0xffffffffu, w, s);
#pragma unroll
    for (int i = 0; i < 5; ++i) {
      acc[i][0] = fmaf(f, v[i].x, acc[i][0]);
      acc[i][1] = fmaf(f, v[i].y, acc[i][1]);
      acc[i][2] = fmaf(f, v[i].z, acc[i][2]);
      acc[i][3] = fmaf(f, v[i].w, acc[i][3]);
    }
  }
#pragma unroll
  for (int i = 0; i < 5; ++i) {
    const int c = lane * 4 + i * 128;
    if (c < R)
      *reinterpret_cast<uint2*>(out + (size_t)row * R + c) =
          make_uint2(pack_bf(acc[i][0], acc[i][1]), pack_bf(acc[i][2], acc[i][3]));
  }
}

template <int NP, int WM, int WN, int KS>
int launch_latent(const LatArgs& a, int B, int max_q, cudaStream_t s) {
  constexpr int R = NP * 64, MT = 16 * WM;
  constexpr int bytes = MT * R * 2 + LatentStages<NP>::value * 64 * R * 2 + MT * 128 + WN * MT * 4 + 128 +
                        (KS == 2 ? WM * WN * (8 / WN) * 512 : 0);
  static bool set = false;
  if (!set) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<NP, WM, WN, KS>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) {
      msgl_set_error("latent_attention smem", e);
      return MSGL_CUDA_ERROR;
    }
    set = true;
  }
  dim3 grid((max_q * a.H + MT - 1) / MT, B, a.splits);
  msgl_launch(latent_attention_kernel<NP, WM, WN, KS>, grid, dim3(32 * WM * WN), bytes, s, a);
  MSGL_CHECK_LAUNCH("latent_attention");
  return MSGL_OK;
}

template <int NP>
int launch_latent_rows(const LatArgs& a, int B, int max_q, bool one_form, cudaStream_t s) {
  const long long rows = one_form ? 64 : (long long)max_q * a.H;
  if constexpr (NP > 8) {                  // 64 rows of queries would not fit beside two tiles
    if (rows <= 16) return launch_latent<NP, 1, 8, 2>(a, B, max_q, s);
    return launch_latent<NP, 2, 8, 2>(a, B, max_q, s);
  } else if constexpr (NP > 4) {                  // a wide latent leaves room for one CTA per SM: sixteen warps of it
    if (rows <= 16) return launch_latent<NP, 1, 8, 2>(a, B, max_q, s);
    if (rows <= 32) return launch_latent<NP, 2, 8, 2>(a, B, max_q, s);
    return launch_latent<NP, 4, 4, 1>(a, B, max_q, s);
  } else {
    if (rows <= 16) return launch_latent<NP, 1, 8, 1>(a, B, max_q, s);
    if (rows <= 32) return launch_latent<NP, 2, 4, 1>(a, B, max_q, s);
    return launch_latent<NP, 4, 2, 1>(a, B, max_q, s);
  }
}

template <typename T>
int launch_simt(const LatArgs& a, int R, int B, int max_q, cudaStream_t s) {
  dim3 grid((max_q * a.H + 3) / 4, B);
  if (R <= 64) msgl_launch(latent_attention_simt_kernel<T, 2>, grid, dim3(128), 0, s, a, R);
  else if (R <= 128) msgl_launch(latent_attention_simt_kernel<T, 4>, grid, dim3(128), 0, s, a, R);
  else if (R <= 256) msgl_launch(latent_attention_simt_kernel<T, 8>, grid, dim3(128), 0, s, a, R);
  else if (R <= 512) msgl_launch(latent_attention_simt_kernel<T, 16>, grid, dim3(128), 0, s, a, R);
  else if (R <= 1024) msgl_launch(latent_attention_simt_kernel<T, 32>, grid, dim3(128), 0, s, a, R);
  else return MSGL_BAD_ARG;
  MSGL_CHECK_LAUNCH("latent_attention_simt");
  return MSGL_OK;
}

}  // namespace

MSGL_API int msgl_latent_norm_store(const void* c, long long ldc, const void* weight, void* pool, const void* out_loc,
                                    int rows, int rank, int width, float eps, long long num_slots, int dtype,
                                    cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (rank <= 0 || rank > width || width % 64 || width > 1024 || ldc % 8 || (uintptr_t)c % 16 || (uintptr_t)pool % 16)
    return MSGL_BAD_ARG;
  dim3 grid((rows + 3) / 4);
#define STORE(T)                                                                                                    \
  msgl_launch(latent_norm_store_kernel<T>, grid, dim3(128), 0, stream,                                              \
              StoreArgs<T>{(const T*)c, ldc, (const float*)weight, (T*)pool, (const int32_t*)out_loc, rows, rank,   \
                           width, eps, num_slots, 0, 0, nullptr, nullptr, 0})
  if (dtype == MSGL_BF16) STORE(__nv_bfloat16);
  else if (dtype == MSGL_F32) STORE(float);
  else return MSGL_BAD_ARG;
#undef STORE
  MSGL_CHECK_LAUNCH("latent_norm_store");
  return MSGL_OK;
}

// q [rows, H, ...] (element strides ldq, hq): channels first .. first + dims of every head are rotated in place by
// cos_sin [table_rows, dims] at positions [rows]. c != null: the rows' latents (and rot_dim channels of shared key behind
// them) are normed, rotated and stored as in msgl_latent_norm_store.
MSGL_API int msgl_latent_rope(void* q, long long ldq, long long hq, int H, int first, int dims, const void* cos_sin,
                              const void* positions, int table_rows, const void* c, long long ldc, const void* weight,
                              void* pool, const void* out_loc, int rows, int rank, int width, int rot_dim, float eps,
                              long long num_slots, int dtype, cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (H <= 0 || dims <= 0 || dims % 2 || first < 0 || table_rows <= 0) return MSGL_BAD_ARG;
  if (c != nullptr && (rank <= 0 || rot_dim < dims || rank + rot_dim > width || width % 64 || width > 1024 || ldc % 8 ||
                       (uintptr_t)c % 16 || (uintptr_t)pool % 16))
    return MSGL_BAD_ARG;
  // many rows: a warp each, the loads in flight come from the grid
  const int per_row = rows <= 1024 ? 4 : 1;
  const int vec = first % 8 == 0 && dims % 8 == 0 && ldq % 8 == 0 && hq % 8 == 0 && (uintptr_t)q % 16 == 0 &&
                  (uintptr_t)cos_sin % 16 == 0;
#define ROPE(T)                                                                                                     \
  msgl_launch(latent_rope_kernel<T>, dim3((rows * per_row + 3) / 4), dim3(128), 0, stream, (T*)q, ldq, hq, H, first, \
              dims, per_row, vec,                                                                                   \
              StoreArgs<T>{(const T*)c, ldc, (const float*)weight, (T*)pool, (const int32_t*)out_loc, rows, rank,   \
                           width, eps, num_slots, rot_dim, dims, (const float*)cos_sin, (const int32_t*)positions,  \
                           table_rows})
  if (dtype == MSGL_BF16) ROPE(__nv_bfloat16);
  else if (dtype == MSGL_F32) ROPE(float);
  else return MSGL_BAD_ARG;
#undef ROPE
  MSGL_CHECK_LAUNCH("latent_rope");
  return MSGL_OK;
}

MSGL_API int msgl_head_gemm(const void* x, long long ldx, long long hx, const void* w, void* out, long long ldo,
                            long long ho, int T, int H, int N, int K, int static_weights, const void* ws_o, const void* ws_lse,
                            int splits, const void* gate, long long ldg, const void* c, long long ldc, const void* norm, void* pool,
                            const void* out_loc, int rank, int width, float eps, long long num_slots,
                            cudaStream_t stream) {
  if (T <= 0) return T == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (H <= 0 || H > 65535 || N % 8 || K % 8 || ldx % 8 || hx % 8 || ldo % 2 || ho % 2 || (uintptr_t)x % 16 ||
      (uintptr_t)w % 16 || (uintptr_t)out % 4 || T > 65535 * 64)
    return MSGL_BAD_ARG;
  HeadGemmArgs a{(const __nv_bfloat16*)x, ldx, hx, (const __nv_bfloat16*)w, (__nv_bfloat16*)out, ldo, ho, T, N, K,
                 static_weights, (const float*)ws_o, (const float*)ws_lse, splits, H, (const __nv_bfloat16*)gate, ldg,
                 StoreArgs<__nv_bfloat16>{(const __nv_bfloat16*)c, ldc, (const float*)norm, (__nv_bfloat16*)pool,
                                          (const int32_t*)out_loc, T, rank, width, eps, num_slots, 0, 0, nullptr, nullptr,
                                          0}};
  if (c != nullptr && (rank <= 0 || rank > width || width % 64 || width > 1024 || ldc % 8 || (uintptr_t)c % 16 ||
                       (uintptr_t)pool % 16 || H > 65000))
    return MSGL_BAD_ARG;
  const int nx = (N + 63) / 64;
  dim3 grid(nx, H + (c != nullptr ? (16 + nx - 1) / nx : 0), (T + 63) / 64);
  if (splits > 1) {
    if (splits > kMaxSplits || ws_o == nullptr || ws_lse == nullptr || (uintptr_t)ws_o % 16) return MSGL_BAD_ARG;
    msgl_launch(head_gemm_kernel<true>, grid, dim3(128), 0, stream, a);
  } else {
    msgl_launch(head_gemm_kernel<false>, grid, dim3(128), 0, stream, a);
  }
  MSGL_CHECK_LAUNCH("head_gemm");
  return MSGL_OK;
}

// one_form: the 64-row form whatever the step's size, for callers whose rows must come out bit for bit the same in
// steps of different sizes.
MSGL_API int msgl_latent_attention(const void* q, const void* pool, void* out, const void* block_table, int bt_stride,
                                   const void* cu_q, const void* seq_lens, void* ws_o, void* ws_lse, int B, int total_q,
                                   int max_q, int H, int R, int page_size, int num_pages, int window, int splits,
                                   float scale, const void* sink, int one_form, int dtype, cudaStream_t stream) {
  if (B <= 0 || total_q <= 0) return B == 0 || total_q == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (max_q <= 0 || H <= 0 || R % 64 || page_size <= 0 || num_pages <= 0 || B > 65535 || splits < 1 || bt_stride < 1 ||
      splits > kMaxSplits || (uintptr_t)q % 16 || (uintptr_t)pool % 16 || (uintptr_t)out % 16 || (out == nullptr && splits == 1))
    return MSGL_BAD_ARG;
  int shift = -1;
  for (int i = 0; i < 31; ++i)
    if ((1 << i) == page_size) shift = i;
  LatArgs a{q, pool, out, (const int32_t*)block_table, bt_stride, (const int32_t*)cu_q, (const int32_t*)seq_lens,
            (float*)ws_o, (float*)ws_lse, H, page_size, shift, num_pages, window, splits, total_q * H, scale,
            (const float*)sink};
  if (dtype == MSGL_F32) return launch_simt<float>(a, R, B, max_q, stream);
  if (dtype != MSGL_BF16) return MSGL_BAD_ARG;
  if (R > 512 && R != 576) {
    a.splits = 1;
    if (splits > 1) return MSGL_BAD_ARG;
    return launch_simt<__nv_bfloat16>(a, R, B, max_q, stream);
  }
  if (splits > 1 && (ws_o == nullptr || ws_lse == nullptr)) return MSGL_BAD_ARG;
  int rc;
  switch (R / 64) {
    case 1: rc = launch_latent_rows<1>(a, B, max_q, one_form != 0, stream); break;
    case 2: rc = launch_latent_rows<2>(a, B, max_q, one_form != 0, stream); break;
    case 3: rc = launch_latent_rows<3>(a, B, max_q, one_form != 0, stream); break;
    case 4: rc = launch_latent_rows<4>(a, B, max_q, one_form != 0, stream); break;
    case 8: rc = launch_latent_rows<8>(a, B, max_q, one_form != 0, stream); break;
    case 9: rc = launch_latent_rows<9>(a, B, max_q, one_form != 0, stream); break;
    default: return MSGL_BAD_ARG;
  }
  // without a destination the ranges stay apart: the projection out of the latent space merges them
  if (rc != MSGL_OK || splits == 1 || out == nullptr) return rc;
  msgl_launch(latent_combine_kernel, dim3((total_q * H + 3) / 4), dim3(128), 0, stream, (const float*)ws_o,
              (const float*)ws_lse, (__nv_bfloat16*)out, total_q * H, R, splits);
  MSGL_CHECK_LAUNCH("latent_combine");
  return MSGL_OK;
}
