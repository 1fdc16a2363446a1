// Decode attention of layers whose heads mix their weights: out[h] = sum_g talk[h, g] (weights of head g on the values of h's
// key / value head), with a distance bias on the scores and a sink in the softmax denominator. Single query rows over the
// paged pool (decode, draft verification, short extends over long prefixes), bf16.
//
// A CTA has one query row, one range of keys (a split) and all query heads, so that keys and values cross HBM once: the
// weights of every head meet the values of every key / value head, and the mixture is taken at the end, when the softmax
// denominators are known. Per block of 64 keys eight consumer warps take three steps: S^T = K Q^T with the keys on the
// 16-row side of the warp MMA and the heads of a group on the 8-column side; softmax, a warp per row; O += P V with the
// heads on the 16-row side, a warp per slice of value columns. Two producer warps stream the block's K tiles, then its V
// tiles, through a ring of shared-memory slots with 16-byte asynchronous copies (a TMA box ends at a page and at 128 bytes,
// and issuing so many small ones takes longer than the copies). Ranges are merged, and heads mixed, by talk_merge_kernel.
#include "common.cuh"
#include "ptx.cuh"

using namespace msgl;
using namespace msgl::ptx;

namespace {

constexpr int TK = 64;            // keys per block
constexpr int kWarps = 8;         // consumer warps
constexpr int kCopyThreads = 64;
constexpr float kLog2e = 1.4426950408889634f;
using bf = __nv_bfloat16;

__device__ int g_talk_status = 0;

struct TalkArgs {
  const bf* q;              // [rows, H, D]
  const bf* k;              // [pages, Hk, page_size, D]
  const bf* v;
  bf* out;                  // [rows, H, D]
  const int32_t* block_table;
  const int32_t* cu_q;
  const int32_t* seq_lens;
  const float* bias;        // [H, reach], or null
  const float* sink;        // [H], or null
  const float* talk;        // [H, H]
  float* ws;                // splits > 1: O [splits][rows][H][Hk * D], then m and l [splits][rows][H]
  int bt_stride, B, rows, H, Hk, page_size, num_pages, reach, window, splits, decode;
  float scale;
  int* status;
};

__device__ __forceinline__ void ldm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void consumers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kWarps * 32) : "memory"); }

// MT: 16-row blocks of heads; GN: key / value heads whose values a CTA takes (grid.y of such groups)
template <int D, int MT, int GN> struct TalkSmem {
  static constexpr int slot = TK * D * 2;
  static constexpr int rows = MT * 16;
  static constexpr int ldq = D * 2 + 16, lds = TK + 4, ldp = TK + 8;     // bytes, floats, elements
  static constexpr int off_q = 0;
  static constexpr int off_s = off_q + rows * ldq;
  static constexpr int off_p = off_s + rows * lds * 4;
  static constexpr int off_row = off_p + rows * ldp * 2;                 // alpha, m, l: [rows] each
  static constexpr int off_bar = off_row + rows * 12;
  static constexpr int off_ring = (off_bar + 512 + 1023) / 1024 * 1024;
  static constexpr int per_sm = MT * GN * (D / 64) <= 8 ? 2 : 1;         // CTAs that fit an SM (registers, too)
  static constexpr int fit = (226 * 1024 / per_sm - 1024 - off_ring - 1024) / slot;
  static constexpr int slots = fit < 24 ? fit : 24;
  static constexpr int bytes = off_ring + slots * slot + 1024;
  // the end of a row that is not split: O of all heads in place of the ring
  static_assert(rows * GN * D * 4 <= slots * slot, "O fits the ring");
};

template <int D, int MT, int GN>
__global__ void __launch_bounds__(kWarps * 32 + kCopyThreads, TalkSmem<D, MT, GN>::per_sm) talk_decode_kernel(const TalkArgs a) {
  using L = TalkSmem<D, MT, GN>;
  constexpr int CW = D / 16, VG = kWarps / CW;       // column slices of 16; groups of warps on different value heads
  constexpr int GW = GN / VG > 0 ? GN / VG : 1;      // value heads per warp
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t base = smem_u32(smem), ring = base + L::off_ring;
  auto full = [&](int s) { return base + L::off_bar + 16u * s; };
  auto empty = [&](int s) { return base + L::off_bar + 16u * s + 8u; };
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + L::off_bar + 16 * L::slots);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, c0 = blockIdx.y * GN, row = blockIdx.z;
  const int H = a.H, Hk = a.Hk, gs = H / Hk, nv = min(GN, Hk - c0);

  int b = row;
  if (!a.decode) {
    b = 0;
    int hi = a.B;
    while (hi - b > 1) {
      const int mid = (b + hi) >> 1;
      if (a.cu_q[mid] <= row) b = mid; else hi = mid;
    }
  }
  const int q_lo = a.cu_q[b], q_hi = a.cu_q[b + 1], kv_len = a.seq_lens[b];
  const bool in = row >= q_lo && row < q_hi;         // not padding of a captured batch
  const int pos = kv_len - (q_hi - row);
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int tile_lo = lo / TK, n_all = in && pos >= 0 ? pos / TK + 1 - tile_lo : 0;
  const int per = (n_all + a.splits - 1) / a.splits;
  const int t0 = tile_lo + split * per, n_tiles = max(min(tile_lo + n_all, t0 + per) - t0, 0);

  if (threadIdx.x == 0) {
    for (int s = 0; s < L::slots; ++s) {
      mbar_init(full(s), kCopyThreads);
      mbar_init(empty(s), kWarps);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  __syncthreads();

  if (warp >= kWarps) {
    // ------------------------------------------------------------------ producers
    // Tables and keys of earlier steps may be read before the kernel ahead has finished; only the blocks with this step's
    // own rows wait for it. A thread copies one 16-byte column of every ROWS-th token.
    constexpr int CH = D / 8, ROWS = kCopyThreads / CH, N = TK / ROWS;
    const int32_t* bt = a.block_table + (size_t)b * a.bt_stride;
    const int ps = a.page_size, pages = TK / ps, newest = max(kv_len - (q_hi - q_lo), 0) / TK;
    const int id = threadIdx.x - kWarps * 32, c = id % CH, r0 = id / CH;
    bool waited = false, ok = true;
    int slot = 0;
    uint32_t phase = 1;
    for (int t = 0; t < n_tiles && ok; ++t) {
      int page = bt[min((t0 + t) * pages + lane % pages, a.bt_stride - 1)];
      (void)MSGL_OOB(page, a.num_pages + 1);
      page = page < 0 ? 0 : (page > a.num_pages ? a.num_pages : page);
      int from[N];                 // row of head 0 in the pool
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int tok = r0 + i * ROWS, p = tok / ps;
        from[i] = __shfl_sync(0xffffffffu, page, p) * Hk * ps + tok - p * ps;
      }
      if (!waited && t0 + t >= newest) {
        pdl_wait();
        waited = true;
      }
      for (int i = 0; i < Hk + nv && ok; ++i) {
        const int h = i < Hk ? i : c0 + i - Hk;
        const bf* src = (i < Hk ? a.k : a.v) + c * 8;
        ok = mbar_wait(empty(slot), phase, abort_flag, a.status, 221);
        if (!ok) break;
        const uint32_t dst = ring + slot * L::slot + (c >> 3) * TK * 128;
#pragma unroll
        for (int k = 0; k < N; ++k) {
          const int tok = r0 + k * ROWS;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + tok * 128 + (((c & 7) ^ (tok & 7)) << 4)),
                       "l"(src + (size_t)(from[k] + h * ps) * D) : "memory");
        }
        asm volatile("cp.async.mbarrier.arrive.noinc.shared::cta.b64 [%0];" ::"r"(full(slot)) : "memory");
        if (++slot == L::slots) { slot = 0; phase ^= 1u; }
      }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    return;
  }

  // -------------------------------------------------------------------- consumers
  pdl_enter();
  const int tid = threadIdx.x, j = lane & 3, r8 = lane >> 2, mi = lane >> 3;
  float* S = reinterpret_cast<float*>(smem + L::off_s);
  bf* P = reinterpret_cast<bf*>(smem + L::off_p);
  float* alpha = reinterpret_cast<float*>(smem + L::off_row);
  float* row_m = alpha + L::rows;
  float* row_l = row_m + L::rows;
  for (int i = tid; i < L::rows * (D / 8); i += kWarps * 32) {
    const int h = i / (D / 8), c = i % (D / 8);
    uint4 x = make_uint4(0, 0, 0, 0);
    if (h < H) x = *reinterpret_cast<const uint4*>(a.q + ((size_t)row * H + h) * D + c * 8);
    *reinterpret_cast<uint4*>(smem + L::off_q + h * L::ldq + c * 16) = x;
  }
  for (int i = tid; i < L::rows * L::ldp; i += kWarps * 32) P[i] = __float2bfloat16(0.f);
  float m[MT * 2], l[MT * 2];              // of the rows warp, warp + 8, ...; l is a lane's part
#pragma unroll
  for (int i = 0; i < MT * 2; ++i) { m[i] = -INFINITY; l[i] = 0.f; }
  float o[GW][MT][2][4];
#pragma unroll
  for (int c = 0; c < GW; ++c)
#pragma unroll
    for (int t = 0; t < MT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[c][t][0][e] = o[c][t][1][e] = 0.f;
  consumers_sync();

  const int mt = warp & 3, half = warp >> 2;      // S: key block of 16, and which of the column blocks in turn
  const int nblk = (gs + 7) / 8;
  const int cw = warp % CW, vg = warp / CW;
  int slot = 0;
  uint32_t phase = 0;
  bool ok = true;
  auto next = [&]() { if (++slot == L::slots) { slot = 0; phase ^= 1u; } };
  for (int t = 0; t < n_tiles; ++t) {
    const int tok0 = (t0 + t) * TK;
    // ---- S^T = K Q^T, scaled, less the bias, in units of log2
    for (int c = 0; c < Hk; ++c) {
      const int nb0 = (half + c) & 1;
      // the bias of the first column block, ahead of its keys
      float bias[4] = {};
      auto load_bias = [&](int nb) {
        if (a.bias == nullptr) return;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int h = min(c * gs + nb * 8 + 2 * j + (e & 1), H - 1), far = pos - tok0 - mt * 16 - r8 - (e >> 1) * 8;
          bias[e] = __ldg(a.bias + (size_t)h * a.reach + min(max(far, 0), a.reach - 1));
        }
      };
      if (nb0 < nblk) load_bias(nb0);
      ok = ok && mbar_wait(full(slot), phase, abort_flag, a.status, 222);
      const uint32_t k_s = ring + slot * L::slot;
      for (int nb = nb0; nb < nblk; nb += 2) {
        if (nb > nb0) load_bias(nb);
        float s[4] = {};
        const int trow = mt * 16 + (lane & 15);
        const uint32_t k_row = k_s + trow * 128, q_row = base + L::off_q + min(c * gs + nb * 8 + (lane & 7), L::rows - 1) * L::ldq;
#pragma unroll
        for (int kk = 0; kk < D / 32; ++kk) {
          uint32_t qf[4];                          // heads x 32 channels
          ldm4(q_row + kk * 64 + mi * 16, qf);
#pragma unroll
          for (int k2 = 0; k2 < 2; ++k2) {
            uint32_t kf[4];
            const int ch = kk * 4 + k2 * 2 + (lane >> 4);
            ldm4(k_row + (ch >> 3) * TK * 128 + (((ch & 7) ^ (trow & 7)) << 4), kf);
            mma16816(s, kf, qf[2 * k2], qf[2 * k2 + 1]);
          }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int k = nb * 8 + 2 * j + (e & 1), h = c * gs + k, key = mt * 16 + r8 + (e >> 1) * 8, tok = tok0 + key;
          if (k < gs) {
            S[h * L::lds + key] = tok > pos || tok < lo ? -INFINITY : fmaf(s[e], a.scale, -bias[e]) * kLog2e;
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty(slot));
      next();
    }
    consumers_sync();
    // ---- softmax of the block, a warp per row
#pragma unroll
    for (int i = 0; i < MT * 2; ++i) {
      const int h = warp + i * 8;
      if (h >= H) break;
      const float2 s = *reinterpret_cast<const float2*>(S + h * L::lds + lane * 2);
      const float mn = fmaxf(m[i], warp_max(fmaxf(s.x, s.y)));
      const float ms = mn == -INFINITY ? 0.f : mn, al = ex2f(m[i] - ms);
      const float p0 = ex2f(s.x - ms), p1 = ex2f(s.y - ms);
      l[i] = l[i] * al + p0 + p1;
      m[i] = mn;
      *reinterpret_cast<__nv_bfloat162*>(P + h * L::ldp + lane * 2) = __floats2bfloat162_rn(p0, p1);
      if (lane == 0) alpha[h] = al;
    }
    consumers_sync();
    // ---- O += P V
    uint32_t pf[MT][TK / 16][4];
#pragma unroll
    for (int k = 0; k < MT; ++k) {
      const float a0 = k * 16 + r8 < H ? alpha[k * 16 + r8] : 0.f, a1 = k * 16 + r8 + 8 < H ? alpha[k * 16 + r8 + 8] : 0.f;
#pragma unroll
      for (int c = 0; c < GW; ++c)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o[c][k][n][0] *= a0; o[c][k][n][1] *= a0;
          o[c][k][n][2] *= a1; o[c][k][n][3] *= a1;
        }
#pragma unroll
      for (int ks = 0; ks < TK / 16; ++ks)
        ldm4(base + L::off_p + ((k * 16 + (lane & 15)) * L::ldp + ks * 16 + (lane >> 4) * 8) * 2, pf[k][ks]);
    }
#pragma unroll
    for (int c = 0; c < GN; ++c) {
      if (c >= nv) break;
      ok = ok && mbar_wait(full(slot), phase, abort_flag, a.status, 223);
      if (VG == 1 || c % VG == vg) {
        const uint32_t v_s = ring + slot * L::slot;
#pragma unroll
        for (int ks = 0; ks < TK / 16; ++ks) {
          const int trow = ks * 16 + (mi & 1) * 8 + (lane & 7), ch = cw * 2 + (mi >> 1);
          uint32_t vf[4];
          ldm4t(v_s + (ch >> 3) * TK * 128 + trow * 128 + (((ch & 7) ^ (trow & 7)) << 4), vf);
#pragma unroll
          for (int k = 0; k < MT; ++k) {
            mma16816(o[c / VG][k][0], pf[k][ks], vf[0], vf[1]);
            mma16816(o[c / VG][k][1], pf[k][ks], vf[2], vf[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty(slot));
      next();
    }
  }

  // ---- the row's maxima and sums
#pragma unroll
  for (int i = 0; i < MT * 2; ++i) {
    const int h = warp + i * 8;
    if (h >= H) break;
    const float sum = warp_sum(l[i]);
    if (a.splits > 1) {
      if (lane == 0 && c0 == 0) {
        const size_t rh = (size_t)a.rows * H, at = split * rh + (size_t)row * H + h;
        float* tail = a.ws + a.splits * rh * Hk * D;
        tail[at] = m[i];
        tail[a.splits * rh + at] = sum;
      }
    } else if (lane == 0) {
      float num = 1.f, den = sum;
      if (a.sink != nullptr) {
        const float sk = a.sink[h] * kLog2e, mn = fmaxf(m[i], sk);
        num = ex2f(m[i] - mn);
        den = sum * num + ex2f(sk - mn);
      }
      row_m[h] = den > 0.f ? num / den : 0.f;
    }
  }
  if (a.splits > 1) {
    if (n_tiles == 0) return;              // its maximum says that there is nothing to read
    float* dst = a.ws + ((size_t)split * a.rows + row) * H * Hk * D;
#pragma unroll
    for (int c = 0; c < GW; ++c) {
      const int cc = c * VG + vg;
      if (cc >= nv) continue;
#pragma unroll
      for (int k = 0; k < MT; ++k)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const int h = k * 16 + r8 + e * 4;
            if (h < H)
              *reinterpret_cast<float2*>(dst + ((size_t)h * Hk + c0 + cc) * D + cw * 16 + n * 8 + 2 * j) =
                  make_float2(o[c][k][n][e], o[c][k][n][e + 1]);
          }
    }
    return;
  }
  // ---- one range: heads are mixed here. Every slot has been read (the copies have landed: each was waited for).
  consumers_sync();
  float* O = reinterpret_cast<float*>(smem + L::off_ring);      // [H][GN * D]
#pragma unroll
  for (int c = 0; c < GW; ++c) {
    const int cc = c * VG + vg;
#pragma unroll
    for (int k = 0; k < MT; ++k)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int h = k * 16 + r8 + e * 4;
          if (h < H && cc < nv)
            *reinterpret_cast<float2*>(O + h * GN * D + cc * D + cw * 16 + n * 8 + 2 * j) =
                make_float2(o[c][k][n][e] * row_m[h], o[c][k][n][e + 1] * row_m[h]);
        }
  }
  consumers_sync();
  // a thread sums one pair of channels of one value head, for four heads at a time
  const int pairs = nv * D / 2, parts = max(kWarps * 32 / pairs, 1);
  for (int id = tid; id < pairs * parts; id += kWarps * 32) {
    const int part = id / pairs, col = (id - part * pairs) * 2, c = c0 + col / D;
    for (int h0 = part * 4; h0 < gs; h0 += parts * 4) {
      float acc[4][2] = {};
      for (int g = 0; g < H; ++g) {
        const float2 x = *reinterpret_cast<const float2*>(O + g * GN * D + col);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float f = h0 + k < gs ? __ldg(a.talk + (size_t)(c * gs + h0 + k) * H + g) : 0.f;
          acc[k][0] = fmaf(f, x.x, acc[k][0]);
          acc[k][1] = fmaf(f, x.y, acc[k][1]);
        }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (h0 + k < gs)
          *reinterpret_cast<__nv_bfloat162*>(a.out + ((size_t)row * H + c * gs + h0 + k) * D + col % D) =
              __floats2bfloat162_rn(acc[k][0], acc[k][1]);
    }
  }
}

// Merge of the ranges and mixture of the heads: grid (rows, Hk, parts of the group), a warp per query head in turn (four
// channels per lane; two heads at a time at D = 64), eight mixed heads in its registers, summed over the warps at the end.
template <int D>
__global__ void __launch_bounds__(256) talk_merge_kernel(const TalkArgs a) {
  pdl_enter();
  extern __shared__ float sm[];              // weight of (split, head): [splits][H]; talk rows [H][8]; sums [8 warps][8][D]
  constexpr int PER = 128 / D;               // heads side by side in a warp
  const int row = blockIdx.x, c = blockIdx.y, H = a.H, gs = H / a.Hk, h0 = blockIdx.z * 8, n = min(8, gs - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t rh = (size_t)a.rows * H, plane = rh * a.Hk * D;
  const float* tm = a.ws + a.splits * plane + (size_t)row * H;
  const float* tl = tm + a.splits * rh;
  float* talk = sm + (a.splits * H + 3) / 4 * 4;
  float* part = talk + H * 8;
  for (int h = tid; h < H; h += 256) {
    const float floor_ = a.sink != nullptr ? a.sink[h] * kLog2e : -INFINITY;
    float mx = floor_;
    for (int s = 0; s < a.splits; ++s) mx = fmaxf(mx, tm[s * rh + h]);
    float den = a.sink != nullptr ? ex2f(floor_ - mx) : 0.f;
    for (int s = 0; s < a.splits; ++s) {
      const float ms = tm[s * rh + h], w = ms == -INFINITY ? 0.f : ex2f(ms - mx);
      sm[s * H + h] = w;
      if (ms != -INFINITY) den = fmaf(w, tl[s * rh + h], den);
    }
    const float inv = den > 0.f ? 1.f / den : 0.f;
    for (int s = 0; s < a.splits; ++s) sm[s * H + h] *= inv;
  }
  for (int i = tid; i < H * 8; i += 256) {
    const int g = i >> 3, k = i & 7;
    talk[i] = k < n ? a.talk[(size_t)(c * gs + h0 + k) * H + g] : 0.f;
  }
  // ranges with keys come first; the others have written nothing but their maximum
  int used = 0;
  for (int s = 0; s < a.splits; ++s) used += tm[s * rh] != -INFINITY;
  __syncthreads();
  const int d = lane * 4 % D;
  float acc[8][4] = {};
  for (int g = warp * PER + lane * 4 / D; g < H; g += 8 * PER) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* src = a.ws + (((size_t)row * H + g) * a.Hk + c) * D + d;
#pragma unroll 4
    for (int s = 0; s < used; ++s) {
      const float w = sm[s * H + g];
      const float4 y = *reinterpret_cast<const float4*>(src + s * plane);
      x.x = fmaf(w, y.x, x.x);
      x.y = fmaf(w, y.y, x.y);
      x.z = fmaf(w, y.z, x.z);
      x.w = fmaf(w, y.w, x.w);
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float f = talk[g * 8 + k];
      acc[k][0] = fmaf(f, x.x, acc[k][0]);
      acc[k][1] = fmaf(f, x.y, acc[k][1]);
      acc[k][2] = fmaf(f, x.z, acc[k][2]);
      acc[k][3] = fmaf(f, x.w, acc[k][3]);
    }
  }
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    if (PER == 2)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[k][e] += __shfl_xor_sync(0xffffffffu, acc[k][e], 16);
    if (PER == 1 || lane < 16)
      *reinterpret_cast<float4*>(part + (warp * 8 + k) * D + d) = make_float4(acc[k][0], acc[k][1], acc[k][2], acc[k][3]);
  }
  __syncthreads();
  for (int i = tid; i < n * D; i += 256) {
    float x = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) x += part[w * 8 * D + i];
    a.out[((size_t)row * H + c * gs + h0) * D + i] = __float2bfloat16(x);
  }
}

template <int D, int MT, int GN> int launch_talk(const TalkArgs& a, cudaStream_t s) {
  using L = TalkSmem<D, MT, GN>;
  static bool set = false;
  if (!set) {
    const cudaError_t e =
        cudaFuncSetAttribute(talk_decode_kernel<D, MT, GN>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::bytes);
    if (e != cudaSuccess) { msgl_set_error("talk attention smem", e); return MSGL_CUDA_ERROR; }
    set = true;
  }
  msgl_launch(talk_decode_kernel<D, MT, GN>, dim3(a.splits, (a.Hk + GN - 1) / GN, a.rows),
              dim3(kWarps * 32 + kCopyThreads), L::bytes, s, a);
  MSGL_CHECK_LAUNCH("talk_decode");
  if (a.splits > 1) {
    const size_t smem = ((size_t)(a.splits * a.H + 3) / 4 * 4 + 8 * a.H + 64 * D) * 4;      // 48 KiB at the most
    msgl_launch(talk_merge_kernel<D>, dim3(a.rows, a.Hk, (a.H / a.Hk + 7) / 8), dim3(256), smem, s, a);
    MSGL_CHECK_LAUNCH("talk_merge");
  }
  return MSGL_OK;
}

template <int D> int dispatch_talk(const TalkArgs& a, cudaStream_t s) {
  const int mt = a.H <= 16 ? 1 : a.H <= 32 ? 2 : 4;
  if (a.Hk <= 2) {
    if (mt == 1) return launch_talk<D, 1, 2>(a, s);
    if (mt == 2) return launch_talk<D, 2, 2>(a, s);
    return launch_talk<D, 4, 2>(a, s);
  }
  if (mt == 1) return launch_talk<D, 1, 4>(a, s);
  if (mt == 2) return launch_talk<D, 2, 4>(a, s);
  return launch_talk<D, 4, D == 64 ? 4 : 2>(a, s);
}

}  // namespace

// Floats of workspace for `splits` partials of `rows` rows.
MSGL_API long long msgl_talk_workspace_floats(int rows, int h, int hk, int d, int splits) {
  return (long long)splits * rows * h * ((long long)hk * d + 2);
}

// q, out [rows, h, d] bf16 (d 64 or 128, up to 64 heads); k, v [pages, hk, page_size, d]. decode: row i is request i. bias [h, reach] fp32 or null; sink [h] or null; talk [h, h].
MSGL_API int msgl_talk_attention(const void* k, const void* v, const void* q, void* out, const void* block_table,
                                 int bt_stride, const void* cu_q, const void* seq_lens, const void* bias, int reach, const void* sink,
                                 const void* talk, void* workspace, int B, int rows, int h, int hk, int d, int page_size,
                                 int num_pages, int window, int splits, int decode, float scale, cudaStream_t stream) {
  if (B == 0 || rows == 0) return MSGL_OK;
  if (hk <= 0 || h % hk || h > 64 || (d != 64 && d != 128) || page_size < 8 || TK % page_size || bt_stride < 1 ||
      (bias != nullptr && reach <= 0) || talk == nullptr || splits < 1 || splits > 16 || rows > 65535 || (uintptr_t)k % 16 || (uintptr_t)v % 16 || (uintptr_t)q % 16 ||
      (splits > 1 && workspace == nullptr) || (decode && rows > B)) {
    msgl_set_error_text("talk attention: rows of 64 or 128, up to 64 heads, pages of 8 to 64");
    return MSGL_BAD_ARG;
  }
  int* status = nullptr;
  cudaGetSymbolAddress((void**)&status, g_talk_status);
  TalkArgs a{(const bf*)q, (const bf*)k, (const bf*)v, (bf*)out, (const int32_t*)block_table, (const int32_t*)cu_q, (const int32_t*)seq_lens,
             (const float*)bias, (const float*)sink, (const float*)talk, (float*)workspace, bt_stride, B, rows, h, hk,
             page_size, num_pages, reach, window, splits, decode, scale, status};
  return d == 64 ? dispatch_talk<64>(a, stream) : dispatch_talk<128>(a, stream);
}

MSGL_API int msgl_talk_status(int reset) {
  int v = 0;
  cudaMemcpyFromSymbol(&v, g_talk_status, sizeof(int));
  if (reset && v != 0) {
    int z = 0;
    cudaMemcpyToSymbol(g_talk_status, &z, sizeof(int));
  }
  return v;
}
