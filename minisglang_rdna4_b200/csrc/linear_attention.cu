// Linear attention with a decaying state: per (request, head) S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, S fp32.
// alpha is one number per head, or comes per key channel from a low-rank input: sigmoid(z)^(1/tau), z = W low + bias.
//
//   linear_attn_recurrent_kernel  token by token; decode, draft verification and the 32-bit mode. The state stays in
//                                 registers, q / k / alpha are staged in shared memory.
//   linear_attn_chunk_kernel      prompts in 16 bits, chunks of 16 tokens on warp-level tensor products with the decays
//                                 factored out of the chunk. The state, decays and scores are fp32: every operand that is
//                                 not a plain 16-bit input is split into two bf16 terms.
//   norm_gate_kernel              RMS norm of the result (per head or over all heads) times a gate
//
// Sequences are packed rows described by cu_q; a sequence without a state (has_state == 0) starts from zeros. Queries and
// keys may be rotated by position first (neighbouring channels are pairs), in fp32.
#include "common.cuh"
#include "ptx.cuh"

using namespace msgl;
using namespace msgl::ptx;

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2a(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2a(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float silu_as(float x) {
  if constexpr (sizeof(T) == 4) return x / (1.f + expf(-x));
  return silu(x);
}

struct LinArgs {
  const void* q;          // [T, H * dk] with row stride ld (k, v, low: the same rows)
  const void* k;
  const void* v;          // [T, H * dv]
  long long ld;
  float* state;           // [slots, H, dk, dv] with slot stride slot_stride
  long long slot_stride;
  const int32_t* cu_q;
  const int32_t* slots;
  const int32_t* has_state;
  void* out;              // [T, H, dv]
  const float* decay;     // [H], or null:
  const void* low;        // [T, rank]
  const void* up;         // [H * dk, rank]
  const float* bias;      // [H * dk]
  int H, dk, dv, rank, act, num_slots;
  float inv_tau, q_scale;
  const float* cos_sin;   // [max_pos, rot]: cosines then sines of the pairs (2 i, 2 i + 1) of q and k, or null
  const int32_t* positions;
  int rot, max_pos;
};

// channel c of a row at a position: its share of the rotation and its partner's
__device__ __forceinline__ float2 turn_of(const LinArgs& a, int pos, int c) {
  pos = pos < 0 ? 0 : (pos < a.max_pos ? pos : a.max_pos - 1);
  const float* cs = a.cos_sin + (size_t)pos * a.rot + (c >> 1);
  const float sn = cs[a.rot >> 1];
  return make_float2(cs[0], (c & 1) ? sn : -sn);
}

// ------------------------------------------------------------------------------------------ recurrent form
// grid (dv / 32, H, B), 128 threads: thread (row group rg of 16, column group cg of 8) owns the rows rg, rg + 16, ... and
// four columns of a 32-column slice of the state.
template <typename T, int RPT>
__global__ void __launch_bounds__(128) linear_attn_recurrent_kernel(const LinArgs a) {
  pdl_enter();
  constexpr int DK = 16 * RPT;
  __shared__ float sq[2][DK], sk[2][DK], sa[2][DK];
  __shared__ float4 red[2][4][8];
  const int tid = threadIdx.x, cg = tid & 7, rg = tid >> 3, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, b = blockIdx.z;
  const int lo = a.cu_q[b], hi = a.cu_q[b + 1];
  if (hi <= lo) return;
  const int col = blockIdx.x * 32 + cg * 4;
  const bool in = col < a.dv;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  float* S = a.state + slot * a.slot_stride + (size_t)h * a.dk * a.dv + col;
  float4 s[RPT];
  const bool keep = a.has_state[b] != 0;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = i * 16 + rg;
    s[i] = keep && in && r < a.dk ? *reinterpret_cast<const float4*>(S + (size_t)r * a.dv) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T* q = reinterpret_cast<const T*>(a.q) + (size_t)h * a.dk;
  const T* k = reinterpret_cast<const T*>(a.k) + (size_t)h * a.dk;
  const T* v = reinterpret_cast<const T*>(a.v) + (size_t)h * a.dv + col;
  const float scalar = a.decay != nullptr ? a.decay[h] : 0.f;
  int buf = 0;
  for (int t = lo; t < hi; ++t, buf ^= 1) {
    for (int c = tid; c < DK; c += 128) {
      float qv = 0.f, kv = 0.f, al = 0.f;
      if (c < a.dk) {
        qv = to_float(q[t * a.ld + c]);
        kv = to_float(k[t * a.ld + c]);
        if (a.act) {
          qv = silu_as<T>(qv);
          kv = silu_as<T>(kv);
        }
        if (a.cos_sin != nullptr && c < a.rot) {
          float qp = to_float(q[t * a.ld + (c ^ 1)]), kp = to_float(k[t * a.ld + (c ^ 1)]);
          if (a.act) {
            qp = silu_as<T>(qp);
            kp = silu_as<T>(kp);
          }
          const float2 f = turn_of(a, a.positions[t], c);
          qv = qv * f.x + qp * f.y;
          kv = kv * f.x + kp * f.y;
        }
        al = scalar;
        if (a.decay == nullptr) {
          const T* low = reinterpret_cast<const T*>(a.low) + t * a.ld;
          const T* up = reinterpret_cast<const T*>(a.up) + (size_t)(h * a.dk + c) * a.rank;
          float z = a.bias[h * a.dk + c];
          int r = 0;
          if (a.rank % 8 == 0) {
            for (; r < a.rank; r += 8) {
              float x[8], w[8];
              load8(low + r, x);
              load8(up + r, w);
#pragma unroll
              for (int e = 0; e < 8; ++e) z = fmaf(w[e], x[e], z);
            }
          }
          for (; r < a.rank; ++r) z = fmaf(to_float(up[r]), to_float(low[r]), z);
          // log sigmoid(z) = min(z, 0) - log(1 + exp(-|z|))
          al = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * a.inv_tau);
        }
      }
      sq[buf][c] = qv * a.q_scale;
      sk[buf][c] = kv;
      sa[buf][c] = al;
    }
    float vv[4] = {};
    if (in) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        vv[e] = to_float(v[t * a.ld + e]);
        if (a.act) vv[e] = silu_as<T>(vv[e]);
      }
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = i * 16 + rg;
      const float al = sa[buf][r], kk = sk[buf][r], qq = sq[buf][r];
      s[i].x = fmaf(s[i].x, al, kk * vv[0]);
      s[i].y = fmaf(s[i].y, al, kk * vv[1]);
      s[i].z = fmaf(s[i].z, al, kk * vv[2]);
      s[i].w = fmaf(s[i].w, al, kk * vv[3]);
      o.x = fmaf(s[i].x, qq, o.x);
      o.y = fmaf(s[i].y, qq, o.y);
      o.z = fmaf(s[i].z, qq, o.z);
      o.w = fmaf(s[i].w, qq, o.w);
    }
#pragma unroll
    for (int m = 8; m <= 16; m <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, m);
      o.y += __shfl_xor_sync(0xffffffffu, o.y, m);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, m);
      o.w += __shfl_xor_sync(0xffffffffu, o.w, m);
    }
    if (lane < 8) red[buf][warp][lane] = o;
    __syncthreads();
    if (tid < 32 && blockIdx.x * 32 + tid < a.dv) {
      float y = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) y += reinterpret_cast<const float*>(red[buf][w])[tid];
      reinterpret_cast<T*>(a.out)[((size_t)t * a.H + h) * a.dv + blockIdx.x * 32 + tid] = from_float<T>(y);
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = i * 16 + rg;
    if (in && r < a.dk) *reinterpret_cast<float4*>(S + (size_t)r * a.dv) = s[i];
  }
}

// ------------------------------------------------------------------------------------------ chunk form
__device__ __forceinline__ void ldm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_hi(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
// what rounding to bf16 left over, as the second term of the pair
__device__ __forceinline__ uint32_t pack_lo(float a, float b, uint32_t hi) {
  return pack_hi(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int n) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ bool bar_any(int id, int n, bool p) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.s32 p, %3, 0;\n\tbarrier.cta.red.or.pred q, %1, %2, p;\n\tselp.s32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(id), "r"(n), "r"((int)p) : "memory");
  return r != 0;
}
__device__ __forceinline__ void cp16z(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

constexpr int kC = 16;        // tokens per chunk
constexpr int kCols = 64;     // value columns per CTA: four warps of 16
constexpr float kMaxLog2 = 80.f;

// G groups of producer warps take the chunks in turn; NS stage buffers and RAW blocks of raw rows per group.
template <int DK> struct ChunkSmem {
  static constexpr int G = DK <= 128 ? 3 : 1;
  static constexpr int NS = G > 1 ? 1 : 2;
  static constexpr int RAW = G > 1 ? 2 : 3;
  static constexpr int LD = DK + 8;                       // row stride in elements: rows on different banks
  static constexpr int LDV = kCols + 8;
  static constexpr int NP = DK / 32;                      // producer warps per group
  // at 0: q hi, q lo, k hi, k lo, [16][LD] each
  static constexpr int off_v = 4 * kC * LD * 2;
  static constexpr int off_dec = off_v + kC * LDV * 2;
  static constexpr int off_score = off_dec + DK * 4;      // [NP][2][32] float4
  static constexpr int off_meta = off_score + NP * 1024;
  static constexpr int stage = off_meta + 16;
  // raw rows as they come: per producer warp and chunk 16 x 32 of q and of k, and 16 x 64 values per chunk
  static constexpr int off_raw = G * NS * stage;
  static constexpr int raw_warp = 2 * kC * 64;
  static constexpr int raw = NP * raw_warp + kC * kCols * 2;
  static constexpr int off_gate = off_raw + G * RAW * raw;
  static constexpr int gate_bytes(int rank) {
    const int r = (rank + 15) / 16 * 16;
    // W transposed [r][DK] fp32, and per producer warp raw blocks [16][r] and one [r][16] in fp32
    return rank > 0 ? r * DK * 4 + G * NP * (RAW * kC * r * 2 + r * kC * 4) : 0;
  }
  static constexpr int bytes(int rank) { return off_gate + gate_bytes(rank); }
};

// Warps 0-3: a slice of 16 value columns each, S^T slice in the accumulators of v^T k, which is also the layout in which
// the tensor core takes S as the right operand of q S. The other warps: 32 key channels each; they turn 16 tokens into
// q 2^(b_i - b_end) and k 2^(b_end - b_j) (b: running sum of log2 alpha in the chunk), so that the state only has to be
// multiplied by 2^b_end once, and the scores q k^T between the chunk's tokens over their channels. None of that depends
// on the chunks before, so groups of such warps work on different chunks at once. A chunk whose decay leaves the range
// of the factors is handed over token by token. Stages go through named barriers.
// ROT: q and k are rotated in fp32 by the producers; a lane holds the cosine (even channel) or sine (odd) of its pair.
template <int DK, bool ROT>
__global__ void __launch_bounds__(128 + ChunkSmem<DK>::G * DK, DK <= 64 ? 2 : 1) linear_attn_chunk_kernel(const LinArgs a) {
  pdl_enter();
  using L = ChunkSmem<DK>;
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int G = L::G, NS = L::NS, RAW = L::RAW, NT = 128 + DK;
  // barriers: a stage is full, a stage is empty, a group's vote, all producers
  constexpr int FULL = 1, EMPTY = FULL + G * NS, VOTE = EMPTY + G * NS, PRODUCERS = VOTE + G;
  static_assert((G == 1 || NS == 1) && PRODUCERS < 16, "stages in order, sixteen barriers");
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z;
  const int lo = a.cu_q[b], len = a.cu_q[b + 1] - lo;
  if (len <= 0) return;
  const int slot = a.slots[b];
  if (MSGL_OOB(slot, a.num_slots) || slot < 0 || slot >= a.num_slots) return;
  const uint32_t base = smem_u32(smem);

  if (warp < 4) {
    // ---------------------------------------------------------------- value columns
    const int n0 = blockIdx.x * kCols + warp * 16;
    const bool active = n0 < a.dv;
    const int g = lane >> 2, t2 = (lane & 3) * 2;
    float* S = a.state + slot * a.slot_stride + (size_t)h * a.dk * a.dv + n0 + g;
    float s[DK / 8][4];
    const bool keep = a.has_state[b] != 0 && active;
#pragma unroll
    for (int kb = 0; kb < DK / 8; ++kb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = kb * 8 + t2 + (e & 1);
        s[kb][e] = keep && row < a.dk ? S[(size_t)row * a.dv + (e >> 1) * 8] : 0.f;
      }
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)lo * a.H + h) * a.dv + n0 + t2;
    const long long ldo = (long long)a.H * a.dv;
    const int chunks = (len + kC - 1) / kC;
    for (int chunk = 0, i = 0; chunk < chunks; ++i) {
      const int st = G > 1 ? chunk % G : i % NS;
      bar_sync(FULL + st, NT);
      const uint32_t sb = base + st * L::stage;
      const uint8_t* sp = smem + st * L::stage;
      const int4 meta = *reinterpret_cast<const int4*>(sp + L::off_meta);      // chunk start, rows [y, z), end of the chunk
      if (active) {
        float o[2][4] = {};
#pragma unroll
        for (int kb = 0; kb < DK / 8; ++kb) {
          const float2 d = *reinterpret_cast<const float2*>(sp + L::off_dec + (kb * 8 + t2) * 4);
          s[kb][0] *= d.x; s[kb][1] *= d.y; s[kb][2] *= d.x; s[kb][3] *= d.y;
        }
        const uint32_t row_a = sb + ((lane & 15) * L::LD + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
          uint32_t qh[4], ql[4];
          ldm4(row_a + ks * 32, qh);
          ldm4(row_a + kC * L::LD * 2 + ks * 32, ql);
#pragma unroll
          for (int nb = 0; nb < 2; ++nb) {
            const float* c0 = &s[2 * ks][2 * nb];
            const float* c1 = &s[2 * ks + 1][2 * nb];
            const uint32_t h0 = pack_hi(c0[0], c0[1]), h1 = pack_hi(c1[0], c1[1]);
            const uint32_t l0 = pack_lo(c0[0], c0[1], h0), l1 = pack_lo(c1[0], c1[1], h1);
            mma16816(o[nb], qh, h0, h1);
            mma16816(o[nb], qh, l0, l1);
            mma16816(o[nb], ql, h0, h1);
          }
        }
        uint32_t vf[4];
        ldm4t(sb + L::off_v + (((lane & 7) + (lane >> 4) * 8) * L::LDV + warp * 16 + ((lane >> 3) & 1) * 8) * 2, vf);
        uint32_t ah[4], al[4];
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int p = 0; p < L::NP; ++p) {
            const float4 y = *reinterpret_cast<const float4*>(sp + L::off_score + ((p * 2 + nb) * 32 + lane) * 16);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
          }
          const int j = nb * 8 + t2;
          x.x = j <= g ? x.x : 0.f;
          x.y = j + 1 <= g ? x.y : 0.f;
          x.z = j <= g + 8 ? x.z : 0.f;
          x.w = j + 1 <= g + 8 ? x.w : 0.f;
          ah[2 * nb] = pack_hi(x.x, x.y);
          ah[2 * nb + 1] = pack_hi(x.z, x.w);
          al[2 * nb] = pack_lo(x.x, x.y, ah[2 * nb]);
          al[2 * nb + 1] = pack_lo(x.z, x.w, ah[2 * nb + 1]);
        }
        mma16816(o[0], ah, vf[0], vf[2]);
        mma16816(o[1], ah, vf[1], vf[3]);
        mma16816(o[0], al, vf[0], vf[2]);
        mma16816(o[1], al, vf[1], vf[3]);
        const uint32_t row_k = row_a + 2 * kC * L::LD * 2;
#pragma unroll
        for (int kb = 0; kb < DK / 8; kb += 2) {
          uint32_t kf[4];
          ldm4t(row_k + kb * 16, kf);
          mma16816(s[kb], vf, kf[0], kf[1]);
          mma16816(s[kb + 1], vf, kf[2], kf[3]);
          ldm4t(row_k + kC * L::LD * 2 + kb * 16, kf);
          mma16816(s[kb], vf, kf[0], kf[1]);
          mma16816(s[kb + 1], vf, kf[2], kf[3]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = g + half * 8;
          if (r >= meta.y && r < meta.z) {
#pragma unroll
            for (int nb = 0; nb < 2; ++nb)
              *reinterpret_cast<uint32_t*>(out + (meta.x + r) * ldo + nb * 8) = pack_hi(o[nb][2 * half], o[nb][2 * half + 1]);
          }
        }
      }
      __syncwarp();
      bar_arrive(EMPTY + st, NT);
      chunk += meta.w;
    }
    if (active) {
#pragma unroll
      for (int kb = 0; kb < DK / 8; ++kb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int row = kb * 8 + t2 + (e & 1);
          if (row < a.dk) S[(size_t)row * a.dv + (e >> 1) * 8] = s[kb][e];
        }
    }
    return;
  }

  // ---------------------------------------------------------------- key channels
  using bf = __nv_bfloat16;
  const int grp = (warp - 4) / L::NP, pw = (warp - 4) % L::NP, ch = pw * 32 + lane;
  const bool live = ch < a.dk;
  const bf* q = reinterpret_cast<const bf*>(a.q) + (size_t)lo * a.ld + (size_t)h * a.dk;
  const bf* k = reinterpret_cast<const bf*>(a.k) + (size_t)lo * a.ld + (size_t)h * a.dk;
  const bf* v = reinterpret_cast<const bf*>(a.v) + (size_t)lo * a.ld + (size_t)h * a.dv + blockIdx.x * kCols;
  const bf* low = reinterpret_cast<const bf*>(a.low) + (size_t)lo * a.ld;
  const int vcols = min(kCols, a.dv - (int)blockIdx.x * kCols);
  const int r16 = (a.rank + 15) / 16 * 16;
  float* up = reinterpret_cast<float*>(smem + L::off_gate);                 // [r16][DK]
  uint8_t* mine = reinterpret_cast<uint8_t*>(up + r16 * DK) +
                  (grp * L::NP + pw) * (RAW * kC * r16 * 2 + r16 * kC * 4);
  float* lowf = reinterpret_cast<float*>(mine + RAW * kC * r16 * 2);        // [r16][16]
  const bool channel = a.decay == nullptr;
  constexpr int NV = L::NP >= 4 ? 1 : 4 / L::NP;       // 16-byte pieces of the value block per thread
  // Raw rows of a chunk: this warp's channels of q and k, this thread's pieces of v (which only it reads), this warp's
  // copy of the low-rank rows. Rows past the end are zeros.
  auto fetch = [&](int start, int buf) {
    if (start < len) {
      const uint32_t dst = base + L::off_raw + (grp * RAW + buf) * L::raw;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int id = lane + (i & 1) * 32, t = id >> 2, c = pw * 32 + (id & 3) * 8;
        const bool ok = start + t < len && c < a.dk;
        cp16z(dst + pw * L::raw_warp + (i >> 1) * kC * 64 + id * 16,
              (i >> 1 ? k : q) + (ok ? (long long)(start + t) * a.ld + c : 0), ok);
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int id = ch + i * DK, t = id >> 3, c = (id & 7) * 8;
        if (id >= 128) break;
        const bool ok = start + t < len && c < vcols;
        cp16z(dst + L::NP * L::raw_warp + id * 16, v + (ok ? (long long)(start + t) * a.ld + c : 0), ok);
      }
      const int per = r16 / 8;
      for (int id = lane; id < kC * per; id += 32) {
        const int t = id / per, c = id - t * per;
        const bool ok = start + t < len;
        cp16z(smem_u32(mine) + (buf * kC * r16 + t * r16 + c * 8) * 2, low + (ok ? (long long)(start + t) * a.ld + c * 8 : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < RAW - 1; ++i) fetch((grp + i * G) * kC, i);
  float bias = 0.f, fixed = 0.f;
  if (channel) {
    const bf* w = reinterpret_cast<const bf*>(a.up) + (size_t)(h * a.dk + (live ? ch : 0)) * a.rank;
    for (int r = grp; r < r16; r += G) up[r * DK + ch] = live && r < a.rank ? to_float(w[r]) : 0.f;
    bias = live ? a.bias[h * a.dk + ch] : 0.f;
    bar_sync(PRODUCERS, G * DK);
  } else {
    fixed = fmaxf(log2f(a.decay[h]), -1e4f);
  }
  float part_of_turn[ROT ? kC : 1];
  const int pos0 = ROT ? a.positions[lo] : 0;
  auto fetch_turns = [&](int start) {
    if constexpr (ROT) {
#pragma unroll
      for (int t = 0; t < kC; ++t) {
        const int pos = min(max(pos0 + min(start + t, len - 1), 0), a.max_pos - 1);
        part_of_turn[t] = ch < a.rot ? a.cos_sin[(size_t)pos * a.rot + (ch >> 1) + (ch & 1) * (a.rot >> 1)]
                                     : (ch & 1) ? 0.f : 1.f;
      }
    }
  };
  fetch_turns(grp * kC);
  int stage = 0, round = 0;
  for (int start = grp * kC; start < len; start += G * kC, ++round) {
    const int n = min(kC, len - start);
    float qf[kC], kf[kC], cum[kC];
    const int raw_buf = round % RAW;
    const uint8_t* raw = smem + L::off_raw + (grp * RAW + raw_buf) * L::raw;
    asm volatile("cp.async.wait_group %0;" ::"n"(RAW - 2) : "memory");
    __syncwarp();                          // this chunk's rows are there, and everyone is done with the one before
    fetch(start + (RAW - 1) * G * kC, (round + RAW - 1) % RAW);
    {
      const bf* qr = reinterpret_cast<const bf*>(raw + pw * L::raw_warp) + lane;
#pragma unroll
      for (int t = 0; t < kC; ++t) {
        qf[t] = to_float(qr[t * 32]);
        kf[t] = to_float(qr[(kC + t) * 32]);
      }
      if (a.act) {                         // (outside the loop over tokens: no branch between independent chains)
#pragma unroll
        for (int t = 0; t < kC; ++t) {
          qf[t] = silu(qf[t]);
          kf[t] = silu(kf[t]);
        }
      }
      if constexpr (ROT) {
#pragma unroll
        for (int t = 0; t < kC; ++t) {
          const float other = __shfl_xor_sync(0xffffffffu, part_of_turn[t], 1);
          const float cs = (lane & 1) ? other : part_of_turn[t], sn = (lane & 1) ? part_of_turn[t] : -other;
          const float qp = __shfl_xor_sync(0xffffffffu, qf[t], 1), kp = __shfl_xor_sync(0xffffffffu, kf[t], 1);
          qf[t] = qf[t] * cs + qp * sn;
          kf[t] = kf[t] * cs + kp * sn;
        }
        fetch_turns(start + G * kC);
      }
#pragma unroll
      for (int t = 0; t < kC; ++t) qf[t] *= a.q_scale;
    }
    if (channel) {
      const bf* lr = reinterpret_cast<const bf*>(mine) + raw_buf * kC * r16;
      for (int id = lane; id < kC * r16; id += 32) lowf[id] = to_float(lr[(id % kC) * r16 + id / kC]);
      __syncwarp();
#pragma unroll
      for (int t = 0; t < kC; ++t) cum[t] = bias;
#pragma unroll 4
      for (int r = 0; r < r16; ++r) {
        const float w = up[r * DK + ch];
#pragma unroll
        for (int t = 0; t < kC; t += 4) {
          const float4 x = *reinterpret_cast<const float4*>(lowf + r * kC + t);
          cum[t] = fmaf(w, x.x, cum[t]);
          cum[t + 1] = fmaf(w, x.y, cum[t + 1]);
          cum[t + 2] = fmaf(w, x.z, cum[t + 2]);
          cum[t + 3] = fmaf(w, x.w, cum[t + 3]);
        }
      }
#pragma unroll
      for (int t = 0; t < kC; ++t) {
        // log2 sigmoid(z) = -log2(1 + 2^(-z log2 e))
        const float y = -cum[t] * kLog2e, soft = lg2a(1.f + ex2a(fminf(y, 64.f)));
        cum[t] = (y > 64.f ? y : soft) * -a.inv_tau;
      }
      __syncwarp();
    } else {
#pragma unroll
      for (int t = 0; t < kC; ++t) cum[t] = fixed;
    }
#pragma unroll
    for (int t = 0; t < kC; ++t) cum[t] = (t > 0 ? cum[t - 1] : 0.f) + (live && t < n ? cum[t] : 0.f);
    const float total = cum[kC - 1];
    const bool far = -total > kMaxLog2;
    const bool slow = bar_any(VOTE + grp, DK, far);
    for (int part = 0; part < (slow ? n : 1); ++part, ++stage) {
      const int st = grp * NS + stage % NS;
      if (stage >= NS) bar_sync(EMPTY + st, NT);
      const uint32_t sb = base + st * L::stage;
      uint8_t* sp = smem + st * L::stage;
      bf* qh = reinterpret_cast<bf*>(sp) + ch;
      float step = total;
      auto put = [&](int t, float x, float y) {
        const bf xh = __float2bfloat16(x), yh = __float2bfloat16(y);
        qh[t * L::LD] = xh;
        qh[(kC + t) * L::LD] = __float2bfloat16(x - to_float(xh));
        qh[(2 * kC + t) * L::LD] = yh;
        qh[(3 * kC + t) * L::LD] = __float2bfloat16(y - to_float(yh));
      };
      if (!slow) {
#pragma unroll
        for (int t = 0; t < kC; ++t) put(t, qf[t] * ex2a(cum[t] - total), kf[t] * ex2a(total - cum[t]));
      } else {
#pragma unroll
        for (int t = 0; t < kC; ++t) {
          if (t == part) step = cum[t] - (t > 0 ? cum[t - 1] : 0.f);
          put(t, t == part ? qf[t] : 0.f, t == part ? kf[t] : 0.f);
        }
      }
      reinterpret_cast<float*>(sp + L::off_dec)[ch] = ex2a(step);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int id = ch + i * DK, t = id >> 3, c = (id & 7) * 8;
        if (id < 128) {
          const bf* src = reinterpret_cast<const bf*>(raw + L::NP * L::raw_warp) + id * 8;
          bf* dst = reinterpret_cast<bf*>(sp + L::off_v) + t * L::LDV + c;
          if (a.act) {
            float x[8];
            load8(src, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = silu(x[e]);
            store8(dst, x);
          } else {
            *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
          }
        }
      }
      __syncwarp();
      float sc[2][4] = {};
      const uint32_t ra = sb + ((lane & 15) * L::LD + (lane >> 4) * 8 + pw * 32) * 2;
      const uint32_t rb = sb + (2 * kC * L::LD + ((lane & 7) + (lane >> 4) * 8) * L::LD + ((lane >> 3) & 1) * 8 + pw * 32) * 2;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        uint32_t xh[4], xl[4], yh[4], yl[4];
        ldm4(ra + ks * 32, xh);
        ldm4(ra + kC * L::LD * 2 + ks * 32, xl);
        ldm4(rb + ks * 32, yh);
        ldm4(rb + kC * L::LD * 2 + ks * 32, yl);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          mma16816(sc[nb], xh, yh[2 * nb], yh[2 * nb + 1]);
          mma16816(sc[nb], xh, yl[2 * nb], yl[2 * nb + 1]);
          mma16816(sc[nb], xl, yh[2 * nb], yh[2 * nb + 1]);
        }
      }
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
        *reinterpret_cast<float4*>(sp + L::off_score + ((pw * 2 + nb) * 32 + lane) * 16) =
            make_float4(sc[nb][0], sc[nb][1], sc[nb][2], sc[nb][3]);
      if (ch == 0)
        *reinterpret_cast<int4*>(sp + L::off_meta) =
            make_int4(start, slow ? part : 0, slow ? part + 1 : n, !slow || part == n - 1);
      __syncwarp();
      bar_arrive(FULL + st, NT);
    }
  }
  // every arrival at an "empty" barrier is matched before the warps leave
  for (int i = max(stage - NS, 0); i < stage; ++i) bar_sync(EMPTY + grp * NS + i % NS, NT);
}

template <int DK, bool ROT> int launch_chunk_form(const LinArgs& a, int B, cudaStream_t s) {
  const int bytes = ChunkSmem<DK>::bytes(a.rank);
  static int set = 0;
  if (bytes > set) {
    const cudaError_t e =
        cudaFuncSetAttribute(linear_attn_chunk_kernel<DK, ROT>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) {
      msgl_set_error("linear_attention smem", e);
      return MSGL_CUDA_ERROR;
    }
    set = bytes;
  }
  msgl_launch(linear_attn_chunk_kernel<DK, ROT>, dim3((a.dv + kCols - 1) / kCols, a.H, B),
              dim3(128 + ChunkSmem<DK>::G * DK), bytes, s, a);
  MSGL_CHECK_LAUNCH("linear_attn_chunk");
  return MSGL_OK;
}
template <int DK> int launch_chunk(const LinArgs& a, int B, cudaStream_t s) {
  return a.cos_sin != nullptr ? launch_chunk_form<DK, true>(a, B, s) : launch_chunk_form<DK, false>(a, B, s);
}

template <typename T> int launch_recurrent(const LinArgs& a, int B, cudaStream_t s) {
  const dim3 grid((a.dv + 31) / 32, a.H, B);
  const int rpt = a.dk / 16;
  if (rpt <= 1) msgl_launch(linear_attn_recurrent_kernel<T, 1>, grid, dim3(128), 0, s, a);
  else if (rpt <= 2) msgl_launch(linear_attn_recurrent_kernel<T, 2>, grid, dim3(128), 0, s, a);
  else if (rpt <= 4) msgl_launch(linear_attn_recurrent_kernel<T, 4>, grid, dim3(128), 0, s, a);
  else if (rpt <= 8) msgl_launch(linear_attn_recurrent_kernel<T, 8>, grid, dim3(128), 0, s, a);
  else if (rpt <= 16) msgl_launch(linear_attn_recurrent_kernel<T, 16>, grid, dim3(128), 0, s, a);
  else if (rpt <= 32) msgl_launch(linear_attn_recurrent_kernel<T, 32>, grid, dim3(128), 0, s, a);
  else {
    msgl_set_error_text("linear_attention: key heads of up to 512 channels");
    return MSGL_BAD_ARG;
  }
  MSGL_CHECK_LAUNCH("linear_attn_recurrent");
  return MSGL_OK;
}

// ------------------------------------------------------------------------------------------ norm and gate
// Groups of `group` channels (a head, or all heads of a row), `width` of which are no padding. CTA: a CTA per group
// instead of a warp.
template <typename T, bool CTA>
__global__ void __launch_bounds__(256) norm_gate_kernel(const T* __restrict__ x, const T* __restrict__ g, long long ldg,
                                                        const float* __restrict__ w, const float* __restrict__ total,
                                                        T* __restrict__ out, long long groups, int per_row, int group,
                                                        float width, float eps, int silu_gate) {
  pdl_enter();
  __shared__ float scratch[32];
  constexpr int V = 8;
  const long long id = CTA ? (long long)blockIdx.x : (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= groups) return;
  const int first = (CTA ? threadIdx.x : (threadIdx.x & 31)) * V, stride = (CTA ? 256 : 32) * V;
  const T* src = x + id * group;
  const T* gs = g + id / per_row * ldg + id % per_row * group;
  float ss = 0.f;
  if (total != nullptr) {
    ss = total[id];
  } else {
    for (int c = first; c < group; c += stride) {
      float v[V];
      load8(src + c, v);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    }
    if constexpr (CTA) ss = block_sum(ss, scratch);
    else ss = warp_sum(ss);
  }
  const float rs = 1.f / sqrtf(ss / width + eps);
  for (int c = first; c < group; c += stride) {
    float v[V], z[V];
    load8(src + c, v);
    load8(gs + c, z);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float sg = 1.f / (1.f + (sizeof(T) == 4 ? expf(-z[e]) : __expf(-z[e])));
      v[e] = v[e] * rs * w[c + e] * (silu_gate ? z[e] * sg : sg);
    }
    store8(out + id * group + c, v);
  }
}

}  // namespace

// chunked: prompts may take the tensor-core form (bf16, key heads of up to 256 channels, 16-byte aligned rows)
MSGL_API int msgl_linear_attention(const void* q, const void* k, const void* v, long long ld, void* state,
                                   long long slot_stride, const void* cu_q, const void* slots, const void* has_state,
                                   void* out, const void* decay, const void* low, const void* up, const void* bias, int B,
                                   int H, int dk, int dv, int rank, int act, int num_slots, float inv_tau, float q_scale,
                                   const void* cos_sin, const void* positions, int rot, int max_pos, int chunked, int dtype,
                                   cudaStream_t stream) {
  if (B <= 0) return B == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (H <= 0 || dk <= 0 || dv <= 0 || dk % 16 || dv % 16 || B > 65535 || H > 65535 || ld % 8 || slot_stride % 4 ||
      (uintptr_t)state % 16 || (uintptr_t)q % 16 || (uintptr_t)k % 16 || (uintptr_t)v % 16 || (uintptr_t)out % 16 ||
      (decay == nullptr && (low == nullptr || up == nullptr || bias == nullptr || rank <= 0 || (uintptr_t)low % 16 ||
                            (uintptr_t)up % 16)) ||
      (cos_sin != nullptr && (positions == nullptr || rot <= 0 || rot % 2 || rot > dk || max_pos <= 0)))
    return MSGL_BAD_ARG;
  LinArgs a{q, k, v, ld, (float*)state, slot_stride, (const int32_t*)cu_q, (const int32_t*)slots,
            (const int32_t*)has_state, out, (const float*)decay, low, up, (const float*)bias, H, dk, dv,
            decay != nullptr ? 0 : rank, act, num_slots, inv_tau, q_scale, (const float*)cos_sin, (const int32_t*)positions, rot,
            max_pos};
  if (dtype == MSGL_F32) return launch_recurrent<float>(a, B, stream);
  if (dtype != MSGL_BF16) return MSGL_BAD_ARG;
  constexpr int kMaxSmem = 225 * 1024;
  if (chunked && dk <= 32 && ChunkSmem<32>::bytes(a.rank) <= kMaxSmem) return launch_chunk<32>(a, B, stream);
  if (chunked && dk <= 64 && ChunkSmem<64>::bytes(a.rank) <= kMaxSmem) return launch_chunk<64>(a, B, stream);
  if (chunked && dk <= 128 && ChunkSmem<128>::bytes(a.rank) <= kMaxSmem) return launch_chunk<128>(a, B, stream);
  if (chunked && dk <= 256 && ChunkSmem<256>::bytes(a.rank) <= kMaxSmem) return launch_chunk<256>(a, B, stream);
  return launch_recurrent<__nv_bfloat16>(a, B, stream);
}

// x [rows * per_row, group]; g [rows, ...] with row stride ldg; w [group]; total [rows * per_row] or null
MSGL_API int msgl_norm_gate(const void* x, const void* g, long long ldg, const void* w, const void* total, void* out,
                            long long rows, int per_row, int group, float width, float eps, int silu_gate, int dtype,
                            cudaStream_t stream) {
  if (rows <= 0) return rows == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (per_row <= 0 || group <= 0 || group % 8 || ldg % 8 || (uintptr_t)x % 16 || (uintptr_t)g % 16 || (uintptr_t)out % 16 ||
      width <= 0.f)
    return MSGL_BAD_ARG;
  const long long groups = rows * per_row;
  const bool cta = group > 512;
  const long long blocks = cta ? groups : (groups + 7) / 8;
  if (blocks > 0x7fffffffLL) return MSGL_BAD_ARG;
#define NORM_GATE(T, C)                                                                                              \
  msgl_launch(norm_gate_kernel<T, C>, dim3((unsigned)blocks), dim3(256), 0, stream, (const T*)x, (const T*)g, ldg,   \
              (const float*)w, (const float*)total, (T*)out, groups, per_row, group, width, eps, silu_gate)
  if (dtype == MSGL_BF16) { if (cta) NORM_GATE(__nv_bfloat16, true); else NORM_GATE(__nv_bfloat16, false); }
  else if (dtype == MSGL_F32) { if (cta) NORM_GATE(float, true); else NORM_GATE(float, false); }
  else return MSGL_BAD_ARG;
#undef NORM_GATE
  MSGL_CHECK_LAUNCH("norm_gate");
  return MSGL_OK;
}
