// True fp32 matrix product (no reduced-precision tensor mode): C[m, n] = sum_k A[m, k] B[n, k], with
// row strides and an optional batch of independent products (one per head) or an expert per block of 128
// rows. The 32-bit serving mode of the models that have one; 64 x 64 tiles, 4 x 4 outputs per thread on the
// FMA pipe.
#include "common.cuh"

using namespace msgl;

namespace {

constexpr int BM = 64, BN = 64, BK = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, long long lda, long long sA,
                                                       const float* __restrict__ B, long long ldb, long long sB,
                                                       float* __restrict__ C, long long ldc, long long sC, int M, int N,
                                                       int K, const float* __restrict__ gate, long long ldg,
                                                       const int* __restrict__ tile_expert) {
  pdl_enter();
  __shared__ float as[BK][BM + 4], bs[BK][BN + 4];
  A += blockIdx.z * sA;
  B += blockIdx.z * sB;
  C += blockIdx.z * sC;
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
  if (tile_expert != nullptr) {            // experts of sB elements each; -1: a block without rows
    const int e = tile_expert[m0 >> 7];
    if (e < 0) return;
    B += e * sB;
  }
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int id = tid + i * 256, r = id >> 4, k = id & 15;
      as[k][r] = m0 + r < M && k0 + k < K ? A[(m0 + r) * lda + k0 + k] : 0.f;
      bs[k][r] = n0 + r < N && k0 + k < K ? B[(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&as[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&bs[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) {
        const float f = gate != nullptr ? 1.f / (1.f + expf(-gate[m * ldg + blockIdx.z])) : 1.f;
        C[m * ldc + n] = acc[i][j] * f;
      }
    }
}

}  // namespace

MSGL_API int msgl_gemm_f32(const void* a, long long lda, long long stride_a, const void* b, long long ldb,
                           long long stride_b, void* c, long long ldc, long long stride_c, int M, int N, int K, int batch,
                           const void* gate, long long ldg, cudaStream_t stream) {
  if (M <= 0) return M == 0 ? MSGL_OK : MSGL_BAD_ARG;
  if (N <= 0 || K <= 0 || batch <= 0 || batch > 65535) return MSGL_BAD_ARG;
  // rows are chunked so that the grid's y extent stays within its limit
  for (int m = 0; m < M; m += 65535 * BM) {
    const int rows = min(M - m, 65535 * BM);
    dim3 grid((N + BN - 1) / BN, (rows + BM - 1) / BM, batch);
    msgl_launch(gemm_f32_kernel, grid, dim3(256), 0, stream, (const float*)a + (long long)m * lda, lda, stride_a,
                (const float*)b, ldb, stride_b, (float*)c + (long long)m * ldc, ldc, stride_c, rows, N, K,
                gate != nullptr ? (const float*)gate + (long long)m * ldg : nullptr, ldg, (const int*)nullptr);
  }
  MSGL_CHECK_LAUNCH("gemm_f32");
  return MSGL_OK;
}

// a [M, K] expert-sorted rows (M % 128 == 0), b [experts, N, K], tile_expert [M / 128] -> c [M, N]
MSGL_API int msgl_gemm_f32_grouped(const void* a, const void* b, void* c, int M, int N, int K, const void* tile_expert,
                                   cudaStream_t stream) {
  if (M == 0) return MSGL_OK;
  if (M < 0 || M % 128 || N <= 0 || K <= 0 || M / BM > 65535 || tile_expert == nullptr) return MSGL_BAD_ARG;
  dim3 grid((N + BN - 1) / BN, M / BM, 1);
  msgl_launch(gemm_f32_kernel, grid, dim3(256), 0, stream, (const float*)a, (long long)K, 0LL, (const float*)b, (long long)K,
              (long long)N * K, (float*)c, (long long)N, 0LL, M, N, K, (const float*)nullptr, 0LL, (const int*)tile_expert);
  MSGL_CHECK_LAUNCH("gemm_f32_grouped");
  return MSGL_OK;
}
