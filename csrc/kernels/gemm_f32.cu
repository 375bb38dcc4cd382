// True fp32 matrix product on the CUDA cores (no reduced-precision tensor mode): the projections of a
// model served in fp32.  C[b, m, n] = sum_k A[b, m, k] * B[b, n, k]  (or B[b, k, n] with b_mn).
// 64 x 64 tiles, 256 threads of 4 x 4 results, operands staged in shared memory 16 k-steps at a time.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "sm100.cuh"

namespace cgk {
namespace {
constexpr int F32_T = 64, F32_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ B, float* __restrict__ C, int M, int N, int K,
                long long lda, long long ldb, long long ldc, long long sA, long long sB, long long sC, int b_mn) {
  __shared__ float as[F32_K][F32_T + 4], bs[F32_K][F32_T + 4];
  A += blockIdx.z * sA; B += blockIdx.z * sB; C += blockIdx.z * sC;
  const int m0 = blockIdx.y * F32_T, n0 = blockIdx.x * F32_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += F32_K) {
    for (int i = threadIdx.x; i < F32_T * F32_K; i += 256) {
      const int r = i / F32_K, k = i % F32_K;
      as[k][r] = (m0 + r < M && k0 + k < K) ? A[(long long)(m0 + r) * lda + k0 + k] : 0.0f;
      if (!b_mn) {
        bs[k][r] = (n0 + r < N && k0 + k < K) ? B[(long long)(n0 + r) * ldb + k0 + k] : 0.0f;
      } else {
        const int rn = i % F32_T, kk = i / F32_T;
        bs[kk][rn] = (n0 + rn < N && k0 + kk < K) ? B[(long long)(k0 + kk) * ldb + n0 + rn] : 0.0f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < F32_K; ++k) {
      const float4 a4 = *reinterpret_cast<const float4*>(&as[k][ty * 4]);
      const float4 b4 = *reinterpret_cast<const float4*>(&bs[k][tx * 4]);
      const float a[4] = {a4.x, a4.y, a4.z, a4.w}, b[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) C[(long long)m * ldc + n] = acc[i][j];
    }
}
}  // namespace
}  // namespace cgk

CGK_API int cgk_gemm_f32(const void* A, const void* B, void* C, int M, int N, int K, int batch, long long lda, long long ldb, long long ldc,
                         long long sA, long long sB, long long sC, int b_mn, void* stream) {
  using namespace cgk;
  CGK_REQUIRE(A && B && C && M >= 0 && N >= 0 && K > 0 && batch >= 1 && batch <= 65535, "cgk_gemm_f32: bad arguments");
  if (M == 0 || N == 0) return 0;
  CGK_REQUIRE((M + F32_T - 1) / F32_T <= 65535, "cgk_gemm_f32: too many rows");
  const dim3 grid((N + F32_T - 1) / F32_T, (M + F32_T - 1) / F32_T, batch);
  gemm_f32_kernel<<<grid, 256, 0, (cudaStream_t)stream>>>((const float*)A, (const float*)B, (float*)C, M, N, K, lda, ldb, ldc, sA, sB, sC, b_mn);
  CGK_LAUNCH_CHECK();
  return 0;
}
