// Matrix products with few rows (decoding): out[m, n] = sum_k x[m, k] W[n, k], m < 8, bf16 weights streamed once with
// plain 16-byte loads, fp32 sums.  A tensor-core tile would compute 128 rows and stream the weights through a
// quarter of the SMs; here every warp owns a few weight rows and keeps several loads in flight per lane.
//   plain   one batch entry per blockIdx.y
//   gated   W holds gate rows then up rows: out = silu(gate) * up (or relu), the feed-forward's first half in one kernel
//   b_mn    W stored [k][n] (the latent image of a query: W_uk^T q per head)
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

constexpr int SK_WARPS = 8;

__device__ __forceinline__ uint4 ld_stream(const __nv_bfloat16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
__device__ __forceinline__ void unpack8f(const uint4& a, float (&f)[8]) {
  float2 t;
  t = unpack_bf16x2(a.x); f[0] = t.x; f[1] = t.y;
  t = unpack_bf16x2(a.y); f[2] = t.x; f[3] = t.y;
  t = unpack_bf16x2(a.z); f[4] = t.x; f[5] = t.y;
  t = unpack_bf16x2(a.w); f[6] = t.x; f[7] = t.y;
}

struct SkinnyDev {
  const __nv_bfloat16* x; long long ldx, sx;
  const __nv_bfloat16* w; long long ldw, sw;
  void* out; long long ldo, so;
  int out_fp32, M, N, K, relu;
};

// MT: rows of x held (M <= MT), RW: output columns per warp; GATED: each column needs weight rows n and N + n
template <int MT, int RW, bool GATED>
__global__ void __launch_bounds__(SK_WARPS * 32)
skinny_kernel(const SkinnyDev a) {
  constexpr int WR = GATED ? 2 * RW : RW;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * SK_WARPS + warp) * RW;
  if (n0 >= a.N) return;
  const __nv_bfloat16* x = a.x + blockIdx.y * a.sx;
  const __nv_bfloat16* w[WR];
#pragma unroll
  for (int r = 0; r < RW; ++r) {
    const long long n = min(n0 + r, a.N - 1);
    w[r] = a.w + blockIdx.y * a.sw + n * a.ldw;
    if (GATED) w[RW + r] = a.w + (a.N + n) * a.ldw;
  }
  float acc[WR][MT];
#pragma unroll
  for (int r = 0; r < WR; ++r)
#pragma unroll
    for (int m = 0; m < MT; ++m) acc[r][m] = 0.0f;
#pragma unroll 2
  for (int k = lane * 8; k < a.K; k += 256) {
    uint4 wv[WR];
#pragma unroll
    for (int r = 0; r < WR; ++r) wv[r] = ld_stream(w[r] + k);
    float xf[MT][8];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (m < a.M) {
        unpack8f(*reinterpret_cast<const uint4*>(x + m * a.ldx + k), xf[m]);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) xf[m][j] = 0.0f;
      }
    }
#pragma unroll
    for (int r = 0; r < WR; ++r) {
      float f[8];
      unpack8f(wv[r], f);
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[r][m] = fmaf(f[j], xf[m][j], acc[r][m]);
    }
  }
#pragma unroll
  for (int r = 0; r < WR; ++r)
#pragma unroll
    for (int m = 0; m < MT; ++m) acc[r][m] = warp_sum(acc[r][m]);
  // lane l stores value l of the RW x MT results
#pragma unroll
  for (int r = 0; r < RW; ++r)
#pragma unroll
    for (int m = 0; m < MT; ++m)
      if (lane == r * MT + m && n0 + r < a.N && m < a.M) {
        float v = acc[r][m];
        if (GATED) v = (a.relu ? fmaxf(v, 0.0f) : v / (1.0f + expf(-v))) * acc[RW + r][m];
        const long long o = blockIdx.y * a.so + m * a.ldo + n0 + r;
        if (a.out_fp32) reinterpret_cast<float*>(a.out)[o] = v;
        else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = __float2bfloat16(v);
      }
}

// W [K][N]: 16 threads cover 128 columns with 16-byte loads, MN_GROUPS groups of threads share the k range
constexpr int MN_COLS = 128;
template <int MT, int MN_GROUPS>
__global__ void __launch_bounds__(16 * MN_GROUPS)
skinny_mn_kernel(const SkinnyDev a) {
  __shared__ float part[MN_GROUPS][MT][MN_COLS + 4];
  const int tx = threadIdx.x & 15, g = threadIdx.x >> 4;
  const int n = blockIdx.x * MN_COLS + tx * 8;
  const __nv_bfloat16* x = a.x + blockIdx.y * a.sx;
  const __nv_bfloat16* w = a.w + blockIdx.y * a.sw + n;
  float acc[MT][8];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[m][j] = 0.0f;
  if (n < a.N) {
#pragma unroll 4
    for (int k = g; k < a.K; k += MN_GROUPS) {
      float f[8];
      unpack8f(ld_stream(w + (long long)k * a.ldw), f);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float xv = m < a.M ? __bfloat162float(x[m * a.ldx + k]) : 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[m][j] = fmaf(f[j], xv, acc[m][j]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 8; ++j) part[g][m][tx * 8 + j] = acc[m][j];
  __syncthreads();
  for (int i = threadIdx.x; i < MT * MN_COLS; i += 16 * MN_GROUPS) {
    const int m = i / MN_COLS, c = i % MN_COLS, nn = blockIdx.x * MN_COLS + c;
    if (m >= a.M || nn >= a.N) continue;
    float v = 0.0f;
#pragma unroll
    for (int q = 0; q < MN_GROUPS; ++q) v += part[q][m][c];
    const long long o = blockIdx.y * a.so + m * a.ldo + nn;
    if (a.out_fp32) reinterpret_cast<float*>(a.out)[o] = v;
    else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = __float2bfloat16(v);
  }
}

template <int MT, bool GATED>
int launch_rw(const SkinnyDev& d, int batch, int sms, cudaStream_t st) {
  // enough warps to fill the machine first, then more columns per warp
  const long long cols = (long long)d.N * batch;
  if (cols >= (long long)sms * 64 && !GATED) {
    constexpr int RW = 4;
    skinny_kernel<MT, RW, GATED><<<dim3((d.N + SK_WARPS * RW - 1) / (SK_WARPS * RW), batch), SK_WARPS * 32, 0, st>>>(d);
  } else if (cols >= (long long)sms * 16) {
    constexpr int RW = 2;
    skinny_kernel<MT, RW, GATED><<<dim3((d.N + SK_WARPS * RW - 1) / (SK_WARPS * RW), batch), SK_WARPS * 32, 0, st>>>(d);
  } else {
    constexpr int RW = 1;
    skinny_kernel<MT, RW, GATED><<<dim3((d.N + SK_WARPS * RW - 1) / (SK_WARPS * RW), batch), SK_WARPS * 32, 0, st>>>(d);
  }
  CGK_LAUNCH_CHECK();
  return 0;
}
template <int MT>
int launch_mn(const SkinnyDev& d, int batch, cudaStream_t st) {
  constexpr int G = MT == 8 ? 8 : 16;
  skinny_mn_kernel<MT, G><<<dim3((d.N + MN_COLS - 1) / MN_COLS, batch), 16 * G, 0, st>>>(d);
  CGK_LAUNCH_CHECK();
  return 0;
}

}  // namespace
}  // namespace cgk

CGK_API int cgk_skinny_gemm(const void* x, long long ldx, long long sx, const void* w, long long ldw, long long sw, void* out, long long ldo,
                            long long so, int out_fp32, int M, int N, int K, int batch, int mode, void* stream) {
  using namespace cgk;
  CGK_REQUIRE(x && w && out && M >= 0 && M <= 8 && N >= 0 && K > 0 && batch >= 1 && batch <= 65535, "cgk_skinny_gemm: 1 to 8 rows");
  CGK_REQUIRE(mode >= 0 && mode <= 3 && ((mode & 1) == 0 || batch == 1), "cgk_skinny_gemm: bad mode");
  auto al = [](const void* p, long long ld, long long s) { return (((uintptr_t)p) & 15) == 0 && ld % 8 == 0 && s % 8 == 0; };
  CGK_REQUIRE(al(w, ldw, sw) && (mode == 2 ? N % 8 == 0 : (K % 8 == 0 && al(x, ldx, sx))), "cgk_skinny_gemm: rows must be 16-byte aligned");
  if (M == 0 || N == 0) return 0;
  int dev = 0;
  CGK_CUDA_CHECK(cudaGetDevice(&dev));
  const int sms = sm_count(dev);
  SkinnyDev d{(const __nv_bfloat16*)x, ldx, sx, (const __nv_bfloat16*)w, ldw, sw, out, ldo, so, out_fp32, M, N, K, mode == 3};
  cudaStream_t st = (cudaStream_t)stream;
  switch (mode) {
    case 0:
      if (M == 1) return launch_rw<1, false>(d, batch, sms, st);
      if (M == 2) return launch_rw<2, false>(d, batch, sms, st);
      if (M <= 4) return launch_rw<4, false>(d, batch, sms, st);
      return launch_rw<8, false>(d, batch, sms, st);
    case 1:
    case 3:
      if (M == 1) return launch_rw<1, true>(d, 1, sms, st);
      if (M == 2) return launch_rw<2, true>(d, 1, sms, st);
      if (M <= 4) return launch_rw<4, true>(d, 1, sms, st);
      return launch_rw<8, true>(d, 1, sms, st);
    default:
      if (M == 1) return launch_mn<1>(d, batch, st);
      if (M == 2) return launch_mn<2>(d, batch, st);
      if (M <= 4) return launch_mn<4>(d, batch, st);
      return launch_mn<8>(d, batch, st);
  }
}
