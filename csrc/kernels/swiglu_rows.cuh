// act(gate) * up (act: silu or relu) over bf16 rows [gate | up] of 2 F elements, F a multiple of 8: four rows at a time per CTA, so every
// thread keeps eight 16-byte loads in flight.  blockIdx.y picks a range of columns (few long rows still fill the GPU).
#pragma once
#include "sm100.cuh"

namespace cgk {

constexpr int SWIGLU_ROWS = 4;

enum : int { GATED_SILU = 0, GATED_RELU = 1 };
template <int ACT>
__device__ __forceinline__ float gated_act(float x) { return ACT == GATED_RELU ? fmaxf(x, 0.0f) : silu_f(x); }

template <int ACT = GATED_SILU>
__device__ __forceinline__ void swiglu_rows_bf16(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ act, long long ldo, long long rows, int F) {
  for (long long row0 = (long long)blockIdx.x * SWIGLU_ROWS; row0 < rows; row0 += (long long)gridDim.x * SWIGLU_ROWS) {
    const int f = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (f < F) {
      uint4 g[SWIGLU_ROWS], u[SWIGLU_ROWS];
#pragma unroll
      for (int j = 0; j < SWIGLU_ROWS; ++j) {
        if (row0 + j >= rows) continue;
        const __nv_bfloat16* p = gu + (row0 + j) * 2 * F + f;
        g[j] = *reinterpret_cast<const uint4*>(p);
        u[j] = *reinterpret_cast<const uint4*>(p + F);
      }
#pragma unroll
      for (int j = 0; j < SWIGLU_ROWS; ++j) {
        if (row0 + j >= rows) continue;
        const uint32_t gw[4] = {g[j].x, g[j].y, g[j].z, g[j].w}, uw[4] = {u[j].x, u[j].y, u[j].z, u[j].w};
        uint32_t o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 a = unpack_bf16x2(gw[e]), b = unpack_bf16x2(uw[e]);
          o[e] = pack_bf16x2(gated_act<ACT>(a.x) * b.x, gated_act<ACT>(a.y) * b.y);
        }
        *reinterpret_cast<uint4*>(act + (row0 + j) * ldo + f) = make_uint4(o[0], o[1], o[2], o[3]);
      }
    }
  }
}

inline int swiglu_rows_threads(int F) { return F / 8 >= 256 ? 256 : (F / 8 + 31) / 32 * 32; }
inline dim3 swiglu_rows_grid(long long rows, int F) {
  const int nt = swiglu_rows_threads(F), cols = (F / 8 + nt - 1) / nt;
  long long n = (rows + SWIGLU_ROWS - 1) / SWIGLU_ROWS, cap = 148 * 16 / (cols < 16 ? cols : 16);
  return dim3((unsigned)(n < 1 ? 1 : (n < cap ? n : cap)), cols);
}

}  // namespace cgk
