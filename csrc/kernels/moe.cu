// Mixture of experts: routing, the permutation to expert order for the grouped GEMM, and expert products for
// few rows.
//   route    router logits (fp32) -> softmax scores; choice = score + correction; the best groups are kept
//            (a group's score is its largest choice score), the best outputs of them chosen; weights are the
//            chosen scores over their sum.  Outputs [experts, experts + identity) stand for the input itself.
//   plan     expert counts -> first row of every expert in the permuted matrix (segments start on multiples
//            of 128, the GEMM's row tile) and the expert of every row tile
//   gather   token rows into their expert's segment
//   rows     (few pairs, fp32, or sizes TMA cannot address) one warp per output element of one (token, choice)
//            pair: silu(gate) * up, then the down-projection
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "sm100.cuh"
#include "swiglu_rows.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

constexpr int RT_WARPS = 4;

__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
}

// One warp per token.  Shared memory per warp: scores [O], choice scores [O].
__global__ void __launch_bounds__(RT_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, const float* __restrict__ corr, int rows, int experts, int O, int top, int groups, int keep,
                 int* __restrict__ idx, float* __restrict__ weight, int* __restrict__ row_of, int* __restrict__ counts) {
  extern __shared__ float rsm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t = (long long)blockIdx.x * RT_WARPS + warp;
  if (t >= rows) return;
  float* sc = rsm + warp * 2 * O;
  float* ch = sc + O;
  const float* z = logits + t * O;
  float m = -INFINITY;
  for (int i = lane; i < O; i += 32) m = fmaxf(m, z[i]);
  m = warp_max(m);
  float sum = 0.0f;
  for (int i = lane; i < O; i += 32) {
    const float e = expf(z[i] - m);
    sc[i] = e;
    sum += e;
  }
  sum = warp_sum(sum);
  for (int i = lane; i < O; i += 32) {
    const float s = sc[i] / sum;
    sc[i] = s;
    ch[i] = s + corr[i];
  }
  __syncwarp();
  if (groups > 1 && keep < groups) {
    const int per = O / groups;
    // group scores live on the lanes: lane l holds groups l, l + 32, ... (up to 128 groups)
    float gs[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int g = lane + j * 32;
      gs[j] = -INFINITY;
      if (g < groups)
        for (int i = 0; i < per; ++i) gs[j] = fmaxf(gs[j], ch[g * per + i]);
    }
    unsigned kept = 0;                                 // bit j: group lane + 32 j is kept
    for (int k = 0; k < keep; ++k) {
      float v = -INFINITY;
      int b = 0x7fffffff;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int g = lane + j * 32;
        if (g < groups && !((kept >> j) & 1u) && (gs[j] > v || b == 0x7fffffff)) { v = gs[j]; b = g; }
      }
      warp_argmax(v, b);
      if (b < groups && (b & 31) == lane) kept |= 1u << (b >> 5);
    }
    __syncwarp();
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int g = lane + j * 32;
      if (g < groups && !((kept >> j) & 1u))
        for (int i = 0; i < per; ++i) ch[g * per + i] = -INFINITY;
    }
    __syncwarp();
  }
  // the largest choice scores, lower index first among equals; a taken output becomes NaN-free "used" by -inf
  float total = 0.0f;
  for (int k = 0; k < top; ++k) {
    float v = -INFINITY;
    int b = 0x7fffffff;
    for (int i = lane; i < O; i += 32)
      if (ch[i] > v) { v = ch[i]; b = i; }
    warp_argmax(v, b);
    b = b < O ? b : 0;
    const float s = sc[b];
    total += s;
    if (lane == 0) {
      idx[t * top + k] = b;
      weight[t * top + k] = s;
      row_of[t * top + k] = b < experts ? (int)(t * top + k) : -1;
      if (counts && b < experts) atomicAdd(counts + b, 1);
      ch[b] = -INFINITY;
    }
    __syncwarp();
  }
  const float inv = 1.0f / (total + 1e-20f);
  for (int k = lane; k < top; k += 32) weight[t * top + k] *= inv;
}

// One block.  counts -> segment starts (cursor), expert of every row tile; counts are cleared for the next call.
__global__ void moe_plan_kernel(int* __restrict__ counts, int E, int* __restrict__ cursor, int* __restrict__ tile_expert, int* __restrict__ tiles,
                                int max_tiles) {
  __shared__ int part[1024];
  const int e = threadIdx.x;
  const int n = e < E ? (counts[e] + 127) / 128 : 0;
  part[e] = n;
  __syncthreads();
  for (int o = 1; o < (int)blockDim.x; o <<= 1) {
    const int v = e >= o ? part[e - o] : 0;
    __syncthreads();
    part[e] += v;
    __syncthreads();
  }
  const int first = part[e] - n;
  if (e < E) {
    cursor[e] = first * 128;
    counts[e] = 0;
    for (int i = 0; i < n; ++i) tile_expert[CGK_IDX(first + i, max_tiles)] = e;
  }
  if (e == (int)blockDim.x - 1) *tiles = part[e];
}

// One warp per (token, choice) pair.
__global__ void moe_gather_kernel(const __nv_bfloat16* __restrict__ h, const int* __restrict__ idx, int pairs, int top, int experts,
                                  int* __restrict__ cursor, int* __restrict__ row_of, __nv_bfloat16* __restrict__ out, int D, int max_rows) {
  const int p = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (p >= pairs) return;
  const int e = idx[p];
  if (e >= experts) {
    if (lane == 0) row_of[p] = -1;
    return;
  }
  int r = 0;
  if (lane == 0) {
    r = (int)CGK_IDX(atomicAdd(cursor + e, 1), max_rows);
    row_of[p] = r;
  }
  r = __shfl_sync(0xffffffffu, r, 0);
  const uint4* src = reinterpret_cast<const uint4*>(h + (long long)(p / top) * D);
  uint4* dst = reinterpret_cast<uint4*>(out + (long long)r * D);
  for (int i = lane; i < D / 8; i += 32) dst[i] = src[i];
}

// act[row][f] = silu(gu[row][f]) * gu[row][F + f] over the rows in use (*tiles * 128)
__global__ void __launch_bounds__(256)
swiglu_tiles_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ act, const int* __restrict__ tiles, int F) {
  swiglu_rows_bf16(gu, act, F, (long long)*tiles * 128, F);
}

template <typename T, int V>
__device__ __forceinline__ float warp_dot(const T* __restrict__ a, const T* __restrict__ b, int n, int lane) {
  float s = 0.0f;
  for (int i = lane * V; i < n; i += 32 * V) {
    float x[V], y[V];
    ldv<V>(a + i, x);
    ldv<V>(b + i, y);
#pragma unroll
    for (int j = 0; j < V; ++j) s = fmaf(x[j], y[j], s);
  }
  return warp_sum(s);
}

// act[p][f] = silu(G_e[f] . h_t) * (U_e[f] . h_t), e the expert of pair p, t its token
template <typename T, int V>
__global__ void __launch_bounds__(256)
expert_gate_up_kernel(const T* __restrict__ h, const int* __restrict__ idx, int top, int experts, const T* __restrict__ w, T* __restrict__ act, int D, int F) {
  const int p = blockIdx.y, e = idx[p];
  if (e >= experts) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* x = h + (long long)(p / top) * D;
  const T* we = w + (long long)e * 2 * F * D;
  for (int f = blockIdx.x * 8 + warp; f < F; f += gridDim.x * 8) {
    const float g = warp_dot<T, V>(we + (long long)f * D, x, D, lane);
    const float u = warp_dot<T, V>(we + (long long)(F + f) * D, x, D, lane);
    if (lane == 0) st1(act + (long long)p * F + f, g / (1.0f + expf(-g)) * u);
  }
}
template <typename T, int V>
__global__ void __launch_bounds__(256)
expert_down_kernel(const T* __restrict__ act, const int* __restrict__ idx, int experts, const T* __restrict__ w, float* __restrict__ y, int D, int F) {
  const int p = blockIdx.y, e = idx[p];
  if (e >= experts) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* we = w + (long long)e * D * F;
  for (int n = blockIdx.x * 8 + warp; n < D; n += gridDim.x * 8) {
    const float v = warp_dot<T, V>(we + (long long)n * F, act + (long long)p * F, F, lane);
    if (lane == 0) y[(long long)p * D + n] = v;
  }
}

template <typename T, int V>
int launch_rows(const void* h, const int* idx, int pairs, int top, int experts, const void* wgu, const void* wd, void* act, void* y, int D, int F,
                cudaStream_t st) {
  expert_gate_up_kernel<T, V><<<dim3((F + 7) / 8, pairs), 256, 0, st>>>((const T*)h, idx, top, experts, (const T*)wgu, (T*)act, D, F);
  expert_down_kernel<T, V><<<dim3((D + 7) / 8, pairs), 256, 0, st>>>((const T*)act, idx, experts, (const T*)wd, (float*)y, D, F);
  CGK_LAUNCH_CHECK();
  return 0;
}

}  // namespace
}  // namespace cgk

using namespace cgk;

CGK_API int cgk_moe_route(const void* logits, const void* correction, int rows, int experts, int outputs, int top, int groups, int keep,
                          void* idx, void* weight, void* row_of, void* counts, void* stream) {
  CGK_REQUIRE(logits && correction && idx && weight && row_of && rows >= 0, "cgk_moe_route: bad arguments");
  CGK_REQUIRE(outputs > 0 && outputs <= 1024 && experts <= outputs && top > 0 && top <= outputs, "cgk_moe_route: up to 1024 router outputs");
  CGK_REQUIRE(groups <= 1 || (groups <= 128 && outputs % groups == 0 && keep > 0 && keep <= groups && keep * (outputs / groups) >= top),
              "cgk_moe_route: groups must be equal, at most 128, and the kept ones must hold the chosen outputs");
  if (rows == 0) return 0;
  moe_route_kernel<<<(rows + RT_WARPS - 1) / RT_WARPS, RT_WARPS * 32, RT_WARPS * 2 * outputs * 4, (cudaStream_t)stream>>>(
      (const float*)logits, (const float*)correction, rows, experts, outputs, top, groups, keep, (int*)idx, (float*)weight, (int*)row_of, (int*)counts);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_moe_plan(void* counts, int experts, void* cursor, void* tile_expert, void* tiles, int max_tiles, void* stream) {
  CGK_REQUIRE(counts && cursor && tile_expert && tiles && experts > 0 && experts <= 1024, "cgk_moe_plan: 1 to 1024 experts");
  moe_plan_kernel<<<1, experts <= 256 ? 256 : 1024, 0, (cudaStream_t)stream>>>((int*)counts, experts, (int*)cursor, (int*)tile_expert, (int*)tiles, max_tiles);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_moe_gather(const void* h, const void* idx, int pairs, int top, int experts, void* cursor, void* row_of, void* out, int D,
                           int max_rows, void* stream) {
  CGK_REQUIRE(h && idx && cursor && row_of && out && D % 8 == 0 && top > 0, "cgk_moe_gather: rows must be multiples of 8 elements");
  if (pairs == 0) return 0;
  moe_gather_kernel<<<(pairs + 3) / 4, 128, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)h, (const int*)idx, pairs, top, experts, (int*)cursor,
                                                                      (int*)row_of, (__nv_bfloat16*)out, D, max_rows);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_swiglu_tiles(const void* gu, void* act, const void* tiles, int F, int max_tiles, void* stream) {
  CGK_REQUIRE(gu && act && tiles && F % 8 == 0 && F > 0, "cgk_swiglu_tiles: rows must be multiples of 8 elements");
  if (max_tiles == 0) return 0;
  swiglu_tiles_kernel<<<swiglu_rows_grid((long long)max_tiles * 128, F), swiglu_rows_threads(F), 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)act, (const int*)tiles, F);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_expert_rows(int fp32, const void* h, const void* idx, int pairs, int top, int experts, const void* w_gate_up, const void* w_down,
                            void* act, void* y, int D, int F, void* stream) {
  CGK_REQUIRE(h && idx && w_gate_up && w_down && act && y && D > 0 && F > 0 && top > 0 && pairs >= 0, "cgk_expert_rows: bad arguments");
  cudaStream_t st = (cudaStream_t)stream;
  auto al = [&](const void* p) { return (((uintptr_t)p) & 15) == 0; };
  const bool vec = D % 4 == 0 && F % 4 == 0 && al(h) && al(w_gate_up) && al(w_down) && al(act);
  const size_t es = fp32 ? 4 : 2;
  for (int p0 = 0; p0 < pairs; ) {                    // a grid's second dimension ends at 65535
    const int step = (65535 / top) * top;
    const int n = pairs - p0 < step ? pairs - p0 : step;
    const void* hp = (const char*)h + (size_t)(p0 / top) * D * es;
    void* ap = (char*)act + (size_t)p0 * F * es;
    void* yp = (float*)y + (size_t)p0 * D;
    const int* ip = (const int*)idx + p0;
    int rc;
    if (fp32) rc = vec ? launch_rows<float, 4>(hp, ip, n, top, experts, w_gate_up, w_down, ap, yp, D, F, st)
                       : launch_rows<float, 1>(hp, ip, n, top, experts, w_gate_up, w_down, ap, yp, D, F, st);
    else rc = vec ? launch_rows<__nv_bfloat16, 4>(hp, ip, n, top, experts, w_gate_up, w_down, ap, yp, D, F, st)
                  : launch_rows<__nv_bfloat16, 1>(hp, ip, n, top, experts, w_gate_up, w_down, ap, yp, D, F, st);
    if (rc) return rc;
    p0 += n;
  }
  return 0;
}

CGK_BOUNDS_READER(moe)
