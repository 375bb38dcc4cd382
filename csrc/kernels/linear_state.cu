// Linear recurrences (linear_state.cuh), token by token: decoding, short portions of prompts, fp32, and shapes the
// tensor-core form (linear_state_tc.cu) does not take.  One CTA per (head, run of consecutive tokens of one
// sequence); the state stays in registers over the run and is read and written once - after every token when the
// cache keeps a history of states (state of p tokens in entry p mod history), so that a caller may go back.
// A run that starts at position 0 starts from zeros whatever its slot holds.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "linear_state.cuh"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {


namespace {

constexpr int LS_THREADS = 256;

// Threads: column groups of CW state columns x row groups; NR rows per thread in registers (0: rows stay in memory).
template <typename T, int NR, int CW>
__global__ void __launch_bounds__(LS_THREADS)
linear_state_scan_kernel(const LinStateDev a, int col_groups, int row_groups) {
  extern __shared__ float sh[];
  __shared__ float red[33];
  const int h = blockIdx.x, D = a.D, V = a.V;
  const int tid = threadIdx.x, cg = tid % col_groups, rg = tid / col_groups;
  const bool active = rg < row_groups;
  float* ad = sh;                                   // decay, key, query, value of the current token; then partial results
  float* kd = ad + D;
  float* qd = kd + D;
  float* vd = qd + D;
  float* part = vd + (V + 3) / 4 * 4;               // [row_groups][V]
  long long t0 = blockIdx.y;
  int count = 1;
  if (a.runs) {
    t0 = a.runs[2 * blockIdx.y];
    count = a.runs[2 * blockIdx.y + 1];
  }
  if (count <= 0) return;
  const int p0 = a.pos[t0];
  const long long slot = CGK_IDX(a.slot[t0], a.slots);
  float* base = a.state + slot * a.history * a.heads * D * V;
  auto entry = [&](int tokens) { return base + ((long long)(tokens % a.history) * a.heads + h) * D * V; };
  float S[NR > 0 ? NR : 1][CW];
  const bool zero = p0 == 0;
  if constexpr (NR > 0) {
    const float* src = entry(p0);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = rg + i * row_groups;
#pragma unroll
      for (int j = 0; j < CW; ++j) S[i][j] = 0.0f;
      if (!zero && active && r < D) ldv<CW>(src + (long long)r * V + cg * CW, S[i]);
    }
  }
  const T* qp = reinterpret_cast<const T*>(a.q);
  const T* kp = reinterpret_cast<const T*>(a.k);
  const T* vp = reinterpret_cast<const T*>(a.v);
  for (int n = 0; n < count; ++n) {
    const long long t = t0 + n;
    for (int c = tid; c < D; c += LS_THREADS) {
      const int ch = h * D + c;
      float one_minus;
      const float g = lin_decay(a, a.z[t * a.ldz + ch], ch, &one_minus);
      ad[c] = expf(g);
      kd[c] = a.k ? ld1(kp + t * a.ldk + ch) : one_minus;
      qd[c] = lin_query(a, ld1(qp + t * a.ldq + ch));
    }
    for (int c = tid; c < V; c += LS_THREADS) vd[c] = ld1(vp + t * a.ldv + (long long)h * V + c);
    __syncthreads();
    if (active) {
      if constexpr (NR > 0) {
        float v[CW], o[CW];
#pragma unroll
        for (int j = 0; j < CW; ++j) { v[j] = vd[cg * CW + j]; o[j] = 0.0f; }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int r = rg + i * row_groups;
          if (r < D) {
            const float ar = ad[r], kr = kd[r], qr = qd[r];
#pragma unroll
            for (int j = 0; j < CW; ++j) {
              S[i][j] = fmaf(ar, S[i][j], kr * v[j]);
              o[j] = fmaf(qr, S[i][j], o[j]);
            }
          }
        }
#pragma unroll
        for (int j = 0; j < CW; ++j) part[rg * V + cg * CW + j] = o[j];
        if (a.history > 1 || n + 1 == count) {
          float* dst = entry(p0 + n + 1);
#pragma unroll
          for (int i = 0; i < NR; ++i) {
            const int r = rg + i * row_groups;
            if (r < D) stv<CW>(dst + (long long)r * V + cg * CW, S[i]);
          }
        }
      } else {
        const float* src = entry(p0 + n);
        float* dst = entry(p0 + n + 1);
        for (int c = cg; c < V; c += col_groups) {
          const float v = vd[c];
          float o = 0.0f;
          for (int r = rg; r < D; r += row_groups) {
            const float s = fmaf(ad[r], zero && n == 0 ? 0.0f : src[(long long)r * V + c], kd[r] * v);
            dst[(long long)r * V + c] = s;
            o = fmaf(qd[r], s, o);
          }
          part[rg * V + c] = o;
        }
      }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int c = tid; c < V; c += LS_THREADS) {
      float o = 0.0f;
      for (int g = 0; g < row_groups; ++g) o += part[g * V + c];
      part[c] = o;                                  // row 0: read by this thread alone
      ss = fmaf(o, o, ss);
    }
    ss = block_sum(ss, red);
    const float r = 1.0f / sqrtf(ss / V + a.eps);
    for (int c = tid; c < V; c += LS_THREADS) {
      float o = part[c] * r * a.w[c];
      if (a.gate) o *= lin_silu(ld1(reinterpret_cast<const T*>(a.gate) + t * a.ldg + (long long)h * V + c));
      st1(reinterpret_cast<T*>(a.out) + t * a.ldo + (long long)h * V + c, o);
    }
    __syncthreads();
  }
}

template <typename T, int NR, int CW>
int launch_scan(const LinStateDev& d, int n_runs, int cols, int groups, cudaStream_t st) {
  const int smem = (3 * d.D + (d.V + 3) / 4 * 4 + groups * d.V) * 4;
  CGK_REQUIRE(smem <= 200 * 1024, "linear state: heads of %d x %d are too large", d.D, d.V);
  if (smem > 48 * 1024)
    CGK_CUDA_CHECK(cudaFuncSetAttribute(linear_state_scan_kernel<T, NR, CW>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  linear_state_scan_kernel<T, NR, CW><<<dim3(d.heads, n_runs), LS_THREADS, smem, st>>>(d, cols, groups);
  CGK_LAUNCH_CHECK();
  return 0;
}
template <typename T, int CW>
int pick_scan(const LinStateDev& d, int n_runs, cudaStream_t st) {
  const int cols = d.V / CW;
  if (cols > LS_THREADS) return launch_scan<T, 0, 1>(d, n_runs, LS_THREADS, 1, st);
  const int groups = LS_THREADS / cols, nr = (d.D + groups - 1) / groups;
  if (nr <= 2) return launch_scan<T, 2, CW>(d, n_runs, cols, groups, st);
  if (nr <= 4) return launch_scan<T, 4, CW>(d, n_runs, cols, groups, st);
  if (nr <= 8) return launch_scan<T, 8, CW>(d, n_runs, cols, groups, st);
  if (nr <= 16) return launch_scan<T, 16, CW>(d, n_runs, cols, groups, st);
  if (nr <= 24) return launch_scan<T, 24, CW>(d, n_runs, cols, groups, st);
  const int c0 = d.V < LS_THREADS ? d.V : LS_THREADS;
  return launch_scan<T, 0, 1>(d, n_runs, c0, LS_THREADS / c0, st);
}

}  // namespace
}  // namespace cgk

using namespace cgk;

CGK_API int cgk_linear_state(const cgk_linear_state_args* pa, int n_runs, void* stream) {
  CGK_REQUIRE(pa, "cgk_linear_state: null args");
  const cgk_linear_state_args& a = *pa;
  CGK_REQUIRE(a.q && a.v && a.z && a.bias && a.w && a.state && a.out && a.slot && a.pos && a.heads > 0 && a.D > 0 && a.V > 0 && a.history > 0 &&
              a.slots > 0 && n_runs >= 0, "cgk_linear_state: bad arguments");
  CGK_REQUIRE(a.mode == GATE_BOUNDED ? (a.low && !a.k) : (a.mode == GATE_ROOT && a.k), "cgk_linear_state: the gate's operands do not fit its kind");
  CGK_REQUIRE(n_runs <= 65535, "cgk_linear_state: too many runs in one call");
  if (n_runs == 0) return 0;
  LinStateDev d{a.q, a.k, a.v, a.gate, a.z, a.ldq, a.ldk, a.ldv, a.ldg, a.ldz, a.bias, a.low, a.w, a.state, a.out, a.ldo, a.slot, a.pos, a.runs,
                a.heads, a.D, a.V, a.history, a.slots, a.mode, a.q_silu, a.q_scale, a.inv_tau, a.eps};
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = a.V % 4 == 0 && (((uintptr_t)a.state) & 15) == 0;
  if (a.fp32) return vec ? pick_scan<float, 4>(d, n_runs, st) : pick_scan<float, 1>(d, n_runs, st);
  return vec ? pick_scan<__nv_bfloat16, 4>(d, n_runs, st) : pick_scan<__nv_bfloat16, 1>(d, n_runs, st);
}

CGK_BOUNDS_READER(linear_state)
