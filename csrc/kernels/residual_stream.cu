// Decoders that keep the residual stream in fp32 and normalise the OUTPUT of a sublayer:
//   * token embedding times a constant plus a sinusoidal position vector -> fp32 stream + operand copy,
//   * stream update x += rms(y) * w, where y is a projection's result, or a weighted sum of expert
//     rows (some of which may stand for the stream itself) plus such a result; the new stream also leaves
//     as the bf16 (or fp32) operand of the next sublayer,
//   * stream start or update x = E[id], x += mult * y, followed by up to two RMS norms of the new stream with weights of their
//     own (layers whose sublayers read one stream side by side),
//   * RMS norm of selected stream rows (before the vocabulary projection), soft cap of logits.
// One CTA per row: a row is read once, kept in shared memory between the statistics and the update.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

template <typename TE, typename TH>
__global__ void embed_sinusoid_kernel(const long long* __restrict__ ids, const int* __restrict__ pos, const TE* __restrict__ table,
                                      float scale, const double* __restrict__ freq, float* __restrict__ x,
                                      TH* __restrict__ h, int D, int vocab) {
  const long long row = blockIdx.x;
  const long long id = CGK_IDX(ids[row], vocab);
  const double p = (double)pos[row];
  const int pairs = (D + 1) / 2;
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    float e0 = 0.0f, e1 = 0.0f;
    if (freq) {
      // The angle is formed and reduced in double: thousands of radians in fp32 would carry an error of
      // a few 1e-4, which the fp32 mode of the model would show.
      const double two_pi = 6.283185307179586;
      double a = p * freq[i];
      a -= two_pi * rint(a / two_pi);
      sincosf((float)a, &e0, &e1);
    }
    const int c = 2 * i;
    const float v0 = ld1(table + id * D + c) * scale + e0;
    x[row * D + c] = v0;
    st1(h + row * D + c, v0);
    if (c + 1 < D) {
      const float v1 = ld1(table + id * D + c + 1) * scale + e1;
      x[row * D + c + 1] = v1;
      st1(h + row * D + c + 1, v1);
    }
  }
}

struct UpdateDev {
  const void* y; long long ldy;
  const void* pairs; long long ldp;
  const int* row_of; const float* weight; int top; int pair_rows;
  const float* w; float* x; void* h;
  int D; float eps;
};

template <typename TY, typename TP, typename TH, int V>
__global__ void stream_update_kernel(const UpdateDev a) {
  extern __shared__ float row_buf[];
  __shared__ float red[33];
  const long long t = blockIdx.x;
  const TY* y = reinterpret_cast<const TY*>(a.y);
  const TP* pairs = reinterpret_cast<const TP*>(a.pairs);
  float* x = a.x + t * a.D;
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < a.D; c += blockDim.x * V) {
    float v[V];
    if (y) {
      ldv<V>(y + t * a.ldy + c, v);
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = 0.0f;
    }
    for (int k = 0; k < a.top; ++k) {
      const int r = a.row_of[t * a.top + k];
      const float wk = a.weight[t * a.top + k];
      float e[V];
      if (r >= 0) ldv<V>(pairs + CGK_IDX(r, a.pair_rows) * a.ldp + c, e);
      else ldv<V>(x + c, e);                          // an expert whose output is its input
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = fmaf(wk, e[j], v[j]);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) { ss = fmaf(v[j], v[j], ss); row_buf[c + j] = v[j]; }
  }
  ss = block_sum(ss, red);
  const float rstd = 1.0f / sqrtf(ss / a.D + a.eps);
  TH* h = reinterpret_cast<TH*>(a.h) + t * a.D;
  for (int c = threadIdx.x * V; c < a.D; c += blockDim.x * V) {
    float xv[V], wv[V];
    ldv<V>(x + c, xv);
    ldv<V>(a.w + c, wv);
#pragma unroll
    for (int j = 0; j < V; ++j) xv[j] += row_buf[c + j] * rstd * wv[j];
    stv<V>(x + c, xv);
    stv<V>(h + c, xv);
  }
}

// The same update with the row in registers: 8 elements per thread and step, the stream requested together with
// the sublayer's result so that one round trip covers both.
template <typename T>
__device__ __forceinline__ void ld8(const T* p, float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    const uint4 t = *reinterpret_cast<const uint4*>(p);
    float2 f;
    f = unpack_bf16x2(t.x); v[0] = f.x; v[1] = f.y;
    f = unpack_bf16x2(t.y); v[2] = f.x; v[3] = f.y;
    f = unpack_bf16x2(t.z); v[4] = f.x; v[5] = f.y;
    f = unpack_bf16x2(t.w); v[6] = f.x; v[7] = f.y;
  } else {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
}
template <typename T>
__device__ __forceinline__ void st8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  } else {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  }
}
template <typename TY, typename TP, typename TH, int ITER>
__global__ void __launch_bounds__(512)
stream_update_regs_kernel(const UpdateDev a) {
  __shared__ float red[16];
  const long long t = blockIdx.x;
  const TY* y = reinterpret_cast<const TY*>(a.y);
  const TP* pairs = reinterpret_cast<const TP*>(a.pairs);
  float* x = a.x + t * a.D;
  float v[ITER][8], xv[ITER][8], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.D) {
      ld8(x + c, xv[i]);
      if (y) {
        ld8(y + t * a.ldy + c, v[i]);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[i][j] = 0.0f;
      }
    }
  }
#pragma unroll 4
  for (int k = 0; k < a.top; ++k) {
    const int r = a.row_of[t * a.top + k];
    const float wk = a.weight[t * a.top + k];
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 8;
      if (c < a.D) {
        if (r >= 0) {
          float e[8];
          ld8(pairs + CGK_IDX(r, a.pair_rows) * a.ldp + c, e);
#pragma unroll
          for (int j = 0; j < 8; ++j) v[i][j] = fmaf(wk, e[j], v[i][j]);
        } else {                                       // an expert whose output is its input
#pragma unroll
          for (int j = 0; j < 8; ++j) v[i][j] = fmaf(wk, xv[i][j], v[i][j]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ITER; ++i)
    if ((i * blockDim.x + threadIdx.x) * 8 < a.D) {
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(v[i][j], v[i][j], ss);
    }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.0f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += red[w];
  const float rstd = 1.0f / sqrtf(ss / a.D + a.eps);
  TH* h = reinterpret_cast<TH*>(a.h) + t * a.D;
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < a.D) {
      float wv[8];
      ld8(a.w + c, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[i][j] += v[i][j] * rstd * wv[j];
      st8(x + c, xv[i]);
      st8(h + c, xv[i]);
    }
  }
}

struct NormsDev {
  const long long* ids; const void* table; const void* y; long long ldy;
  const float* w1; const float* w2; float* x; void* h1; void* h2;
  int D, vocab;
  float mult, eps;
};

// V elements per thread and step, the row in registers (ITER steps) or, with ITER 0, in shared memory.
template <typename TE, typename TY, typename TH, int V, int ITER>
__global__ void __launch_bounds__(512)
stream_norms_kernel(const NormsDev a) {
  extern __shared__ float row_buf[];
  __shared__ float red[33];
  const long long t = blockIdx.x;
  float* x = a.x + t * a.D;
  const TE* e = a.ids ? reinterpret_cast<const TE*>(a.table) + CGK_IDX(a.ids[t], a.vocab) * a.D : nullptr;
  const TY* y = reinterpret_cast<const TY*>(a.y) + t * a.ldy;
  float xv[ITER > 0 ? ITER : 1][V], ss = 0.0f;
  auto take = [&](int c, float (&v)[V]) {
    if constexpr (V == 8) {
      if (e) { ld8(e + c, v); } else { ld8(x + c, v); }
    } else {
      v[0] = e ? ld1(e + c) : x[c];
    }
    if (a.y) {
      float u[V];
      if constexpr (V == 8) ld8(y + c, u); else u[0] = ld1(y + c);
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = fmaf(a.mult, u[j], v[j]);
    }
    if (a.y || e) {
      if constexpr (V == 8) st8(x + c, v); else x[c] = v[0];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(v[j], v[j], ss);
  };
  if constexpr (ITER > 0) {
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < a.D) take(c, xv[i]);
    }
  } else {
    for (int c = threadIdx.x * V; c < a.D; c += blockDim.x * V) {
      take(c, xv[0]);
#pragma unroll
      for (int j = 0; j < V; ++j) row_buf[c + j] = xv[0][j];
    }
  }
  if (!a.h1 && !a.h2) return;
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / a.D + a.eps);
  auto give = [&](int c, const float (&v)[V], const float* w, void* h) {
    if (!h) return;
    float o[V];
    if constexpr (V == 8) {
      ld8(w + c, o);
    } else {
      o[0] = w[c];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] *= v[j] * r;
    TH* p = reinterpret_cast<TH*>(h) + t * a.D + c;
    if constexpr (V == 8) st8(p, o); else st1(p, o[0]);
  };
  if constexpr (ITER > 0) {
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < a.D) { give(c, xv[i], a.w1, a.h1); give(c, xv[i], a.w2, a.h2); }
    }
  } else {
    for (int c = threadIdx.x * V; c < a.D; c += blockDim.x * V) {
#pragma unroll
      for (int j = 0; j < V; ++j) xv[0][j] = row_buf[c + j];
      give(c, xv[0], a.w1, a.h1);
      give(c, xv[0], a.w2, a.h2);
    }
  }
}

__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap, float inv) {
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) x[i] = cap * tanhf(x[i] * inv);
}

template <typename TO>
__global__ void rms_rows_kernel(const float* __restrict__ x, const long long* __restrict__ rows, int n_rows, const float* __restrict__ w,
                                TO* __restrict__ out, int D, float eps) {
  __shared__ float red[33];
  const long long i = blockIdx.x;
  const float* xr = x + CGK_IDX(rows ? rows[i] : i, n_rows) * D;
  float ss = 0.0f;
  for (int c = threadIdx.x; c < D; c += blockDim.x) ss = fmaf(xr[c], xr[c], ss);
  ss = block_sum(ss, red);
  const float rstd = 1.0f / sqrtf(ss / D + eps);
  for (int c = threadIdx.x; c < D; c += blockDim.x) st1(out + i * D + c, xr[c] * rstd * w[c]);
}

// threads for a row of n work items
int row_threads(int n) { return n <= 64 ? 64 : (n >= 512 ? 512 : (n + 31) / 32 * 32); }

template <typename TY, typename TP, typename TH>
int launch_update(const UpdateDev& d, int rows, bool vec, cudaStream_t st) {
  auto a16 = [](const void* p, long long row_bytes) { return !p || ((((uintptr_t)p) & 15) == 0 && row_bytes % 16 == 0); };
  if (d.D % 8 == 0 && d.D <= 512 * 8 * 4 && a16(d.y, d.ldy * sizeof(TY)) && a16(d.pairs, d.ldp * sizeof(TP)) && a16(d.x, 0) && a16(d.w, 0) &&
      a16(d.h, 0)) {
    const int vecs = d.D / 8, iter = vecs <= 512 ? 1 : (vecs <= 1024 ? 2 : 4), nt = ((vecs + iter - 1) / iter + 31) / 32 * 32;
    if (iter == 1) stream_update_regs_kernel<TY, TP, TH, 1><<<rows, nt, 0, st>>>(d);
    else if (iter == 2) stream_update_regs_kernel<TY, TP, TH, 2><<<rows, nt, 0, st>>>(d);
    else stream_update_regs_kernel<TY, TP, TH, 4><<<rows, nt, 0, st>>>(d);
    CGK_LAUNCH_CHECK();
    return 0;
  }
  const int smem = d.D * 4;
  const int nt = row_threads(vec ? d.D / 4 : d.D);
  if (vec) {
    if (smem > 48 * 1024)
      CGK_CUDA_CHECK(cudaFuncSetAttribute(stream_update_kernel<TY, TP, TH, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    stream_update_kernel<TY, TP, TH, 4><<<rows, nt, smem, st>>>(d);
  } else {
    if (smem > 48 * 1024)
      CGK_CUDA_CHECK(cudaFuncSetAttribute(stream_update_kernel<TY, TP, TH, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    stream_update_kernel<TY, TP, TH, 1><<<rows, nt, smem, st>>>(d);
  }
  CGK_LAUNCH_CHECK();
  return 0;
}

template <typename TE, typename TY, typename TH>
int launch_norms(const NormsDev& d, int rows, bool vec, cudaStream_t st) {
  if (vec && d.D <= 512 * 8 * 4) {
    const int vecs = d.D / 8, iter = vecs <= 512 ? 1 : (vecs <= 1024 ? 2 : 4), nt = ((vecs + iter - 1) / iter + 31) / 32 * 32;
    if (iter == 1) stream_norms_kernel<TE, TY, TH, 8, 1><<<rows, nt, 0, st>>>(d);
    else if (iter == 2) stream_norms_kernel<TE, TY, TH, 8, 2><<<rows, nt, 0, st>>>(d);
    else stream_norms_kernel<TE, TY, TH, 8, 4><<<rows, nt, 0, st>>>(d);
  } else {
    const int smem = d.D * 4;
    if (smem > 48 * 1024)
      CGK_CUDA_CHECK(cudaFuncSetAttribute(stream_norms_kernel<TE, TY, TH, 1, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    stream_norms_kernel<TE, TY, TH, 1, 0><<<rows, row_threads(d.D), smem, st>>>(d);
  }
  CGK_LAUNCH_CHECK();
  return 0;
}

}  // namespace
}  // namespace cgk

using namespace cgk;

CGK_API int cgk_stream_norms(const cgk_stream_norms_args* pa, void* stream) {
  CGK_REQUIRE(pa, "cgk_stream_norms: null args");
  const cgk_stream_norms_args& a = *pa;
  CGK_REQUIRE(a.x && a.rows >= 0 && a.D > 0 && (!a.ids || (a.table && a.vocab > 0)) && !(a.ids && a.y) && (!a.h1 || a.w1) && (!a.h2 || a.w2),
              "cgk_stream_norms: bad arguments");
  CGK_REQUIRE(a.D * 4 <= 200 * 1024, "cgk_stream_norms: rows of %d elements are too long", a.D);
  if (a.rows == 0) return 0;
  NormsDev d{(const long long*)a.ids, a.table, a.y, a.ldy, a.w1, a.w2, a.x, a.h1, a.h2, a.D, a.vocab, a.mult, a.eps};
  auto al = [](const void* p) { return (((uintptr_t)p) & 15) == 0; };
  const bool vec = a.D % 8 == 0 && a.ldy % 8 == 0 && al(a.table) && al(a.y) && al(a.w1) && al(a.w2) && al(a.x) && al(a.h1) && al(a.h2);
  cudaStream_t st = (cudaStream_t)stream;
  typedef __nv_bfloat16 bf;
  if (a.h_fp32) {
    CGK_REQUIRE((!a.ids || a.table_fp32) && (!a.y || a.y_fp32), "cgk_stream_norms: the fp32 form takes fp32 inputs");
    return launch_norms<float, float, float>(d, a.rows, vec, st);
  }
  CGK_REQUIRE(!a.ids || !a.table_fp32, "cgk_stream_norms: table and norms must have one type");
  return a.y_fp32 ? launch_norms<bf, float, bf>(d, a.rows, vec, st) : launch_norms<bf, bf, bf>(d, a.rows, vec, st);
}

CGK_API int cgk_softcap(void* x, long long n, float cap, void* stream) {
  CGK_REQUIRE((x || n == 0) && n >= 0 && cap > 0.0f, "cgk_softcap: bad arguments");
  if (n == 0) return 0;
  const long long blocks = (n + 1023) / 1024;
  softcap_kernel<<<(unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, (cudaStream_t)stream>>>((float*)x, n, cap, 1.0f / cap);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_embed_sinusoid(const void* ids, const void* pos, const void* table, int table_fp32, float scale, const void* freq,
                               void* x, void* h, int h_fp32, int rows, int D, int vocab, void* stream) {
  CGK_REQUIRE(ids && pos && table && x && h && rows >= 0 && D > 0 && vocab > 0, "cgk_embed_sinusoid: bad arguments");
  if (rows == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const int nt = (D + 1) / 2 < 256 ? 128 : 256;
  const long long* i = (const long long*)ids;
  const int* p = (const int*)pos;
  const double* f = (const double*)freq;
  if (table_fp32 && h_fp32)
    embed_sinusoid_kernel<float, float><<<rows, nt, 0, st>>>(i, p, (const float*)table, scale, f, (float*)x, (float*)h, D, vocab);
  else if (!table_fp32 && !h_fp32)
    embed_sinusoid_kernel<__nv_bfloat16, __nv_bfloat16><<<rows, nt, 0, st>>>(i, p, (const __nv_bfloat16*)table, scale, f, (float*)x,
                                                                             (__nv_bfloat16*)h, D, vocab);
  else
    CGK_REQUIRE(false, "cgk_embed_sinusoid: table and operand copy must have one type");
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_stream_update(const cgk_stream_update_args* pa, void* stream) {
  CGK_REQUIRE(pa, "cgk_stream_update: null args");
  const cgk_stream_update_args& a = *pa;
  CGK_REQUIRE(a.x && a.h && a.w && a.rows >= 0 && a.D > 0 && (a.y || a.pairs), "cgk_stream_update: bad arguments");
  CGK_REQUIRE(a.D * 4 <= 200 * 1024, "cgk_stream_update: rows of %d elements are too long", a.D);
  CGK_REQUIRE(!a.pairs || (a.row_of && a.weight && a.top > 0), "cgk_stream_update: expert rows need their index and weight tables");
  if (a.rows == 0) return 0;
  UpdateDev d{a.y, a.ldy, a.pairs, a.ldp, a.row_of, a.weight, a.pairs ? a.top : 0, a.pair_rows, a.w, a.x, a.h, a.D, a.eps};
  auto ok = [](const void* p, long long ld, int es) { return !p || ((((uintptr_t)p) % (4 * es)) == 0 && ld % 4 == 0); };
  const bool vec = a.D % 4 == 0 && ok(a.y, a.ldy, a.y_fp32 ? 4 : 2) && ok(a.pairs, a.ldp, a.pairs_fp32 ? 4 : 2) &&
                   ok(a.x, a.D, 4) && ok(a.w, a.D, 4) && ok(a.h, a.D, a.h_fp32 ? 4 : 2);
  cudaStream_t st = (cudaStream_t)stream;
  typedef __nv_bfloat16 bf;
  if (a.h_fp32) {
    CGK_REQUIRE((!a.y || a.y_fp32) && (!a.pairs || a.pairs_fp32), "cgk_stream_update: the fp32 form takes fp32 inputs");
    return launch_update<float, float, float>(d, a.rows, vec, st);
  }
  const bool yf = a.y && a.y_fp32, pf = a.pairs && a.pairs_fp32;
  if (yf && pf) return launch_update<float, float, bf>(d, a.rows, vec, st);
  if (yf) return launch_update<float, bf, bf>(d, a.rows, vec, st);
  if (pf) return launch_update<bf, float, bf>(d, a.rows, vec, st);
  return launch_update<bf, bf, bf>(d, a.rows, vec, st);
}

CGK_API int cgk_rms_rows(const void* x, const void* rows, int n_out, int n_rows, const void* w, void* out, int out_fp32, int D, float eps,
                         void* stream) {
  CGK_REQUIRE(x && w && out && n_out >= 0 && D > 0, "cgk_rms_rows: bad arguments");
  if (n_out == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const int nt = row_threads(D);
  if (out_fp32)
    rms_rows_kernel<float><<<n_out, nt, 0, st>>>((const float*)x, (const long long*)rows, n_rows, (const float*)w, (float*)out, D, eps);
  else
    rms_rows_kernel<__nv_bfloat16><<<n_out, nt, 0, st>>>((const float*)x, (const long long*)rows, n_rows, (const float*)w,
                                                        (__nv_bfloat16*)out, D, eps);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_BOUNDS_READER(residual_stream)
