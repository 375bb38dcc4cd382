// Latent attention: keys and values of all heads are linear images of one short vector per token (the
// latent c), so the cache holds c alone, in pages.  This file has
//   * the step between the down-projections and everything else: RMS norm of the query latent and of the
//     key/value latent, the latter written into its cache page (one pass),
//   * the gather of a sequence's latents into a contiguous matrix (prompt path: keys and values are then
//     expanded by one matrix product),
//   * attention in the latent space on the CUDA cores: scores q'.c with q' = W_uk^T q, result sum p c
//     (W_uv is applied afterwards).  The form for fp32, and for shapes the tensor-core kernel
//     (latent_attn_tc.cu) does not take,
//   * the merge of partial results of key ranges, shared with the tensor-core kernel.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "latent_dev.cuh"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

// One CTA per token; the row stays in shared memory between the sums of squares and the scaling.
template <typename TI, typename T, int V>
__global__ void __launch_bounds__(256)
latent_norm_append_kernel(const TI* __restrict__ in, long long ld, const float* __restrict__ wq, const float* __restrict__ wc, int q_rank, int R,
                          float eps, T* __restrict__ cq, T* __restrict__ c_out, T* __restrict__ pages, const int* __restrict__ slot,
                          const int* __restrict__ pos, const int* __restrict__ page_table, int slots, int max_pages, int page_size, int n_pages) {
  extern __shared__ float row_buf[];
  __shared__ float red[64];
  const long long t = blockIdx.x;
  const int n = q_rank + R, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int p = (int)CGK_IDX(pos[t], (long long)max_pages * page_size), s = (int)CGK_IDX(slot[t], slots);
  const long long page = CGK_IDX(page_table[(long long)s * max_pages + p / page_size], n_pages);
  float sq = 0.0f, sc = 0.0f;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {        // q_rank is a multiple of V: no vector straddles
    float v[V], ss = 0.0f;
    ldv<V>(in + t * ld + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) { ss = fmaf(v[j], v[j], ss); row_buf[i + j] = v[j]; }
    if (i < q_rank) sq += ss; else sc += ss;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) { red[warp] = sq; red[32 + warp] = sc; }
  __syncthreads();
  sq = sc = 0.0f;
  for (int w = 0; w < nw; ++w) { sq += red[w]; sc += red[32 + w]; }
  const float rq = 1.0f / sqrtf(sq / q_rank + eps), rc = 1.0f / sqrtf(sc / R + eps);
  T* dst = pages + (page * page_size + p % page_size) * R;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    float v[V], w[V];
    const bool isq = i < q_rank;
    ldv<V>(isq ? wq + i : wc + i - q_rank, w);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = row_buf[i + j] * (isq ? rq : rc) * w[j];
    if (isq) {
      stv<V>(cq + t * q_rank + i, v);
    } else {
      stv<V>(dst + i - q_rank, v);
      if (c_out) stv<V>(c_out + t * R + i - q_rank, v);
    }
  }
}

// One warp per row.
template <typename T>
__global__ void latent_gather_kernel(const T* __restrict__ pages, const int* __restrict__ table_row, T* __restrict__ out, int len, int R, int page_size,
                                     int max_pages, int n_pages) {
  const int p = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (p >= len) return;
  const long long page = CGK_IDX(table_row[CGK_IDX(p / page_size, max_pages)], n_pages);
  const T* src = pages + (page * page_size + p % page_size) * R;
  T* dst = out + (long long)p * R;
  if ((R * (int)sizeof(T)) % 16 == 0) {
    for (int i = lane; i < R * (int)sizeof(T) / 16; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (int i = lane; i < R; i += 32) dst[i] = src[i];
  }
}

// One CTA per (head, query token); warp w walks keys w, w + 4, ... with a running maximum of its own, the
// four warps are merged at the end.  NR: latent elements per lane.
constexpr int LAT_WARPS = 4;
template <typename T, int NR>
__global__ void __launch_bounds__(LAT_WARPS * 32)
latent_attention_kernel(const LatentDev c, const T* __restrict__ q, T* __restrict__ out) {
  extern __shared__ float sh[];                       // [warps][R] accumulators, then [warps] maxima, [warps] sums
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t = blockIdx.y;
  const int h = blockIdx.x, R = c.R;
  const T* pages = reinterpret_cast<const T*>(c.pages);
  const T* qr = q + (t * c.heads + h) * R;
  float qv[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = lane + i * 32;
    qv[i] = r < R ? ld1(qr + r) * c.scale : 0.0f;
    acc[i] = 0.0f;
  }
  const int len = (int)CGK_IDX(c.pos[t], (long long)c.max_pages * c.page_size) + 1;
  const int* row = c.page_table + CGK_IDX(c.slot[t], c.slots) * c.max_pages;
  float m = -INFINITY, l = 0.0f;
  for (int key = warp; key < len; key += LAT_WARPS) {
    const long long page = CGK_IDX(row[key / c.page_size], c.n_pages);
    const T* kr = pages + (page * c.page_size + key % c.page_size) * R;
    float kv[NR], s = 0.0f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int r = lane + i * 32;
      kv[i] = r < R ? ld1(kr + r) : 0.0f;
      s = fmaf(qv[i], kv[i], s);
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s), corr = expf(m - mn), p = expf(s - mn);
    l = l * corr + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] = fmaf(p, kv[i], acc[i] * corr);
  }
  float* stat = sh + LAT_WARPS * R;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = lane + i * 32;
    if (r < R) sh[warp * R + r] = acc[i];
  }
  if (lane == 0) { stat[warp] = m; stat[LAT_WARPS + warp] = l; }
  __syncthreads();
  float mm = -INFINITY;
  for (int w = 0; w < LAT_WARPS; ++w) mm = fmaxf(mm, stat[w]);
  float f[LAT_WARPS], ll = 0.0f;
  for (int w = 0; w < LAT_WARPS; ++w) {
    f[w] = stat[w] > -INFINITY ? expf(stat[w] - mm) : 0.0f;
    ll = fmaf(stat[LAT_WARPS + w], f[w], ll);
  }
  const float inv = 1.0f / ll;
  for (int r = threadIdx.x; r < R; r += blockDim.x) {
    float v = 0.0f;
    for (int w = 0; w < LAT_WARPS; ++w) v = fmaf(sh[w * R + r], f[w], v);
    st1(out + (t * c.heads + h) * R + r, v * inv);
  }
}

// Partials of up to 32 key ranges -> result: out[row][r] = sum_s acc[row][s][r] 2^(m_s - m) / sum_s l_s 2^(m_s - m)
__global__ void latent_merge_kernel(const float* __restrict__ part, const float* __restrict__ ml, __nv_bfloat16* __restrict__ out, int splits, int R) {
  __shared__ float weight[32];
  const long long row = blockIdx.x;
  const int lane = threadIdx.x & 31, r = blockIdx.y * blockDim.x + threadIdx.x;
  const float* p = part + row * splits * R + r;
  float e[16];                                       // the first ranges' sums travel while the weights are worked out
#pragma unroll
  for (int s = 0; s < 16; ++s) e[s] = (s < splits && r < R) ? p[(long long)s * R] : 0.0f;
  if (threadIdx.x < 32) {
    const float2 v = lane < splits ? reinterpret_cast<const float2*>(ml)[row * splits + lane] : make_float2(-INFINITY, 0.0f);
    const float m = warp_max(v.x);
    const float f = v.x > -INFINITY ? exp2f(v.x - m) : 0.0f;
    weight[lane] = f / warp_sum(v.y * f);
  }
  __syncthreads();
  if (r >= R) return;
  // a range without keys has weight 0 and wrote no sums: whatever its memory holds is not used
  float v = 0.0f;
#pragma unroll
  for (int s = 0; s < 16; ++s) {
    const float w = weight[s];
    v += w > 0.0f ? w * e[s] : 0.0f;
  }
  for (int s = 16; s < splits; ++s) {
    const float w = weight[s];
    v += w > 0.0f ? w * p[(long long)s * R] : 0.0f;
  }
  out[row * R + r] = __float2bfloat16(v);
}

template <typename T, int NR>
int launch_simt(const LatentDev& d, const void* q, void* out, int n, cudaStream_t st) {
  const int smem = (LAT_WARPS * d.R + 2 * LAT_WARPS) * 4;
  latent_attention_kernel<T, NR><<<dim3(d.heads, n), LAT_WARPS * 32, smem, st>>>(d, (const T*)q, (T*)out);
  CGK_LAUNCH_CHECK();
  return 0;
}
template <typename T>
int pick_simt(const LatentDev& d, const void* q, void* out, int n, cudaStream_t st) {
  const int nr = (d.R + 31) / 32;
  if (nr <= 2) return launch_simt<T, 2>(d, q, out, n, st);
  if (nr <= 4) return launch_simt<T, 4>(d, q, out, n, st);
  if (nr <= 8) return launch_simt<T, 8>(d, q, out, n, st);
  if (nr <= 16) return launch_simt<T, 16>(d, q, out, n, st);
  return launch_simt<T, 32>(d, q, out, n, st);
}

int fill_latent(const cgk_latent_args& a, LatentDev* d) {
  CGK_REQUIRE(a.pages && a.page_table && a.slot && a.pos && a.R > 0 && a.page_size > 0 && a.max_pages > 0 && a.slots > 0 && a.n_pages > 0,
              "latent cache: bad arguments");
  *d = LatentDev{a.pages, (const int*)a.page_table, (const int*)a.slot, (const int*)a.pos, a.R, a.page_size, a.max_pages,
                 a.slots, a.n_pages, a.heads, a.scale};
  return 0;
}

}  // namespace

cudaError_t launch_latent_merge(const float* part, const float* ml, __nv_bfloat16* out, int rows, int splits, int R, cudaStream_t st) {
  latent_merge_kernel<<<dim3(rows, (R + 127) / 128), 128, 0, st>>>(part, ml, out, splits, R);
  return cudaGetLastError();
}

}  // namespace cgk

using namespace cgk;

CGK_API int cgk_latent_norm_append(const cgk_latent_args* pa, const void* in, int in_fp32, long long ld, const void* wq, const void* wc,
                                   int q_rank, float eps, void* cq, void* c_out, int rows, void* stream) {
  CGK_REQUIRE(pa && in && wq && wc && cq && q_rank > 0 && rows >= 0, "cgk_latent_norm_append: bad arguments");
  LatentDev d;
  int rc = fill_latent(*pa, &d);
  if (rc) return rc;
  if (rows == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  typedef __nv_bfloat16 bf;
  const int n = q_rank + d.R, smem = n * 4;
  CGK_REQUIRE(smem <= 48 * 1024, "cgk_latent_norm_append: rows of %d elements are too long", n);
  auto al = [](const void* p) { return (((uintptr_t)p) & 15) == 0; };
  const bool vec = q_rank % 4 == 0 && d.R % 4 == 0 && ld % 4 == 0 && al(in) && al(wq) && al(wc) && al(cq) && al(c_out) && al(d.pages);
  const int nt = n >= 2048 ? 256 : 128;
#define CGK_LNA(TI, T)                                                                                                              \
  do {                                                                                                                             \
    if (vec)                                                                                                                       \
      latent_norm_append_kernel<TI, T, 4><<<rows, nt, smem, st>>>((const TI*)in, ld, (const float*)wq, (const float*)wc, q_rank,   \
                                                                  d.R, eps, (T*)cq, (T*)c_out, (T*)d.pages, d.slot, d.pos,         \
                                                                  d.page_table, d.slots, d.max_pages, d.page_size, d.n_pages);     \
    else                                                                                                                           \
      latent_norm_append_kernel<TI, T, 1><<<rows, nt, smem, st>>>((const TI*)in, ld, (const float*)wq, (const float*)wc, q_rank,   \
                                                                  d.R, eps, (T*)cq, (T*)c_out, (T*)d.pages, d.slot, d.pos,         \
                                                                  d.page_table, d.slots, d.max_pages, d.page_size, d.n_pages);     \
  } while (0)
  if (pa->fp32) {
    CGK_REQUIRE(in_fp32, "cgk_latent_norm_append: the fp32 form takes fp32 inputs");
    CGK_LNA(float, float);
  } else if (in_fp32) {
    CGK_LNA(float, bf);
  } else {
    CGK_LNA(bf, bf);
  }
#undef CGK_LNA
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_latent_gather(const cgk_latent_args* pa, int slot, int len, void* out, void* stream) {
  CGK_REQUIRE(pa && out && pa->pages && pa->page_table && len >= 0 && len <= pa->max_pages * pa->page_size && slot >= 0 && slot < pa->slots,
              "cgk_latent_gather: bad arguments");
  if (len == 0) return 0;
  const int* row = (const int*)pa->page_table + (long long)slot * pa->max_pages;
  cudaStream_t st = (cudaStream_t)stream;
  if (pa->fp32) latent_gather_kernel<float><<<(len + 3) / 4, 128, 0, st>>>((const float*)pa->pages, row, (float*)out, len, pa->R, pa->page_size, pa->max_pages, pa->n_pages);
  else latent_gather_kernel<__nv_bfloat16><<<(len + 3) / 4, 128, 0, st>>>((const __nv_bfloat16*)pa->pages, row, (__nv_bfloat16*)out, len, pa->R, pa->page_size, pa->max_pages, pa->n_pages);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_latent_attention_tc_ok(int R, int page_size, int heads) { return latent_tc_ok(R, page_size, heads) ? 1 : 0; }

CGK_API long long cgk_latent_attention_scratch_floats(int rows, int heads, int R, int splits) {
  return splits > 1 ? (long long)rows * heads * splits * (R + 2) : 0;
}

CGK_API int cgk_latent_attention(const cgk_latent_args* pa, const void* q, void* out, int rows, int splits, void* scratch, int force_simt,
                                 void* stream) {
  CGK_REQUIRE(pa && q && out && rows >= 0 && pa->heads > 0, "cgk_latent_attention: bad arguments");
  LatentDev d;
  int rc = fill_latent(*pa, &d);
  if (rc) return rc;
  if (rows == 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  if (!pa->fp32 && !force_simt && latent_tc_ok(d.R, d.page_size, d.heads)) {
    CGK_REQUIRE(splits >= 1 && splits <= 32 && (splits == 1 || scratch), "cgk_latent_attention: up to 32 key ranges, with scratch space");
    return launch_latent_tc(d, (const __nv_bfloat16*)q, (__nv_bfloat16*)out, rows, splits, (float*)scratch, st);
  }
  CGK_REQUIRE(d.R <= 1024, "cgk_latent_attention: latents of %d elements are longer than the 1024 supported", d.R);
  CGK_REQUIRE(rows <= 65535, "cgk_latent_attention: too many query tokens in one call");
  return pa->fp32 ? pick_simt<float>(d, q, out, rows, st) : pick_simt<__nv_bfloat16>(d, q, out, rows, st);
}

CGK_BOUNDS_READER(latent_kv)
