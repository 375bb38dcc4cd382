// Attention over paged keys and values with rotary positions, for models served by the layer-stack engine:
//   * the angles of a step's tokens (cosine, sine per pair), formed and reduced in fp64 and shared by all layers
//     with the same rotation,
//   * the step between the q / k / v products and attention: rotation of queries and keys (interleaved pairs),
//     RMS norm of each value head, rotation of values by their position, append to the pages, and contiguous
//     copies with padded heads for the prompt kernel - one pass,
//   * the gather of part of a sequence into contiguous keys / values (a prompt portion that continues a block),
//   * attention of single query tokens over the pages: causal, optionally inside blocks of positions, optionally
//     with a sink (a key of score 0 without a value), the result turned back by the query's own position.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "kv_rows.cuh"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

__global__ void rotary_angles_kernel(const int* __restrict__ pos, const double* __restrict__ freq, float2* __restrict__ cs, int rows, int pairs) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)rows * pairs) return;
  const long long t = i / pairs;
  const double two_pi = 6.283185307179586;
  double a = (double)pos[t] * freq[i - t * pairs];
  a -= two_pi * rint(a / two_pi);
  float s, c;
  sincosf((float)a, &s, &c);
  cs[i] = make_float2(c, s);
}

struct PrepDev {
  KvRowsDev c;
  const void* q; const void* k; const void* v; long long ldq, ldk, ldv;   // rows of the products; k and v null: queries only
  const float2* cs_k; const float2* cs_v;                                // [rows][rot / 2], [rows][vdim / 2] or null (values stay)
  void* q_out; void* k_out; void* v_out;                                 // [rows][heads][wide]; k_out, v_out may be null
  int heads, rot, wide, norm_v;
  float eps;
};

// V consecutive columns of a head row, pairs (2i, 2i + 1) turned by the angles in cs
template <typename T, int V>
__device__ __forceinline__ void load_cols(const T* p, int col, int n, float (&x)[V]) {
  if constexpr (V == 8) {
    if (col + 8 <= n) {
      float a[4], b[4];
      ldv<4>(p + col, a);
      ldv<4>(p + col + 4, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) { x[j] = a[j]; x[4 + j] = b[j]; }
      return;
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) x[j] = col + j < n ? ld1(p + col + j) : 0.0f;
}
template <typename T, int V>
__device__ __forceinline__ void store_cols(T* p, int col, int n, const float (&x)[V]) {
  if constexpr (V == 8) {
    if (col + 8 <= n) {
      const float a[4] = {x[0], x[1], x[2], x[3]}, b[4] = {x[4], x[5], x[6], x[7]};
      stv<4>(p + col, a);
      stv<4>(p + col + 4, b);
      return;
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j)
    if (col + j < n) st1(p + col + j, x[j]);
}
template <int V>
__device__ __forceinline__ void turn_cols(const float2* __restrict__ cs, int col, int rot, float sign, float (&x)[V]) {
#pragma unroll
  for (int j = 0; j < V; j += 2)
    if (col + j + 1 < rot) {
      const float2 a = cs[(col + j) >> 1];
      const float u = x[j], v = x[j + 1], s = a.y * sign;
      x[j] = u * a.x - v * s;
      x[j + 1] = v * a.x + u * s;
    }
}

// One CTA per token: queries and keys by column groups of all threads, value heads by warps.
template <typename T, int V>
__global__ void __launch_bounds__(256)
rotate_append_kernel(const PrepDev a) {
  const KvRowsDev& c = a.c;
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const float2* cs_k = a.cs_k + t * (a.rot >> 1);
  {
    const T* q = reinterpret_cast<const T*>(a.q) + t * a.ldq;
    T* out = reinterpret_cast<T*>(a.q_out) + t * a.heads * a.wide;
    const int per = a.wide / V;
    for (int i = threadIdx.x; i < a.heads * per; i += blockDim.x) {
      const int h = i / per, col = (i - h * per) * V;
      float x[V];
      load_cols<T, V>(q + h * c.dim, col, c.dim, x);
      turn_cols<V>(cs_k, col, a.rot, 1.0f, x);
      store_cols<T, V>(out + h * a.wide, col, a.wide, x);
    }
  }
  if (!a.k) return;
  const int p = (int)CGK_IDX(c.pos[t], (long long)c.max_pages * c.page_size), s = (int)CGK_IDX(c.slot[t], c.slots);
  const long long page = CGK_IDX(c.page_table[(long long)s * c.max_pages + c.page_of(p)], c.n_pages);
  {
    const T* k = reinterpret_cast<const T*>(a.k) + t * a.ldk;
    const int wide = a.k_out ? max(a.wide, c.ld_k) : c.ld_k, per = wide / V;
    for (int i = threadIdx.x; i < c.kv_heads * per; i += blockDim.x) {
      const int g = i / per, col = (i - g * per) * V;
      float x[V];
      load_cols<T, V>(k + g * c.dim, col, c.dim, x);
      turn_cols<V>(cs_k, col, a.rot, 1.0f, x);
      store_cols<T, V>(reinterpret_cast<T*>(c.k_pages) + c.row_of(page, g, p) * c.ld_k, col, c.ld_k, x);
      if (a.k_out) store_cols<T, V>(reinterpret_cast<T*>(a.k_out) + (t * c.kv_heads + g) * a.wide, col, a.wide, x);
    }
  }
  const float2* cs_v = a.cs_v ? a.cs_v + t * (c.vdim >> 1) : nullptr;
  for (int g = warp; g < c.kv_heads; g += nw) {
    const T* v = reinterpret_cast<const T*>(a.v) + t * a.ldv + g * c.vdim;
    float r = 1.0f;
    if (a.norm_v) {
      float ss = 0.0f;
      for (int col = lane * V; col < c.vdim; col += 32 * V) {
        float x[V];
        load_cols<T, V>(v, col, c.vdim, x);
#pragma unroll
        for (int j = 0; j < V; ++j) ss = fmaf(x[j], x[j], ss);
      }
      r = 1.0f / sqrtf(warp_sum(ss) / c.vdim + a.eps);
    }
    const int wide = a.v_out ? max(a.wide, c.ld_v) : c.ld_v;
    for (int col = lane * V; col < wide; col += 32 * V) {
      float x[V];
      load_cols<T, V>(v, col, c.vdim, x);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= r;
      if (cs_v) turn_cols<V>(cs_v, col, c.vdim, 1.0f, x);
      store_cols<T, V>(reinterpret_cast<T*>(c.v_pages) + c.row_of(page, g, p) * c.ld_v, col, c.ld_v, x);
      if (a.v_out) store_cols<T, V>(reinterpret_cast<T*>(a.v_out) + (t * c.kv_heads + g) * a.wide, col, a.wide, x);
    }
  }
}

// Positions first .. first + len of one sequence -> [len][kv_heads][wide] for keys and for values; 16 bytes per thread.
__global__ void kv_gather_kernel(const KvRowsDev c, int slot, int first, int len, int esize, int wide, uint4* __restrict__ k_out, uint4* __restrict__ v_out) {
  const int per = wide * esize / 16;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)len * c.kv_heads * per) return;
  const int col = (int)(i % per);
  const long long r = i / per;
  const int g = (int)(r % c.kv_heads), key = first + (int)(r / c.kv_heads);
  const long long page = CGK_IDX(c.page_table[(long long)slot * c.max_pages + c.page_of(key)], c.n_pages);
  const long long row = c.row_of(page, g, key);
  const int kc = c.ld_k * esize / 16, vc = c.ld_v * esize / 16;
  const uint4 z = make_uint4(0, 0, 0, 0);
  k_out[i] = col < kc ? reinterpret_cast<const uint4*>(c.k_pages)[row * kc + col] : z;
  v_out[i] = col < vc ? reinterpret_cast<const uint4*>(c.v_pages)[row * vc + col] : z;
}

struct RowsDev {
  KvRowsDev c;
  const void* q; long long ldq; int wide;          // [rows][heads][wide]
  void* out; long long ldo;                        // [rows][heads * vdim]
  const float2* turn;                              // [rows][vdim / 2]: the result is turned back by these; null: left alone
  float* part; float* ml;                          // partial results of key ranges
  int heads, block, sink, splits, hgroups;
  float scale_log2;
};

// EPL elements of a row, kept as loaded until they are used; groups of 8 beyond the row's ld elements are zero
template <typename T, int EPL>
struct RawRow {
  static constexpr int Q = 8 * sizeof(T) / 16;             // 16-byte words per 8 elements
  uint4 w[EPL / 8 * Q];
  __device__ __forceinline__ void load(const T* p, int e0, int ld) {
#pragma unroll
    for (int i = 0; i < EPL / 8; ++i)
#pragma unroll
      for (int j = 0; j < Q; ++j)
        w[i * Q + j] = e0 + 8 * i < ld ? reinterpret_cast<const uint4*>(p + e0 + 8 * i)[j] : make_uint4(0, 0, 0, 0);
  }
  __device__ __forceinline__ void get(float (&x)[EPL]) const {
#pragma unroll
    for (int i = 0; i < EPL / 8 * Q; ++i) {
      const uint32_t u[4] = {w[i].x, w[i].y, w[i].z, w[i].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if constexpr (sizeof(T) == 2) {
          const float2 f = unpack_bf16x2(u[j]);
          x[8 * i + 2 * j] = f.x;
          x[8 * i + 2 * j + 1] = f.y;
        } else {
          x[4 * i + j] = __uint_as_float(u[j]);
        }
      }
    }
  }
};

// a pair of result columns, turned back and stored
template <typename T>
__device__ __forceinline__ void finish_pair(const RowsDev& a, long long t, int h, int col, float u, float v) {
  if (a.turn) {
    const float2 cs = a.turn[t * (a.c.vdim >> 1) + (col >> 1)];
    const float u0 = u;
    u = u0 * cs.x + v * cs.y;
    v = v * cs.x - u0 * cs.y;
  }
  T* o = reinterpret_cast<T*>(a.out) + t * a.ldo + (long long)h * a.c.vdim + col;
  st1(o, u);
  if (col + 1 < a.c.vdim) st1(o + 1, v);
}

// One CTA = (key range, kv head with up to R of its query heads, query token).  LPK lanes share a key, EPL elements each;
// a warp takes U keys per group of lanes at a time, the next ones on their way while it works.  The U * R scores are summed
// over the lanes so that every lane ends with its share of them (and one exponential per score is computed); maxima are
// the warp's, and stay until a score passes one by more than 2^8.  The four warps are merged at the end.
constexpr int KR_WARPS = 4;
template <int N, int LPK>
struct Shares {                                         // N sums over LPK lanes: C per lane, or DUP lanes with the same one
  static constexpr int C = N > LPK ? N / LPK : 1, DUP = N < LPK ? LPK / N : 1;
  static __device__ __forceinline__ int index(int sub, int c) { return DUP > 1 ? sub / DUP : sub * C + c; }
  static __device__ __forceinline__ int lane_of(int i) { return DUP > 1 ? i * DUP : i / C; }
  template <int M, int OFF>
  static __device__ __forceinline__ void step(float (&v)[N], int sub) {
    if constexpr (OFF >= 1) {
      if constexpr (M > 1) {
        const bool upper = (sub & OFF) != 0;
#pragma unroll
        for (int i = 0; i < M / 2; ++i) {
          const float send = upper ? v[i] : v[i + M / 2];
          v[i] = (upper ? v[i + M / 2] : v[i]) + __shfl_xor_sync(0xffffffffu, send, OFF);
        }
        step<M / 2, OFF / 2>(v, sub);
      } else {
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], OFF);
        step<1, OFF / 2>(v, sub);
      }
    }
  }
  static __device__ __forceinline__ void sum(float (&v)[N], int sub) { step<N, LPK / 2>(v, sub); }
};

template <typename T, int LPK, int EPL, int R>
__global__ void __launch_bounds__(KR_WARPS * 32, sizeof(T) == 2 && EPL == 8 ? 3 : 1)
kv_rows_kernel(const RowsDev a) {
  constexpr int KPW = 32 / LPK, W = LPK * EPL, U = EPL == 8 ? 4 : 1, N = U * R;
  typedef Shares<N, LPK> Sh;
  __shared__ float sh[KR_WARPS][R][W];
  __shared__ float stat[KR_WARPS][R][2];
  const KvRowsDev& c = a.c;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane % LPK, kg = lane / LPK, e0 = sub * EPL;
  const long long t = blockIdx.y;
  const int split = blockIdx.x % a.splits, hg = (int)(blockIdx.x / a.splits) % a.hgroups, g = (int)(blockIdx.x / a.splits) / a.hgroups;
  const int group = a.heads / c.kv_heads, h0 = g * group + hg * R, nh = min(R, group - hg * R);
  const int p = (int)CGK_IDX(c.pos[t], (long long)c.max_pages * c.page_size);
  const int lo = a.block > 0 ? p / a.block * a.block : 0, n = p + 1 - lo;
  constexpr int STEP = KR_WARPS * KPW * U;
  const int per = ((n + a.splits - 1) / a.splits + STEP - 1) / STEP * STEP;
  const int k_begin = lo + split * per, k_end = min(p + 1, k_begin + per);
  const int* row = c.page_table + CGK_IDX(c.slot[t], c.slots) * c.max_pages;
  const T* kp = reinterpret_cast<const T*>(c.k_pages);
  const T* vp = reinterpret_cast<const T*>(c.v_pages);

  float q[R][EPL], acc[R][EPL], m[R], l[Sh::C], mo[Sh::C];
#pragma unroll
  for (int i = 0; i < Sh::C; ++i) { l[i] = 0.0f; mo[i] = -INFINITY; }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    m[r] = -INFINITY;
#pragma unroll
    for (int e = 0; e < EPL; ++e) { q[r][e] = 0.0f; acc[r][e] = 0.0f; }
    if (r < nh) {
      RawRow<T, EPL> x;
      x.load(reinterpret_cast<const T*>(a.q) + t * a.ldq + (long long)(h0 + r) * a.wide, e0, c.ld_k);
      x.get(q[r]);
#pragma unroll
      for (int e = 0; e < EPL; ++e) q[r][e] *= a.scale_log2;
    }
  }
  RawRow<T, EPL> kk[U], vv[U];
  auto load = [&](int k0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int key = min(k0 + u * KPW + kg, k_end - 1);
      const long long at = c.row_of(CGK_IDX(row[c.page_of(key)], c.n_pages), g, key);
      kk[u].load(kp + at * c.ld_k, e0, c.ld_k);
      vv[u].load(vp + at * c.ld_v, e0, c.ld_v);
    }
  };
  int k0 = k_begin + warp * KPW * U;
  if (k0 < k_end) load(k0);
  for (; k0 < k_end; k0 += STEP) {
    float s[N];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float x[EPL];
      kk[u].get(x);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float d0 = 0.0f, d1 = 0.0f;
#pragma unroll
        for (int e = 0; e < EPL; e += 2) ffma2(d0, d1, q[r][e], q[r][e + 1], x[e], x[e + 1], d0, d1);
        s[u * R + r] = d0 + d1;
      }
    }
    RawRow<T, EPL> v0[U];
#pragma unroll
    for (int u = 0; u < U; ++u) v0[u] = vv[u];
    const int k1 = k0;
    if (k0 + STEP < k_end) load(k0 + STEP);
    Sh::sum(s, sub);
    bool grown = false;
#pragma unroll
    for (int i = 0; i < Sh::C; ++i) {
      if (k1 + Sh::index(sub, i) / R * KPW + kg >= k_end) s[i] = -INFINITY;
      grown |= s[i] > mo[i] + 8.0f;
    }
    if (__any_sync(0xffffffffu, grown)) {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float x = -INFINITY;
#pragma unroll
        for (int i = 0; i < Sh::C; ++i) x = Sh::index(sub, i) % R == r ? fmaxf(x, s[i]) : x;
        x = fmaxf(warp_max(x), m[r]);
        const float corr = x > -INFINITY ? exp2f(m[r] - x) : 1.0f;
        m[r] = x;
#pragma unroll
        for (int e = 0; e < EPL; ++e) acc[r][e] *= corr;
#pragma unroll
        for (int i = 0; i < Sh::C; ++i)
          if (Sh::index(sub, i) % R == r) { l[i] *= corr; mo[i] = x; }
      }
    }
    float w[Sh::C];
#pragma unroll
    for (int i = 0; i < Sh::C; ++i) {
      w[i] = sizeof(T) == 2 ? fast_exp2(s[i] - mo[i]) : exp2f(s[i] - mo[i]);
      l[i] += w[i];
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float x[EPL];
      v0[u].get(x);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const float pw = __shfl_sync(0xffffffffu, w[(u * R + r) % Sh::C], kg * LPK + Sh::lane_of(u * R + r));
#pragma unroll
        for (int e = 0; e < EPL; e += 2) ffma2(acc[r][e], acc[r][e + 1], pw, pw, x[e], x[e + 1], acc[r][e], acc[r][e + 1]);
      }
    }
  }
  // key groups of the warp, then the warps
#pragma unroll
  for (int r = 0; r < R; ++r) {
#pragma unroll
    for (int e = 0; e < EPL; ++e)
#pragma unroll
      for (int o = LPK; o < 32; o <<= 1) acc[r][e] += __shfl_xor_sync(0xffffffffu, acc[r][e], o);
    float lr = 0.0f;
#pragma unroll
    for (int i = 0; i < Sh::C; ++i)
      if (Sh::index(sub, i) % R == r && sub % Sh::DUP == 0) lr += l[i];
    lr = warp_sum(lr);
    if (kg == 0) {
#pragma unroll
      for (int e = 0; e < EPL; ++e) sh[warp][r][e0 + e] = acc[r][e];
    }
    if (lane == 0) { stat[warp][r][0] = m[r]; stat[warp][r][1] = lr; }
  }
  __syncthreads();
  const int pairs = (c.vdim + 1) / 2;
  for (int i = threadIdx.x; i < nh * pairs; i += KR_WARPS * 32) {
    const int r = i / pairs, col = (i - r * pairs) * 2;
    float mm = -INFINITY, ll = 0.0f, u = 0.0f, v = 0.0f;
#pragma unroll
    for (int w = 0; w < KR_WARPS; ++w) mm = fmaxf(mm, stat[w][r][0]);
#pragma unroll
    for (int w = 0; w < KR_WARPS; ++w) {
      const float f = stat[w][r][0] > -INFINITY ? exp2f(stat[w][r][0] - mm) : 0.0f;
      ll = fmaf(stat[w][r][1], f, ll);
      u = fmaf(sh[w][r][col], f, u);
      v = fmaf(sh[w][r][col + 1], f, v);
    }
    if (a.splits == 1) {
      if (a.sink) ll += exp2f(-mm);
      const float inv = 1.0f / ll;
      finish_pair<T>(a, t, h0 + r, col, u * inv, v * inv);
    } else {
      const long long at = (t * a.heads + h0 + r) * a.splits + split;
      float* o = a.part + at * 2 * pairs + col;
      o[0] = u;
      o[1] = v;
      if (col == 0) { a.ml[at * 2] = mm; a.ml[at * 2 + 1] = ll; }
    }
  }
}

// Partial results of up to 32 key ranges of one (token, head) -> result
template <typename T>
__global__ void kv_rows_merge_kernel(const RowsDev a) {
  __shared__ float weight[32];
  const long long t = blockIdx.y;
  const int h = blockIdx.x, lane = threadIdx.x & 31, pairs = (a.c.vdim + 1) / 2;
  const long long at = (t * a.heads + h) * a.splits;
  if (threadIdx.x < 32) {
    const float2 v = lane < a.splits ? reinterpret_cast<const float2*>(a.ml)[at + lane] : make_float2(-INFINITY, 0.0f);
    const float m = warp_max(v.x);
    const float f = v.x > -INFINITY ? exp2f(v.x - m) : 0.0f;
    weight[lane] = f / (warp_sum(v.y * f) + (a.sink ? exp2f(-m) : 0.0f));
  }
  __syncthreads();
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    float u = 0.0f, v = 0.0f;
    for (int s = 0; s < a.splits; ++s) {
      const float w = weight[s];
      if (w > 0.0f) {
        const float2 x = reinterpret_cast<const float2*>(a.part)[(at + s) * pairs + i];
        u = fmaf(w, x.x, u);
        v = fmaf(w, x.y, v);
      }
    }
    finish_pair<T>(a, t, h, 2 * i, u, v);
  }
}

template <typename T, int LPK, int EPL, int R>
int launch_rows(const RowsDev& d, int rows, cudaStream_t st) {
  const dim3 grid(d.splits * d.c.kv_heads * d.hgroups, rows);
  kv_rows_kernel<T, LPK, EPL, R><<<grid, KR_WARPS * 32, 0, st>>>(d);
  CGK_LAUNCH_CHECK();
  if (d.splits > 1) {
    kv_rows_merge_kernel<T><<<dim3(d.heads, rows), d.c.vdim >= 128 ? 64 : 32, 0, st>>>(d);
    CGK_LAUNCH_CHECK();
  }
  return 0;
}
template <typename T, int LPK, int EPL>
int pick_heads(RowsDev& d, int rows, cudaStream_t st) {
  const int group = d.heads / d.c.kv_heads;
  constexpr int RMAX = EPL == 8 ? 4 : 1;
  if (group == 1 || RMAX == 1) { d.hgroups = group; return launch_rows<T, LPK, EPL, 1>(d, rows, st); }
  if (group == 2) { d.hgroups = 1; return launch_rows<T, LPK, EPL, 2>(d, rows, st); }
  d.hgroups = (group + RMAX - 1) / RMAX;
  return launch_rows<T, LPK, EPL, RMAX>(d, rows, st);
}
template <typename T>
int pick_rows(RowsDev& d, int rows, cudaStream_t st) {
  const int w = max(d.c.ld_k, d.c.ld_v);
  if (w <= 32) return pick_heads<T, 4, 8>(d, rows, st);
  if (w <= 64) return pick_heads<T, 8, 8>(d, rows, st);
  if (w <= 128) return pick_heads<T, 16, 8>(d, rows, st);
  if (w <= 256) return pick_heads<T, 32, 8>(d, rows, st);
  if (w <= 512) return pick_heads<T, 32, 16>(d, rows, st);
  return pick_heads<T, 32, 32>(d, rows, st);
}

int fill_kv(const cgk_kv_rows_args& a, KvRowsDev* d) {
  CGK_REQUIRE(a.k_pages && a.v_pages && a.page_table && a.kv_heads > 0 && a.dim > 0 && a.vdim > 0 && a.page_size > 0 && a.max_pages > 0 &&
              a.slots > 0 && a.n_pages > 0, "paged keys and values: bad arguments");
  const int shift = (a.page_size & (a.page_size - 1)) == 0 ? __builtin_ctz(a.page_size) : -1;
  *d = KvRowsDev{a.k_pages, a.v_pages, a.page_table, a.slot, a.pos, a.kv_heads, a.dim, a.vdim, (a.dim + 7) / 8 * 8, (a.vdim + 7) / 8 * 8,
                 a.page_size, shift, a.max_pages, a.slots, a.n_pages};
  return 0;
}

}  // namespace
}  // namespace cgk

using namespace cgk;

CGK_API int cgk_rotary_angles(const void* pos, const void* freq, void* cs, int rows, int pairs, void* stream) {
  CGK_REQUIRE(pos && freq && cs && rows >= 0 && pairs > 0, "cgk_rotary_angles: bad arguments");
  if (rows == 0) return 0;
  const long long n = (long long)rows * pairs;
  rotary_angles_kernel<<<(unsigned)((n + 127) / 128), 128, 0, (cudaStream_t)stream>>>((const int*)pos, (const double*)freq, (float2*)cs, rows, pairs);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_kv_rotate_append(const cgk_kv_rows_args* pc, const cgk_kv_prep_args* pa, int rows, void* stream) {
  CGK_REQUIRE(pc && pa && rows >= 0, "cgk_kv_rotate_append: bad arguments");
  const cgk_kv_prep_args& a = *pa;
  PrepDev d;
  int rc = fill_kv(*pc, &d.c);
  if (rc) return rc;
  CGK_REQUIRE(a.q && a.q_out && a.heads > 0 && a.rot >= 0 && a.rot <= pc->dim && a.rot % 2 == 0 && (a.rot == 0 || a.cs_k) && a.wide % 8 == 0 &&
              a.wide >= pc->dim && (!a.k == !a.v) && (!a.k || (pc->slot && pc->pos)) && (!a.cs_v || pc->vdim % 2 == 0) &&
              (!a.k_out == !a.v_out) && (!a.k_out || a.wide >= pc->vdim), "cgk_kv_rotate_append: bad arguments");
  if (rows == 0) return 0;
  d.q = a.q; d.k = a.k; d.v = a.v; d.ldq = a.ldq; d.ldk = a.ldk; d.ldv = a.ldv;
  d.cs_k = (const float2*)a.cs_k; d.cs_v = (const float2*)a.cs_v;
  d.q_out = a.q_out; d.k_out = a.k_out; d.v_out = a.v_out;
  d.heads = a.heads; d.rot = a.rot; d.wide = a.wide; d.norm_v = a.norm_v; d.eps = a.eps;
  cudaStream_t st = (cudaStream_t)stream;
  auto al = [](const void* p) { return (((uintptr_t)p) & 15) == 0; };
  const bool vec = d.c.dim % 8 == 0 && d.c.vdim % 8 == 0 && a.ldq % 8 == 0 && a.ldk % 8 == 0 && a.ldv % 8 == 0 && al(a.q) && al(a.k) && al(a.v) &&
                   al(a.q_out) && al(a.k_out) && al(a.v_out) && al(pc->k_pages) && al(pc->v_pages);
  const int work = a.heads * a.wide / (vec ? 8 : 2);
  const int nt = work >= 256 ? 256 : (work > 64 ? 128 : 64);
  if (pc->fp32) {
    if (vec) rotate_append_kernel<float, 8><<<rows, nt, 0, st>>>(d);
    else rotate_append_kernel<float, 2><<<rows, nt, 0, st>>>(d);
  } else {
    if (vec) rotate_append_kernel<__nv_bfloat16, 8><<<rows, nt, 0, st>>>(d);
    else rotate_append_kernel<__nv_bfloat16, 2><<<rows, nt, 0, st>>>(d);
  }
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API int cgk_kv_gather(const cgk_kv_rows_args* pc, int slot, int first, int len, int wide, void* k_out, void* v_out, void* stream) {
  CGK_REQUIRE(pc && k_out && v_out && first >= 0 && len >= 0 && first + len <= pc->max_pages * pc->page_size && slot >= 0 && slot < pc->slots && wide % 8 == 0,
              "cgk_kv_gather: bad arguments");
  KvRowsDev d;
  int rc = fill_kv(*pc, &d);
  if (rc) return rc;
  CGK_REQUIRE(wide >= d.ld_k && wide >= d.ld_v, "cgk_kv_gather: rows are longer than the output's");
  if (len == 0) return 0;
  const int es = pc->fp32 ? 4 : 2;
  const long long n = (long long)len * d.kv_heads * (wide * es / 16);
  kv_gather_kernel<<<(unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream>>>(d, slot, first, len, es, wide, (uint4*)k_out, (uint4*)v_out);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_API long long cgk_kv_rows_scratch_floats(int rows, int heads, int vdim, int splits) {
  return splits > 1 ? (long long)rows * heads * splits * (2 * ((vdim + 1) / 2) + 2) : 0;
}

CGK_API int cgk_kv_rows_attention(const cgk_kv_rows_args* pc, const void* q, long long ldq, int wide, void* out, long long ldo, const void* turn,
                                  int rows, int heads, float scale, int block, int sink, int splits, void* scratch, void* stream) {
  CGK_REQUIRE(pc && q && out && rows >= 0 && heads > 0 && heads % pc->kv_heads == 0 && pc->slot && pc->pos && splits >= 1 && splits <= 32 &&
              (splits == 1 || scratch) && (!turn || pc->vdim % 2 == 0), "cgk_kv_rows_attention: bad arguments");
  RowsDev d;
  int rc = fill_kv(*pc, &d.c);
  if (rc) return rc;
  CGK_REQUIRE(d.c.ld_k <= 1024 && d.c.ld_v <= 1024, "cgk_kv_rows_attention: heads of more than 1024 elements");
  CGK_REQUIRE(rows <= 65535, "cgk_kv_rows_attention: too many query tokens in one call");
  CGK_REQUIRE(wide % 8 == 0 && ldq % 8 == 0 && wide >= d.c.ld_k && (((uintptr_t)q) & 15) == 0 && (((uintptr_t)pc->k_pages) & 15) == 0 &&
              (((uintptr_t)pc->v_pages) & 15) == 0, "cgk_kv_rows_attention: rows must be 16-byte aligned");
  if (rows == 0) return 0;
  d.q = q; d.ldq = ldq; d.wide = wide; d.out = out; d.ldo = ldo; d.turn = (const float2*)turn;
  d.heads = heads; d.block = block; d.sink = sink; d.splits = splits; d.hgroups = 1;
  d.part = (float*)scratch;
  d.ml = splits > 1 ? (float*)scratch + (long long)rows * heads * splits * 2 * ((pc->vdim + 1) / 2) : nullptr;
  d.scale_log2 = scale * 1.4426950408889634f;
  cudaStream_t st = (cudaStream_t)stream;
  return pc->fp32 ? pick_rows<float>(d, rows, st) : pick_rows<__nv_bfloat16>(d, rows, st);
}

CGK_BOUNDS_READER(kv_rows)
