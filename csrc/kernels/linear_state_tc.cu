// Linear recurrences (linear_state.cuh) over prompt portions, 64 tokens at a time on the tcgen05 tensor cores.
//
// With b_t the logarithm of the decay since the start of a chunk (per state row), r its value in the chunk's middle,
//     Q = q 2^(b - r),  K = k 2^(r - b),  A = tril(Q K^T),  O = A V + Q (2^r S),  S' = 2^(b_end - r) (2^r S + K^T V)
// so a chunk takes four products.  The state stays in TMEM in fp32 from chunk to chunk (times a factor per row that is kept
// beside it); every fp32 operand enters the tensor core as the sum of two bf16 numbers (three products for two such
// operands, the smallest one is dropped), so the sums see 16 bits of each factor.  Where a decay is so strong that
// the exponents could leave fp32's range, A is formed term by term with b_t - b_s <= 0, and Q and K take the
// chunk's ends as their references.
//
// One CTA walks the chunks of one (stretch of a run, head).  A long run is cut into stretches that run side by side: a
// first pass sums up what each stretch adds to the state, a second one turns that into the stretches' first states.
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "linear_state.cuh"
#include "sm100.cuh"
#include "typed_io.cuh"

namespace cgk {
namespace {

constexpr int LC = 64, LC_THREADS = 512;
constexpr float LC_LIMIT = 100.0f;                        // largest exponent (base 2) of a factor
// shared memory: operand tiles of 128-byte rows in blocks of 64 columns (bytes)
constexpr uint32_t T_K = 0, T_V = 32768, T_Q = 49152, T_A = 81920, T_S = 98304, T_END = 163840;
constexpr uint32_t T_END_SUM = T_Q;                       // the summing pass has K and V only
constexpr uint32_t T_SPLIT = 16384;                       // high part -> low part of Q and K
constexpr uint32_t LC_MISC = (8 * 128 + 5 * 128 + 4 * LC) * 4 + 64 + LC_THREADS * 8 * 12;      // and staged rows
constexpr uint32_t TM_S = 0, TM_O = 128, TM_A = 256;      // TMEM columns

struct ChunksDev {
  LinStateDev a;
  const int* items;          // [n_items][4]: first row, tokens, run, last stretch of the run
  float* start;              // [n_items][heads][D][V]: sums, then first states; null: every run is one stretch
  float* total;              // [n_items][heads][D]: logarithm (base 2) of a stretch's whole decay
  int* status;
};

__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x0, x1);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x0 - h.x, x1 - h.y);
}
// byte offset of a 4-byte pair of columns in a tile with `rows` rows per block
__device__ __forceinline__ uint32_t pair_at(int row, int col, int rows) {
  return (col >> 6) * (rows * 128) + sw128_offset(row, (col & 63) >> 3) + (col & 7) * 2;
}

// operand descriptors of consecutive 16-wide steps differ by constants in the address field
__device__ __forceinline__ uint64_t k_major(uint64_t d, int kk) { return d + (uint64_t)(((kk >> 2) * (LC * 128) + (kk & 3) * 32) >> 4); }
__device__ __forceinline__ uint64_t mn_major(uint64_t d, int kk) { return d + (uint64_t)((kk * 2048) >> 4); }

// meeting point of the sixteen worker warps, plain and with a vote
__device__ __forceinline__ void lc_meet() { asm volatile("bar.sync 1, 512;" ::: "memory"); }
__device__ __forceinline__ bool lc_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "bar.red.or.pred q, 1, 512, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"((uint32_t)v) : "memory");
  return r != 0;
}

// Warps 0 .. 15 prepare operands and read results, warp 16 issues the products.
template <bool OUT, int MODE>
__global__ void __launch_bounds__(LC_THREADS + 32, 1)
linear_chunks_kernel(const ChunksDev c) {
  const LinStateDev& a = c.a;
  extern __shared__ uint8_t lc_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lc_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sb = smem_u32(sm);
  constexpr uint32_t END = OUT ? T_END : T_END_SUM;
  float* part = reinterpret_cast<float*>(sm + END);       // [8][128] decay of eight tokens
  float* rq = part + 8 * 128;                             // [128] references of Q and K
  float* rk = rq + 128;
  float* pend = rk + 128;                                 // [2][128] factor of the state in TMEM, by parity of the chunk
  float* tot = pend + 256;                                // [128] decay of all chunks
  float* red = tot + 128;                                 // [4][64]
  uint32_t* bars = reinterpret_cast<uint32_t*>(red + 4 * LC);
  const uint32_t b_qk = smem_u32(bars), b_sa = b_qk + 8, bar_a = b_qk + 16, bar_o = b_qk + 24, bar_s = b_qk + 32;
  volatile uint32_t* tmem_slot = bars + 10;
  volatile int* dead = reinterpret_cast<volatile int*>(bars + 11);
  volatile int* far_flag = reinterpret_cast<volatile int*>(bars + 12);

  const int* item = c.items + 4 * blockIdx.y;
  const int row0 = item[0], count = item[1], last = item[3], h = blockIdx.x;
  if (!OUT && last) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = a.D, V = a.V, n_chunks = (count + LC - 1) / LC;
  constexpr uint32_t COLS = OUT ? 512 : 128;

  if (tid == 0) {
    mbar_init(b_qk, 16);
    mbar_init(b_sa, 16);
    mbar_init(bar_a, 1);
    mbar_init(bar_o, 1);
    mbar_init(bar_s, 1);
    *dead = 0;
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32((const void*)tmem_slot), COLS);
    tmem_relinquish();
  }
  if (V < 128 && tid < LC_THREADS)                        // columns that are not loaded
    for (uint32_t i = tid; i < 1024; i += LC_THREADS) reinterpret_cast<uint4*>(sm + T_V)[i] = make_uint4(0, 0, 0, 0);
  if (tid < 128) { pend[tid] = 0.0f; tot[tid] = 0.0f; }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 16) {
    // ------------------------------ issuer ------------------------------
    const uint32_t mine = lane == 0;
    const int ksteps = (D + 15) / 16;
    const uint64_t dq = make_smem_desc_sw128(sb + T_Q, 16, 1024), dk = make_smem_desc_sw128(sb + T_K, 16, 1024);
    const uint64_t da = make_smem_desc_sw128(sb + T_A, 16, 1024), ds = make_smem_desc_sw128(sb + T_S, 16384, 1024);
    const uint64_t dv = make_smem_desc_sw128(sb + T_V, 8192, 1024), dkt = make_smem_desc_sw128(sb + T_K, 8192, 1024);
    const uint32_t id_a = make_idesc_bf16(128, LC, 0, 0);   // rows 64 .. 127 of A and O are not used
    const uint32_t id_o = make_idesc_bf16(128, 128, 0, 1), id_s = make_idesc_bf16(128, 128, 1, 1);
    const uint32_t tm = __shfl_sync(0xffffffffu, tmem, 0);
    for (int n = 0; n < n_chunks; ++n) {
      if (OUT) {
        if (!__all_sync(0xffffffffu, mbar_wait(b_qk, n & 1, dead, c.status, 810))) break;
        tc_fence_after();
        if (*far_flag) {
          if (mine) mbar_arrive(bar_a);
          __syncwarp();
        } else {
#pragma unroll
          for (int p3 = 0; p3 < 3; ++p3) {
            const uint64_t q = dq + (p3 == 2 ? T_SPLIT >> 4 : 0), k = dk + (p3 == 1 ? T_SPLIT >> 4 : 0);
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              if (kk < ksteps) umma_f16_lane(mine, tm + TM_A, k_major(q, kk), k_major(k, kk), id_a, (p3 | kk) != 0);
          }
          umma_commit_lane(mine, bar_a);
        }
      }
      if (!__all_sync(0xffffffffu, mbar_wait(b_sa, n & 1, dead, c.status, 811))) break;
      tc_fence_after();
      if (OUT) {
#pragma unroll
        for (int p3 = 0; p3 < 3; ++p3) {
          const uint64_t q = dq + (p3 == 2 ? T_SPLIT >> 4 : 0), s = ds + (p3 == 1 ? 32768 >> 4 : 0);
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            if (kk < ksteps) umma_f16_lane(mine, tm + TM_O, k_major(q, kk), mn_major(s, kk), id_o, (p3 | kk) != 0);
        }
#pragma unroll
        for (int kk = 0; kk < 2 * LC / 16; ++kk)
          umma_f16_lane(mine, tm + TM_O, da + (uint64_t)(((kk >> 2) * 8192 + (kk & 3) * 32) >> 4), mn_major(dv, kk & 3), id_o, 1);
        umma_commit_lane(mine, bar_o);
      }
#pragma unroll
      for (int kk = 0; kk < 2 * LC / 16; ++kk)
        umma_f16_lane(mine, tm + TM_S, mn_major(dkt + (kk >= 4 ? T_SPLIT >> 4 : 0), kk & 3), mn_major(dv, kk & 3), id_s, 1);
      umma_commit_lane(mine, bar_s);
    }
  } else {
    // ------------------------------ workers ------------------------------
    const int quad = warp & 3, cg = warp >> 2, srow = quad * 32 + lane;
    const uint32_t lanes = (uint32_t)(quad * 32) << 16;
    const int p0 = a.pos[row0];
    const long long slot = CGK_IDX(a.slot[row0], a.slots);
    {
      // first state -> TMEM: lane = state row, this warp's 32 columns
      const float* src = nullptr;
      if (OUT && c.start) src = c.start + ((long long)blockIdx.y * a.heads + h) * D * V;
      else if (OUT && p0 > 0) src = a.state + ((slot * a.history + p0 % a.history) * a.heads + h) * (long long)D * V;
      uint32_t r[32];
#pragma unroll
      for (int j = 0; j < 32; j += 4) {
        float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        if (src && srow < D && cg * 32 + j < V) ldv<4>(src + (long long)srow * V + cg * 32 + j, v);
#pragma unroll
        for (int e = 0; e < 4; ++e) r[j + e] = __float_as_uint(v[e]);
      }
      tmem_st32(tmem + TM_S + lanes + cg * 32, r);
      tmem_st_wait();
    }
    const __nv_bfloat16* qp = reinterpret_cast<const __nv_bfloat16*>(a.q) + (long long)row0 * a.ldq + h * D;
    const __nv_bfloat16* kp = reinterpret_cast<const __nv_bfloat16*>(a.k) + (MODE == GATE_ROOT ? (long long)row0 * a.ldk + h * D : 0);
    const __nv_bfloat16* vp = reinterpret_cast<const __nv_bfloat16*>(a.v) + (long long)row0 * a.ldv + h * V;
    const __nv_bfloat16* gp = reinterpret_cast<const __nv_bfloat16*>(a.gate) + (a.gate ? (long long)row0 * a.ldg + h * V : 0);
    const float* zp = a.z + (long long)row0 * a.ldz + h * D;
    const int ch = (tid & 63) * 2, tg = tid >> 6;         // two state rows, eight tokens
    const bool mine = ch < D;
    const float bias0 = mine ? a.bias[h * D + ch] : 0.0f, bias1 = mine ? a.bias[h * D + ch + 1] : 0.0f;
    const float low0 = MODE == GATE_BOUNDED && mine ? a.low[h * D + ch] : 0.0f, low1 = MODE == GATE_BOUNDED && mine ? a.low[h * D + ch + 1] : 0.0f;

    // A chunk's rows: gates and one of keys and queries go to slots of this thread in shared memory, the others are
    // asked for in L2 (128 bytes per prefetch).
    constexpr bool STAGE_Q = OUT && MODE == GATE_BOUNDED;
    const uint32_t st_z = smem_u32(bars) + 64 + tid * 8, st_w = smem_u32(bars) + 64 + 32768 + tid * 4;
    const float2* sz = reinterpret_cast<const float2*>(bars + 16) + tid;
    const uint32_t* sw = bars + 16 + 8192 + tid;
    auto fetch = [&](int n) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int t = n * LC + tg * 8 + i;
        if (mine && t < count) {
          cp_async<8>(st_z + i * (LC_THREADS * 8), zp + (long long)t * a.ldz + ch);
          if (STAGE_Q) cp_async<4>(st_w + i * (LC_THREADS * 4), qp + (long long)t * a.ldq + ch);
          else if (MODE == GATE_ROOT) cp_async<4>(st_w + i * (LC_THREADS * 4), kp + (long long)t * a.ldk + ch);
        }
      }
      const int t = n * LC + (tid >> 3), i = tid & 7;
      if (t < count) {
        if (i < 2) {
          if (i * 64 < V) asm volatile("prefetch.global.L2 [%0];" ::"l"(vp + (long long)t * a.ldv + i * 64));
        } else if (OUT && i < 4) {
          if (a.gate && (i - 2) * 64 < V) asm volatile("prefetch.global.L2 [%0];" ::"l"(gp + (long long)t * a.ldg + (i - 2) * 64));
        } else if (OUT && !STAGE_Q && i < 6) {
          if ((i - 4) * 64 < D) asm volatile("prefetch.global.L2 [%0];" ::"l"(qp + (long long)t * a.ldq + (i - 4) * 64));
        }
      }
    };
    float b[8][2], kv[8][2], qv[8][2];
    auto gates = [&](int n) {                             // decays and their sums over eight tokens, keys, queries
      uint32_t raw_q[8];
      if (OUT && !STAGE_Q) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int t = n * LC + tg * 8 + i;
          raw_q[i] = mine && t < count ? *reinterpret_cast<const uint32_t*>(qp + (long long)t * a.ldq + ch) : 0u;
        }
      }
      cp_async_wait_all();
      float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const bool in = mine && n * LC + tg * 8 + i < count;      // otherwise the slot holds an earlier chunk's row
        const float2 z = in ? sz[i * LC_THREADS] : make_float2(0.0f, 0.0f);
        const uint32_t w = in && (STAGE_Q || MODE == GATE_ROOT) ? sw[i * LC_THREADS] : 0u;
        float k0 = 0.0f, k1 = 0.0f;
        const float g0 = lin_decay_log2<MODE>(z.x + bias0, low0, a.inv_tau, &k0);
        const float g1 = lin_decay_log2<MODE>(z.y + bias1, low1, a.inv_tau, &k1);
        if (MODE == GATE_ROOT) {
          const float2 k = unpack_bf16x2(w);
          k0 = k.x;
          k1 = k.y;
        }
        kv[i][0] = in ? k0 : 0.0f;
        kv[i][1] = in ? k1 : 0.0f;
        if (OUT) {
          const float2 q = unpack_bf16x2(STAGE_Q ? w : raw_q[i]);
          qv[i][0] = (a.q_silu ? lin_silu_fast(q.x) : q.x) * a.q_scale;
          qv[i][1] = (a.q_silu ? lin_silu_fast(q.y) : q.y) * a.q_scale;
        }
        sum0 += in ? g0 : 0.0f;
        sum1 += in ? g1 : 0.0f;
        b[i][0] = sum0;
        b[i][1] = sum1;
      }
      *reinterpret_cast<float2*>(part + tg * 128 + ch) = make_float2(sum0, sum1);
    };
    fetch(0);
    gates(0);
    bool ok = true;                                       // after a wait that ran out a warp still comes to every meeting point

    for (int n = 0; n < n_chunks; ++n) {
      const int t0 = n * LC, left = min(LC, count - t0);
      // values: two 16-byte pieces per thread
      uint4 vv[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int j = tid + i * LC_THREADS, t = j >> 4, col = (j & 15) * 8;
        vv[i] = make_uint4(0, 0, 0, 0);
        if (t < left && col < V) vv[i] = *reinterpret_cast<const uint4*>(vp + (long long)(t0 + t) * a.ldv + col);
      }
      if (n + 1 < n_chunks) fetch(n + 1);
      // the previous chunk's products are done with the tiles and the state
      if (n > 0) ok &= mbar_wait(bar_s, (n - 1) & 1, dead, c.status, 802);
      tc_fence_after();
      lc_meet();
      float before[2] = {0.0f, 0.0f}, mid[2] = {0.0f, 0.0f}, end[2] = {0.0f, 0.0f};
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        const float2 s = *reinterpret_cast<const float2*>(part + g * 128 + ch);
        if (g == tg) { before[0] = end[0]; before[1] = end[1]; }
        end[0] += s.x;
        end[1] += s.y;
        if (g == 3) { mid[0] = end[0]; mid[1] = end[1]; }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) { b[i][0] += before[0]; b[i][1] += before[1]; }
      bool far = false;
      if (OUT) far = lc_any(fmaxf(-mid[0], -mid[1]) > LC_LIMIT || fmaxf(mid[0] - end[0], mid[1] - end[1]) > LC_LIMIT);
      if (far) {
        // A term by term, into its tile at once: row tid / 8, columns 8 (tid % 8) ..
        float* fb = reinterpret_cast<float*>(sm + T_S);
        float* fq = fb + LC * 128;
        float* fk = reinterpret_cast<float*>(sm + T_K);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int at = (tg * 8 + i) * 128 + ch;
          *reinterpret_cast<float2*>(fb + at) = make_float2(b[i][0], b[i][1]);
          *reinterpret_cast<float2*>(fq + at) = make_float2(qv[i][0], qv[i][1]);
          *reinterpret_cast<float2*>(fk + at) = make_float2(kv[i][0], kv[i][1]);
        }
        lc_meet();
        const int t = tid >> 3, s0 = (tid & 7) * 8;
#pragma unroll 1
        for (int j = 0; j < 4; ++j) {
          float x[2] = {0.0f, 0.0f};
#pragma unroll
          for (int e2 = 0; e2 < 2; ++e2) {
            const int s = s0 + 2 * j + e2;
            if (s <= t)
              for (int e = 0; e < D; ++e) x[e2] = fmaf(fq[t * 128 + e] * fk[s * 128 + e], exp2f(fb[t * 128 + e] - fb[s * 128 + e]), x[e2]);
          }
          uint32_t hh, ll;
          split2(x[0], x[1], hh, ll);
          *reinterpret_cast<uint32_t*>(sm + T_A + pair_at(t, s0 + 2 * j, LC)) = hh;
          *reinterpret_cast<uint32_t*>(sm + T_A + 8192 + pair_at(t, s0 + 2 * j, LC)) = ll;
        }
        lc_meet();
      }
      const float ref_q[2] = {far ? 0.0f : mid[0], far ? 0.0f : mid[1]};
      const float ref_k[2] = {far || !OUT ? end[0] : mid[0], far || !OUT ? end[1] : mid[1]};
      if (tg == 0) {
        rq[ch] = ref_q[0]; rq[ch + 1] = ref_q[1];
        rk[ch] = ref_k[0]; rk[ch + 1] = ref_k[1];
        float* next = pend + ((n + 1) & 1) * 128 + ch;
        next[0] = end[0] - ref_k[0];
        next[1] = end[1] - ref_k[1];
        tot[ch] += end[0];
        tot[ch + 1] += end[1];
        if (tid == 0) *far_flag = far;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const uint32_t at = pair_at(tg * 8 + i, ch, LC);
        uint32_t hi, lo;
        split2(kv[i][0] * fast_exp2(ref_k[0] - b[i][0]), kv[i][1] * fast_exp2(ref_k[1] - b[i][1]), hi, lo);
        *reinterpret_cast<uint32_t*>(sm + T_K + at) = hi;
        *reinterpret_cast<uint32_t*>(sm + T_K + T_SPLIT + at) = lo;
        if (OUT) {
          split2(qv[i][0] * fast_exp2(b[i][0] - ref_q[0]), qv[i][1] * fast_exp2(b[i][1] - ref_q[1]), hi, lo);
          *reinterpret_cast<uint32_t*>(sm + T_Q + at) = hi;
          *reinterpret_cast<uint32_t*>(sm + T_Q + T_SPLIT + at) = lo;
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int j = tid + i * LC_THREADS, t = j >> 4, col = (j & 15) * 8;
        if (col < V) *reinterpret_cast<uint4*>(sm + T_V + pair_at(t, col, LC)) = vv[i];
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive_warp(b_qk);
      lc_meet();                                          // references and factors
      // ---- state: operand of the product with Q, and the sum that K^T V is added to
      {
        uint32_t r[32];
        __syncwarp();
        tmem_ld32(tmem + TM_S + lanes + cg * 32, r);
        tmem_ld_wait();
        const float f = exp2f(pend[(n & 1) * 128 + srow]), fq = exp2f(rq[srow]), fk = exp2f(rk[srow]);
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
          float s[8];
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            s[e] = __uint_as_float(r[j + e]) * f;
            r[j + e] = __float_as_uint(s[e] * fk);
            s[e] *= fq;
          }
          if (OUT) {
#pragma unroll
            for (int e = 0; e < 4; ++e) split2(s[2 * e], s[2 * e + 1], hi[e], lo[e]);
            const uint32_t at = T_S + pair_at(srow, cg * 32 + j, 128);
            *reinterpret_cast<uint4*>(sm + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(sm + at + 32768) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
        __syncwarp();
        tmem_st32(tmem + TM_S + lanes + cg * 32, r);
        tmem_st_wait();
      }
      if (OUT && quad < 2 && !far) {
        // ---- A, lower triangle, as two bf16 parts
        ok &= mbar_wait(bar_a, n & 1, dead, c.status, 800);
        tc_fence_after();
        const int t = srow;
        uint32_t r[16];
        __syncwarp();
        tmem_ld16(tmem + TM_A + lanes + cg * 16, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; j += 8) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int s = cg * 16 + j + 2 * e;
            split2(s <= t ? __uint_as_float(r[j + 2 * e]) : 0.0f, s + 1 <= t ? __uint_as_float(r[j + 2 * e + 1]) : 0.0f, hi[e], lo[e]);
          }
          const uint32_t at = T_A + sw128_offset(t, (cg * 16 + j) >> 3);
          *reinterpret_cast<uint4*>(sm + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(sm + at + 8192) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive_warp(b_sa);
      if (n + 1 < n_chunks) gates(n + 1);                 // while the tensor core works
      if (OUT && quad < 2) {
        // ---- result: lane = token, this warp's 32 columns; norm over the head, gate
        ok &= mbar_wait(bar_o, n & 1, dead, c.status, 801);
        tc_fence_after();
        const int t = srow;
        uint32_t r[32];
        __syncwarp();
        tmem_ld32(tmem + TM_O + lanes + cg * 32, r);
        tmem_ld_wait();
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < 32; ++j) ss = fmaf(__uint_as_float(r[j]), __uint_as_float(r[j]), ss);
        red[cg * LC + t] = ss;
        asm volatile("bar.sync 2, 256;" ::: "memory");
        if (t < left) {
          const float rs = 1.0f / sqrtf((red[t] + red[LC + t] + red[2 * LC + t] + red[3 * LC + t]) / V + a.eps);
          const long long row = t0 + t;
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.out) + (row0 + row) * a.ldo + (long long)h * V + cg * 32;
          const __nv_bfloat16* g = gp + row * a.ldg + cg * 32;
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (cg * 32 + j >= V) continue;
            float x[8];
#pragma unroll
            for (int e = 0; e < 8; e += 4) {
              const float4 w = *reinterpret_cast<const float4*>(a.w + cg * 32 + j + e);
              x[e] = __uint_as_float(r[j + e]) * rs * w.x;
              x[e + 1] = __uint_as_float(r[j + e + 1]) * rs * w.y;
              x[e + 2] = __uint_as_float(r[j + e + 2]) * rs * w.z;
              x[e + 3] = __uint_as_float(r[j + e + 3]) * rs * w.w;
            }
            if (a.gate) {
              const uint4 u = *reinterpret_cast<const uint4*>(g + j);
              const uint32_t gu[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 f = unpack_bf16x2(gu[e]);
                x[2 * e] *= lin_silu_fast(f.x);
                x[2 * e + 1] *= lin_silu_fast(f.y);
              }
            }
            *reinterpret_cast<uint4*>(o + j) = make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
          }
        }
        tc_fence_before();
      }
    }
    // ---- last state: to the cache, or as the stretch's sum
    if (n_chunks > 0) ok &= mbar_wait(bar_s, (n_chunks - 1) & 1, dead, c.status, 803);
    tc_fence_after();
    if (ok && (!OUT || last)) {
      uint32_t r[32];
      __syncwarp();
      tmem_ld32(tmem + TM_S + lanes + cg * 32, r);
      tmem_ld_wait();
      const float f = exp2f(pend[(n_chunks & 1) * 128 + srow]);
      float* dst = OUT ? a.state + ((slot * a.history + (p0 + count) % a.history) * a.heads + h) * (long long)D * V
                       : c.start + ((long long)blockIdx.y * a.heads + h) * D * V;
      if (srow < D) {
#pragma unroll
        for (int j = 0; j < 32; j += 4)
          if (cg * 32 + j < V) {
            const float v[4] = {__uint_as_float(r[j]) * f, __uint_as_float(r[j + 1]) * f, __uint_as_float(r[j + 2]) * f, __uint_as_float(r[j + 3]) * f};
            stv<4>(dst + (long long)srow * V + cg * 32 + j, v);
          }
      }
      if (!OUT && tid < D) c.total[((long long)blockIdx.y * a.heads + h) * D + tid] = tot[tid];
    }
  }
  if (*dead) __nanosleep(100000);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, COLS);
  }
}

// Sums of a run's stretches -> their first states.  grid (state elements / 1024, heads, runs); four columns per thread.
__global__ void __launch_bounds__(256)
linear_starts_kernel(const ChunksDev c, const int* __restrict__ run_items) {
  const LinStateDev& a = c.a;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4, h = blockIdx.y, n0 = run_items[2 * blockIdx.z], n = run_items[2 * blockIdx.z + 1];
  const int size = a.D * a.V, row = c.items[4 * n0], p0 = a.pos[row], d = e / a.V;
  if (e >= size) return;
  float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
  if (p0 > 0) ldv<4>(a.state + ((CGK_IDX(a.slot[row], a.slots) * a.history + p0 % a.history) * a.heads + h) * (long long)size + e, s);
  const long long step = (long long)a.heads * size;
  float* at = c.start + ((long long)n0 * a.heads + h) * size + e;
  const float* tot = c.total + ((long long)n0 * a.heads + h) * a.D + d;
  float next[4] = {0.0f, 0.0f, 0.0f, 0.0f};
  if (n > 1) ldv<4>(at, next);
  for (int j = 0; j < n; ++j) {
    const float add[4] = {next[0], next[1], next[2], next[3]};
    if (j + 2 < n) ldv<4>(at + (j + 1) * step, next);
    stv<4>(at + j * step, s);
    if (j + 1 < n) {
      const float f = exp2f(tot[(long long)j * a.heads * a.D]);
#pragma unroll
      for (int i = 0; i < 4; ++i) s[i] = fmaf(f, s[i], add[i]);
    }
  }
}

}  // namespace
}  // namespace cgk

using namespace cgk;

CGK_API int cgk_linear_chunks_ok(int D, int V) { return D % 8 == 0 && V % 8 == 0 && D > 0 && V > 0 && D <= 128 && V <= 128; }

CGK_API long long cgk_linear_chunks_scratch_floats(int n_items, int heads, int D, int V) { return (long long)n_items * heads * D * (V + 1); }

CGK_API int cgk_linear_chunks(const cgk_linear_state_args* pa, const int* items, int n_items, const int* run_items, int n_runs, void* scratch,
                              void* stream) {
  CGK_REQUIRE(pa && items && n_items >= 0 && (!scratch || (run_items && n_runs > 0)), "cgk_linear_chunks: bad arguments");
  const cgk_linear_state_args& a = *pa;
  CGK_REQUIRE(a.q && a.v && a.z && a.bias && a.w && a.state && a.out && a.slot && a.pos && a.heads > 0 && a.history > 0 && a.slots > 0 && !a.fp32,
              "cgk_linear_chunks: bad arguments");
  CGK_REQUIRE(a.mode == GATE_BOUNDED ? (a.low && !a.k) : (a.mode == GATE_ROOT && a.k), "cgk_linear_chunks: the gate's operands do not fit its kind");
  auto al = [](const void* p, long long ld) { return (((uintptr_t)p) & 15) == 0 && ld % 8 == 0; };
  CGK_REQUIRE(cgk_linear_chunks_ok(a.D, a.V) && al(a.q, a.ldq) && al(a.k, a.k ? a.ldk : 0) && al(a.v, a.ldv) && al(a.gate, a.gate ? a.ldg : 0) &&
              al(a.z, a.ldz) && al(a.out, a.ldo) && al(a.state, 0) && al(a.w, 0) && al(scratch, 0), "cgk_linear_chunks: sizes or alignment not supported");
  CGK_REQUIRE(n_items <= 65535 && n_runs <= 65535, "cgk_linear_chunks: too many stretches in one call");
  if (n_items == 0) return 0;
  int dev = 0;
  CGK_CUDA_CHECK(cudaGetDevice(&dev));
  ChunksDev d;
  d.a = LinStateDev{a.q, a.k, a.v, a.gate, a.z, a.ldq, a.ldk, a.ldv, a.ldg, a.ldz, a.bias, a.low, a.w, a.state, a.out, a.ldo, a.slot, a.pos, nullptr,
                    a.heads, a.D, a.V, a.history, a.slots, a.mode, a.q_silu, a.q_scale, a.inv_tau, a.eps};
  d.items = items;
  d.start = (float*)scratch;
  d.total = scratch ? (float*)scratch + (long long)n_items * a.heads * a.D * a.V : nullptr;
  d.status = device_status(dev);
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 grid(a.heads, n_items);
  auto sums = a.mode == GATE_BOUNDED ? linear_chunks_kernel<false, GATE_BOUNDED> : linear_chunks_kernel<false, GATE_ROOT>;
  auto results = a.mode == GATE_BOUNDED ? linear_chunks_kernel<true, GATE_BOUNDED> : linear_chunks_kernel<true, GATE_ROOT>;
  if (scratch) {
    const int smem = T_END_SUM + LC_MISC + 1024;
    CGK_CUDA_CHECK(cudaFuncSetAttribute(sums, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    sums<<<grid, LC_THREADS + 32, smem, st>>>(d);
    CGK_LAUNCH_CHECK();
    linear_starts_kernel<<<dim3((a.D * a.V / 4 + 255) / 256, a.heads, n_runs), 256, 0, st>>>(d, run_items);
    CGK_LAUNCH_CHECK();
  }
  const int smem = T_END + LC_MISC + 1024;
  CGK_CUDA_CHECK(cudaFuncSetAttribute(results, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  results<<<grid, LC_THREADS + 32, smem, st>>>(d);
  CGK_LAUNCH_CHECK();
  return 0;
}

CGK_BOUNDS_READER(linear_state_tc)
