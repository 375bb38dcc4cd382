// Linear recurrences (linear_state.cuh) over prompt portions, 64 tokens at a time on the tcgen05 tensor cores.
//
// With b_t the logarithm of the decay since the start of a chunk (per state row), r its value in the chunk's middle,
//     Q = q 2^(b - r),  K = k 2^(r - b),  A = tril(Q K^T),  O = A V + Q (2^r S),  S' = 2^(b_end - r) (2^r S + K^T V)
// so a chunk takes four products.  The state stays in TMEM in fp32 from chunk to chunk (transposed: lanes are the elements
// of v; times a factor per state row that is kept beside it).  Every fp32 operand enters the tensor core as the sum of
// two bf16 numbers, so the sums see 16 bits of each factor; the two parts of Q, K and A are stacked in one tile, which
// makes the partial products one wider instruction:
//     [Qh; Ql] [Kh; Kl]^T  -> A in four quarters        Sh [Qh; Ql]^T, Sl Qh^T, V^T [Ah; Al]^T  -> O^T in two halves
// Where a state row's decay is so strong that its exponents could leave fp32's range, the row's part of A is formed term by
// term with b_t - b_s <= 0, and its columns of Q and K take the chunk's ends as their references (what the product
// makes of them is below 2^-100 of the truth).
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

constexpr int LC = 64, LC_THREADS = 512;                  // tokens of a chunk; worker threads
constexpr float LC_LIMIT = 100.0f;                        // largest exponent (base 2) of a factor
// shared memory (bytes): operand tiles of 128-byte rows in blocks of 64 columns, then rows as they come from memory
constexpr uint32_t T_Q = 0, T_K = 32768, T_V = 65536, T_A = 81920, T_A2 = 98304, R_Z = 106496, R_W = R_Z + 32768, R_X = R_W + 16384, LC_MISC = R_X + 16384;
constexpr int FAR_N = 24;                                 // strongly decaying state rows handled at a time
constexpr uint32_t LC_SMEM = LC_MISC + (8 * 128 + 3 * 128 + 4 * LC + LC * LC + FAR_N * 3 * LC) * 4 + 128 + 1024;
constexpr uint32_t T_SPLIT = 8192;                        // high part -> low part of Q, K and A: 64 rows further
// TMEM columns: state, its two parts, O in two halves, A in four quarters
constexpr uint32_t TM_S = 0, TM_SH = 128, TM_SL = 192, TM_O = 256, TM_A = 384;

struct ChunksDev {
  LinStateDev a;
  const int* items;          // [n_items][4]: first row, tokens, run, last stretch of the run
  float* start;              // [n_items][heads][D][V]: sums, then first states; null: every run is one stretch
  float* total;              // [n_items][heads][D]: logarithm (base 2) of a stretch's whole decay
  int* status;
};

__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x0, x1);
  const Pair rest = pfma(Pair{__uint_as_float(hi << 16), __uint_as_float(hi & 0xffff0000u)}, pall(-1.0f), Pair{x0, x1});
  lo = pack_bf16x2(rest.x, rest.y);
}
// byte offset of a 4-byte pair of columns in a tile with `rows` rows per block
__device__ __forceinline__ uint32_t pair_at(int row, int col, int rows) {
  return (col >> 6) * (rows * 128) + sw128_offset(row, (col & 63) >> 3) + (col & 7) * 2;
}

// operand descriptors of consecutive 16-wide steps differ by constants in the address field
__device__ __forceinline__ uint64_t k_major(uint64_t d, int kk) { return d + (uint64_t)(((kk >> 2) * 16384 + (kk & 3) * 32) >> 4); }
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

// 16 values per lane -> their sums over the warp: lane l gets the sum of value (l >> 1).
__device__ __forceinline__ float sum_over_lanes(float (&v)[16], int lane) {
#pragma unroll
  for (int half = 8; half >= 1; half >>= 1) {
    const bool upper = (lane & (2 * half)) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? v[i] : v[i + half];
      v[i] = (upper ? v[i + half] : v[i]) + __shfl_xor_sync(0xffffffffu, send, 2 * half);
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

// Warps 0 .. 15 prepare operands and read results, warp 16 issues the products, warp 17 brings gates, queries and keys.
template <bool OUT, int MODE>
__global__ void __launch_bounds__(LC_THREADS + 128, 1)
linear_chunks_kernel(const __grid_constant__ CUtensorMap tm_z, const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                     const __grid_constant__ CUtensorMap tm_v, const ChunksDev c) {
  const LinStateDev& a = c.a;
  extern __shared__ uint8_t lc_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lc_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sb = smem_u32(sm);
  float* part = reinterpret_cast<float*>(sm + LC_MISC);   // [8][128] decay of eight tokens
  float* f0 = part + 8 * 128;                             // [128] factors of the state: pending, of K's and Q's references
  float* fk = f0 + 128;
  float* fq = fk + 128;
  float* red = fq + 128;                                  // [4][64]
  float* far_a = red + 4 * LC;                            // [64][64] what strongly decaying rows give to A
  float* far_rows = far_a + LC * LC;                      // [FAR_N][q, k, b][64]
  uint32_t* bars = reinterpret_cast<uint32_t*>(far_rows + FAR_N * 3 * LC);
  const uint32_t b_qk = smem_u32(bars), b_sa = b_qk + 8, bar_a = b_qk + 16, bar_o = b_qk + 24, bar_s = b_qk + 32, b_raw = b_qk + 40, b_free = b_qk + 48, b_v = b_qk + 56;
  volatile uint32_t* tmem_slot = bars + 16;
  volatile int* dead = reinterpret_cast<volatile int*>(bars + 17);
  uint32_t* far_mask = bars + 18;                         // [4]

  const int* item = c.items + 4 * blockIdx.y;
  const int row0 = item[0], count = item[1], last = item[3], h = blockIdx.x;
  if (!OUT && last) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = a.D, V = a.V, n_chunks = (count + LC - 1) / LC;

  if (tid == 0) {
    mbar_init(b_qk, 16);
    mbar_init(b_sa, 16);
    mbar_init(bar_a, 1);
    mbar_init(bar_o, 1);
    mbar_init(bar_s, 1);
    mbar_init(b_raw, 1);
    mbar_init(b_free, 16);
    mbar_init(b_v, 1);
    *dead = 0;
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(smem_u32((const void*)tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  // 640 threads are launched with 96 registers each; the last warpgroup leaves some of its share to the workers
  if (warp >= 16) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 32;");
   if (warp == 17) {
    // ------------------------------ loader ------------------------------
    // 64 rows at a time; what lies behind the end of the run is another run's (or zero) and is not used
    if (lane == 0) {
      const int v_blocks = (V + 63) / 64;
      for (int n = 0; n < n_chunks; ++n) {
        const int row = row0 + (OUT ? n : n_chunks - 1 - n) * LC;
        if (n > 0 && !mbar_wait(b_free, (n - 1) & 1, dead, c.status, 820)) break;
        mbar_expect_tx(b_raw, LC * D * (4 + (OUT ? 2 : 0) + (MODE == GATE_ROOT ? 2 : 0)));
        tma_load_2d(sb + R_Z, &tm_z, b_raw, h * D, row);
        if (OUT) tma_load_2d(sb + R_W, &tm_q, b_raw, h * D, row);
        if (MODE == GATE_ROOT) tma_load_2d(sb + R_X, &tm_k, b_raw, h * D, row);
        if (n > 0 && !mbar_wait(bar_s, (n - 1) & 1, dead, c.status, 822)) break;
        mbar_expect_tx(b_v, v_blocks * 8192);
        for (int i = 0; i < v_blocks; ++i) tma_load_2d(sb + T_V + i * 8192, &tm_v, b_v, h * V + i * 64, row);
      }
    }
  } else if (warp == 16) {
    // ------------------------------ issuer ------------------------------
    const uint32_t mine = lane == 0;
    const int ksteps = (D + 15) / 16;
    const uint64_t dq = make_smem_desc_sw128(sb + T_Q, 16, 1024), dk = make_smem_desc_sw128(sb + T_K, 16, 1024);
    const uint64_t da = make_smem_desc_sw128(sb + T_A, 16, 1024), da2 = make_smem_desc_sw128(sb + T_A2, 16, 1024);
    const uint64_t dv = make_smem_desc_sw128(sb + T_V, 8192, 1024), dkt = make_smem_desc_sw128(sb + T_K, 16384, 1024);
    const uint32_t id_kk = make_idesc_bf16(128, 128, 0, 0), id_kk64 = make_idesc_bf16(128, 64, 0, 0);
    const uint32_t id_mk = make_idesc_bf16(128, 128, 1, 0), id_mk64 = make_idesc_bf16(128, 64, 1, 0), id_mm = make_idesc_bf16(128, 128, 1, 1);
    const uint32_t tm = __shfl_sync(0xffffffffu, tmem, 0);
    for (int n = 0; n < n_chunks; ++n) {
      if (OUT) {
        if (!__all_sync(0xffffffffu, mbar_wait(b_qk, n & 1, dead, c.status, 810))) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          if (kk < ksteps) umma_f16_lane(mine, tm + TM_A, k_major(dq, kk), k_major(dk, kk), id_kk, kk != 0);
        umma_commit_lane(mine, bar_a);
      }
      if (!__all_sync(0xffffffffu, mbar_wait(b_v, n & 1, dead, c.status, 812) && mbar_wait(b_sa, n & 1, dead, c.status, 811))) break;
      tc_fence_after();
      if (OUT) {
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          if (kk < ksteps) umma_f16_ts_lane(mine, tm + TM_O, tm + TM_SH + kk * 8, k_major(dq, kk), id_kk, kk != 0);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          if (kk < ksteps) umma_f16_ts_lane(mine, tm + TM_O, tm + TM_SL + kk * 8, k_major(dq, kk), id_kk64, 1);
#pragma unroll
        for (int kk = 0; kk < LC / 16; ++kk) umma_f16_lane(mine, tm + TM_O, mn_major(dv, kk), da + kk * 2, id_mk, 1);
#pragma unroll
        for (int kk = 0; kk < LC / 16; ++kk) umma_f16_lane(mine, tm + TM_O, mn_major(dv, kk), da2 + kk * 2, id_mk64, 1);
        umma_commit_lane(mine, bar_o);
      }
#pragma unroll
      for (int kk = 0; kk < 2 * LC / 16; ++kk)
        umma_f16_lane(mine, tm + TM_S, mn_major(dv, kk & 3), mn_major(dkt + (kk >= 4 ? T_SPLIT >> 4 : 0), kk & 3), id_mm, OUT || n > 0 || kk > 0);
      umma_commit_lane(mine, bar_s);
    }
   }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 112;");
    // ------------------------------ workers ------------------------------
    const int quad = warp & 3, cg = warp >> 2, lrow = quad * 32 + lane;       // TMEM lane: an element of v, or a row of A
    const uint32_t lanes = (uint32_t)(quad * 32) << 16;
    const int p0 = a.pos[row0];
    const long long slot = CGK_IDX(a.slot[row0], a.slots);
    if (OUT) {
      // first state -> TMEM: this warp's 32 state rows
      const float* src = nullptr;
      if (c.start) src = c.start + ((long long)blockIdx.y * a.heads + h) * D * V;
      else if (p0 > 0) src = a.state + ((slot * a.history + p0 % a.history) * a.heads + h) * (long long)D * V;
      uint32_t r[32];
#pragma unroll
      for (int j = 0; j < 32; ++j)
        r[j] = src && lrow < V && cg * 32 + j < D ? __float_as_uint(src[(long long)(cg * 32 + j) * V + lrow]) : 0u;
      tmem_st32(tmem + TM_S + lanes + cg * 32, r);
      tmem_st_wait();
    }
    // results leave with two 16-byte pieces per thread: rows cg * 16 + (0, 8) + .., columns o_col ..
    const int o_row = cg * 16 + (quad * 32 + lane) / 16, o_col = (lane & 15) * 8;
    const bool o_mine = o_col < V;
    const float inv_v = 1.0f / V;
    const __nv_bfloat16* gp = reinterpret_cast<const __nv_bfloat16*>(a.gate) + (a.gate ? (long long)row0 * a.ldg + h * V + o_col : 0);
    __nv_bfloat16* op = reinterpret_cast<__nv_bfloat16*>(a.out) + (long long)row0 * a.ldo + h * V + o_col;
    const int ch = (tid & 63) * 2, tg = tid >> 6;         // two state rows, eight tokens
    const bool mine = ch < D;
    const Pair bias = mine ? Pair{a.bias[h * D + ch], a.bias[h * D + ch + 1]} : pall(0.0f);
    const Pair low = MODE == GATE_BOUNDED && mine ? Pair{a.low[h * D + ch], a.low[h * D + ch + 1]} : pall(0.0f);
    bool ok = true;                                       // after a wait that ran out a warp still comes to every meeting point

    Pair kv[8], qv[8], pend = pall(0.0f), tot = pall(0.0f);
    auto gates = [&](int n, int at) {                     // the n-th chunk of the loop is the at-th of the stretch: decays
      ok &= mbar_wait(b_raw, n & 1, dead, c.status, 821);  // and their sums over eight tokens, keys, queries
      Pair sum = pall(0.0f);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int t = tg * 8 + i;
        const bool in = mine && at * LC + t < count;      // what lies behind the run does not count
        Pair* place = reinterpret_cast<Pair*>(sm + R_Z + (t * D + (mine ? ch : 0)) * 4);
        Pair k = pall(0.0f);
        const Pair g = lin_decay_log2<MODE>(padd(*place, bias), low, a.inv_tau, &k);
        if (MODE == GATE_ROOT) {
          const float2 w = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm + R_X + (t * D + (mine ? ch : 0)) * 2));
          k = Pair{w.x, w.y};
        }
        kv[i] = Pair{in ? k.x : 0.0f, in ? k.y : 0.0f};
        if (OUT) {
          const float2 w = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sm + R_W + (t * D + (mine ? ch : 0)) * 2));
          const Pair q = {in ? w.x : 0.0f, in ? w.y : 0.0f};
          qv[i] = pmul(a.q_silu ? lin_silu_fast(q) : q, pall(a.q_scale));
        }
        sum = padd(sum, Pair{in ? g.x : 0.0f, in ? g.y : 0.0f});
        if (mine) *place = sum;                           // read back by this thread
      }
      *reinterpret_cast<Pair*>(part + tg * 128 + ch) = sum;
    };
    auto chunk_of = [&](int n) { return OUT ? n : n_chunks - 1 - n; };      // the sums are taken from the end
    if (n_chunks > 0) gates(0, chunk_of(0));

    for (int n = 0; n < n_chunks; ++n) {
      const int t0 = n * LC, left = min(LC, count - t0);
      // the previous chunk's products are done with the tiles and the state
      if (n > 0) ok &= mbar_wait(bar_s, (n - 1) & 1, dead, c.status, 802);
      tc_fence_after();
      lc_meet();
      Pair before = pall(0.0f), mid = pall(0.0f), end = pall(0.0f);
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        const Pair s = *reinterpret_cast<const Pair*>(part + g * 128 + ch);
        if (g == tg) before = end;
        end = padd(end, s);
        if (g == 3) mid = end;
      }
      auto sum_at = [&](int i) {                          // decay up to and with this thread's token i
        return mine ? padd(*reinterpret_cast<const Pair*>(sm + R_Z + ((tg * 8 + i) * D + ch) * 4), before) : pall(0.0f);
      };
      const bool far_x = OUT && (-mid.x > LC_LIMIT || mid.x - end.x > LC_LIMIT), far_y = OUT && (-mid.y > LC_LIMIT || mid.y - end.y > LC_LIMIT);
      const bool far = OUT && lc_any(far_x || far_y);
      if (far) {
        // number the rows, bring theirs together, and work out their part of A: row tid / 8, columns 8 (tid % 8) ..
        if (warp < 2) {
          const uint32_t mx = __ballot_sync(0xffffffffu, far_x), my = __ballot_sync(0xffffffffu, far_y);
          if (lane == 0) { far_mask[2 * warp] = mx; far_mask[2 * warp + 1] = my; }
        }
        lc_meet();
        const int w = (tid >> 5) & 1, below0 = w ? __popc(far_mask[0]) + __popc(far_mask[1]) : 0;
        const uint32_t below = (1u << lane) - 1u;
        const int ix = below0 + __popc(far_mask[2 * w] & below) + __popc(far_mask[2 * w + 1] & below), iy = ix + far_x;
        const int n_far = __popc(far_mask[0]) + __popc(far_mask[1]) + __popc(far_mask[2]) + __popc(far_mask[3]);
        const int t = tid >> 3, s0 = (tid & 7) * 8;
        float acc[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = 0.0f;
        for (int g0 = 0; g0 < n_far; g0 += FAR_N) {
          const bool put_x = far_x && ix >= g0 && ix < g0 + FAR_N, put_y = far_y && iy >= g0 && iy < g0 + FAR_N;
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const Pair b = sum_at(i);
            float* px = far_rows + (ix - g0) * 3 * LC + tg * 8 + i;
            float* py = far_rows + (iy - g0) * 3 * LC + tg * 8 + i;
            if (put_x) { px[0] = qv[i].x; px[LC] = kv[i].x; px[2 * LC] = b.x; }
            if (put_y) { py[0] = qv[i].y; py[LC] = kv[i].y; py[2 * LC] = b.y; }
          }
          lc_meet();
          if (s0 <= t)
            for (int r = 0; r < min(FAR_N, n_far - g0); ++r) {
              const float* row = far_rows + r * 3 * LC;
              const float q = row[t], b = row[2 * LC + t];
#pragma unroll
              for (int j = 0; j < 8; ++j)
                if (s0 + j <= t) acc[j] = fmaf(q * row[LC + s0 + j], fast_exp2(b - row[2 * LC + s0 + j]), acc[j]);
            }
          lc_meet();
        }
        *reinterpret_cast<float4*>(far_a + t * LC + s0) = make_float4(acc[0], acc[1], acc[2], acc[3]);
        *reinterpret_cast<float4*>(far_a + t * LC + s0 + 4) = make_float4(acc[4], acc[5], acc[6], acc[7]);
      }
      // K's factors refer to the chunk's middle or end; the summing pass comes from the end and adds what follows
      const Pair ref_q = {far_x ? 0.0f : mid.x, far_y ? 0.0f : mid.y};
      const Pair ref_k = OUT ? Pair{far_x ? end.x : mid.x, far_y ? end.y : mid.y} : padd(end, tot);
      if (OUT && tg == 0) {
        f0[ch] = exp2f(pend.x);
        f0[ch + 1] = exp2f(pend.y);
        fk[ch] = exp2f(ref_k.x);
        fk[ch + 1] = exp2f(ref_k.y);
        if (far) {                                        // otherwise Q has K's references
          fq[ch] = exp2f(ref_q.x);
          fq[ch + 1] = exp2f(ref_q.y);
        }
      }
      pend = padd(end, Pair{-ref_k.x, -ref_k.y});
      tot = padd(tot, end);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const uint32_t at = pair_at(tg * 8 + i, ch, 128);
        const Pair b = sum_at(i), bk = pfma(b, pall(-1.0f), ref_k);
        uint32_t hi, lo;
        const Pair k = pmul(kv[i], Pair{fast_exp2(bk.x), fast_exp2(bk.y)});
        split2(k.x, k.y, hi, lo);
        *reinterpret_cast<uint32_t*>(sm + T_K + at) = hi;
        *reinterpret_cast<uint32_t*>(sm + T_K + T_SPLIT + at) = lo;
        if (OUT) {
          const Pair bq = padd(b, Pair{-ref_q.x, -ref_q.y}), q = pmul(qv[i], Pair{fast_exp2(bq.x), fast_exp2(bq.y)});
          split2(q.x, q.y, hi, lo);
          *reinterpret_cast<uint32_t*>(sm + T_Q + at) = hi;
          *reinterpret_cast<uint32_t*>(sm + T_Q + T_SPLIT + at) = lo;
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      if (OUT) {
        mbar_arrive_warp(b_qk);
        mbar_arrive_warp(b_free);
        lc_meet();                                        // factors of the state
      } else {
        mbar_arrive_warp(b_free);
      }
      if (OUT) {
        // ---- state: operand of the product with Q, and the sum that K^T V is added to
        uint32_t r[32], hi[16], lo[16];
        __syncwarp();
        tmem_ld32(tmem + TM_S + lanes + cg * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; j += 4) {
          const float4 w0 = *reinterpret_cast<const float4*>(f0 + cg * 32 + j), wk = *reinterpret_cast<const float4*>(fk + cg * 32 + j);
          const Pair x0 = pmul(Pair{__uint_as_float(r[j]), __uint_as_float(r[j + 1])}, Pair{w0.x, w0.y});
          const Pair x1 = pmul(Pair{__uint_as_float(r[j + 2]), __uint_as_float(r[j + 3])}, Pair{w0.z, w0.w});
          const Pair y0 = pmul(x0, Pair{wk.x, wk.y}), y1 = pmul(x1, Pair{wk.z, wk.w});
          Pair z0 = y0, z1 = y1;
          if (far) {
            const float4 wq = *reinterpret_cast<const float4*>(fq + cg * 32 + j);
            z0 = pmul(x0, Pair{wq.x, wq.y});
            z1 = pmul(x1, Pair{wq.z, wq.w});
          }
          split2(z0.x, z0.y, hi[j / 2], lo[j / 2]);
          split2(z1.x, z1.y, hi[j / 2 + 1], lo[j / 2 + 1]);
          r[j] = __float_as_uint(y0.x);
          r[j + 1] = __float_as_uint(y0.y);
          r[j + 2] = __float_as_uint(y1.x);
          r[j + 3] = __float_as_uint(y1.y);
        }
        __syncwarp();
        tmem_st32(tmem + TM_S + lanes + cg * 32, r);
        tmem_st16(tmem + TM_SH + lanes + cg * 16, hi);
        tmem_st16(tmem + TM_SL + lanes + cg * 16, lo);
        tmem_st_wait();
      }
      if (OUT) {
        // ---- A, lower triangle: the quarters of Qh (lanes 0 .. 63) as two bf16 parts, those of Ql as one
        ok &= mbar_wait(bar_a, n & 1, dead, c.status, 800);
        tc_fence_after();
        const int t = lrow & 63;
        uint32_t r[16], r2[16];
        __syncwarp();
        tmem_ld16(tmem + TM_A + lanes + cg * 16, r);
        tmem_ld16(tmem + TM_A + LC + lanes + cg * 16, r2);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 16; j += 8) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = j + 2 * e, s = cg * 16 + i;
            Pair x = {s <= t ? __uint_as_float(r[i]) + __uint_as_float(r2[i]) : 0.0f, s + 1 <= t ? __uint_as_float(r[i + 1]) + __uint_as_float(r2[i + 1]) : 0.0f};
            if (far && quad < 2) x = padd(x, *reinterpret_cast<const Pair*>(far_a + t * LC + s));
            split2(x.x, x.y, hi[e], lo[e]);
          }
          const uint32_t at = sw128_offset(t, (cg * 16 + j) >> 3);
          *reinterpret_cast<uint4*>(sm + (quad < 2 ? T_A : T_A2) + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          if (quad < 2) *reinterpret_cast<uint4*>(sm + T_A + T_SPLIT + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive_warp(b_sa);
      if (n + 1 < n_chunks) gates(n + 1, chunk_of(n + 1));                 // while the tensor core works
      if (OUT) {
        // ---- result: lane = element of v, this warp's 16 tokens; norm over the head, gate.  Rows go through the tile of Q
        // (its products are done) to leave in 16-byte pieces.
        uint4 g[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          g[i] = make_uint4(0, 0, 0, 0);
          if (a.gate && o_mine && o_row + 8 * i < left) g[i] = *reinterpret_cast<const uint4*>(gp + (long long)(t0 + o_row + 8 * i) * a.ldg);
        }
        ok &= mbar_wait(bar_o, n & 1, dead, c.status, 801);
        tc_fence_after();
        float* rows = reinterpret_cast<float*>(sm + T_Q);
        {
          float sq[16];
          uint32_t r[16], r2[16];
          __syncwarp();
          tmem_ld16(tmem + TM_O + lanes + cg * 16, r);
          tmem_ld16(tmem + TM_O + LC + lanes + cg * 16, r2);
          tmem_ld_wait();
          tc_fence_before();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float o = __uint_as_float(r[j]) + __uint_as_float(r2[j]);
            rows[(cg * 16 + j) * 128 + lrow] = o;
            sq[j] = lrow < V ? o * o : 0.0f;              // lanes behind the head hold other columns of the rows
          }
          const float mine_sum = sum_over_lanes(sq, lane);
          if ((lane & 1) == 0) red[quad * LC + cg * 16 + (lane >> 1)] = mine_sum;
        }
        asm volatile("bar.sync %0, 128;" ::"r"(2 + cg) : "memory");
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = o_row + 8 * i;
          if (!o_mine || t >= left) continue;
          const float scale = rsqrtf(fmaf(red[t] + red[LC + t] + red[2 * LC + t] + red[3 * LC + t], inv_v, a.eps));
          const float4 x0 = *reinterpret_cast<const float4*>(rows + t * 128 + o_col), x1 = *reinterpret_cast<const float4*>(rows + t * 128 + o_col + 4);
          const float4 w0 = *reinterpret_cast<const float4*>(a.w + o_col), w1 = *reinterpret_cast<const float4*>(a.w + o_col + 4);
          float x[8] = {x0.x * scale * w0.x, x0.y * scale * w0.y, x0.z * scale * w0.z, x0.w * scale * w0.w,
                        x1.x * scale * w1.x, x1.y * scale * w1.y, x1.z * scale * w1.z, x1.w * scale * w1.w};
          if (a.gate) {
            const uint32_t gu[4] = {g[i].x, g[i].y, g[i].z, g[i].w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 f = unpack_bf16x2(gu[e]);
              x[2 * e] *= lin_silu_fast(f.x);
              x[2 * e + 1] *= lin_silu_fast(f.y);
            }
          }
          *reinterpret_cast<uint4*>(op + (long long)(t0 + t) * a.ldo) =
              make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
        }
      }
    }
    // ---- last state: to the cache, or as the stretch's sum
    if (n_chunks > 0) ok &= mbar_wait(bar_s, (n_chunks - 1) & 1, dead, c.status, 803);
    tc_fence_after();
    lc_meet();
    if (tg == 0) {
      f0[ch] = OUT ? exp2f(pend.x) : 1.0f;
      f0[ch + 1] = OUT ? exp2f(pend.y) : 1.0f;
    }
    lc_meet();
    if (ok && (!OUT || last)) {
      uint32_t r[32];
      __syncwarp();
      tmem_ld32(tmem + TM_S + lanes + cg * 32, r);
      tmem_ld_wait();
      float* dst = OUT ? a.state + ((slot * a.history + (p0 + count) % a.history) * a.heads + h) * (long long)D * V
                       : c.start + ((long long)blockIdx.y * a.heads + h) * D * V;
#pragma unroll
      for (int j = 0; j < 32; ++j)
        if (lrow < V && cg * 32 + j < D) dst[(long long)(cg * 32 + j) * V + lrow] = __uint_as_float(r[j]) * f0[cg * 32 + j];
      if (!OUT && tg == 0 && mine) {
        float* total = c.total + ((long long)blockIdx.y * a.heads + h) * D + ch;
        total[0] = tot.x;
        total[1] = tot.y;
      }
    }
  }
  if (*dead) __nanosleep(100000);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
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

CGK_API int cgk_linear_chunks(const cgk_linear_state_args* pa, int n_rows, const int* items, int n_items, const int* run_items, int n_runs,
                              void* scratch, void* stream) {
  CGK_REQUIRE(pa && items && n_rows > 0 && n_items >= 0 && (!scratch || (run_items && n_runs > 0)), "cgk_linear_chunks: bad arguments");
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
  // rows as the kernels read them: all tokens of the call, one head's columns at a time
  CUtensorMap tz, tq, tk, tv;
  auto rows_map = [&](CUtensorMap* m, const void* p, bool fp32, long long ld, int width, int box_cols, Swz swz) {
    const int es = fp32 ? 4 : 2;
    uint64_t dims[2] = {(uint64_t)width, (uint64_t)n_rows}, strides[1] = {(uint64_t)ld * es};
    uint32_t box[2] = {(uint32_t)box_cols, LC};
    return encode_tmap(m, p, fp32 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT32 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, dims, strides, box, swz);
  };
  int rc;
  if ((rc = rows_map(&tz, a.z, true, a.ldz, a.heads * a.D, a.D, Swz::None)) || (rc = rows_map(&tq, a.q, false, a.ldq, a.heads * a.D, a.D, Swz::None)) ||
      (rc = rows_map(&tk, a.k ? a.k : a.q, false, a.k ? a.ldk : a.ldq, a.heads * a.D, a.D, Swz::None)) ||
      (rc = rows_map(&tv, a.v, false, a.ldv, a.heads * a.V, 64, Swz::B128)))
    return rc;
  for (auto kernel : {scratch ? sums : nullptr, results}) {
    if (!kernel) continue;
    CGK_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LC_SMEM));
    kernel<<<grid, LC_THREADS + 128, LC_SMEM, st>>>(tz, tq, tk, tv, d);
    CGK_LAUNCH_CHECK();
    if (kernel == sums) {
      linear_starts_kernel<<<dim3((a.D * a.V / 4 + 255) / 256, a.heads, n_runs), 256, 0, st>>>(d, run_items);
      CGK_LAUNCH_CHECK();
    }
  }
  return 0;
}

CGK_BOUNDS_READER(linear_state_tc)
