// Attention in the latent space on the tcgen05 tensor cores: one query token, all heads, one shared row of
// R elements per key that serves as key AND value (multi-query attention whose K and V are the same matrix).
//
// One CTA = (key range, group of NP heads, query token); 128 keys at a time:
//   1. warp 8 brings the block in by TMA, page by page, as slices of 128 latent columns; the slices live in
//      a ring, so those of the next block arrive while this block's products run,
//   2. S^T[128 keys, NP] = C . Q^T          (tcgen05.mma by warp 9, keys on the TMEM lanes),
//   3. warps 0..7: scale, mask, row maxima through a row-major copy in shared memory, p = 2^(s - m); p is
//      stored as the sum of two bf16 numbers (two column groups of one operand tile), so the product below sees
//      the weight to 16 bits at the price of a wider instruction,
//   4. O^T[R, 2 NP] += C^T . P^T            (the same slices read MN-major); O stays in TMEM, is rescaled only
//      when a row maximum grows by more than 2^8, and its two column groups are added at the end.  A slice goes back
//      to the ring when its product is done.
// The kernel is bound by reading the latents (R * 2 bytes per key for all heads of the group).
#include "../../include/cogito_kernels.h"
#include "host_common.h"
#include "latent_dev.cuh"
#include "sm100.cuh"

namespace cgk {
namespace {

constexpr int LT_KB = 128, LT_SOFT = 256, LT_THREADS = 320, LT_MAX_SLOTS = 4;
constexpr uint32_t LT_SLICE = LT_KB * 128 * 2;            // 128 keys x 128 columns: two 64-column blocks of 16 KiB

struct LatentTcDev {
  LatentDev c;
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  float* part;               // [token][head][split][R], then (m, l) pairs; null with one split
  float* ml;
  int splits, ns, slots_c;
  float scale_log2;
  int* status;
};

template <int N>
__device__ __forceinline__ void lt_ld(uint32_t taddr, uint32_t (&r)[N]) {
  if constexpr (N == 8) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr)
                 : "memory");
  } else {
    static_assert(N == 16, "8 or 16 columns");
    tmem_ld16(taddr, r);
  }
}
template <int N>
__device__ __forceinline__ void lt_st(uint32_t taddr, const uint32_t (&r)[N]) {
  if constexpr (N == 8) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};"
                 ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
                 : "memory");
  } else {
    static_assert(N == 16, "8 or 16 columns");
    tmem_st16(taddr, r);
  }
}
// meeting point of the eight softmax warps
__device__ __forceinline__ void lt_meet() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int NP>
struct LtSmem {
  static constexpr uint32_t T_STRIDE = LT_KB + 4;                  // floats per row of the row-major score copy
  static constexpr uint32_t T_BYTES = NP * T_STRIDE * 4;           // later overwritten by P (2 * NP * 256 bytes)
  // offsets after the slice ring
  static __host__ __device__ uint32_t off_q(int slots) { return slots * LT_SLICE; }
  static __host__ __device__ uint32_t off_t(int slots, int ns) { return off_q(slots) + ns * NP * 256; }
  static __host__ __device__ uint32_t off_stat(int slots, int ns) { return off_t(slots, ns) + T_BYTES; }          // float [3][NP]
  static __host__ __device__ uint32_t off_lred(int slots, int ns) { return off_stat(slots, ns) + 3 * NP * 4; }    // float [4][NP]
  static __host__ __device__ uint32_t off_bar(int slots, int ns) { return off_lred(slots, ns) + 4 * NP * 4; }     // full, empty, s_full, p_ready, o_full, q_full
  static __host__ __device__ uint32_t off_misc(int slots, int ns) { return off_bar(slots, ns) + (2 * LT_MAX_SLOTS + 4) * 8; }
  static __host__ __device__ uint32_t total(int slots, int ns) { return off_misc(slots, ns) + 32 + 1024; }
};

template <int NP>
__global__ void __launch_bounds__(LT_THREADS, 2)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_pages, const LatentTcDev a) {
  using S = LtSmem<NP>;
  constexpr int CPT = NP / 2, TS = (int)S::T_STRIDE;
  extern __shared__ uint8_t lt_raw[];
  uint8_t* sm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sb = smem_u32(sm);
  const LatentDev& c = a.c;
  const int ns = a.ns, slots = a.slots_c, R = c.R;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x % a.splits, h0 = (int)(blockIdx.x / a.splits) * NP;
  const long long t = blockIdx.y;
  const int nh = min(NP, c.heads - h0);
  const int len = (int)CGK_IDX(c.pos[t], (long long)c.max_pages * c.page_size) + 1;
  const int per = ((len + a.splits - 1) / a.splits + LT_KB - 1) / LT_KB * LT_KB;
  const int k_begin = split * per, k_end = min(len, k_begin + per);
  if (k_begin >= k_end) {                                   // nothing in this range (never with one split)
    if (tid < nh) {
      float* ml = a.ml + ((t * c.heads + h0 + tid) * a.splits + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.0f;
    }
    return;
  }
  const int nblk = (k_end - k_begin + LT_KB - 1) / LT_KB;

  const uint32_t o_t = S::off_t(slots, ns), o_bar = S::off_bar(slots, ns), o_misc = S::off_misc(slots, ns), o_q = S::off_q(slots);
  float* tsc = reinterpret_cast<float*>(sm + o_t);
  float* stat = reinterpret_cast<float*>(sm + S::off_stat(slots, ns));     // [0] maximum in use, [NP] rescale factor
  float* lred = reinterpret_cast<float*>(sm + S::off_lred(slots, ns));
  auto full_bar = [&](int s) { return sb + o_bar + 8u * s; };
  auto empty_bar = [&](int s) { return sb + o_bar + 8u * (LT_MAX_SLOTS + s); };
  const uint32_t s_full = sb + o_bar + 8u * (2 * LT_MAX_SLOTS), p_ready = s_full + 8, o_full = s_full + 16, q_full = s_full + 24;
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(sm + o_misc);
  volatile int* dead = reinterpret_cast<volatile int*>(sm + o_misc + 4);
  volatile int* go = reinterpret_cast<volatile int*>(sm + o_misc + 8);
  volatile int* grew = reinterpret_cast<volatile int*>(sm + o_misc + 12);
  uint32_t cols = 32;
  while (cols < (uint32_t)(NP * (2 * ns + 1))) cols <<= 1;

  if (tid == 0) {
    for (int s = 0; s < slots; ++s) { mbar_init(full_bar(s), 1); mbar_init(empty_bar(s), 1); }
    mbar_init(s_full, 1);
    mbar_init(p_ready, 8);
    mbar_init(o_full, 1);
    mbar_init(q_full, 8);
    *dead = 0;
    mbar_fence_init();
  }
  if (warp == 8) {
    tmem_alloc(sb + o_misc, cols);
    tmem_relinquish();
  }
  if (tid < NP) stat[tid] = -INFINITY;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 8) {
    if (lane == 0) {
      const int* row = c.page_table + CGK_IDX(c.slot[t], c.slots) * c.max_pages;
      int it = 0;
      bool ok = true;
      for (int b = 0; b < nblk && ok; ++b) {
        const int kb = k_begin + b * LT_KB;
        int page[2], y[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int key = kb + i * 64, pi = key / c.page_size;
          // keys beyond the sequence are masked; any page will do for them
          page[i] = key < k_end ? (int)CGK_IDX(row[pi], c.n_pages) : 0;
          y[i] = key % c.page_size;
        }
        for (int m = 0; m < ns; ++m, ++it) {
          const int s = it % slots;
          if (!mbar_wait(empty_bar(s), ((it / slots) & 1) ^ 1, dead, a.status, 700)) { ok = false; break; }
          mbar_expect_tx(full_bar(s), LT_SLICE);
#pragma unroll
          for (int half = 0; half < 2; ++half)
#pragma unroll
            for (int i = 0; i < 2; ++i)
              tma_load_3d(sb + s * LT_SLICE + half * 16384 + i * 8192, &tm_pages, full_bar(s), m * 128 + half * 64, y[i], page[i]);
        }
      }
    }
  } else if (warp == 9) {
    if (lane == 0) {
      const uint32_t id_s = make_idesc_bf16(128, NP, 0, 0), id_o = make_idesc_bf16(128, 2 * NP, 1, 0);
      bool ok = mbar_wait(q_full, 0, dead, a.status, 712);
      tc_fence_after();
      for (int b = 0; b < nblk && ok; ++b) {
        for (int m = 0; m < ns; ++m) {
          const int it = b * ns + m, s = it % slots;
          if (!mbar_wait(full_bar(s), (it / slots) & 1, dead, a.status, 710)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            umma_f16(tmem, make_smem_desc_sw128(sb + s * LT_SLICE + (kk >> 2) * 16384 + (kk & 3) * 32, 16, 1024),
                     make_smem_desc_sw128(sb + o_q + (m * 2 + (kk >> 2)) * (NP * 128) + (kk & 3) * 32, 16, 1024), id_s,
                     (m | kk) != 0);
        }
        if (!ok) break;
        umma_commit(s_full);
        if (!mbar_wait(p_ready, b & 1, dead, a.status, 711)) break;
        tc_fence_after();
        for (int m = 0; m < ns; ++m) {
          const int it = b * ns + m, s = it % slots;
#pragma unroll
          for (int kk = 0; kk < LT_KB / 16; ++kk)
            umma_f16(tmem + NP * (1 + 2 * m), make_smem_desc_sw128(sb + s * LT_SLICE + kk * 2048, 16384, 1024),
                     make_smem_desc_sw128(sb + o_t + (kk >> 2) * (NP * 256) + (kk & 3) * 32, 16, 1024), id_o, b != 0 || kk != 0);
          umma_commit(empty_bar(s));
        }
        if (b + 1 == nblk) umma_commit(o_full);
      }
    }
  } else {
    // queries -> K-major operand tiles [NP][64] per 64 latent columns, zeros beyond the heads and beyond R; the
    // first key block is already on its way
#pragma unroll 4
    for (int i = tid; i < ns * NP * 16; i += LT_SOFT) {
      const int ch = i & 15, r = (i >> 4) % NP, m = (i >> 4) / NP, col = m * 128 + ch * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nh && col < R) v = *reinterpret_cast<const uint4*>(a.q + (t * c.heads + h0 + r) * R + col);
      *reinterpret_cast<uint4*>(sm + o_q + (m * 2 + (ch >> 3)) * (NP * 128) + sw128_offset(r, ch & 7)) = v;
    }
    fence_proxy_async_smem();
    mbar_arrive_warp(q_full);
    const int quad = warp & 3, half = warp >> 2;
    const uint32_t t_s = tmem + ((uint32_t)(quad * 32) << 16) + half * CPT;
    const int kin = quad * 32 + lane;
    float l_part[CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) l_part[j] = 0.0f;
    bool ok = true;
    for (int b = 0; b < nblk; ++b) {
      // one thread polls; the meeting point releases the rest, who read its verdict
      if (tid == 0) {
        go[0] = mbar_wait(s_full, b & 1, dead, a.status, 720);
        grew[0] = 0;
      }
      lt_meet();
      ok = go[0] != 0;
      if (!ok) break;
      tc_fence_after();
      uint32_t sr[CPT];
      lt_ld<CPT>(t_s, sr);
      tmem_ld_wait();
      const bool vis = k_begin + b * LT_KB + kin < k_end;
      float s[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        s[j] = vis ? __uint_as_float(sr[j]) * a.scale_log2 : -INFINITY;
        tsc[(half * CPT + j) * TS + kin] = s[j];
      }
      lt_meet();
      {
        constexpr int TPR = LT_SOFT / NP, F4 = LT_KB / 4 / TPR;
        const int r = tid / TPR, seg = tid % TPR;
        const float4* row4 = reinterpret_cast<const float4*>(tsc + r * TS);
        float mb = -INFINITY;
#pragma unroll
        for (int i = 0; i < F4; ++i) {
          const float4 v = row4[i * TPR + seg];
          mb = fmaxf(fmaxf(mb, fmaxf(v.x, v.y)), fmaxf(v.z, v.w));
        }
#pragma unroll
        for (int o = 1; o < TPR; o <<= 1) mb = fmaxf(mb, __shfl_xor_sync(0xffffffffu, mb, o));
        if (seg == 0) {
          const float mo = stat[r];
          float corr = 1.0f;
          if (mb > mo + 8.0f) {                        // also the first block: mo is -infinity
            corr = mo > -INFINITY ? exp2f(mo - mb) : 0.0f;
            stat[r] = mb;
            grew[0] = 1;
          }
          stat[NP + r] = corr;
        }
      }
      lt_meet();
      float corr[CPT];
      uint8_t* pbase = sm + o_t + (kin >> 6) * (NP * 256) + (kin & 7) * 2;
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        const int r = half * CPT + j;
        corr[j] = stat[NP + r];
        const float p = vis ? exp2f(s[j] - stat[r]) : 0.0f;
        l_part[j] = l_part[j] * corr[j] + p;
        const __nv_bfloat16 hi = __float2bfloat16(p);
        const uint32_t off = sw128_offset(r, (kin & 63) >> 3);
        *reinterpret_cast<__nv_bfloat16*>(pbase + off) = hi;
        *reinterpret_cast<__nv_bfloat16*>(pbase + NP * 128 + off) = __float2bfloat16(p - __bfloat162float(hi));
      }
      if (b > 0 && grew[0]) {
        // s_full of this block was committed after the products of the previous one: O is at rest
        for (int m = 0; m < 2 * ns; ++m) {
          uint32_t o[CPT];
          __syncwarp();
          lt_ld<CPT>(t_s + NP * (1 + m), o);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < CPT; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * corr[j]);
          lt_st<CPT>(t_s + NP * (1 + m), o);
        }
        tmem_st_wait();
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive_warp(p_ready);
    }
    if (ok) {
      if (tid == 0) go[0] = mbar_wait(o_full, 0, dead, a.status, 721);
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        const float v = warp_sum(l_part[j]);
        if (lane == 0) lred[quad * NP + half * CPT + j] = v;
      }
      lt_meet();
      ok = go[0] != 0;
    }
    if (ok) {
      tc_fence_after();
      // everything that depends on the column alone is worked out once; the stores below are an addition each
      float inv[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        const int hr = half * CPT + j;
        const float l = lred[hr] + lred[NP + hr] + lred[2 * NP + hr] + lred[3 * NP + hr];
        inv[j] = 1.0f / l;
        if (a.splits > 1 && kin == 0 && hr < nh) {
          float* ml = a.ml + ((t * c.heads + h0 + hr) * a.splits + split) * 2;
          ml[0] = stat[hr];
          ml[1] = l;
        }
      }
      const long long row0 = t * c.heads + h0 + half * CPT;
      __nv_bfloat16* out = a.out + row0 * R + kin;
      float* part = a.part + (row0 * a.splits + split) * R + kin;
      const int step = a.splits * R, mine = nh - half * CPT;         // columns of this half that are heads
      for (int m = 0; m < ns; ++m) {
        uint32_t o[CPT], lo[CPT];
        __syncwarp();
        lt_ld<CPT>(t_s + NP * (1 + 2 * m), o);
        lt_ld<CPT>(t_s + NP * (2 + 2 * m), lo);
        tmem_ld_wait();
        if (m * 128 + kin >= R) continue;
        if (a.splits == 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j)
            if (j < mine) out[m * 128 + j * R] = __float2bfloat16((__uint_as_float(o[j]) + __uint_as_float(lo[j])) * inv[j]);
        } else {
#pragma unroll
          for (int j = 0; j < CPT; ++j)
            if (j < mine) part[m * 128 + j * step] = __uint_as_float(o[j]) + __uint_as_float(lo[j]);
        }
      }
    }
  }
  if (*dead) __nanosleep(100000);
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tmem, cols);
  }
}

template <int NP>
int launch_np(const CUtensorMap& tm, const LatentTcDev& a, int rows, cudaStream_t st) {
  const uint32_t smem = LtSmem<NP>::total(a.slots_c, a.ns);
  CGK_CUDA_CHECK(cudaFuncSetAttribute(latent_attn_tc_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid(a.splits * ((a.c.heads + NP - 1) / NP), rows);
  latent_attn_tc_kernel<NP><<<grid, LT_THREADS, smem, st>>>(tm, a);
  CGK_LAUNCH_CHECK();
  return 0;
}

}  // namespace

bool latent_tc_ok(int R, int page_size, int heads) { return R % 8 == 0 && R > 0 && R <= 512 && page_size % 64 == 0 && heads > 0; }

int launch_latent_tc(const LatentDev& d, const __nv_bfloat16* q, __nv_bfloat16* out, int rows, int splits, float* scratch, cudaStream_t st) {
  CGK_REQUIRE(rows <= 65535, "latent attention: too many query tokens in one call");
  CGK_REQUIRE((((uintptr_t)q) & 15) == 0 && (((uintptr_t)d.pages) & 15) == 0, "latent attention: operands must be 16-byte aligned");
  int dev = 0;
  CGK_CUDA_CHECK(cudaGetDevice(&dev));
  LatentTcDev a;
  a.c = d;
  a.q = q;
  a.out = out;
  a.splits = splits;
  a.part = splits > 1 ? scratch : nullptr;
  a.ml = splits > 1 ? scratch + (long long)rows * d.heads * splits * d.R : nullptr;
  a.ns = (d.R + 127) / 128;
  a.slots_c = a.ns == 1 ? 2 : LT_MAX_SLOTS;
  a.scale_log2 = d.scale * 1.4426950408889634f;
  a.status = device_status(dev);
  CUtensorMap tm;
  uint64_t dims[3] = {(uint64_t)d.R, (uint64_t)d.page_size, (uint64_t)d.n_pages};
  uint64_t strides[2] = {(uint64_t)d.R * 2, (uint64_t)d.R * d.page_size * 2};
  uint32_t box[3] = {64, 64, 1};
  int rc = encode_tmap(&tm, d.pages, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, strides, box, Swz::B128);
  if (rc) return rc;
  // 16 heads per CTA while that leaves every CTA an SM (a CTA's time grows with its heads), else 32: more heads share
  // one pass over the latents, and the per-thread state of a wider tile no longer fits in registers
  if (d.heads <= 16 || (long long)rows * ((d.heads + 15) / 16) * splits <= sm_count(dev)) rc = launch_np<16>(tm, a, rows, st);
  else rc = launch_np<32>(tm, a, rows, st);
  if (rc) return rc;
  if (splits > 1) CGK_CUDA_CHECK(launch_latent_merge(a.part, a.ml, out, rows * d.heads, splits, d.R, st));
  return 0;
}

}  // namespace cgk

CGK_BOUNDS_READER(latent_attn_tc)
