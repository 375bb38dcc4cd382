// Linear recurrences with a decay per state row:  S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t   per head,
// state rows belong to the D elements of q and k, columns to the V elements of v.
//   o leaves RMS-normed over V with a weight, optionally times silu(gate), in the operand's type.
// Two ways to the decay, both from z (fp32) + bias:
//   GATE_BOUNDED  a = low + (1 - low) sigmoid(z), k = 1 - a        (the forget gate decides what is written)
//   GATE_ROOT     a = sigmoid(z)^(1 / tau), k given
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "sm100.cuh"

namespace cgk {

enum : int { GATE_BOUNDED = 0, GATE_ROOT = 1 };

struct LinStateDev {
  const void* q; const void* k; const void* v; const void* gate;      // bf16 or fp32 rows; k null with GATE_BOUNDED, gate may be null
  const float* z;
  long long ldq, ldk, ldv, ldg, ldz;
  const float* bias; const float* low; const float* w;                // [heads * D], [heads * D] or null, [V]
  float* state;                                                       // [slots][history][heads][D][V]
  void* out; long long ldo;
  const int* slot; const int* pos;                                    // [tokens]
  const int* runs;                                                    // [n_runs][2]: first token, tokens; null: every token by itself
  int heads, D, V, history, slots, mode, q_silu;
  float q_scale, inv_tau, eps;
};

// z -> natural logarithm of the decay; *one_minus gets 1 - decay without cancellation (GATE_BOUNDED)
__device__ __forceinline__ float lin_decay(const LinStateDev& a, float z, int channel, float* one_minus) {
  z += a.bias[channel];
  if (a.mode == GATE_ROOT) {
    *one_minus = 0.0f;
    return (fminf(z, 0.0f) - log1pf(expf(-fabsf(z)))) * a.inv_tau;
  }
  const float low = a.low[channel], e = expf(-fabsf(z)), big = 1.0f / (1.0f + e), small = e * big;
  const float s = z >= 0.0f ? big : small, ns = z >= 0.0f ? small : big;
  *one_minus = (1.0f - low) * ns;
  return logf(fmaxf(fmaf(1.0f - low, s, low), 1e-37f));
}

// The same in base 2 with the hardware's exponential and reciprocal, for the tensor-core form: bias and low are the
// channel's.  Logarithms near 1 come from 2 artanh(u) = 2 (u + u^3 / 3 + ...), which keeps their relative error at
// fp32's resolution (lg2.approx bounds the absolute error, and thousands of tokens would add that up).
__device__ __forceinline__ float lin_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lin_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lin_lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two channels at once, in packed fp32 arithmetic
struct Pair { float x, y; };
__device__ __forceinline__ Pair pfma(Pair a, Pair b, Pair c) { Pair d; ffma2(d.x, d.y, a.x, a.y, b.x, b.y, c.x, c.y); return d; }
__device__ __forceinline__ Pair pmul(Pair a, Pair b) { Pair d; fmul2(d.x, d.y, a.x, a.y, b.x, b.y); return d; }
__device__ __forceinline__ Pair padd(Pair a, Pair b) { fadd2(a.x, a.y, b.x, b.y); return a; }
__device__ __forceinline__ Pair pall(float v) { return Pair{v, v}; }
// y: gate with its bias; low: lower bounds; returns the logarithms, *key the keys of GATE_BOUNDED
template <int MODE>
__device__ __forceinline__ Pair lin_decay_log2(Pair y, Pair low, float inv_tau, Pair* key) {
  constexpr float LOG2E = 1.4426950408889634f;
  const Pair e = {lin_ex2(-fabsf(y.x) * LOG2E), lin_ex2(-fabsf(y.y) * LOG2E)};
  if constexpr (MODE == GATE_ROOT) {                       // -(max(-y, 0) log2 e + log2(1 + e)) / tau, u = e / (2 + e) <= 1/3
    const Pair d = padd(e, pall(2.0f)), u = pmul(e, Pair{lin_rcp(d.x), lin_rcp(d.y)}), u2 = pmul(u, u);
    Pair p = pfma(u2, pall(1.0f / 13), pall(1.0f / 11));
    p = pfma(u2, p, pall(1.0f / 9));
    p = pfma(u2, p, pall(1.0f / 7));
    p = pfma(u2, p, pall(1.0f / 5));
    p = pfma(u2, p, pall(1.0f / 3));
    p = pfma(pmul(u2, u), p, u);
    const Pair m = {fminf(y.x, 0.0f), fminf(y.y, 0.0f)};
    return pfma(p, pall(-2.0f * LOG2E * inv_tau), pmul(m, pall(LOG2E * inv_tau)));
  } else {
    // one reciprocal for 1 / (1 + e) and for u = k / (2 - k), k = room * num / (1 + e)
    const bool px = y.x >= 0.0f, py = y.y >= 0.0f;
    const Pair room = padd(pall(1.0f), Pair{-low.x, -low.y}), num = {px ? e.x : 1.0f, py ? e.y : 1.0f}, rest = {px ? 1.0f : e.x, py ? 1.0f : e.y};
    const Pair one = padd(e, pall(1.0f)), rn = pmul(room, num), den = pfma(one, pall(2.0f), Pair{-rn.x, -rn.y}), od = pmul(one, den);
    const Pair r = {lin_rcp(od.x), lin_rcp(od.y)}, inv = pmul(r, den), k = pmul(rn, inv), f = pfma(pmul(room, inv), rest, low);
    const Pair u = pmul(rn, pmul(one, r)), u2 = pmul(u, u);   // k <= 1/4: u <= 1/7
    Pair p = pfma(u2, pall(1.0f / 7), pall(1.0f / 5));
    p = pfma(u2, p, pall(1.0f / 3));
    p = pmul(pfma(pmul(u2, u), p, u), pall(-2.0f * LOG2E));
    *key = k;
    return Pair{k.x <= 0.25f ? p.x : lin_lg2(fmaxf(f.x, 1e-37f)), k.y <= 0.25f ? p.y : lin_lg2(fmaxf(f.y, 1e-37f))};
  }
}
__device__ __forceinline__ Pair lin_silu_fast(Pair x) {
  const Pair t = pmul(x, pall(-1.4426950408889634f)), d = padd(Pair{lin_ex2(t.x), lin_ex2(t.y)}, pall(1.0f));
  return pmul(x, Pair{lin_rcp(d.x), lin_rcp(d.y)});
}
__device__ __forceinline__ float lin_silu_fast(float x) { return x * lin_rcp(1.0f + lin_ex2(-1.4426950408889634f * x)); }

__device__ __forceinline__ float lin_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float lin_query(const LinStateDev& a, float q) { return (a.q_silu ? lin_silu(q) : q) * a.q_scale; }

}  // namespace cgk
