// Linear recurrences with a decay per state row:  S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t   per head,
// state rows belong to the D elements of q and k, columns to the V elements of v.
//   o leaves RMS-normed over V with a weight, optionally times silu(gate), in the operand's type.
// Two ways to the decay, both from z (fp32) + bias:
//   GATE_BOUNDED  a = low + (1 - low) sigmoid(z), k = 1 - a        (the forget gate decides what is written)
//   GATE_ROOT     a = sigmoid(z)^(1 / tau), k given
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

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
__device__ __forceinline__ float lin_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float lin_query(const LinStateDev& a, float q) { return (a.q_silu ? lin_silu(q) : q) * a.q_scale; }

}  // namespace cgk
