// Shared between latent_kv.cu and latent_attn_tc.cu: the paged latent cache as the kernels see it.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace cgk {

struct LatentDev {
  void* pages;               // [n_pages][page_size][R]
  const int* page_table;     // [slots][max_pages]
  const int* slot;           // [tokens] sequence slot of every query token
  const int* pos;            // [tokens] its position; it sees keys 0 .. pos
  int R, page_size, max_pages, slots, n_pages, heads;
  float scale;
};

bool latent_tc_ok(int R, int page_size, int heads);
int launch_latent_tc(const LatentDev& d, const __nv_bfloat16* q, __nv_bfloat16* out, int rows, int splits, float* scratch, cudaStream_t st);
cudaError_t launch_latent_merge(const float* part, const float* ml, __nv_bfloat16* out, int rows, int splits, int R, cudaStream_t st);

}  // namespace cgk
