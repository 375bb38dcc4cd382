// Paged keys and values as the kernels see them: k_pages[n_pages][kv_heads][page_size][ld_k], v_pages likewise with ld_v;
// ld_k and ld_v are the head sizes rounded up to 8 elements (the rest of a row is zero).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace cgk {

struct KvRowsDev {
  void* k_pages;
  void* v_pages;
  const int* page_table;     // [slots][max_pages]
  const int* slot;           // [tokens]
  const int* pos;            // [tokens]
  int kv_heads, dim, vdim, ld_k, ld_v, page_size, shift, max_pages, slots, n_pages;

  __device__ __forceinline__ int page_of(int key) const { return shift >= 0 ? key >> shift : key / page_size; }
  __device__ __forceinline__ int place_of(int key) const { return shift >= 0 ? key & (page_size - 1) : key % page_size; }
  // row number of a key of one head, in units of rows
  __device__ __forceinline__ long long row_of(long long page, int head, int key) const {
    return (page * kv_heads + head) * page_size + place_of(key);
  }
};

}  // namespace cgk
