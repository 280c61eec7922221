// Rows of cached keys and values inside the pages of an attention layer.
#pragma once
#include "device_util.cuh"
#include "layered_kernels.cuh"

namespace pg {
namespace {

// First element of the key (which = 0) or value row of cache index c of one kv head; a latent row is both.
template <typename T>
__device__ __forceinline__ T* page_row(const AttentionLayer& l, T* pool, const int* table_row, int c, int head, int which) {
  const size_t page_elems = (size_t)l.kv_heads * l.page_tokens * (l.dimp + l.vrow);
  T* page = pool + (size_t)table_row[c / l.page_tokens] * page_elems;
  const int off = c % l.page_tokens;
  if (which == 0 || l.vrow == 0) return page + ((size_t)head * l.page_tokens + off) * l.dimp;
  return page + (size_t)l.kv_heads * l.page_tokens * l.dimp + ((size_t)head * l.page_tokens + off) * l.vrow;
}

}  // namespace
}  // namespace pg
