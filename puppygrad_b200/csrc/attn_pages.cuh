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
  const bool value = which != 0 && l.vrow != 0;
  const int off = c % l.page_tokens, width = value ? l.vrow : l.dimp;
  T* page = pool + (size_t)table_row[c / l.page_tokens] * page_elems + (value ? (size_t)l.kv_heads * l.page_tokens * l.dimp : 0);
  return page + (l.wide ? (size_t)off * l.kv_heads + head : (size_t)head * l.page_tokens + off) * width;
}

}  // namespace
}  // namespace pg
