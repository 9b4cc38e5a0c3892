// kv_rows.cuh -- where the rows of a paged key/value cache lie (KvRowCache, fosavik.h): a token's row, a block's pooled row, and
// how many pooled rows a position sees.
#pragma once
#include "fosavik.h"

namespace qie {

__device__ __forceinline__ const char* kv_row_ptr(const KvRowCache& c, const int* block_table, int max_pages, int slot, int pos) {
  const int page = block_table[(size_t)slot * max_pages + pos / c.page_size];
  const size_t off = (size_t)page * c.page_elems + c.layer_off + (size_t)(pos % c.page_size) * (c.kw + c.vw);
  return static_cast<const char*>(c.pool) + off * c.elt_bytes;
}
// pooled row of block b
__device__ __forceinline__ const char* kv_pool_ptr(const KvRowCache& c, const int* block_table, int max_pages, int slot, int b) {
  const int pi = (b * c.block + c.block - 1) / c.page_size;
  const int page = block_table[(size_t)slot * max_pages + pi];
  const size_t off = (size_t)page * c.page_elems + c.pool_off + (size_t)(b - pi * c.page_size / c.block) * (c.kw + c.vw);
  return static_cast<const char*>(c.pool) + off * c.elt_bytes;
}
// the first position that a row at pos sees below itself: its window's edge or its chunk's start (kept first tokens aside)
__host__ __device__ __forceinline__ int first_seen(int pos, int window, int chunk) {
  if (chunk > 0) return pos / chunk * chunk;
  return window > 0 && pos >= window ? pos - window + 1 : 0;
}
// blocks that end before the window of position pos begins: (b + 1) * block - 1 <= pos - window
__host__ __device__ __forceinline__ int pooled_seen(int pos, int window, int block) { return block > 0 && pos >= window ? (pos - window + 1) / block : 0; }

}  // namespace qie
