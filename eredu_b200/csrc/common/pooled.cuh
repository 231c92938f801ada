// Where the mean key and value of a block of cached tokens lie: beside the page of the block's last token.
#pragma once
#include <cuda_runtime.h>

namespace eredu {

struct PooledRow {
  int page, row;   // page of the sequence (16 tokens), row among the means kept beside that page
};

// Block b holds the positions b pool .. b pool + pool - 1.
__host__ __device__ __forceinline__ PooledRow pooled_row(int block, int pool) {
  PooledRow r;
  r.page = (block * pool + pool - 1) >> 4;
  r.row = block - (r.page << 4) / pool;
  return r;
}
// Whole blocks a query at `pos` sees behind its window: those that end at pos - window or before.
__host__ __device__ __forceinline__ int pooled_seen(int pos, int window, int pool) {
  return pos >= window ? (pos - window + 1) / pool : 0;
}

}  // namespace eredu
