// Means of the keys and values of whole blocks of `size` tokens, counted from a sequence's first, beside the paged cache
// [blocks][G][block_size][..]: caches [blocks][G][rows][..] with rows = ceil(block_size / size).  The entry of a block lies in the page of the
// block's last token, which holds the blocks that end in it, in order: everything in a page depends on the tokens up to its end alone.
#pragma once

#include "scalar.cuh"

namespace forge {

template <typename T>
struct PoolCache {
  T* k;
  T* v;
  int size, rows;           // tokens of a block, entries of a page; size 0: no pooled blocks
};

__device__ __forceinline__ int pool_page(int block, int size, int block_size) {
  return static_cast<int>((static_cast<long long>(block + 1) * size - 1) / block_size);
}
__device__ __forceinline__ int pool_row(int block, int page, int size, int block_size) {
  return block - static_cast<int>(static_cast<long long>(page) * block_size / size);
}
// Blocks that end before key `oldest`, the oldest of a query's window.
__device__ __forceinline__ int pool_visible(int oldest, int size) { return oldest / size; }

}  // namespace forge
