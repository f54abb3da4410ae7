// What stands around attention over pooled blocks and over a window of a step's keys:
//
//   pool_blocks   the means of the blocks that end among the step's tokens, to their places in the cache (pooled.cuh); with a gather buffer
//                 also all entries of the step's sequences, one after another: [rows][G][d / dv], as TMA wants them
//   row_offsets   where the rows of the step's sequences begin in such a buffer: running sums of min(keys, queries + window - 1) or of
//                 floor(keys / size)
#include "../include/launch.cuh"
#include "../include/pooled.cuh"

namespace forge {

template <typename T>
struct PoolArgs {
  const T* k_cache;         // [blocks][G][block_size][d]
  const T* v_cache;
  PoolCache<T> pool;
  const int* cu;            // [seqs + 1] rows of the sequences' queries
  const int* lens;          // [seqs] keys
  const int* tables;        // [seqs][width]
  const int* offsets;       // [seqs + 1] first gathered row of a sequence; null: nothing is gathered
  T* gk;                    // [bound][G][d]
  T* gv;                    // [bound][G][dv]
  int bound, seqs, width, num_blocks, block_size, G, d, dv, own;
  unsigned* status;
};

// CTA = (blocks x, x + gridDim.x, .. of a sequence's, or of those that end in this step; sequence).  The last row of the grid zeroes what
// remains of the gather buffer.  A thread takes N neighbouring columns of a head.
template <typename T, int N>
__global__ void __launch_bounds__(128) pool_blocks_kernel(const PoolArgs<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y, ku = p.d / N, vu = p.dv / N, items = p.G * (ku + vu), size = p.pool.size;
  if (s == p.seqs) {
    float zero[N];
#pragma unroll
    for (int e = 0; e < N; ++e) zero[e] = 0.f;
    for (int row = p.offsets[p.seqs] + blockIdx.x; row < p.bound; row += gridDim.x) {
      for (int i = threadIdx.x * N; i < p.G * p.d; i += blockDim.x * N) store_n<N>(p.gk + static_cast<size_t>(row) * p.G * p.d + i, zero);
      for (int i = threadIdx.x * N; i < p.G * p.dv; i += blockDim.x * N) store_n<N>(p.gv + static_cast<size_t>(row) * p.G * p.dv + i, zero);
    }
    return;
  }
  int len = p.lens[s];
  if (len > p.width * p.block_size) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    len = p.width * p.block_size;
  }
  const int start = max(len - (p.cu[s + 1] - p.cu[s]), 0), fresh = start / size, end = max(len, 0) / size;
  const bool gather = p.offsets != nullptr;
  const int* table = p.tables + static_cast<size_t>(s) * p.width;
  auto block_of = [&](int page) {
    int blk = table[page];
    if (blk < 0 || blk >= p.num_blocks) {
      set_status(p.status, kStatusBadIndex);
      blk = 0;
    }
    return blk;
  };
  for (int b = (gather ? 0 : fresh) + blockIdx.x; b < end; b += gridDim.x) {
    const int page = pool_page(b, size, p.block_size), row = pool_row(b, page, size, p.block_size), blk = block_of(page);
    const bool made = b >= fresh && p.own;                 // its tokens are summed; else the entry exists
    if (!made && !gather) continue;
    for (int i = threadIdx.x; i < items; i += blockDim.x) {
      const bool value = i >= p.G * ku;
      const int j = value ? i - p.G * ku : i, w = value ? p.dv : p.d, g = j / (w / N), c = j % (w / N) * N;
      T* place = (value ? p.pool.v : p.pool.k) + ((static_cast<size_t>(blk) * p.G + g) * p.pool.rows + row) * w + c;
      float m[N];
      if (made) {
        const T* cache = value ? p.v_cache : p.k_cache;
#pragma unroll
        for (int e = 0; e < N; ++e) m[e] = 0.f;
#pragma unroll 8
        for (int t = b * size; t < (b + 1) * size; ++t) {
          float x[N];
          load_n<N>(cache + ((static_cast<size_t>(block_of(t / p.block_size)) * p.G + g) * p.block_size + t % p.block_size) * w + c, x);
#pragma unroll
          for (int e = 0; e < N; ++e) m[e] += x[e];
        }
#pragma unroll
        for (int e = 0; e < N; ++e) m[e] /= static_cast<float>(size);
        store_n<N>(place, m);
      } else {
        load_n<N>(place, m);
      }
      if (!gather) continue;
      const int at = p.offsets[s] + b;
      if (at < p.bound) store_n<N>((value ? p.gv : p.gk) + (static_cast<size_t>(at) * p.G + g) * w + c, m);
    }
  }
}

template <typename T>
static int pool_blocks(const PoolArgs<T>& p, int max_q, int max_k, cudaStream_t stream) {
  const bool gather = p.offsets != nullptr;
  int x = gather ? max_k / p.pool.size : (max_q + p.pool.size - 1) / p.pool.size;
  x = x < 1 ? 1 : (x > 65535 ? 65535 : x);
  const dim3 grid(x, p.seqs + (gather ? 1 : 0));
  if (grid.y > 65535) return -1;
  const int all = p.d | p.dv;
  auto k = (all & 7) == 0 ? pool_blocks_kernel<T, 8> : (all & 3) == 0 ? pool_blocks_kernel<T, 4> : pool_blocks_kernel<T, 1>;
  return launch_kernel(k, grid, dim3(128), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
}

// own: this call makes the entries of the blocks that end in the step (else they exist).  offsets, gk, gv (or null): gathered entries, `bound`
// rows in all.  max_q, max_k: most queries and keys of a sequence.
extern "C" int forge_pool_blocks(int fp32, const void* k_cache, const void* v_cache, void* pool_k, void* pool_v, int size, int own, const int* cu,
                                 const int* lens, const int* tables, int seqs, int max_q, int max_k, const int* offsets, void* gk, void* gv, int bound,
                                 int width, int num_blocks, int block_size, int G, int d, int dv, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0 || (offsets == nullptr && !own)) return 0;
  if (size < 1) return -1;
  const int rows = (block_size + size - 1) / size;
#define FORGE_POOL(T)                                                                                                                             \
  return pool_blocks<T>({static_cast<const T*>(k_cache), static_cast<const T*>(v_cache), {static_cast<T*>(pool_k), static_cast<T*>(pool_v), size, rows}, \
                         cu, lens, tables, offsets, static_cast<T*>(gk), static_cast<T*>(gv), bound, seqs, width, num_blocks, block_size, G, d, dv, own, \
                         status}, max_q, max_k, stream)
  if (fp32) FORGE_POOL(float);
  FORGE_POOL(bf16);
#undef FORGE_POOL
}

// One warp: out[s] = rows of the sequences ahead of s.
__global__ void __launch_bounds__(32) row_offsets_kernel(const int* __restrict__ cu, const int* __restrict__ lens, int seqs, int window, int size,
                                                         int* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  int base = 0;
  for (int s0 = 0; s0 < seqs; s0 += 32) {
    const int s = s0 + threadIdx.x;
    int v = 0;
    if (s < seqs) {
      const int len = max(lens[s], 0);
      v = size > 0 ? len / size : min(len, cu[s + 1] - cu[s] + window - 1);
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, v, o);
      if (threadIdx.x >= o) v += u;
    }
    if (s < seqs) out[s + 1] = base + v;
    base += __shfl_sync(0xffffffffu, v, 31);
  }
  if (threadIdx.x == 0) out[0] = 0;
}

// size > 0: rows = floor(keys / size); else rows = min(keys, queries + window - 1).
extern "C" int forge_row_offsets(const int* cu, const int* lens, int seqs, int window, int size, int* out, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  return launch_kernel(row_offsets_kernel, dim3(1), dim3(32), 0, stream, 0, cu, lens, seqs, window, size, out) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
