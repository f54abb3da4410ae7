// The fp32 residual stream of a decoder whose sublayers are normed on their way out, in groups of columns, in one pass over a row:
//
//   y = a row of a, the weighted sum of a token's expert outputs, or the embedding row of a token (the stream then begins at zero)
//   x += mult * norm(y) * (offset + post)
//   h  = norm(x) * (offset + w), or x itself where no weight is given
//
// norm divides every one of `groups` equal parts of a row by its own root mean square.  One CTA per row, the row in registers: thread i
// holds pieces i, i + threads, ... of N neighbouring columns, none of which straddles two groups.  Squares are added over 2^k neighbouring
// lanes as far as a group's pieces divide, the rest through shared memory in a fixed order.
// With `rows` only those rows are emitted and x is left as it was (the last norm of a step).
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct GroupStream {
  float* x;
  const T* a;               // [rows][W], or with a_rows a buffer of rows
  const int* a_rows;        // [rows][top]
  const float* a_weights;   // [rows][top]; null: all 1
  int top;
  const T* post;
  float mult, offset;
  const int* ids;           // with ids: y is the row of embed
  const T* embed;
  int vocab;
  const T* w;
  T* h;                     // null: nothing is emitted
  const int* rows;
  int n_rows, W, start, groups, per, seg_log2, segs;      // per: pieces of a group; segs: sums of 2^seg_log2 pieces in a group
  float eps;
};

// Sum of squares of the group that piece i belongs to, from every thread's sums v[q] over its pieces; part: one entry per 2^seg_log2 pieces.
template <int R, typename Args>
__device__ __forceinline__ void group_scales(const Args& p, int pieces, float (&v)[R], const int (&group)[R], float* part) {
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = q * blockDim.x + threadIdx.x;
    for (int o = 1; o < (1 << p.seg_log2); o <<= 1) v[q] += __shfl_xor_sync(0xffffffffu, v[q], o);
    if (i < pieces && (i & ((1 << p.seg_log2) - 1)) == 0) part[i >> p.seg_log2] = v[q];
  }
  __syncthreads();
  const float n = 1.f / static_cast<float>(p.W / p.groups);
#pragma unroll
  for (int q = 0; q < R; ++q) {
    float s = 0.f;
    for (int k = 0; k < p.segs; ++k) s += part[group[q] * p.segs + k];
    v[q] = rsqrtf(fmaf(s, n, p.eps));
  }
}

template <typename T, int N, int R, int kThreads>
__global__ void __launch_bounds__(kThreads) stream_group_kernel(const GroupStream<T> p) {
  extern __shared__ float part[];           // [2][groups * segs]
  const int pieces = p.W / N;
  int group[R];
#pragma unroll
  for (int q = 0; q < R; ++q) group[q] = min(static_cast<int>(q * blockDim.x + threadIdx.x), pieces - 1) / p.per;
  pdl_launch_dependents();
  pdl_wait();
  int r = blockIdx.x;
  if (p.rows != nullptr) {
    r = p.rows[r];
    r = r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
  }
  const size_t base = static_cast<size_t>(r) * p.W;
  const T* src = p.a + base;
  if (p.ids != nullptr) {
    int id = p.ids[r];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    src = p.embed + static_cast<size_t>(id) * p.W;
  }
  float x[R][N], y[R][N], ss[R];
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
#pragma unroll
    for (int e = 0; e < N; ++e) x[q][e] = y[q][e] = 0.f;
    ss[q] = 0.f;
    if (i >= p.W) continue;
    if (!p.start) load_n<N>(p.x + base + i, x[q]);
    if (p.a_rows == nullptr) load_n<N>(src + i, y[q]);
  }
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    if (p.a_rows != nullptr) {
#pragma unroll 4
      for (int j = 0; j < p.top; ++j) {
        const size_t at = static_cast<size_t>(r) * p.top + j;
        const float s = p.a_weights != nullptr ? p.a_weights[at] : 1.f;
        float v[N];
        load_n<N>(p.a + static_cast<size_t>(p.a_rows[at]) * p.W + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) y[q][e] = fmaf(s, v[e], y[q][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < N; ++e) ss[q] = fmaf(y[q][e], y[q][e], ss[q]);
  }
  group_scales<R>(p, pieces, ss, group, part);
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    const float f = p.mult * ss[q];
    ss[q] = 0.f;
    if (i >= p.W) continue;
    float g[N];
    load_n<N>(p.post + i, g);
#pragma unroll
    for (int e = 0; e < N; ++e) {
      x[q][e] = fmaf(f * y[q][e], g[e] + p.offset, x[q][e]);
      ss[q] = fmaf(x[q][e], x[q][e], ss[q]);
    }
    if (p.rows == nullptr) store_n<N>(p.x + base + i, x[q]);
  }
  if (p.h == nullptr) return;
  if (p.w != nullptr) group_scales<R>(p, pieces, ss, group, part + p.groups * p.segs);
  const size_t out = static_cast<size_t>(blockIdx.x) * p.W;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    if (p.w != nullptr) {
      float g[N];
      load_n<N>(p.w + i, g);
#pragma unroll
      for (int e = 0; e < N; ++e) x[q][e] *= ss[q] * (g[e] + p.offset);
    }
    store_n<N>(p.h + out + i, x[q]);
  }
}

template <typename T, int N, int R, int kThreads>
static int launch_stream_group(int out_rows, GroupStream<T> p, cudaStream_t stream) {
  const int pieces = p.W / N, threads = ((pieces + R - 1) / R + 31) / 32 * 32;
  p.per = pieces / p.groups;
  p.seg_log2 = 0;
  while (p.seg_log2 < 5 && p.per % (2 << p.seg_log2) == 0) ++p.seg_log2;
  p.segs = p.per >> p.seg_log2;
  const size_t smem = static_cast<size_t>(2) * p.groups * p.segs * 4;
  auto k = stream_group_kernel<T, N, R, kThreads>;
  FORGE_ENSURE_DYN_SMEM(k, 128 * 1024);
  return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
}

template <typename T>
static int stream_group(int out_rows, const GroupStream<T>& p, cudaStream_t stream) {
  if (p.groups < 1 || p.W % p.groups || p.W > 16384) return -1;
  if ((p.W / p.groups) % 8 == 0) {
    if (p.W <= 2048) return launch_stream_group<T, 8, 1, 256>(out_rows, p, stream);
    if (p.W <= 4096) return launch_stream_group<T, 8, 2, 256>(out_rows, p, stream);
    return launch_stream_group<T, 8, 2, 1024>(out_rows, p, stream);
  }
  if (p.W <= 1024) return launch_stream_group<T, 1, 1, 1024>(out_rows, p, stream);
  return launch_stream_group<T, 1, 16, 1024>(out_rows, p, stream);
}

// x fp32 [n_rows][W]; ids and embed, or a (with a_rows: any rows of it); out_rows rows of h.
extern "C" int forge_stream_group(int fp32, float* x, const void* a, const int* a_rows, const float* a_weights, int top, const void* post, float mult,
                                  float offset, const int* ids, const void* embed, int vocab, const void* w, void* h, const int* rows, int out_rows,
                                  int n_rows, int W, int groups, int start, float eps, cudaStream_t stream) {
  if (out_rows <= 0) return 0;
#define FORGE_GROUP(T)                                                                                                              \
  return stream_group<T>(out_rows, GroupStream<T>{x, static_cast<const T*>(a), a_rows, a_weights, top, static_cast<const T*>(post), mult, offset, ids, \
                                                  static_cast<const T*>(embed), vocab, static_cast<const T*>(w), static_cast<T*>(h), rows, n_rows, W, start, \
                                                  groups, 0, 0, 0, eps}, stream)
  if (fp32) FORGE_GROUP(float);
  FORGE_GROUP(bf16);
#undef FORGE_GROUP
}

}  // namespace forge
