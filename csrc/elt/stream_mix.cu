// Several fp32 residual streams between two sublayers of a decoder, in one pass over a token's rows:
//
//   x_t <- sum_s mix[s, t] x_s + out[t] y        a sublayer's result y is taken up by all streams at once, or
//   x_t <- scale * embed[id] + pairs[row]        every stream begins as the embedding; row = (prev * mul_prev + id * mul_cur) mod buckets,
//                                                the last row for a sequence's first token (prev < 0)
//   h   = layer_norm(sum_s into[s] x_s) * w + b  the normed input of the sublayer after
//
// One CTA per token.  With `rows` only those tokens are normed and x is left as it was (the last norm of a step: only rows whose
// logits are wanted).
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kMaxStreams = 16;

template <typename T>
struct MixArgs {
  float* x;                 // [n_rows][S][W]
  const T* y;               // [n_rows][W]; null: the streams begin
  const float* mix;         // [S from][S to]
  const float* out;         // [S]
  const int* ids;
  const int* prev;
  const T* embed;           // [vocab][W]
  const T* pairs;           // [buckets + 1][W]
  int vocab, buckets;
  long long mul_prev, mul_cur;
  float scale;
  const float* into;        // [S]
  const T* w;               // null: no result
  const T* b;
  T* h;
  const int* rows;
  int n_rows, W, S;
  float eps;
};

template <typename T>
__device__ __forceinline__ int mix_row(const MixArgs<T>& p) {
  if (p.rows == nullptr) return blockIdx.x;
  const int r = p.rows[blockIdx.x];
  return r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
}

template <typename T>
__device__ __forceinline__ void mix_embedding(const MixArgs<T>& p, int r, const T*& emb, const T*& pair) {
  const int id = min(max(p.ids[r], 0), p.vocab - 1), prev = p.prev[r];
  long long row = p.buckets;
  if (prev >= 0) {
    row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
    if (row < 0) row += p.buckets;
  }
  emb = p.embed + static_cast<size_t>(id) * p.W;
  pair = p.pairs + static_cast<size_t>(row) * p.W;
}

// Rows that fit the registers of a CTA: R pieces of N entries of every stream per thread.
template <typename T, int N, int R, int S>
__global__ void __launch_bounds__(256) stream_mix_reg_kernel(const MixArgs<T> p) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int r = mix_row(p);
  float* x = p.x + static_cast<size_t>(r) * S * p.W;
  float u[R][N], sum = 0.f;
  float into[S];
#pragma unroll
  for (int s = 0; s < S; ++s) into[s] = p.into[s];
  if (p.y != nullptr) {
    float mix[S][S], out[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      out[s] = p.out[s];
#pragma unroll
      for (int t = 0; t < S; ++t) mix[s][t] = p.mix[s * S + t];
    }
    float v[R][S][N], y[R][N];
#pragma unroll
    for (int q = 0; q < R; ++q) {
      const int i = (q * blockDim.x + threadIdx.x) * N;
      if (i >= p.W) continue;
      load_n<N>(p.y + static_cast<size_t>(r) * p.W + i, y[q]);
#pragma unroll
      for (int s = 0; s < S; ++s) load_n<N>(x + static_cast<size_t>(s) * p.W + i, v[q][s]);
    }
#pragma unroll
    for (int q = 0; q < R; ++q) {
      const int i = (q * blockDim.x + threadIdx.x) * N;
#pragma unroll
      for (int e = 0; e < N; ++e) u[q][e] = 0.f;
      if (i >= p.W) continue;
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float n[N];
#pragma unroll
        for (int e = 0; e < N; ++e) {
          n[e] = out[t] * y[q][e];
#pragma unroll
          for (int s = 0; s < S; ++s) n[e] = fmaf(mix[s][t], v[q][s][e], n[e]);
          u[q][e] = fmaf(into[t], n[e], u[q][e]);
        }
        if (p.rows == nullptr) store_n<N>(x + static_cast<size_t>(t) * p.W + i, n);
      }
    }
  } else {
    const T *emb, *pair;
    mix_embedding(p, r, emb, pair);
    float all = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) all += into[s];
#pragma unroll
    for (int q = 0; q < R; ++q) {
      const int i = (q * blockDim.x + threadIdx.x) * N;
#pragma unroll
      for (int e = 0; e < N; ++e) u[q][e] = 0.f;
      if (i >= p.W) continue;
      float n[N], v[N];
      load_n<N>(emb + i, n);
      load_n<N>(pair + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        n[e] = fmaf(p.scale, n[e], v[e]);
        u[q][e] = all * n[e];
      }
      if (p.rows == nullptr)
#pragma unroll
        for (int s = 0; s < S; ++s) store_n<N>(x + static_cast<size_t>(s) * p.W + i, n);
    }
  }
  if (p.w == nullptr) return;
#pragma unroll
  for (int q = 0; q < R; ++q)
#pragma unroll
    for (int e = 0; e < N; ++e) sum += u[q][e];
  const float mean = block_sum_f(sum, red) / static_cast<float>(p.W);
  float ss = 0.f;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    if ((q * blockDim.x + threadIdx.x) * N >= p.W) continue;
#pragma unroll
    for (int e = 0; e < N; ++e) {
      u[q][e] -= mean;
      ss = fmaf(u[q][e], u[q][e], ss);
    }
  }
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  T* h = p.h + static_cast<size_t>(blockIdx.x) * p.W;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    float w[N], b[N];
    load_n<N>(p.w + i, w);
    load_n<N>(p.b + i, b);
#pragma unroll
    for (int e = 0; e < N; ++e) w[e] = fmaf(u[q][e] * inv, w[e], b[e]);
    store_n<N>(h + i, w);
  }
}

// Any width and up to kMaxStreams streams; the joined row passes through shared memory.
template <typename T>
__global__ void __launch_bounds__(256) stream_mix_any_kernel(const MixArgs<T> p) {
  extern __shared__ float srow[];           // [W]
  __shared__ float red[32];
  __shared__ float sc[kMaxStreams * (kMaxStreams + 2)];
  pdl_launch_dependents();
  pdl_wait();
  const int r = mix_row(p), S = p.S;
  float* x = p.x + static_cast<size_t>(r) * S * p.W;
  float* into = sc + S * S;
  float* out = into + S;
  const T *emb = nullptr, *pair = nullptr;
  if (p.y == nullptr) mix_embedding(p, r, emb, pair);
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) sc[i] = p.y != nullptr ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    into[i] = p.into[i];
    out[i] = p.y != nullptr ? p.out[i] : 0.f;
  }
  __syncthreads();
  float sum = 0.f;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
    float v[kMaxStreams], u = 0.f;
    const float y = p.y != nullptr ? load_f(p.y + static_cast<size_t>(r) * p.W + i) : fmaf(p.scale, load_f(emb + i), load_f(pair + i));
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) v[s] = s < S && p.y != nullptr ? x[static_cast<size_t>(s) * p.W + i] : 0.f;
    for (int t = 0; t < S; ++t) {
      float n = y;
      if (p.y != nullptr) {
        n *= out[t];
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s)
          if (s < S) n = fmaf(sc[s * S + t], v[s], n);
      }
      u = fmaf(into[t], n, u);
      if (p.rows == nullptr) x[static_cast<size_t>(t) * p.W + i] = n;
    }
    srow[i] = u;
    sum += u;
  }
  if (p.w == nullptr) return;
  const float mean = block_sum_f(sum, red) / static_cast<float>(p.W);
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
    const float u = srow[i] - mean;
    ss = fmaf(u, u, ss);
  }
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  T* h = p.h + static_cast<size_t>(blockIdx.x) * p.W;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) store_f(h + i, fmaf((srow[i] - mean) * inv, load_f(p.w + i), load_f(p.b + i)));
}

template <typename T, int S>
static int stream_mix_reg(int out_rows, const MixArgs<T>& p, cudaStream_t stream) {
  const int pieces = p.W <= 2048 ? 1 : 2, per = 8 * pieces;
  const int threads = ((p.W + per - 1) / per + 31) / 32 * 32;
  auto k = pieces == 1 ? stream_mix_reg_kernel<T, 8, 1, S> : stream_mix_reg_kernel<T, 8, 2, S>;
  return launch_kernel(k, dim3(out_rows), dim3(threads), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
}

template <typename T>
static int stream_mix(int out_rows, const MixArgs<T>& p, cudaStream_t stream) {
  if (p.S < 1 || p.S > kMaxStreams) return -1;
  if ((p.W & 7) == 0 && p.W <= 4096) {
    if (p.S == 1) return stream_mix_reg<T, 1>(out_rows, p, stream);
    if (p.S == 2) return stream_mix_reg<T, 2>(out_rows, p, stream);
    if (p.S == 3) return stream_mix_reg<T, 3>(out_rows, p, stream);
    if (p.S == 4) return stream_mix_reg<T, 4>(out_rows, p, stream);
  }
  const size_t smem = static_cast<size_t>(p.W) * 4;
  if (smem > 200 * 1024) return -1;
  auto k = stream_mix_any_kernel<T>;
  FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
  const int threads = p.W >= 256 ? 256 : (p.W + 31) / 32 * 32;
  return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
}

// y == null: the streams begin (ids, prev, embed, pairs given); else mix and out are.  w == null: no result.
extern "C" int forge_stream_mix(int fp32, float* x, const void* y, const float* mix, const float* out, const int* ids, const int* prev,
                                const void* embed, int vocab, float scale, const void* pairs, int buckets, long long mul_prev, long long mul_cur,
                                const float* into, const void* w, const void* b, void* h, const int* rows, int out_rows, int n_rows, int W, int S,
                                float eps, cudaStream_t stream) {
  if (out_rows <= 0) return 0;
  if (y == nullptr && (ids == nullptr || buckets < 1)) return -1;
#define FORGE_MIX(T)                                                                                                                          \
  return stream_mix<T>(out_rows, MixArgs<T>{x, static_cast<const T*>(y), mix, out, ids, prev, static_cast<const T*>(embed),                   \
                                            static_cast<const T*>(pairs), vocab, buckets, mul_prev, mul_cur, scale, into,                     \
                                            static_cast<const T*>(w), static_cast<const T*>(b), static_cast<T*>(h), rows, n_rows, W, S, eps}, stream)
  if (fp32) FORGE_MIX(float);
  FORGE_MIX(bf16);
#undef FORGE_MIX
}

}  // namespace forge
