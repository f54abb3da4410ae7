// The fp32 residual stream between two layers of a decoder with parallel branches, in one pass over a row:
//
//   x += a + b                    both branches of the layer before (b dense, or the sum of a token's expert outputs)
//   x += embed[id], x += vec      ahead of a pass of a looped range of layers (and at the start, where x begins at zero)
//   h_i = rms_norm(x) * w_i       the norms of the layer after (they share the row's mean square)
//
// A decoder that norms a sublayer's result on its way out uses stream_sandwich instead:
//
//   x += mult * rms_norm(y) * (offset + post),   y = a + bias, or the weighted sum of a token's expert outputs
//   h  = rms_norm(x) * (offset + w)              norm weights stored around `offset`
//
// One CTA per row; the row stays in shared memory between the two halves.  With `rows` only those rows are normed and x is
// left as it was (the last norm of a step: only rows whose logits are wanted).
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct StreamArgs {
  float* x;
  const T* a;
  const T* b;
  const int* b_rows;     // null: b is [rows][W]; else b is indexed by b_rows[row * top + j], j < top
  int top;
  const int* ids;
  const T* embed;
  int vocab;
  const T* vec;
  const T* w1;
  const T* w2;
  T* h1;
  T* h2;
  const int* rows;
  int n_rows, W, start;
  float eps;
};

template <typename T, int N>
__global__ void __launch_bounds__(256) stream_update_kernel(const StreamArgs<T> p) {
  extern __shared__ float srow[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  int r = blockIdx.x;
  if (p.rows != nullptr) {
    r = p.rows[r];
    r = r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
  }
  const size_t base = static_cast<size_t>(r) * p.W;
  const T* emb = nullptr;
  if (p.ids != nullptr) {
    int id = p.ids[r];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    emb = p.embed + static_cast<size_t>(id) * p.W;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * N; i < p.W; i += blockDim.x * N) {
    float s[N], v[N];
    if (p.start) {
#pragma unroll
      for (int e = 0; e < N; ++e) s[e] = 0.f;
    } else {
      load_n<N>(p.x + base + i, s);
    }
    if (p.a != nullptr) {
      load_n<N>(p.a + base + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) s[e] += v[e];
    }
    if (p.b != nullptr) {
      if (p.b_rows == nullptr) {
        load_n<N>(p.b + base + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) s[e] += v[e];
      } else {
        for (int j = 0; j < p.top; ++j) {
          load_n<N>(p.b + static_cast<size_t>(p.b_rows[static_cast<size_t>(r) * p.top + j]) * p.W + i, v);
#pragma unroll
          for (int e = 0; e < N; ++e) s[e] += v[e];
        }
      }
    }
    if (emb != nullptr) {
      load_n<N>(emb + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) s[e] += v[e];
    }
    if (p.vec != nullptr) {
      load_n<N>(p.vec + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) s[e] += v[e];
    }
    if (p.rows == nullptr) store_n<N>(p.x + base + i, s);
#pragma unroll
    for (int e = 0; e < N; ++e) ss += s[e] * s[e];
    store_n<N>(srow + i, s);
  }
  if (p.w1 == nullptr) return;
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  const size_t out = static_cast<size_t>(blockIdx.x) * p.W;
  for (int i = threadIdx.x * N; i < p.W; i += blockDim.x * N) {
    float s[N], w[N], y[N];
    load_n<N>(srow + i, s);
    load_n<N>(p.w1 + i, w);
#pragma unroll
    for (int e = 0; e < N; ++e) {
      s[e] *= inv;
      y[e] = s[e] * w[e];
    }
    store_n<N>(p.h1 + out + i, y);
    if (p.w2 != nullptr) {
      load_n<N>(p.w2 + i, w);
#pragma unroll
      for (int e = 0; e < N; ++e) y[e] = s[e] * w[e];
      store_n<N>(p.h2 + out + i, y);
    }
  }
}

template <typename T>
struct SandwichArgs {
  float* x;
  const T* a;               // null: nothing to add (the embedding starts the stream)
  const int* a_rows;        // null: a is [rows][W]; else a row's result is sum_j a_weights[row, j] a[a_rows[row, j]]
  const float* a_weights;   // null: all 1
  int top;
  const float* a_bias;
  const T* post;            // null: a is added as it is
  float mult, offset;
  const int* ids;
  const T* embed;
  int vocab;
  const T* w;
  T* h;
  const int* rows;
  int n_rows, W, start;
  float eps;
};

template <typename T, int N>
__global__ void __launch_bounds__(256) stream_sandwich_kernel(const SandwichArgs<T> p) {
  extern __shared__ float srow[];           // [2][W]: the sublayer's result, then the new row; the row before
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  float* sx = srow + p.W;
  int r = blockIdx.x;
  if (p.rows != nullptr) {
    r = p.rows[r];
    r = r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
  }
  const size_t base = static_cast<size_t>(r) * p.W;
  const T* emb = nullptr;
  if (p.ids != nullptr) {
    int id = p.ids[r];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    emb = p.embed + static_cast<size_t>(id) * p.W;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * N; i < p.W; i += blockDim.x * N) {
    float y[N], v[N];
#pragma unroll
    for (int e = 0; e < N; ++e) y[e] = 0.f;
    if (p.a != nullptr) {
      if (p.a_rows == nullptr) {
        load_n<N>(p.a + base + i, y);
      } else {
        for (int j = 0; j < p.top; ++j) {
          const size_t at = static_cast<size_t>(r) * p.top + j;
          const float s = p.a_weights != nullptr ? p.a_weights[at] : 1.f;
          load_n<N>(p.a + static_cast<size_t>(p.a_rows[at]) * p.W + i, v);
#pragma unroll
          for (int e = 0; e < N; ++e) y[e] = fmaf(s, v[e], y[e]);
        }
      }
      if (p.a_bias != nullptr) {
        load_n<N>(p.a_bias + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) y[e] += v[e];
      }
    }
    if (p.start) {
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] = 0.f;
    } else {
      load_n<N>(p.x + base + i, v);
    }
    if (emb != nullptr) {
      float m[N];
      load_n<N>(emb + i, m);
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] += m[e];
    }
    store_n<N>(sx + i, v);
    store_n<N>(srow + i, y);
#pragma unroll
    for (int e = 0; e < N; ++e) ss += y[e] * y[e];
  }
  float f = 1.f;                                        // block-uniform choices below
  if (p.a != nullptr && p.post != nullptr) f = p.mult * rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  ss = 0.f;
  for (int i = threadIdx.x * N; i < p.W; i += blockDim.x * N) {
    float y[N], v[N], g[N];
    load_n<N>(srow + i, y);
    load_n<N>(sx + i, v);
#pragma unroll
    for (int e = 0; e < N; ++e) g[e] = 1.f;
    if (p.post != nullptr) {
      load_n<N>(p.post + i, g);
#pragma unroll
      for (int e = 0; e < N; ++e) g[e] += p.offset;
    }
#pragma unroll
    for (int e = 0; e < N; ++e) {
      v[e] = fmaf(f * y[e], g[e], v[e]);
      ss += v[e] * v[e];
    }
    if (p.rows == nullptr) store_n<N>(p.x + base + i, v);
    store_n<N>(srow + i, v);
  }
  if (p.w == nullptr) return;
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  const size_t out = static_cast<size_t>(blockIdx.x) * p.W;
  for (int i = threadIdx.x * N; i < p.W; i += blockDim.x * N) {
    float v[N], g[N];
    load_n<N>(srow + i, v);
    load_n<N>(p.w + i, g);
#pragma unroll
    for (int e = 0; e < N; ++e) v[e] *= inv * (g[e] + p.offset);
    store_n<N>(p.h + out + i, v);
  }
}

// The same for rows that fit the registers of a CTA: R pieces of N entries per thread, no pass through shared memory.
template <typename T, int N, int R>
__global__ void __launch_bounds__(256) stream_sandwich_reg_kernel(const SandwichArgs<T> p) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  int r = blockIdx.x;
  if (p.rows != nullptr) {
    r = p.rows[r];
    r = r < 0 ? 0 : (r >= p.n_rows ? p.n_rows - 1 : r);
  }
  const size_t base = static_cast<size_t>(r) * p.W;
  const T* emb = nullptr;
  if (p.ids != nullptr) {
    int id = p.ids[r];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    emb = p.embed + static_cast<size_t>(id) * p.W;
  }
  float x[R][N], y[R][N], ss = 0.f;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
#pragma unroll
    for (int e = 0; e < N; ++e) x[q][e] = y[q][e] = 0.f;
    if (i >= p.W) continue;
    if (!p.start) load_n<N>(p.x + base + i, x[q]);
    if (p.a != nullptr && p.a_rows == nullptr) load_n<N>(p.a + base + i, y[q]);
  }
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    float v[N];
    if (p.a != nullptr && p.a_rows != nullptr) {
#pragma unroll 4
      for (int j = 0; j < p.top; ++j) {
        const size_t at = static_cast<size_t>(r) * p.top + j;
        const float s = p.a_weights != nullptr ? p.a_weights[at] : 1.f;
        load_n<N>(p.a + static_cast<size_t>(p.a_rows[at]) * p.W + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) y[q][e] = fmaf(s, v[e], y[q][e]);
      }
    }
    if (p.a_bias != nullptr) {
      load_n<N>(p.a_bias + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) y[q][e] += v[e];
    }
    if (emb != nullptr) {
      load_n<N>(emb + i, v);
#pragma unroll
      for (int e = 0; e < N; ++e) x[q][e] += v[e];
    }
#pragma unroll
    for (int e = 0; e < N; ++e) ss += y[q][e] * y[q][e];
  }
  float f = 1.f;
  if (p.a != nullptr && p.post != nullptr) f = p.mult * rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  ss = 0.f;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    float g[N];
#pragma unroll
    for (int e = 0; e < N; ++e) g[e] = 1.f;
    if (p.post != nullptr) {
      load_n<N>(p.post + i, g);
#pragma unroll
      for (int e = 0; e < N; ++e) g[e] += p.offset;
    }
#pragma unroll
    for (int e = 0; e < N; ++e) {
      x[q][e] = fmaf(f * y[q][e], g[e], x[q][e]);
      ss += x[q][e] * x[q][e];
    }
    if (p.rows == nullptr) store_n<N>(p.x + base + i, x[q]);
  }
  if (p.w == nullptr) return;
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.W) + p.eps);
  const size_t out = static_cast<size_t>(blockIdx.x) * p.W;
#pragma unroll
  for (int q = 0; q < R; ++q) {
    const int i = (q * blockDim.x + threadIdx.x) * N;
    if (i >= p.W) continue;
    float g[N];
    load_n<N>(p.w + i, g);
#pragma unroll
    for (int e = 0; e < N; ++e) g[e] = x[q][e] * inv * (g[e] + p.offset);
    store_n<N>(p.h + out + i, g);
  }
}

template <typename T>
static int stream_sandwich(int out_rows, const SandwichArgs<T>& p, cudaStream_t stream) {
  if ((p.W & 7) == 0 && p.W <= 4096) {
    const int pieces = p.W <= 2048 ? 1 : 2, per = 8 * pieces;
    const int threads = ((p.W + per - 1) / per + 31) / 32 * 32;
    auto k = pieces == 1 ? stream_sandwich_reg_kernel<T, 8, 1> : stream_sandwich_reg_kernel<T, 8, 2>;
    return launch_kernel(k, dim3(out_rows), dim3(threads), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
  }
  const size_t smem = static_cast<size_t>(p.W) * 8;
  if (smem > 200 * 1024) return -1;
  const bool v4 = (p.W & 3) == 0;
  int threads = ((p.W / (v4 ? 4 : 1) + 31) / 32) * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  if (v4) {
    auto k = stream_sandwich_kernel<T, 4>;
    FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
    return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
  }
  auto k = stream_sandwich_kernel<T, 1>;
  FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
  return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_stream_sandwich(int fp32, float* x, const void* a, const int* a_rows, const float* a_weights, int top, const float* a_bias,
                                     const void* post, float mult, float offset, const int* ids, const void* embed, int vocab, const void* w,
                                     void* h, const int* rows, int out_rows, int n_rows, int W, int start, float eps, cudaStream_t stream) {
  if (out_rows <= 0) return 0;
#define FORGE_SANDWICH(T)                                                                                                              \
  return stream_sandwich<T>(out_rows, SandwichArgs<T>{x, static_cast<const T*>(a), a_rows, a_weights, top, a_bias,                     \
                                                      static_cast<const T*>(post), mult, offset, ids, static_cast<const T*>(embed), vocab, \
                                                      static_cast<const T*>(w), static_cast<T*>(h), rows, n_rows, W, start, eps}, stream)
  if (fp32) FORGE_SANDWICH(float);
  FORGE_SANDWICH(bf16);
#undef FORGE_SANDWICH
}

template <typename T>
static int stream_update(int out_rows, const StreamArgs<T>& p, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(p.W) * 4;
  if (smem > 200 * 1024) return -1;
  const bool v4 = (p.W & 3) == 0;
  int threads = ((p.W / (v4 ? 4 : 1) + 31) / 32) * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  if (v4) {
    auto k = stream_update_kernel<T, 4>;
    FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
    return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
  }
  auto k = stream_update_kernel<T, 1>;
  FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
  return launch_kernel(k, dim3(out_rows), dim3(threads), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_stream_update(int fp32, float* x, const void* a, const void* b, const int* b_rows, int top, const int* ids,
                                   const void* embed, int vocab, const void* vec, const void* w1, const void* w2, void* h1, void* h2,
                                   const int* rows, int out_rows, int n_rows, int W, int start, float eps, cudaStream_t stream) {
  if (out_rows <= 0) return 0;
  if (fp32) {
    using T = float;
    const StreamArgs<T> p = {x, static_cast<const T*>(a), static_cast<const T*>(b), b_rows, top, ids, static_cast<const T*>(embed), vocab,
                             static_cast<const T*>(vec), static_cast<const T*>(w1), static_cast<const T*>(w2), static_cast<T*>(h1),
                             static_cast<T*>(h2), rows, n_rows, W, start, eps};
    return stream_update<T>(out_rows, p, stream);
  }
  using T = bf16;
  const StreamArgs<T> p = {x, static_cast<const T*>(a), static_cast<const T*>(b), b_rows, top, ids, static_cast<const T*>(embed), vocab,
                           static_cast<const T*>(vec), static_cast<const T*>(w1), static_cast<const T*>(w2), static_cast<T*>(h1),
                           static_cast<T*>(h2), rows, n_rows, W, start, eps};
  return stream_update<T>(out_rows, p, stream);
}

// x <- act(x) elementwise (PlainAct), bf16 or fp32; logits <- cap tanh(scale logits / cap).
template <typename T, int N>
__global__ void __launch_bounds__(256) act_any_kernel(T* __restrict__ x, long long n, int act, bool logits, float scale, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  const long long step = static_cast<long long>(gridDim.x) * blockDim.x * N;
  for (long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * N; i < n; i += step) {
    float v[N];
    load_n<N>(x + i, v);
#pragma unroll
    for (int e = 0; e < N; ++e) v[e] = logits ? bound_logit<sizeof(T) == 4>(v[e], scale, cap) : plain_act<sizeof(T) == 4>(act, v[e]);
    store_n<N>(x + i, v);
  }
}

template <typename T>
static int act_any(T* x, long long n, int act, int logits, float scale, float cap, cudaStream_t stream) {
  const bool wide = n % 8 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0;
  long long grid = (n / (wide ? 8 : 1) + 255) / 256;
  if (grid > device_sm_count() * 16) grid = device_sm_count() * 16;
  auto k = wide ? act_any_kernel<T, 8> : act_any_kernel<T, 1>;
  return launch_kernel(k, dim3(static_cast<unsigned>(grid)), dim3(256), 0, stream, 0, x, n, act, logits != 0, scale, cap) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_act_any(int fp32, void* x, long long n, int act, int logits, float scale, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  return fp32 ? act_any(static_cast<float*>(x), n, act, logits, scale, cap, stream) : act_any(static_cast<bf16*>(x), n, act, logits, scale, cap, stream);
}

// out[r, :I] = act(x[r, :I], x[r, I:2I]) (GateAct), any I, bf16 or fp32 (the fused epilogue of the tcgen05 GEMMs needs no such pass).
template <typename T>
__global__ void __launch_bounds__(256) act_mul_any_kernel(const T* __restrict__ x, T* __restrict__ out, long long rows, int I, int act,
                                                          float limit) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long idx = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; idx < rows * I;
       idx += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = idx / I;
    const int c = static_cast<int>(idx % I);
    store_f(out + idx, gated_act<sizeof(T) == 4>(act, limit, load_f(x + r * 2 * I + c), load_f(x + r * 2 * I + I + c)));
  }
}

extern "C" int forge_act_mul_any(int fp32, const void* x, void* out, long long rows, int I, int act, float limit, cudaStream_t stream) {
  if (rows <= 0) return 0;
  long long grid = (rows * I + 255) / 256;
  if (grid > device_sm_count() * 16) grid = device_sm_count() * 16;
  const dim3 g(static_cast<unsigned>(grid));
  if (fp32)
    return launch_kernel(act_mul_any_kernel<float>, g, dim3(256), 0, stream, 0, static_cast<const float*>(x), static_cast<float*>(out), rows, I, act, limit) == cudaSuccess ? 0 : -2;
  return launch_kernel(act_mul_any_kernel<bf16>, g, dim3(256), 0, stream, 0, static_cast<const bf16*>(x), static_cast<bf16*>(out), rows, I, act, limit) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
