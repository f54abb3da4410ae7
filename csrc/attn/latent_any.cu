// Latent attention, element types bf16 and fp32, any sizes.
//
//   latent_prepare    one pass over a token's [query latent | key/value latent | rotated key part]: both RMS norms, the
//                     rotation, and the store into the paged cache [blocks][block_size][kv_rank + rot].  Queries that do not come
//                     from a latent stand in its place and are passed over
//   latent_rotate_q   the rotated query parts of a range of tokens, next to the folded queries: row [kv_rank | rot] per head
//   latent_attend_any softmax attention of folded queries straight over the cached latents (scores against [c | k_rot],
//                     weighted sum of c): four heads per CTA share the key tile, one warp per head.  This is the path of
//                     fp32 models and of sizes the tensor-core kernels do not take, for prompts and single tokens alike.
//
// window: a token sees the last `window` tokens; 0: all.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T, int N>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const T* __restrict__ proj, long long ld, int q_rank, int kv_rank, int rot,
                                                             const T* __restrict__ qw, const T* __restrict__ kw, float eps,
                                                             const float* __restrict__ rope, int rope_rows,
                                                             const int* __restrict__ positions, const int* __restrict__ slots,
                                                             T* __restrict__ cq, T* __restrict__ cache, long long num_slots,
                                                             unsigned* status) {
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const T* row = proj + static_cast<size_t>(t) * ld;
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x * N; qw != nullptr && i < q_rank; i += blockDim.x * N) {
    float v[N];
    load_n<N>(row + i, v);
#pragma unroll
    for (int e = 0; e < N; ++e) ssq += v[e] * v[e];
  }
  for (int i = threadIdx.x * N; i < kv_rank; i += blockDim.x * N) {
    float v[N];
    load_n<N>(row + q_rank + i, v);
#pragma unroll
    for (int e = 0; e < N; ++e) ssk += v[e] * v[e];
  }
  ssq = warp_sum_f(ssq);
  ssk = warp_sum_f(ssk);
  if ((threadIdx.x & 31) == 0) {
    red[threadIdx.x >> 5] = ssq;
    red[4 + (threadIdx.x >> 5)] = ssk;
  }
  __syncthreads();                                 // four warps
  const float inv_q = rsqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(q_rank) + eps);
  const float inv_k = rsqrtf((red[4] + red[5] + red[6] + red[7]) / static_cast<float>(kv_rank) + eps);
  T* q_out = cq + static_cast<size_t>(t) * q_rank;
  for (int i = threadIdx.x * N; qw != nullptr && i < q_rank; i += blockDim.x * N) {
    float v[N], w[N];
    load_n<N>(row + i, v);
    load_n<N>(qw + i, w);
#pragma unroll
    for (int e = 0; e < N; ++e) v[e] *= inv_q * w[e];
    store_n<N>(q_out + i, v);
  }
  const long long slot = slots[t];
  if (slot < 0) return;
  if (slot >= num_slots) {
    if (threadIdx.x == 0) set_status(status, kStatusBadIndex);
    return;
  }
  T* dst = cache + static_cast<size_t>(slot) * (kv_rank + rot);
  for (int i = threadIdx.x * N; i < kv_rank; i += blockDim.x * N) {
    float v[N], w[N];
    load_n<N>(row + q_rank + i, v);
    load_n<N>(kw + i, w);
#pragma unroll
    for (int e = 0; e < N; ++e) v[e] *= inv_k * w[e];
    store_n<N>(dst + i, v);
  }
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= rope_rows ? rope_rows - 1 : pos);
  const float* cs = rope + static_cast<size_t>(pos) * rot;
  const int half = rot / 2;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float u = load_f(row + q_rank + kv_rank + i), v = load_f(row + q_rank + kv_rank + half + i);
    const float c = cs[i], s = cs[half + i];
    store_f(dst + kv_rank + i, u * c - v * s);
    store_f(dst + kv_rank + half + i, v * c + u * s);
  }
}

template <typename T>
static int latent_prepare(const void* proj, long long ld, int T_, int q_rank, int kv_rank, int rot, const void* qw, const void* kw, float eps,
                          const float* rope, int rope_rows, const int* positions, const int* slots, void* cq, void* cache,
                          long long num_slots, unsigned* status, cudaStream_t stream) {
  const bool v4 = ((q_rank | kv_rank | rot | static_cast<int>(ld & 3)) & 3) == 0;
  auto k = v4 ? latent_prepare_kernel<T, 4> : latent_prepare_kernel<T, 1>;
  return launch_kernel(k, dim3(T_), dim3(128), 0, stream, 0, static_cast<const T*>(proj), ld, q_rank, kv_rank, rot, static_cast<const T*>(qw),
                       static_cast<const T*>(kw), eps, rope, rope_rows, positions, slots, static_cast<T*>(cq), static_cast<T*>(cache),
                       num_slots, status) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_latent_prepare(int fp32, const void* proj, long long ld, int T_, int q_rank, int kv_rank, int rot, const void* qw, const void* kw,
                                    float eps, const float* rope, int rope_rows, const int* positions, const int* slots, void* cq,
                                    void* cache, long long num_slots, unsigned* status, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  return fp32 ? latent_prepare<float>(proj, ld, T_, q_rank, kv_rank, rot, qw, kw, eps, rope, rope_rows, positions, slots, cq, cache, num_slots, status, stream)
              : latent_prepare<bf16>(proj, ld, T_, q_rank, kv_rank, rot, qw, kw, eps, rope, rope_rows, positions, slots, cq, cache, num_slots, status, stream);
}

// q [tokens][heads][dim + rot], tokens ld elements apart -> qa [tokens][heads][kv_rank + rot], last `rot` entries of every head rotated.
template <typename T>
__global__ void __launch_bounds__(128) latent_rotate_q_kernel(const T* __restrict__ q, long long ld, T* __restrict__ qa, int heads, int dim, int rot,
                                                              int kv_rank, const float* __restrict__ rope, int rope_rows,
                                                              const int* __restrict__ positions) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, half = rot / 2;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= rope_rows ? rope_rows - 1 : pos);
  const float* cs = rope + static_cast<size_t>(pos) * rot;
  for (int i = threadIdx.x; i < heads * half; i += blockDim.x) {
    const int h = i / half, j = i % half;
    const T* src = q + static_cast<size_t>(t) * ld + static_cast<size_t>(h) * (dim + rot) + dim;
    T* dst = qa + (static_cast<size_t>(t) * heads + h) * (kv_rank + rot) + kv_rank;
    const float u = load_f(src + j), v = load_f(src + half + j), c = cs[j], s = cs[half + j];
    store_f(dst + j, u * c - v * s);
    store_f(dst + half + j, v * c + u * s);
  }
}

extern "C" int forge_latent_rotate_q(int fp32, const void* q, long long ld, void* qa, int tokens, int heads, int dim, int rot, int kv_rank,
                                     const float* rope, int rope_rows, const int* positions, cudaStream_t stream) {
  if (tokens <= 0 || rot <= 0) return 0;
  if (fp32)
    return launch_kernel(latent_rotate_q_kernel<float>, dim3(tokens), dim3(128), 0, stream, 0, static_cast<const float*>(q), ld,
                         static_cast<float*>(qa), heads, dim, rot, kv_rank, rope, rope_rows, positions) == cudaSuccess ? 0 : -2;
  return launch_kernel(latent_rotate_q_kernel<bf16>, dim3(tokens), dim3(128), 0, stream, 0, static_cast<const bf16*>(q), ld,
                       static_cast<bf16*>(qa), heads, dim, rot, kv_rank, rope, rope_rows, positions) == cudaSuccess ? 0 : -2;
}

// Which sequence token t of the step belongs to: cu[s] <= t < cu[s + 1]; -1 for the padding of a graph bucket.
__device__ __forceinline__ int sequence_of(const int* cu, int num_seqs, int t) {
  if (t >= cu[num_seqs]) return -1;
  int lo = 0, hi = num_seqs;                 // cu[lo] <= t < cu[hi]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid;
  }
  return lo;
}

constexpr int kLKeys = 32;          // keys per tile
constexpr int kLHeads = 4;          // heads (= warps) per CTA
constexpr int kLRegs = 32;          // latent entries per lane: kv_rank <= 1024

// qa [tokens][heads][D], D = kv_rank + rot; o [tokens][heads][kv_rank]; token i of both is token tok0 + i of the step.
template <typename T>
__global__ void __launch_bounds__(32 * kLHeads) latent_attend_any_kernel(const T* __restrict__ qa, const T* __restrict__ cache,
                                                                         T* __restrict__ o, int tok0, const int* __restrict__ cu,
                                                                         int num_seqs, const int* __restrict__ positions,
                                                                         const int* __restrict__ block_tables, int table_width,
                                                                         int num_blocks, int block_size, int heads, int kv_rank, int rot,
                                                                         int window, float scale, unsigned* status) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int D = kv_rank + rot, pitch = D | 1;
  float* sq = sm;                              // [kLHeads][D]
  float* skv = sm + kLHeads * D;               // [kLKeys][pitch]
  const int i = blockIdx.x, t = tok0 + i;
  const int seq = sequence_of(cu, num_seqs, t);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * kLHeads + warp;
  T* out = o + (static_cast<size_t>(i) * heads + h) * kv_rank;
  if (seq < 0) {                               // padding: defined values for whoever multiplies them
    if (h < heads)
      for (int d = lane; d < kv_rank; d += 32) store_f(out + d, 0.f);
    return;
  }
  const int n = positions[t] + 1, lo = window > 0 ? max(n - window, 0) : 0;          // visible keys: [lo, n)
  for (int d = lane; d < D; d += 32)
    sq[warp * D + d] = h < heads ? load_f(qa + (static_cast<size_t>(i) * heads + h) * D + d) * scale : 0.f;
  float acc[kLRegs];
#pragma unroll
  for (int j = 0; j < kLRegs; ++j) acc[j] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = lo; k0 < n; k0 += kLKeys) {
    __syncthreads();
    const int keys = min(kLKeys, n - k0);
    for (int kk = warp; kk < keys; kk += kLHeads) {
      const int key = k0 + kk;
      int blk = block_tables[static_cast<size_t>(seq) * table_width + min(key / block_size, table_width - 1)];
      if (blk < 0 || blk >= num_blocks) {
        if (lane == 0) set_status(status, kStatusBadIndex);
        blk = 0;
      }
      const T* src = cache + (static_cast<size_t>(blk) * block_size + key % block_size) * D;
      for (int d = lane; d < D; d += 32) skv[kk * pitch + d] = load_f(src + d);
    }
    __syncthreads();
    float s = -INFINITY;
    if (lane < keys) {
      s = 0.f;
      const float* kr = skv + lane * pitch;
      const float* qr = sq + warp * D;
      for (int d = 0; d < D; ++d) s = fmaf(qr[d], kr[d], s);
    }
    float mx = s;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    const float m_new = fmaxf(m, mx);
    const float alpha = expf(m - m_new), p = lane < keys ? expf(s - m_new) : 0.f;
    l = l * alpha + warp_sum_f(p);
    m = m_new;
#pragma unroll
    for (int j = 0; j < kLRegs; ++j) acc[j] *= alpha;
    for (int kk = 0; kk < keys; ++kk) {
      const float pk = __shfl_sync(0xffffffffu, p, kk);
      const float* vr = skv + kk * pitch + lane;
#pragma unroll
      for (int j = 0; j < kLRegs; ++j)
        if (j * 32 + lane < kv_rank) acc[j] = fmaf(pk, vr[j * 32], acc[j]);
    }
  }
  if (h >= heads) return;
  const float inv = 1.f / l;
#pragma unroll
  for (int j = 0; j < kLRegs; ++j)
    if (j * 32 + lane < kv_rank) store_f(out + j * 32 + lane, acc[j] * inv);
}

template <typename T>
static int latent_attend_any(const void* qa, const void* cache, void* o, int tok0, int tokens, const int* cu, int num_seqs,
                             const int* positions, const int* block_tables, int table_width, int num_blocks, int block_size, int heads,
                             int kv_rank, int rot, int window, float scale, unsigned* status, cudaStream_t stream) {
  const int D = kv_rank + rot;
  const size_t smem = (static_cast<size_t>(kLHeads) * D + static_cast<size_t>(kLKeys) * (D | 1)) * 4;
  if (kv_rank > 32 * kLRegs || smem > 220 * 1024) return -1;
  auto k = latent_attend_any_kernel<T>;
  FORGE_ENSURE_DYN_SMEM(k, 220 * 1024);
  return launch_kernel(k, dim3(tokens, (heads + kLHeads - 1) / kLHeads), dim3(32 * kLHeads), smem, stream, 0, static_cast<const T*>(qa),
                       static_cast<const T*>(cache), static_cast<T*>(o), tok0, cu, num_seqs, positions, block_tables, table_width,
                       num_blocks, block_size, heads, kv_rank, rot, window, scale, status) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_latent_attend_any(int fp32, const void* qa, const void* cache, void* o, int tok0, int tokens, const int* cu,
                                       int num_seqs, const int* positions, const int* block_tables, int table_width, int num_blocks,
                                       int block_size, int heads, int kv_rank, int rot, int window, float scale, unsigned* status,
                                       cudaStream_t stream) {
  if (tokens <= 0) return 0;
  return fp32 ? latent_attend_any<float>(qa, cache, o, tok0, tokens, cu, num_seqs, positions, block_tables, table_width, num_blocks, block_size, heads, kv_rank, rot, window, scale, status, stream)
              : latent_attend_any<bf16>(qa, cache, o, tok0, tokens, cu, num_seqs, positions, block_tables, table_width, num_blocks, block_size, heads, kv_rank, rot, window, scale, status, stream);
}

}  // namespace forge
