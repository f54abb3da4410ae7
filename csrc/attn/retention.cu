// Retention: S <- decay_h S + k v^T, o = S^T q per head, with the state S [dim][vdim] in fp32, one per sequence and head.
// q, k, v and the output gate come packed from one projection, row [heads x dim | heads x dim | heads x vdim | heads x vdim].
// The rotation of q and k (first rd entries of a head, entry i with i + rd / 2) is done where they are read, and k carries
// the factor dim^-1/2.  A sequence's first token (position 0) starts from S = 0, so a state slot needs no clearing.
//
//   retention_decode   one token of many sequences: the state is read, updated and written once; the head's output is
//                      normed (no weight), gated and stored in the same kernel
//   retention_scan     a run of tokens per sequence, token by token, any sizes, bf16 or fp32 operands
//   retention_gate     o / rms(o) * silu(gate) for the outputs of the prompt kernels
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct RetentionIn {
  const T* qkvg;          // [tokens][ld]
  int ld;
  const float* decay;     // [heads]
  float* state;           // [slots][heads][dk][dv]
  const int* slots;       // [sequences]
  const int* positions;   // [tokens]
  const float* rope;      // [rope_rows][rd]
  int rope_rows, rd, heads, dk, dv, num_slots;
  unsigned* status;
};

// Entry i of a head's q or k after rotation; `cs` is the token's row of the table.
template <typename T>
__device__ __forceinline__ float rotated(const T* v, int i, const float* cs, int rd) {
  const float x = load_f(v + i);
  const int half = rd >> 1;
  if (i < half) return x * cs[i] - load_f(v + i + half) * cs[half + i];
  if (i < rd) return x * cs[i - half] + load_f(v + i - half) * cs[i];
  return x;
}

template <typename T>
__device__ __forceinline__ const float* rope_row(const RetentionIn<T>& p, int t) {
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.rope_rows ? p.rope_rows - 1 : pos);
  return p.rope + static_cast<size_t>(pos) * p.rd;
}

// CTA = (head, sequence).  A thread owns N columns of the state and every `groups`-th row.
template <typename T, int N>
__global__ void __launch_bounds__(256) retention_decode_kernel(const RetentionIn<T> p, T* __restrict__ y, float eps) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y, t = s;
  const int slot = p.slots[s];
  T* out = y + (static_cast<size_t>(t) * p.heads + h) * p.dv;
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    for (int c = threadIdx.x; c < p.dv; c += blockDim.x) store_f(out + c, 0.f);
    return;
  }
  const int cols = (p.dv + N - 1) / N;                                  // column groups
  const int groups = cols < static_cast<int>(blockDim.x) ? static_cast<int>(blockDim.x) / cols : 1;
  float* sq = sm;                       // [dk]
  float* sk = sm + p.dk;                // [dk]
  float* so = sk + p.dk;                // [groups][dv], then the sum in row 0
  const T* row = p.qkvg + static_cast<size_t>(t) * p.ld;
  const float* cs = rope_row(p, t);
  const float ks = rsqrtf(static_cast<float>(p.dk));
  for (int i = threadIdx.x; i < p.dk; i += blockDim.x) {
    sq[i] = rotated(row + h * p.dk, i, cs, p.rd);
    sk[i] = rotated(row + (p.heads + h) * p.dk, i, cs, p.rd) * ks;
  }
  __syncthreads();
  const T* v = row + 2 * p.heads * p.dk + h * p.dv;
  float* S = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dk * p.dv;
  const float g = p.decay[h];
  const bool fresh = p.positions[t] == 0;
  const int grp = threadIdx.x / cols < groups ? threadIdx.x / cols : groups;   // threads past the last whole group idle
  for (int c0 = cols < static_cast<int>(blockDim.x) ? threadIdx.x % cols : threadIdx.x; grp < groups && c0 < cols;
       c0 += cols < static_cast<int>(blockDim.x) ? cols : blockDim.x) {
    const int c = c0 * N;
    float vv[N], acc[N];
    load_n<N>(v + c, vv);
#pragma unroll
    for (int e = 0; e < N; ++e) acc[e] = 0.f;
#pragma unroll 8
    for (int i = grp; i < p.dk; i += groups) {
      float* sp = S + static_cast<size_t>(i) * p.dv + c;
      float st[N];
      if (fresh) {
#pragma unroll
        for (int e = 0; e < N; ++e) st[e] = 0.f;
      } else {
        load_n<N>(sp, st);
      }
      const float ki = sk[i], qi = sq[i];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        st[e] = fmaf(g, st[e], ki * vv[e]);
        acc[e] = fmaf(st[e], qi, acc[e]);
      }
      store_n<N>(sp, st);
    }
#pragma unroll
    for (int e = 0; e < N; ++e) so[grp * p.dv + c + e] = acc[e];
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.dv; c += blockDim.x) {
    float o = 0.f;
    for (int r = 0; r < groups; ++r) o += so[r * p.dv + c];
    so[c] = o;
    ss += o * o;
  }
  const float inv = rsqrtf(block_sum_f(ss, red) / static_cast<float>(p.dv) + eps);
  const T* gate = v + p.heads * p.dv;
  for (int c = threadIdx.x; c < p.dv; c += blockDim.x) store_f(out + c, so[c] * inv * silu_t<T>(load_f(gate + c)));
}

// CTA = (32 columns of the state, head, sequence); eight adjacent lanes share a column and own every eighth row of it.
constexpr int kRScanCols = 32, kRScanTok = 16;

template <typename T, int R>
__global__ void __launch_bounds__(256) retention_scan_kernel(const RetentionIn<T> p, const int* __restrict__ cu, float* __restrict__ o) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, s = blockIdx.z, c0 = blockIdx.x * kRScanCols;
  const int t_begin = cu[s], t_end = cu[s + 1];
  if (t_begin >= t_end) return;
  const int slot = p.slots[s];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    return;
  }
  float* sq = sm;                                  // [kRScanTok][dk]
  float* sk = sq + kRScanTok * p.dk;
  float* sv = sk + kRScanTok * p.dk;               // [kRScanTok][kRScanCols]
  const int grp = threadIdx.x & 7, col = threadIdx.x >> 3;
  const bool live = c0 + col < p.dv;
  float* S = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dk * p.dv + c0 + col;
  const bool fresh = p.positions[t_begin] == 0;
  const float g = p.decay[h], ks = rsqrtf(static_cast<float>(p.dk));
  float st[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * 8 + grp;
    st[j] = (live && !fresh && i < p.dk) ? S[static_cast<size_t>(i) * p.dv] : 0.f;
  }
  for (int t0 = t_begin; t0 < t_end; t0 += kRScanTok) {
    const int n = min(kRScanTok, t_end - t0);
    __syncthreads();
    for (int idx = threadIdx.x; idx < n * p.dk; idx += blockDim.x) {
      const int tt = idx / p.dk, i = idx % p.dk;
      const T* row = p.qkvg + static_cast<size_t>(t0 + tt) * p.ld;
      const float* cs = rope_row(p, t0 + tt);
      sq[idx] = rotated(row + h * p.dk, i, cs, p.rd);
      sk[idx] = rotated(row + (p.heads + h) * p.dk, i, cs, p.rd) * ks;
    }
    for (int idx = threadIdx.x; idx < n * kRScanCols; idx += blockDim.x) {
      const int tt = idx / kRScanCols, c = idx % kRScanCols;
      sv[idx] = c0 + c < p.dv ? load_f(p.qkvg + static_cast<size_t>(t0 + tt) * p.ld + 2 * p.heads * p.dk + h * p.dv + c0 + c) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      const float v = sv[tt * kRScanCols + col];
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < R; ++j) {
        const int i = j * 8 + grp;
        if (i < p.dk) {
          st[j] = fmaf(g, st[j], sk[tt * p.dk + i] * v);
          acc = fmaf(st[j], sq[tt * p.dk + i], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (grp == 0 && live) o[(static_cast<size_t>(t0 + tt) * p.heads + h) * p.dv + c0 + col] = acc;
    }
  }
  if (!live) return;
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * 8 + grp;
    if (i < p.dk) S[static_cast<size_t>(i) * p.dv] = st[j];
  }
}

// y = o / rms(o over the head) * silu(gate); one warp per (token, head).  o fp32 [tokens][heads][dv], tokens from tok0 on.
template <typename T, int N>
__global__ void __launch_bounds__(256) retention_gate_kernel(const float* __restrict__ o, const T* __restrict__ qkvg, int ld, int gate_at,
                                                             T* __restrict__ y, int tok0, long long n, int heads, int dv, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const long long w = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= n) return;
  const int lane = threadIdx.x & 31, h = static_cast<int>(w % heads);
  const long long t = tok0 + w / heads;
  const float* src = o + (t * heads + h) * dv;
  const T* gate = qkvg + t * ld + gate_at + h * dv;
  T* dst = y + (t * heads + h) * dv;
  float ss = 0.f;
  for (int c = lane * N; c < dv; c += 32 * N) {
    float v[N];
    load_n<N>(src + c, v);
#pragma unroll
    for (int e = 0; e < N; ++e) ss += v[e] * v[e];
  }
  const float inv = rsqrtf(warp_sum_f(ss) / static_cast<float>(dv) + eps);
  for (int c = lane * N; c < dv; c += 32 * N) {
    float v[N], g[N];
    load_n<N>(src + c, v);
    load_n<N>(gate + c, g);
#pragma unroll
    for (int e = 0; e < N; ++e) v[e] *= inv * silu_t<T>(g[e]);
    store_n<N>(dst + c, v);
  }
}

template <typename T>
static RetentionIn<T> retention_in(const void* qkvg, int ld, const float* decay, float* state, const int* slots, const int* positions,
                                   const float* rope, int rope_rows, int rd, int heads, int dk, int dv, int num_slots, unsigned* status) {
  return RetentionIn<T>{static_cast<const T*>(qkvg), ld, decay, state, slots, positions, rope, rope_rows, rd, heads, dk, dv, num_slots, status};
}

template <typename T>
static int retention_decode(const RetentionIn<T>& p, int seqs, void* y, float eps, cudaStream_t stream) {
  const bool v4 = (p.dv & 3) == 0 && (p.ld & 3) == 0 && ((p.heads * p.dk) & 1) == 0;
  const int cols = v4 ? p.dv / 4 : p.dv;
  const int groups = cols < 256 ? 256 / cols : 1;
  const size_t smem = (2 * static_cast<size_t>(p.dk) + static_cast<size_t>(groups) * p.dv) * 4;
  if (smem > 200 * 1024) return -1;
  const dim3 grid(p.heads, seqs);
  if (v4) {
    auto k = retention_decode_kernel<T, 4>;
    FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
    return launch_kernel(k, grid, dim3(256), smem, stream, 0, p, static_cast<T*>(y), eps) == cudaSuccess ? 0 : -2;
  }
  auto k = retention_decode_kernel<T, 1>;
  FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
  return launch_kernel(k, grid, dim3(256), smem, stream, 0, p, static_cast<T*>(y), eps) == cudaSuccess ? 0 : -2;
}

// Token s of the step is sequence s's (s < seqs).  y [seqs][heads * dv].
extern "C" int forge_retention_decode(int fp32, const void* qkvg, int ld, const float* decay, float* state, const int* slots,
                                      const int* positions, const float* rope, int rope_rows, int rd, int seqs, int heads, int dk, int dv,
                                      int num_slots, void* y, float eps, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (seqs > 65535) return -1;
  return fp32 ? retention_decode(retention_in<float>(qkvg, ld, decay, state, slots, positions, rope, rope_rows, rd, heads, dk, dv, num_slots, status), seqs, y, eps, stream)
              : retention_decode(retention_in<bf16>(qkvg, ld, decay, state, slots, positions, rope, rope_rows, rd, heads, dk, dv, num_slots, status), seqs, y, eps, stream);
}

template <typename T>
static int retention_scan(const RetentionIn<T>& p, int seqs, const int* cu, float* o, cudaStream_t stream) {
  const size_t smem = (2 * static_cast<size_t>(kRScanTok) * p.dk + kRScanTok * kRScanCols) * 4;
  const dim3 grid((p.dv + kRScanCols - 1) / kRScanCols, p.heads, seqs);
#define FORGE_SCAN(R)                                                                                                     \
  {                                                                                                                       \
    auto k = retention_scan_kernel<T, R>;                                                                                 \
    FORGE_ENSURE_DYN_SMEM(k, 100 * 1024);                                                                                 \
    return launch_kernel(k, grid, dim3(256), smem, stream, 0, p, cu, o) == cudaSuccess ? 0 : -2;                          \
  }
  if (p.dk <= 64) FORGE_SCAN(8)
  if (p.dk <= 128) FORGE_SCAN(16)
  if (p.dk <= 256) FORGE_SCAN(32)
  if (p.dk <= 512) FORGE_SCAN(64)
#undef FORGE_SCAN
  return -1;
}

// Sequence s takes the step's tokens cu[s] .. cu[s + 1]; o fp32 [tokens][heads][dv] (before norm and gate).
extern "C" int forge_retention_scan(int fp32, const void* qkvg, int ld, const float* decay, float* state, const int* slots,
                                    const int* positions, const float* rope, int rope_rows, int rd, const int* cu, int seqs, int heads,
                                    int dk, int dv, int num_slots, float* o, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (seqs > 65535) return -1;
  return fp32 ? retention_scan(retention_in<float>(qkvg, ld, decay, state, slots, positions, rope, rope_rows, rd, heads, dk, dv, num_slots, status), seqs, cu, o, stream)
              : retention_scan(retention_in<bf16>(qkvg, ld, decay, state, slots, positions, rope, rope_rows, rd, heads, dk, dv, num_slots, status), seqs, cu, o, stream);
}

template <typename T>
static int retention_gate(const float* o, const void* qkvg, int ld, int gate_at, void* y, int tok0, int tokens, int heads, int dv, float eps,
                          cudaStream_t stream) {
  const long long n = static_cast<long long>(tokens) * heads;
  const dim3 grid(static_cast<unsigned>((n + 7) / 8));
  const bool v4 = ((dv | ld | gate_at) & 3) == 0;
  auto k = v4 ? retention_gate_kernel<T, 4> : retention_gate_kernel<T, 1>;
  return launch_kernel(k, grid, dim3(256), 0, stream, 0, o, static_cast<const T*>(qkvg), ld, gate_at, static_cast<T*>(y), tok0, n, heads, dv,
                       eps) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_retention_gate(int fp32, const float* o, const void* qkvg, int ld, int gate_at, void* y, int tok0, int tokens, int heads,
                                    int dv, float eps, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  return fp32 ? retention_gate<float>(o, qkvg, ld, gate_at, y, tok0, tokens, heads, dv, eps, stream)
              : retention_gate<bf16>(o, qkvg, ld, gate_at, y, tok0, tokens, heads, dv, eps, stream);
}

}  // namespace forge
