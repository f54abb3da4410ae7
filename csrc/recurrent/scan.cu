// Linear recurrences with a decay per token and head (recurrence.cuh), token by token.
//
//   recurrence_scan     a run of tokens per sequence, any sizes, bf16 or fp32 operands
//   recurrence_decode   one token of many sequences: the state is read, updated and written once
//   gated_norm          what follows: the state-space mixer's (y silu(z)) / rms per group, or the delta rule's o / rms per head
//                       times silu(gate); both times a weight and a factor
//
// A sequence's first token (position 0) starts from S = 0, so a state slot needs no clearing.
#include "../include/launch.cuh"
#include "../include/recurrence.cuh"

namespace forge {

constexpr int kSTok = 16, kSCols = 32;

// CTA = (32 value columns, head, sequence); thread = one column and every eighth row of the state, R rows at most.
template <typename T, int R, bool kDelta>
__global__ void __launch_bounds__(256) recurrence_scan_kernel(const Recurrence<T> p, const int* __restrict__ cu, float* __restrict__ o) {
  extern __shared__ float sm[];
  float* sq = sm;                            // [16][dk]
  float* sk = sq + kSTok * p.dk;             // [16][dk]
  float* sv = sk + kSTok * p.dk;             // [16][32]
  float* sg = sv + kSTok * kSCols;           // [16] decay
  float* sw = sg + kSTok;                    // [16] dt or beta
  pdl_launch_dependents();
  pdl_wait();
  const int c0 = blockIdx.x * kSCols, h = blockIdx.y, s = blockIdx.z;
  const int t_begin = cu[s], t_end = cu[s + 1], slot = p.slots[s];
  if (t_begin >= t_end) return;
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    return;
  }
  const int grp = threadIdx.x & 7, col = threadIdx.x >> 3, hk = h / p.share;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool live = c0 + col < p.dv;
  float* S = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dk * p.dv + c0 + col;
  float st[R];
  const bool fresh = p.positions[t_begin] == 0;
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * 8 + grp;
    st[j] = !fresh && live && i < p.dk ? S[static_cast<size_t>(i) * p.dv] : 0.f;
  }
  const float skip = kDelta ? 0.f : p.D[h];
  for (int t0 = t_begin; t0 < t_end; t0 += kSTok) {
    const int n = min(kSTok, t_end - t0);
    __syncthreads();
    for (int tt = warp; tt < n; tt += 8) {                       // a warp brings a token's q and k, as unit vectors for the delta rule
      const size_t at = static_cast<size_t>(t0 + tt) * p.ld + static_cast<size_t>(hk) * p.dk;
      float qq = 0.f, kk = 0.f;
      for (int i = lane; i < p.dk; i += 32) {
        const float a = load_f(p.q + at + i), b = load_f(p.k + at + i);
        sq[tt * p.dk + i] = a;
        sk[tt * p.dk + i] = b;
        qq += a * a;
        kk += b * b;
      }
      if (kDelta) {
        qq = rsqrtf(warp_sum_f(qq) + kUnitEps) * rsqrtf(static_cast<float>(p.dk));
        kk = rsqrtf(warp_sum_f(kk) + kUnitEps);
        for (int i = lane; i < p.dk; i += 32) {
          sq[tt * p.dk + i] *= qq;
          sk[tt * p.dk + i] *= kk;
        }
      }
      if (lane == 0) {
        const TokenGates g = token_gates(p, t0 + tt, h);
        sg[tt] = expf(g.log_g);
        sw[tt] = g.w;
      }
    }
    for (int idx = threadIdx.x; idx < n * kSCols; idx += blockDim.x) {
      const int tt = idx / kSCols, c = idx % kSCols;
      sv[idx] = c0 + c < p.dv ? load_f(p.v + static_cast<size_t>(t0 + tt) * p.ld + static_cast<size_t>(h) * p.dv + c0 + c) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      const float v = sv[tt * kSCols + col], g = sg[tt], w = sw[tt];
      const float* k = sk + tt * p.dk;
      const float* q = sq + tt * p.dk;
      float u = w * v, acc = 0.f;
      if (kDelta) {
        float seen = 0.f;
#pragma unroll
        for (int j = 0; j < R; ++j) {
          const int i = j * 8 + grp;
          st[j] *= g;
          if (i < p.dk) seen = fmaf(st[j], k[i], seen);
        }
        seen += __shfl_xor_sync(0xffffffffu, seen, 1);
        seen += __shfl_xor_sync(0xffffffffu, seen, 2);
        seen += __shfl_xor_sync(0xffffffffu, seen, 4);
        u = w * (v - seen);
      }
#pragma unroll
      for (int j = 0; j < R; ++j) {
        const int i = j * 8 + grp;
        if (i < p.dk) {
          st[j] = kDelta ? fmaf(k[i], u, st[j]) : fmaf(g, st[j], k[i] * u);
          acc = fmaf(st[j], q[i], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (grp == 0 && live) o[(static_cast<size_t>(t0 + tt) * p.heads + h) * p.dv + c0 + col] = fmaf(skip, v, acc);
    }
  }
  if (!live) return;
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * 8 + grp;
    if (i < p.dk) S[static_cast<size_t>(i) * p.dv] = st[j];
  }
}

// CTA = (head, sequence), one token each: token s is sequence s's.  A thread owns four columns and every `groups`-th row, R
// rows at most, and holds them in registers between reading and writing.  dv a multiple of 4.
template <typename T, int R, bool kDelta, int kThreads>
__global__ void __launch_bounds__(kThreads) recurrence_decode_kernel(const Recurrence<T> p, float* __restrict__ o) {
  extern __shared__ float sm[];
  __shared__ float red[2];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y, slot = p.slots[s];
  float* out = o + (static_cast<size_t>(s) * p.heads + h) * p.dv;
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    for (int c = threadIdx.x; c < p.dv; c += kThreads) out[c] = 0.f;
    return;
  }
  const int cols = p.dv >> 2, groups = kThreads / cols;
  float* sq = sm;                            // [dk]
  float* sk = sq + p.dk;                     // [dk]
  float* part = sk + p.dk;                   // [groups][dv]
  float* su = part + groups * p.dv;          // [dv]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t at = static_cast<size_t>(s) * p.ld + static_cast<size_t>(h / p.share) * p.dk;
  const int cg = threadIdx.x % cols, rg = threadIdx.x / cols, c = cg * 4;
  const bool live = rg < groups;
  float* S = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dk * p.dv + c;
  const bool fresh = p.positions[s] == 0;
  float4 st[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * groups + rg;
    st[j] = live && !fresh && i < p.dk ? *reinterpret_cast<const float4*>(S + static_cast<size_t>(i) * p.dv) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int i = threadIdx.x; i < p.dk; i += kThreads) {
    sq[i] = load_f(p.q + at + i);
    sk[i] = load_f(p.k + at + i);
  }
  const TokenGates gates = token_gates(p, s, h);
  const float g = expf(gates.log_g);
  __syncthreads();
  float nq = 1.f, nk = 1.f;
  if (kDelta) {
    if (warp < 2) {
      const float* x = warp == 0 ? sq : sk;
      float ss = 0.f;
      for (int i = lane; i < p.dk; i += 32) ss += x[i] * x[i];
      ss = warp_sum_f(ss);
      if (lane == 0) red[warp] = rsqrtf(ss + kUnitEps) * (warp == 0 ? rsqrtf(static_cast<float>(p.dk)) : 1.f);
    }
    __syncthreads();
    nq = red[0];
    nk = red[1];
  }
  float v[4];
  const T* vrow = p.v + static_cast<size_t>(s) * p.ld + static_cast<size_t>(h) * p.dv;
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = live ? load_f(vrow + c + e) : 0.f;
  float4 u = make_float4(gates.w * v[0], gates.w * v[1], gates.w * v[2], gates.w * v[3]);
  if (kDelta) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int i = j * groups + rg;
      st[j].x *= g; st[j].y *= g; st[j].z *= g; st[j].w *= g;
      if (live && i < p.dk) {
        const float k = sk[i];
        a.x = fmaf(st[j].x, k, a.x); a.y = fmaf(st[j].y, k, a.y); a.z = fmaf(st[j].z, k, a.z); a.w = fmaf(st[j].w, k, a.w);
      }
    }
    if (live) *reinterpret_cast<float4*>(part + rg * p.dv + c) = a;
    __syncthreads();
    for (int i = threadIdx.x; i < p.dv; i += kThreads) {
      float seen = 0.f;
      for (int r = 0; r < groups; ++r) seen += part[r * p.dv + i];
      su[i] = gates.w * (load_f(vrow + i) - nk * seen) * nk;      // carries the factor of the unit vector k
    }
    __syncthreads();
    if (live) u = *reinterpret_cast<const float4*>(su + c);
  }
  float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int i = j * groups + rg;
    if (live && i < p.dk) {
      const float k = sk[i], q = sq[i];
      if (!kDelta) { st[j].x *= g; st[j].y *= g; st[j].z *= g; st[j].w *= g; }
      st[j].x = fmaf(k, u.x, st[j].x); st[j].y = fmaf(k, u.y, st[j].y); st[j].z = fmaf(k, u.z, st[j].z); st[j].w = fmaf(k, u.w, st[j].w);
      *reinterpret_cast<float4*>(S + static_cast<size_t>(i) * p.dv) = st[j];
      y.x = fmaf(st[j].x, q, y.x); y.y = fmaf(st[j].y, q, y.y); y.z = fmaf(st[j].z, q, y.z); y.w = fmaf(st[j].w, q, y.w);
    }
  }
  if (live) *reinterpret_cast<float4*>(part + rg * p.dv + c) = y;
  __syncthreads();
  for (int i = threadIdx.x; i < p.dv; i += kThreads) {
    float a = 0.f;
    for (int r = 0; r < groups; ++r) a += part[r * p.dv + i];
    out[i] = kDelta ? nq * a : fmaf(p.D[h], load_f(vrow + i), a);
  }
}

template <typename T>
static int scan(const Recurrence<T>& p, int seqs, const int* cu, float* o, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(kSTok) * (2 * p.dk + kSCols + 2) * 4;
  const dim3 grid((p.dv + kSCols - 1) / kSCols, p.heads, seqs);
  if (p.heads > 65535 || seqs > 65535) return -1;
#define FORGE_SCAN(R)                                                                                                \
  {                                                                                                                  \
    auto k = p.beta != nullptr ? recurrence_scan_kernel<T, R, true> : recurrence_scan_kernel<T, R, false>;           \
    if (p.beta != nullptr) FORGE_ENSURE_DYN_SMEM((recurrence_scan_kernel<T, R, true>), 100 * 1024);                  \
    else FORGE_ENSURE_DYN_SMEM((recurrence_scan_kernel<T, R, false>), 100 * 1024);                                   \
    return launch_kernel(k, grid, dim3(256), smem, stream, 0, p, cu, o) == cudaSuccess ? 0 : -2;                     \
  }
  if (p.dk <= 64) FORGE_SCAN(8)
  if (p.dk <= 128) FORGE_SCAN(16)
  if (p.dk <= 256) FORGE_SCAN(32)
  if (p.dk <= 512) FORGE_SCAN(64)
#undef FORGE_SCAN
  return -1;
}

// Threads and rows per thread of the decode kernel for these sizes; 0: no instance (use the scan).
static int decode_shape(int dk, int dv, int* rows) {
  if ((dv & 3) || dv > 1024) return 0;
  for (int threads = 256; threads <= 512; threads *= 2) {
    const int groups = threads / (dv >> 2);
    if (groups < 1) continue;
    const int r = (dk + groups - 1) / groups;
    if (r <= 32) {
      *rows = r <= 8 ? 8 : r <= 16 ? 16 : 32;
      return threads;
    }
  }
  return 0;
}

template <typename T, bool kDelta>
static int decode(const Recurrence<T>& p, int seqs, float* o, cudaStream_t stream) {
  int rows = 0;
  const int threads = decode_shape(p.dk, p.dv, &rows);
  if (threads == 0 || seqs > 65535) return -1;
  const size_t smem = (2 * static_cast<size_t>(p.dk) + static_cast<size_t>(threads / (p.dv >> 2) + 1) * p.dv) * 4;
  const dim3 grid(p.heads, seqs);
#define FORGE_DEC(R, TH) return launch_kernel(recurrence_decode_kernel<T, R, kDelta, TH>, grid, dim3(TH), smem, stream, 0, p, o) == cudaSuccess ? 0 : -2
  if (threads == 256) {
    if (rows == 8) FORGE_DEC(8, 256);
    if (rows == 16) FORGE_DEC(16, 256);
    FORGE_DEC(32, 256);
  }
  FORGE_DEC(32, 512);
#undef FORGE_DEC
}

template <typename T>
static Recurrence<T> operands(const void* q, const void* k, const void* v, long long ld, const void* dt, const void* beta, long long ld_raw,
                              const float* A_log, const float* dt_bias, const float* D, float* state, const int* slots, const int* positions,
                              int heads, int share, int dk, int dv, int num_slots, unsigned* status) {
  return {static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v), ld, static_cast<const T*>(dt), static_cast<const T*>(beta),
          ld_raw, A_log, dt_bias, D, state, slots, positions, heads, share, dk, dv, num_slots, status};
}

extern "C" int forge_recurrence_decode_ok(int dk, int dv) {
  int rows = 0;
  return decode_shape(dk, dv, &rows) != 0;
}

// o fp32 [tokens][heads][dv].  cu null: one token per sequence (decode), else sequence s has the step's tokens cu[s] .. cu[s + 1].
extern "C" int forge_recurrence(int fp32, const void* q, const void* k, const void* v, long long ld, const void* dt, const void* beta,
                                long long ld_raw, const float* A_log, const float* dt_bias, const float* D, float* state, const int* slots,
                                const int* positions, const int* cu, int seqs, int heads, int share, int dk, int dv, int num_slots, float* o,
                                unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (beta == nullptr && D == nullptr) return -1;
#define FORGE_REC(T)                                                                                                                            \
  {                                                                                                                                             \
    const Recurrence<T> p = operands<T>(q, k, v, ld, dt, beta, ld_raw, A_log, dt_bias, D, state, slots, positions, heads, share, dk, dv, num_slots, \
                                        status);                                                                                                \
    if (cu != nullptr) return scan(p, seqs, cu, o, stream);                                                                                     \
    return beta != nullptr ? decode<T, true>(p, seqs, o, stream) : decode<T, false>(p, seqs, o, stream);                                        \
  }
  if (fp32) FORGE_REC(float)
  FORGE_REC(bf16)
#undef FORGE_REC
}

// One warp per (token, group of n entries).  kGateFirst: a = o silu(z), out = a / rms(a) weight; else out = o / rms(o) weight silu(z).
// A lane holds up to R pieces of N entries; R = 0: any n, read twice.
template <typename T, int N, int R, bool kGateFirst>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long ldg,
                                                         const float* __restrict__ weight, int weight_period, T* __restrict__ out, long long ldo,
                                                         long long work, int groups, int n, float factor, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const long long w = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= work) return;
  const int lane = threadIdx.x & 31;
  const long long t = w / groups;
  const int g = static_cast<int>(w - t * groups);
  const float* src = o + w * n;
  const float* w0 = weight + static_cast<long long>(g) * n % weight_period;
  const T* z = gate + t * ldg + static_cast<long long>(g) * n;
  T* dst = out + t * ldo + static_cast<long long>(g) * n;
  float ss = 0.f;
  if constexpr (R > 0) {
    float v[R][N], s[R][N], m[R][N];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int c = (r * 32 + lane) * N;
      if (c < n) {
        load_n<N>(src + c, v[r]);
        load_n<N>(z + c, s[r]);
        load_n<N>(w0 + c, m[r]);
      } else {
#pragma unroll
        for (int e = 0; e < N; ++e) v[r][e] = s[r][e] = m[r][e] = 0.f;
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int e = 0; e < N; ++e) {
        if (kGateFirst) v[r][e] *= silu_t<T>(s[r][e]);
        ss += v[r][e] * v[r][e];
        m[r][e] *= kGateFirst ? v[r][e] : v[r][e] * silu_t<T>(s[r][e]);
      }
    const float inv = factor * rsqrtf(warp_sum_f(ss) / static_cast<float>(n) + eps);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int c = (r * 32 + lane) * N;
#pragma unroll
      for (int e = 0; e < N; ++e) m[r][e] *= inv;
      if (c < n) store_n<N>(dst + c, m[r]);
    }
  } else {
    for (int c = lane * N; c < n; c += 32 * N) {
      float v[N], s[N];
      load_n<N>(src + c, v);
      load_n<N>(z + c, s);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        if (kGateFirst) v[e] *= silu_t<T>(s[e]);
        ss += v[e] * v[e];
      }
    }
    const float inv = factor * rsqrtf(warp_sum_f(ss) / static_cast<float>(n) + eps);
    for (int c = lane * N; c < n; c += 32 * N) {
      float v[N], s[N], m[N];
      load_n<N>(src + c, v);
      load_n<N>(z + c, s);
      load_n<N>(w0 + c, m);
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] *= inv * m[e] * silu_t<T>(s[e]);
      store_n<N>(dst + c, v);
    }
  }
}

// o fp32 [tokens][groups n], gate [tokens][ldg], out [tokens][ldo]; the weight repeats every weight_period entries, a multiple of n.
template <typename T>
static int gated_norm(const float* o, const T* gate, long long ldg, const float* weight, int weight_period, T* out, long long ldo, int tokens,
                      int groups, int n, bool gate_first, float factor, float eps, cudaStream_t stream) {
  const long long work = static_cast<long long>(tokens) * groups;
  const dim3 grid(static_cast<unsigned>((work + 7) / 8));
  const uintptr_t mask = 4 * sizeof(T) - 1;
  const bool v4 = ((n | weight_period) & 3) == 0 && ((ldg | ldo) & 3) == 0 && (reinterpret_cast<uintptr_t>(gate) & mask) == 0 && (reinterpret_cast<uintptr_t>(out) & mask) == 0;
#define FORGE_GN(N, R)                                                                                                                         \
  return launch_kernel(gate_first ? gated_norm_kernel<T, N, R, true> : gated_norm_kernel<T, N, R, false>, grid, dim3(256), 0, stream, 0, o, gate, \
                       ldg, weight, weight_period, out, ldo, work, groups, n, factor, eps) == cudaSuccess ? 0 : -2
  if (!v4) FORGE_GN(1, 0);
  if (n <= 128) FORGE_GN(4, 1);
  if (n <= 256) FORGE_GN(4, 2);
  FORGE_GN(4, 0);
#undef FORGE_GN
}

extern "C" int forge_gated_norm(int fp32, const float* o, const void* gate, long long ldg, const float* weight, int weight_period, void* out,
                                long long ldo, int tokens, int groups, int n, int gate_first, float factor, float eps, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (groups < 1 || n < 1 || weight_period < n || weight_period % n) return -1;
  return fp32 ? gated_norm<float>(o, static_cast<const float*>(gate), ldg, weight, weight_period, static_cast<float*>(out), ldo, tokens, groups, n, gate_first != 0, factor, eps, stream)
              : gated_norm<bf16>(o, static_cast<const bf16*>(gate), ldg, weight, weight_period, static_cast<bf16*>(out), ldo, tokens, groups, n, gate_first != 0, factor, eps, stream);
}

}  // namespace forge
