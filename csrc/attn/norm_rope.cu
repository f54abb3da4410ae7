// What stands before the attention of a decoder that norms its queries and keys: q | k | v of a token -> q and k normed (RMS over each
// head with a weight of d entries, or over all rows of the projection at once with a weight per row) and rotated (first rd entries of
// a head, entry i with i + rd / 2); q to [token][head][q_pitch] (padding columns zero), k and v to the caches
// [block][kv_head][block_size][d / dv].
//
// CTA = one token.  L lanes (a power of two) share a head: a lane owns an item of N rotated pairs or of N entries that pass, of one
// head or of several.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct NormRope {
  const T* proj;            // [tokens][ld]
  long long ld;
  const float* q_norm;      // [d], or [H d] with `whole`
  const float* k_norm;      // [d], or [G d]
  const float* rope;        // [rope_rows][rd]
  int rope_rows, rd;
  const int* positions;
  const int* slots;
  T* q;
  T* k_cache;
  T* v_cache;
  long long num_slots;
  int H, G, d, dv, q_pitch, block_size, whole, lanes_log2;
  float eps;
  unsigned* status;
};

template <typename T, int N>
struct alignas(sizeof(T) * N) Piece {       // N consecutive elements as they lie in memory
  T v[N];
};
template <typename T, int N>
__device__ __forceinline__ Piece<T, N> load_piece(const T* p) { return *reinterpret_cast<const Piece<T, N>*>(p); }
template <typename T, int N>
__device__ __forceinline__ Piece<T, N> zero_piece() {
  Piece<T, N> r;
#pragma unroll
  for (int e = 0; e < N; ++e) store_f(&r.v[e], 0.f);
  return r;
}

// One token's sums of squares over all rows of q and of k -> their reciprocal root mean squares, for all threads.
__device__ __forceinline__ void whole_norms(float& sq, float& sk, float (*red)[32], float nq, float nk, float eps) {
  const int wl = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  sq = warp_sum_f(sq);
  sk = warp_sum_f(sk);
  if (wl == 0) {
    red[0][warp] = sq;
    red[1][warp] = sk;
  }
  __syncthreads();
  sq = rsqrtf(warp_sum_f(wl < nw ? red[0][wl] : 0.f) / nq + eps);
  sk = rsqrtf(warp_sum_f(wl < nw ? red[1][wl] : 0.f) / nk + eps);
}

template <typename T>
struct TokenPlace {
  bool stored;
  size_t blk, off;
  const float* rope;
};
template <typename T>
__device__ __forceinline__ TokenPlace<T> token_place(const NormRope<T>& p, int t) {
  const long long slot = p.slots[t];
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.rope_rows ? p.rope_rows - 1 : pos);
  TokenPlace<T> r;
  r.stored = slot >= 0 && slot < p.num_slots;
  if (slot >= p.num_slots && threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
  const unsigned s = r.stored ? static_cast<unsigned>(slot) : 0u;      // num_slots fits 31 bits
  r.blk = s / static_cast<unsigned>(p.block_size);
  r.off = s % static_cast<unsigned>(p.block_size);
  r.rope = p.rope + static_cast<size_t>(pos) * p.rd;
  return r;
}

// R > 0: every lane has one item at most of each of up to R heads; all of the token's loads are under way before the first
// sum.  R = 0: any sizes, items are read again after the norm's sum.
template <typename T, int N, int R>
__global__ void __launch_bounds__(512) norm_rope_kernel(const NormRope<T> p) {
  __shared__ float red[2][32];
  const int lane = threadIdx.x & ((1 << p.lanes_log2) - 1), L = 1 << p.lanes_log2;
  const int group = threadIdx.x >> p.lanes_log2, groups = blockDim.x >> p.lanes_log2, heads = p.H + p.G;
  const int half = p.rd >> 1, pairs = half / N, items = pairs + (p.d - p.rd) / N, padded = items + (p.q_pitch - p.d) / N;
  const int rounds = (heads + groups - 1) / groups;                    // the same for all threads: shuffles stay converged
  const int t = blockIdx.x;
  const T* src = p.proj + static_cast<size_t>(t) * p.ld;
  auto first = [&](int i) { return i < pairs ? i * N : p.rd + (i - pairs) * N; };
  pdl_launch_dependents();
  pdl_wait();
  using P = Piece<T, N>;
  auto load = [&](int h, int i, P& a, P& b) {                          // item i of head h
    const T* row = src + static_cast<size_t>(h) * p.d + first(i);
    a = i < items ? load_piece<T, N>(row) : zero_piece<T, N>();
    b = i < pairs ? load_piece<T, N>(row + half) : zero_piece<T, N>();
  };
  auto squares = [&](const P& a, const P& b) {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < N; ++e) s = fmaf(load_f(&a.v[e]), load_f(&a.v[e]), fmaf(load_f(&b.v[e]), load_f(&b.v[e]), s));
    return s;
  };
  auto store = [&](const TokenPlace<T>& at, int h, int i, const P& a, const P& b, float inv) {
    const bool query = h < p.H;
    if (i >= (query ? padded : items) || (!query && !at.stored)) return;
    T* dst = (query ? p.q + (static_cast<size_t>(t) * p.H + h) * p.q_pitch : p.k_cache + ((at.blk * p.G + (h - p.H)) * p.block_size + at.off) * p.d) + first(i);
    const float* w = (query ? p.q_norm + (p.whole ? h * p.d : 0) : p.k_norm + (p.whole ? (h - p.H) * p.d : 0)) + first(i);
    float x[N], g[N];
    if (i < items) load_n<N>(w, g);
#pragma unroll
    for (int e = 0; e < N; ++e) x[e] = i < items ? load_f(&a.v[e]) * inv * g[e] : 0.f;
    if (i < pairs) {
      float co[N], si[N], y[N];
      load_n<N>(w + half, g);
      load_n<N>(at.rope + i * N, co);
      load_n<N>(at.rope + i * N + half, si);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const float z = load_f(&b.v[e]) * inv * g[e];
        y[e] = z * co[e] + x[e] * si[e];
        x[e] = x[e] * co[e] - z * si[e];
      }
      store_n<N>(dst + half, y);
    }
    store_n<N>(dst, x);
  };
  const T* values = src + static_cast<size_t>(heads) * p.d;
  const int n_values = p.G * p.dv;
  auto value_at = [&](const TokenPlace<T>& at, int i) { return p.v_cache + ((at.blk * p.G + i / p.dv) * p.block_size + at.off) * p.dv + i % p.dv; };

  if constexpr (R > 0) {
    P a[R], b[R], v;
    float s[R], sq = 0.f, sk = 0.f;
    const int vi = threadIdx.x * N;
#pragma unroll
    for (int k = 0; k < R; ++k) {
      const int h = k * groups + group;
      if (h < heads) load(h, lane, a[k], b[k]);
      else a[k] = b[k] = zero_piece<T, N>();
    }
    v = vi < n_values ? load_piece<T, N>(values + vi) : zero_piece<T, N>();
    const TokenPlace<T> at = token_place(p, t);
#pragma unroll
    for (int k = 0; k < R; ++k) {
      s[k] = squares(a[k], b[k]);
      if (k * groups + group < p.H) sq += s[k];
      else sk += s[k];
    }
    if (at.stored) {
      if (vi < n_values) *reinterpret_cast<P*>(value_at(at, vi)) = v;
      for (int i = vi + blockDim.x * N; i < n_values; i += blockDim.x * N) *reinterpret_cast<P*>(value_at(at, i)) = load_piece<T, N>(values + i);
    }
    if (p.whole) whole_norms(sq, sk, red, static_cast<float>(p.H * p.d), static_cast<float>(p.G * p.d), p.eps);
#pragma unroll
    for (int k = 0; k < R; ++k) {
      const int h = k * groups + group;
      float inv = h < p.H ? sq : sk;
      if (!p.whole) {
        for (int o = L >> 1; o > 0; o >>= 1) s[k] += __shfl_xor_sync(0xffffffffu, s[k], o);
        inv = rsqrtf(s[k] / static_cast<float>(p.d) + p.eps);
      }
      if (h < heads) store(at, h, lane, a[k], b[k], inv);
    }
  } else {
    const TokenPlace<T> at = token_place(p, t);
    P a, b;
    auto head_sum = [&](int h) {
      float s = 0.f;
      if (h < heads)
        for (int i = lane; i < items; i += L) {
          load(h, i, a, b);
          s += squares(a, b);
        }
      return s;
    };
    float sq = 0.f, sk = 0.f;
    if (p.whole) {
      for (int k = 0; k < rounds; ++k) {
        const int h = k * groups + group;
        const float s = head_sum(h);
        if (h < p.H) sq += s;
        else sk += s;
      }
      whole_norms(sq, sk, red, static_cast<float>(p.H * p.d), static_cast<float>(p.G * p.d), p.eps);
    }
    for (int k = 0; k < rounds; ++k) {
      const int h = k * groups + group;
      float inv = h < p.H ? sq : sk;
      if (!p.whole) {
        float s = head_sum(h);
        for (int o = L >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        inv = rsqrtf(s / static_cast<float>(p.d) + p.eps);
      }
      if (h >= heads) continue;
      for (int i = lane; i < (h < p.H ? padded : items); i += L) {
        load(h, i, a, b);
        store(at, h, i, a, b, inv);
      }
    }
    if (at.stored)
      for (int i = threadIdx.x * N; i < n_values; i += blockDim.x * N) *reinterpret_cast<P*>(value_at(at, i)) = load_piece<T, N>(values + i);
  }
}

template <typename T, int N>
static int norm_rope_n(NormRope<T> p, int tokens, cudaStream_t stream) {
  const int items = (p.rd >> 1) / N + (p.q_pitch - p.rd) / N, heads = p.H + p.G;
  p.lanes_log2 = 0;
  while ((1 << p.lanes_log2) < items && p.lanes_log2 < 5) ++p.lanes_log2;
  const int L = 1 << p.lanes_log2;
  // heads per lane: few threads and many tokens per SM where there are many tokens
  int r = tokens >= 1024 ? 4 : 1;
  auto threads_for = [&](int rounds) { return static_cast<int>((static_cast<long long>((heads + rounds - 1) / rounds) * L + 31) / 32 * 32); };
  if (items > L) r = 0;
  while (r > 0 && r < 4 && threads_for(r) > 512) r *= 2;
  if (r > 0 && threads_for(r) > 512) r = 0;
  const int threads = r > 0 ? threads_for(r) : heads >= 512 / L ? 512 : static_cast<int>((static_cast<long long>(heads) * L + 31) / 32 * 32);
  auto k = r == 0 ? norm_rope_kernel<T, N, 0> : r == 1 ? norm_rope_kernel<T, N, 1> : r == 2 ? norm_rope_kernel<T, N, 2> : norm_rope_kernel<T, N, 4>;
  return launch_kernel(k, dim3(tokens), dim3(threads), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
}

template <typename T>
static int norm_rope(const NormRope<T>& p, int tokens, cudaStream_t stream) {
  const uintptr_t proj = reinterpret_cast<uintptr_t>(p.proj);
  const int all = (p.rd >> 1) | p.d | p.dv | p.q_pitch | static_cast<int>(p.ld & 7);
  if (sizeof(T) == 2 && (all & 7) == 0 && (proj & 15) == 0) return norm_rope_n<T, 8>(p, tokens, stream);
  if ((all & 3) == 0 && (proj & (4 * sizeof(T) - 1)) == 0) return norm_rope_n<T, 4>(p, tokens, stream);
  return norm_rope_n<T, 1>(p, tokens, stream);
}

// whole: the norms run over all rows of q and of k at once (weights [H d] and [G d]), else over each head (weights [d]).
extern "C" int forge_norm_rope_store(int fp32, const void* proj, long long ld, int tokens, const float* q_norm, const float* k_norm, int whole,
                                     float eps, const float* rope, int rope_rows, int rd, const int* positions, const int* slots, void* q,
                                     int q_pitch, void* k_cache, void* v_cache, long long num_slots, int block_size, int H, int G, int d, int dv,
                                     unsigned* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (rd < 0 || (rd & 1) || rd > d || q_pitch < d || (rd > 0 && rope_rows < 1) || num_slots >= (1ll << 31)) return -1;
#define FORGE_NORM_ROPE(T)                                                                                                             \
  return norm_rope<T>({static_cast<const T*>(proj), ld, q_norm, k_norm, rope, rope_rows, rd, positions, slots, static_cast<T*>(q),     \
                       static_cast<T*>(k_cache), static_cast<T*>(v_cache), num_slots, H, G, d, dv, q_pitch, block_size, whole, 0, eps, status}, tokens, stream)
  if (fp32) FORGE_NORM_ROPE(float);
  FORGE_NORM_ROPE(bf16);
#undef FORGE_NORM_ROPE
}

}  // namespace forge
