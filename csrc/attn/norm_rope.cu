// What stands before the attention of a decoder that norms its queries and keys: q | k | v of a token -> q and k normed (RMS over each
// head with a weight of d entries, or over all rows of the projection at once with a weight per row) and rotated (first rd entries of
// a head, entry i with i + rd / 2); q to [token][head][q_pitch] (padding columns zero), k and v to the caches
// [block][kv_head][block_size][d / dv].
//
// CTA = a few tokens, one after the other.  L lanes (a power of two) share a head: a lane owns an item of N rotated pairs or of N
// entries that pass.  Where every lane has one item at most and all heads fit the CTA (kOnce), weights stay in registers and the
// row is read once; else rows are read again after the norm's sum.
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
struct RopeItem {
  float a[N], b[N];
};

template <typename T, int N, bool kOnce, int kTok>
__global__ void __launch_bounds__(512) norm_rope_kernel(const NormRope<T> p, int tokens) {
  __shared__ float red[2][32];
  const int lane = threadIdx.x & ((1 << p.lanes_log2) - 1), L = 1 << p.lanes_log2;
  const int group = threadIdx.x >> p.lanes_log2, groups = blockDim.x >> p.lanes_log2, heads = p.H + p.G;
  const int half = p.rd >> 1, pairs = half / N, items = pairs + (p.d - p.rd) / N, padded = items + (p.q_pitch - p.d) / N;
  const int rounds = (heads + groups - 1) / groups;                    // the same for all threads: shuffles stay converged
  auto load = [&](const T* row, int i, float* a, float* b) {           // item i of a head's row
#pragma unroll
    for (int e = 0; e < N; ++e) a[e] = b[e] = 0.f;
    if (i < pairs) {
      load_n<N>(row + i * N, a);
      load_n<N>(row + i * N + half, b);
    } else if (i < items) {
      load_n<N>(row + p.rd + (i - pairs) * N, a);
    }
  };
  auto weight = [&](int h, int i, float* wa, float* wb) {
    const float* w = h < p.H ? p.q_norm + (p.whole ? static_cast<size_t>(h) * p.d : 0) : p.k_norm + (p.whole ? static_cast<size_t>(h - p.H) * p.d : 0);
    if (i < pairs) {
      load_n<N>(w + i * N, wa);
      load_n<N>(w + i * N + half, wb);
    } else if (i < items) {
      load_n<N>(w + p.rd + (i - pairs) * N, wa);
    }
  };
  float wa[N], wb[N];
#pragma unroll
  for (int e = 0; e < N; ++e) wa[e] = wb[e] = 0.f;
  if (kOnce && group < heads) weight(group, lane, wa, wb);             // weights do not come from the kernel before
  pdl_launch_dependents();
  pdl_wait();
  for (int u = 0; u < kTok; ++u) {
    const int t = blockIdx.x * kTok + u;
    if (t >= tokens) break;                                            // uniform for the CTA
    const T* src = p.proj + static_cast<size_t>(t) * p.ld;
    const long long slot = p.slots[t];
    int pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.rope_rows ? p.rope_rows - 1 : pos);
    const bool stored = slot >= 0 && slot < p.num_slots;
    if (slot >= p.num_slots && threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    const size_t blk = stored ? slot / p.block_size : 0, off = stored ? slot % p.block_size : 0;
    float a[N], b[N];
    float sq = 0.f, sk = 0.f;
    if (kOnce && group < heads) load(src + static_cast<size_t>(group) * p.d, lane, a, b);
    if (p.whole) {                                                     // uniform
      for (int k = 0; k < rounds; ++k) {
        const int h = k * groups + group;
        if (h >= heads) break;
        float s = 0.f;
        for (int i = lane; i < items; i += L) {
          if (!kOnce) load(src + static_cast<size_t>(h) * p.d, i, a, b);
#pragma unroll
          for (int e = 0; e < N; ++e) s = fmaf(a[e], a[e], fmaf(b[e], b[e], s));
        }
        if (h < p.H) sq += s;
        else sk += s;
      }
      const int wl = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
      sq = warp_sum_f(sq);
      sk = warp_sum_f(sk);
      if (wl == 0) {
        red[0][warp] = sq;
        red[1][warp] = sk;
      }
      __syncthreads();
      sq = rsqrtf(warp_sum_f(wl < nw ? red[0][wl] : 0.f) / static_cast<float>(p.H * p.d) + p.eps);
      sk = rsqrtf(warp_sum_f(wl < nw ? red[1][wl] : 0.f) / static_cast<float>(p.G * p.d) + p.eps);
      if (u + 1 < kTok) __syncthreads();
    }
    for (int k = 0; k < rounds; ++k) {
      const int h = k * groups + group;
      const bool live = h < heads;
      const T* row = src + static_cast<size_t>(live ? h : 0) * p.d;
      float inv = h < p.H ? sq : sk;
      if (!p.whole) {
        float s = 0.f;
        if (live)
          for (int i = lane; i < items; i += L) {
            if (!kOnce) load(row, i, a, b);
#pragma unroll
            for (int e = 0; e < N; ++e) s = fmaf(a[e], a[e], fmaf(b[e], b[e], s));
          }
        for (int o = L >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        inv = rsqrtf(s / static_cast<float>(p.d) + p.eps);
      }
      if (!live || (h >= p.H && !stored)) continue;
      T* dst = h < p.H ? p.q + (static_cast<size_t>(t) * p.H + h) * p.q_pitch
                       : p.k_cache + ((blk * p.G + (h - p.H)) * p.block_size + off) * p.d;
      for (int i = lane; i < (h < p.H ? padded : items); i += L) {
        if (!kOnce) {
          load(row, i, a, b);
          weight(h, i, wa, wb);
        }
        if (i < pairs) {
          const float* cs = p.rope + static_cast<size_t>(pos) * p.rd + i * N;
          float co[N], si[N], x[N], y[N];
          load_n<N>(cs, co);
          load_n<N>(cs + half, si);
#pragma unroll
          for (int e = 0; e < N; ++e) {
            const float v = a[e] * inv * wa[e], z = b[e] * inv * wb[e];
            x[e] = v * co[e] - z * si[e];
            y[e] = z * co[e] + v * si[e];
          }
          store_n<N>(dst + i * N, x);
          store_n<N>(dst + i * N + half, y);
        } else {
          float x[N];
#pragma unroll
          for (int e = 0; e < N; ++e) x[e] = i < items ? a[e] * inv * wa[e] : 0.f;
          store_n<N>(dst + p.rd + (i - pairs) * N, x);
        }
      }
    }
    if (stored)
      for (int i = threadIdx.x * N; i < p.G * p.dv; i += blockDim.x * N) {
        float x[N];
        load_n<N>(src + static_cast<size_t>(heads) * p.d + i, x);
        store_n<N>(p.v_cache + ((blk * p.G + i / p.dv) * p.block_size + off) * p.dv + i % p.dv, x);
      }
  }
}

template <typename T, int N>
static int norm_rope_n(NormRope<T> p, int tokens, cudaStream_t stream) {
  const int items = (p.rd >> 1) / N + (p.q_pitch - p.rd) / N, heads = p.H + p.G;
  p.lanes_log2 = 0;
  while ((1 << p.lanes_log2) < items && p.lanes_log2 < 5) ++p.lanes_log2;
  const int L = 1 << p.lanes_log2;
  const long long all = static_cast<long long>(heads) * L;
  const bool once = items <= L && all <= 512;
  const int threads = all >= 512 ? 512 : static_cast<int>((all + 31) / 32 * 32);
  const bool four = tokens >= 2048;
  auto k = once ? (four ? norm_rope_kernel<T, N, true, 4> : norm_rope_kernel<T, N, true, 1>)
                : (four ? norm_rope_kernel<T, N, false, 4> : norm_rope_kernel<T, N, false, 1>);
  return launch_kernel(k, dim3(four ? (tokens + 3) / 4 : tokens), dim3(threads), 0, stream, 0, p, tokens) == cudaSuccess ? 0 : -2;
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
  if (rd < 0 || (rd & 1) || rd > d || q_pitch < d || (rd > 0 && rope_rows < 1)) return -1;
#define FORGE_NORM_ROPE(T)                                                                                                             \
  return norm_rope<T>({static_cast<const T*>(proj), ld, q_norm, k_norm, rope, rope_rows, rd, positions, slots, static_cast<T*>(q),     \
                       static_cast<T*>(k_cache), static_cast<T*>(v_cache), num_slots, H, G, d, dv, q_pitch, block_size, whole, 0, eps, status}, tokens, stream)
  if (fp32) FORGE_NORM_ROPE(float);
  FORGE_NORM_ROPE(bf16);
#undef FORGE_NORM_ROPE
}

}  // namespace forge
