// What stands before the attention of a decoder that norms its queries and keys: q | k | v of a token -> q and k normed (RMS over each
// head with a weight of d entries, or over all rows of the projection at once with a weight per row) and rotated (first rd entries of
// a head, entry i with i + rd / 2); q to [token][head][q_pitch] (padding columns zero), k and v to the caches
// [block][kv_head][block_size][d / dv].  Without key/value heads (G = 0) there is q alone.  temper: one more factor per query head.
//
// The work of a token is a list of items: N rotated pairs or 2 N entries that pass of a head, or N values.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct NormRope {
  const T* proj;            // [tokens][ld]
  long long ld;
  const T* q_norm;          // [d], or [H d] with `whole`
  const T* k_norm;          // [d], or [G d]
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
  const float* temper;      // [H]; null: none
  unsigned* status;
};

template <typename T>
__device__ __forceinline__ float head_factor(const NormRope<T>& p, int h) { return p.temper != nullptr && h < p.H ? p.temper[h] : 1.f; }

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
  if (slot >= p.num_slots && p.G > 0) set_status(p.status, kStatusBadIndex);
  const unsigned s = r.stored ? static_cast<unsigned>(slot) : 0u;      // num_slots fits 31 bits
  r.blk = s / static_cast<unsigned>(p.block_size);
  r.off = s % static_cast<unsigned>(p.block_size);
  r.rope = p.rope + static_cast<size_t>(pos) * p.rd;
  return r;
}

// The items of a head, two pieces of N entries each: item i < pairs is N rotated pairs, i < items two neighbouring pieces that pass (the
// second may be missing), i < padded (queries) reaches into the padding columns.
__host__ __device__ __forceinline__ int items_of(int pairs, int passing) { return pairs + ((passing + 1) >> 1); }

template <typename T, int N>
struct HeadItems {
  int pairs, items, padded;
  __device__ explicit HeadItems(const NormRope<T>& p)
      : pairs((p.rd >> 1) / N), items(items_of(pairs, (p.d - p.rd) / N)), padded(items_of(pairs, (p.q_pitch - p.rd) / N)) {}
};

template <typename T, int N>
struct Item {
  Piece<T, N> a, b;         // entries at c and at c2
  Piece<T, N> wa, wb;       // their norm weights
  int c, c2;

  __device__ __forceinline__ void place(const NormRope<T>& p, const HeadItems<T, N>& z, int i) {
    c = i < z.pairs ? i * N : p.rd + 2 * (i - z.pairs) * N;
    c2 = c + (i < z.pairs ? p.rd >> 1 : N);
  }
  __device__ __forceinline__ void weights(const NormRope<T>& p, int h) {
    const T* w = h < p.H ? p.q_norm + (p.whole ? h * p.d : 0) : p.k_norm + (p.whole ? (h - p.H) * p.d : 0);
    wa = c < p.d ? load_piece<T, N>(w + c) : zero_piece<T, N>();
    wb = c2 < p.d ? load_piece<T, N>(w + c2) : zero_piece<T, N>();
  }
  __device__ __forceinline__ void load(const NormRope<T>& p, const T* head) {
    a = c < p.d ? load_piece<T, N>(head + c) : zero_piece<T, N>();
    b = c2 < p.d ? load_piece<T, N>(head + c2) : zero_piece<T, N>();
  }
  __device__ __forceinline__ float squares() const {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < N; ++e) s = fmaf(load_f(&a.v[e]), load_f(&a.v[e]), fmaf(load_f(&b.v[e]), load_f(&b.v[e]), s));
    return s;
  }
  // co, si: 1 and 0 where the entries pass; cols: columns of a row at dst
  __device__ __forceinline__ void store(T* dst, int cols, float inv, const float* co, const float* si) const {
    float x[N], y[N];
#pragma unroll
    for (int e = 0; e < N; ++e) {
      const float u = load_f(&a.v[e]) * inv * load_f(&wa.v[e]), v = load_f(&b.v[e]) * inv * load_f(&wb.v[e]);
      x[e] = u * co[e] - v * si[e];
      y[e] = v * co[e] + u * si[e];
    }
    if (c < cols) store_n<N>(dst + c, x);
    if (c2 < cols) store_n<N>(dst + c2, y);
  }
};

// Cos and sin of item i.
template <typename T, int N>
__device__ __forceinline__ void item_rotation(const NormRope<T>& p, const HeadItems<T, N>& z, const float* row, int i, float* co, float* si) {
#pragma unroll
  for (int e = 0; e < N; ++e) {
    co[e] = 1.f;
    si[e] = 0.f;
  }
  if (i < z.pairs) {
    load_n<N>(row + i * N, co);
    load_n<N>(row + i * N + (p.rd >> 1), si);
  }
}

template <typename T>
__device__ __forceinline__ T* head_place(const NormRope<T>& p, const TokenPlace<T>& at, int t, int h) {
  return h < p.H ? p.q + (static_cast<size_t>(t) * p.H + h) * p.q_pitch : p.k_cache + ((at.blk * p.G + (h - p.H)) * p.block_size + at.off) * p.d;
}
template <typename T>
__device__ __forceinline__ T* value_place(const NormRope<T>& p, const TokenPlace<T>& at, int i) {
  return p.v_cache + ((at.blk * p.G + i / p.dv) * p.block_size + at.off) * p.dv + i % p.dv;
}

// A norm per head: L lanes take a head of a token (or its share of the values), whatever the token.  kOnce: one item per lane.
template <typename T, int N, bool kOnce>
__global__ void __launch_bounds__(256) norm_rope_heads_kernel(const NormRope<T> p, int units) {
  const HeadItems<T, N> z(p);
  const int L = 1 << p.lanes_log2, lane = threadIdx.x & (L - 1), all = p.H + 2 * p.G;
  const int unit = blockIdx.x * (blockDim.x >> p.lanes_log2) + (threadIdx.x >> p.lanes_log2);
  const bool live = unit < units;
  const int t = live ? unit / all : 0, h = live ? unit % all : all;
  const bool value = h >= p.H + p.G;
  Item<T, N> it;
  it.place(p, z, lane);
  if (kOnce && !value) it.weights(p, h);                               // weights do not come from the kernel before
  pdl_launch_dependents();
  pdl_wait();
  const T* src = p.proj + static_cast<size_t>(t) * p.ld + (value ? static_cast<size_t>(p.H + p.G) * p.d + static_cast<size_t>(h - p.H - p.G) * p.dv
                                                                 : static_cast<size_t>(h) * p.d);
  float s = 0.f;
  TokenPlace<T> at = {};
  if (live) {
    if (kOnce && !value) {
      it.load(p, src);
      s = it.squares();
    }
    if (!kOnce && !value)
      for (int i = lane; i < z.items; i += L) {
        it.place(p, z, i);
        it.load(p, src);
        s += it.squares();
      }
    at = token_place(p, t);
  }
  float co[N], si[N];
  if (kOnce) item_rotation(p, z, at.rope, live && !value ? lane : z.pairs, co, si);
  for (int o = L >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if (!live || (h >= p.H && !at.stored)) return;
  if (value) {
    for (int i = lane * N; i < p.dv; i += L * N)
      *reinterpret_cast<Piece<T, N>*>(value_place(p, at, (h - p.H - p.G) * p.dv + i)) = load_piece<T, N>(src + i);
    return;
  }
  const float inv = rsqrtf(s / static_cast<float>(p.d) + p.eps) * head_factor(p, h);
  T* dst = head_place(p, at, t, h);
  const int cols = h < p.H ? p.q_pitch : p.d;
  if (kOnce) {
    it.store(dst, cols, inv, co, si);
    return;
  }
  for (int i = lane; i < z.padded; i += L) {
    it.place(p, z, i);
    it.load(p, src);
    it.weights(p, h);
    item_rotation(p, z, at.rope, i, co, si);
    it.store(dst, cols, inv, co, si);
  }
}

// A norm over all rows of q and one over all rows of k: CTA = one token.  kOnce: a thread has one item (or one piece of the values).
template <typename T, int N, bool kOnce>
__global__ void __launch_bounds__(kOnce ? 1024 : 512) norm_rope_whole_kernel(const NormRope<T> p) {
  __shared__ float red[2][32];
  const HeadItems<T, N> z(p);
  const int heads = p.H + p.G, head_items = p.H * z.padded + p.G * z.items, items = head_items + p.G * p.dv / N, t = blockIdx.x;
  auto split = [&](int k, int& h, int& i) {                            // item k of the token: of which head
    const int kk = k - p.H * z.padded;
    h = kk < 0 ? k / z.padded : p.H + kk / z.items;
    i = kk < 0 ? k % z.padded : kk % z.items;
  };
  Item<T, N> it;
  int h = 0, i = 0;
  const int mine = threadIdx.x;
  if (kOnce && mine < head_items) {
    split(mine, h, i);
    it.place(p, z, i);
    it.weights(p, h);
  }
  pdl_launch_dependents();
  pdl_wait();
  const T* src = p.proj + static_cast<size_t>(t) * p.ld;
  const T* values = src + static_cast<size_t>(heads) * p.d;
  float sq = 0.f, sk = 0.f;
  for (int k = mine; k < (kOnce ? min(items, mine + 1) : head_items); k += blockDim.x) {
    if (k < head_items) {
      if (!kOnce) {
        split(k, h, i);
        it.place(p, z, i);
      }
      it.load(p, src + static_cast<size_t>(h) * p.d);
      const float s = it.squares();
      if (h < p.H) sq += s;
      else sk += s;
    } else {
      it.a = load_piece<T, N>(values + (k - head_items) * N);
    }
  }
  const TokenPlace<T> at = token_place(p, t);
  float co[N], si[N];
  if (kOnce) item_rotation(p, z, at.rope, mine < head_items ? i : z.pairs, co, si);
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
  for (int k = mine; k < (kOnce ? min(items, mine + 1) : items); k += blockDim.x) {
    if (k >= head_items) {
      const int v = (k - head_items) * N;
      if (!kOnce) it.a = load_piece<T, N>(values + v);
      if (at.stored) *reinterpret_cast<Piece<T, N>*>(value_place(p, at, v)) = it.a;
      continue;
    }
    if (!kOnce) {
      split(k, h, i);
      it.place(p, z, i);
      it.load(p, src + static_cast<size_t>(h) * p.d);
      it.weights(p, h);
      item_rotation(p, z, at.rope, i, co, si);
    }
    if (h < p.H || at.stored) it.store(head_place(p, at, t, h), h < p.H ? p.q_pitch : p.d, (h < p.H ? sq : sk) * head_factor(p, h), co, si);
  }
}

// Many tokens: a warp takes a token, L lanes a head at a time, one item per lane; the rotation and a head's weights stay in registers, the
// next heads' entries are under way while these are stored.  With kWhole a first pass over the heads takes the sums.
template <typename T, int N, bool kWhole>
__global__ void __launch_bounds__(256, sizeof(T) == 2 ? 3 : 2) norm_rope_warp_kernel(const NormRope<T> p, int tokens) {
  const HeadItems<T, N> z(p);
  const int L = 1 << p.lanes_log2, warp_lane = threadIdx.x & 31, lane = warp_lane & (L - 1), group = warp_lane >> p.lanes_log2, step = 32 >> p.lanes_log2;
  const int heads = p.H + p.G, t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  Item<T, N> it, next;
  it.place(p, z, lane);
  next.place(p, z, lane);
  if (!kWhole) it.weights(p, 0);                                       // weights do not come from the kernel before
  pdl_launch_dependents();
  pdl_wait();
  if (t >= tokens) return;                                             // uniform for the warp
  const T* src = p.proj + static_cast<size_t>(t) * p.ld;
  const TokenPlace<T> at = token_place(p, t);
  float sq = 0.f, sk = 0.f;
  if (kWhole) {
#pragma unroll 4
    for (int h = group; h < heads; h += step) {
      next.load(p, src + static_cast<size_t>(h) * p.d);
      const float s = next.squares();
      if (h < p.H) sq += s;
      else sk += s;
    }
    sq = rsqrtf(warp_sum_f(sq) / static_cast<float>(p.H * p.d) + p.eps);
    sk = rsqrtf(warp_sum_f(sk) / static_cast<float>(p.G * p.d) + p.eps);
  }
  float co[N], si[N];
  item_rotation(p, z, at.rope, lane, co, si);
  next.load(p, src + static_cast<size_t>(min(group, heads - 1)) * p.d);
  bool keys = false;
  for (int h0 = 0; h0 < heads; h0 += step) {                           // the same for all lanes: shuffles stay converged
    const int h = h0 + group;
    it.a = next.a;
    it.b = next.b;
    if (h0 + step < heads) next.load(p, src + static_cast<size_t>(min(h + step, heads - 1)) * p.d);
    float inv = h < p.H ? sq : sk;
    if (!kWhole) {
      float s = it.squares();
      for (int o = L >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      inv = rsqrtf(s / static_cast<float>(p.d) + p.eps);
    }
    if (h >= heads || (h >= p.H && !at.stored)) continue;
    if (kWhole || (h >= p.H && !keys)) {
      it.weights(p, h);
      keys = h >= p.H;
    }
    it.store(head_place(p, at, t, h), h < p.H ? p.q_pitch : p.d, inv * head_factor(p, h), co, si);
  }
  if (!at.stored) return;
  const T* values = src + static_cast<size_t>(heads) * p.d;
  for (int i = warp_lane * N; i < p.G * p.dv; i += 32 * N) *reinterpret_cast<Piece<T, N>*>(value_place(p, at, i)) = load_piece<T, N>(values + i);
}

template <typename T, int N>
static int norm_rope_n(NormRope<T> p, int tokens, cudaStream_t stream) {
  const int pairs = (p.rd >> 1) / N, items = items_of(pairs, (p.d - p.rd) / N), padded = items_of(pairs, (p.q_pitch - p.rd) / N);
  p.lanes_log2 = 0;
  while ((1 << p.lanes_log2) < padded && p.lanes_log2 < 5) ++p.lanes_log2;
  if (tokens >= 2048 && padded <= (1 << p.lanes_log2)) {
    auto k = p.whole ? norm_rope_warp_kernel<T, N, true> : norm_rope_warp_kernel<T, N, false>;
    return launch_kernel(k, dim3((tokens + 7) / 8), dim3(256), 0, stream, 0, p, tokens) == cudaSuccess ? 0 : -2;
  }
  if (p.whole) {
    const long long all = static_cast<long long>(p.H) * padded + static_cast<long long>(p.G) * items + static_cast<long long>(p.G) * p.dv / N;
    if (all >= (1ll << 31)) return -1;
    const bool once = all <= 1024;
    const int threads = all >= 512 && !once ? 512 : static_cast<int>((all + 31) / 32 * 32);
    auto k = once ? norm_rope_whole_kernel<T, N, true> : norm_rope_whole_kernel<T, N, false>;
    return launch_kernel(k, dim3(tokens), dim3(threads), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
  }
  const long long units = static_cast<long long>(tokens) * (p.H + 2 * p.G);
  const int per = 256 >> p.lanes_log2;
  if (units >= (1ll << 31) - 256) return -1;
  auto k = padded <= (1 << p.lanes_log2) ? norm_rope_heads_kernel<T, N, true> : norm_rope_heads_kernel<T, N, false>;
  return launch_kernel(k, dim3(static_cast<unsigned>((units + per - 1) / per)), dim3(256), 0, stream, 0, p, static_cast<int>(units)) == cudaSuccess ? 0 : -2;
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
extern "C" int forge_norm_rope_store(int fp32, const void* proj, long long ld, int tokens, const void* q_norm, const void* k_norm, int whole,
                                     float eps, const float* rope, int rope_rows, int rd, const int* positions, const int* slots, void* q,
                                     int q_pitch, void* k_cache, void* v_cache, long long num_slots, int block_size, int H, int G, int d, int dv,
                                     const float* temper, unsigned* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (rd < 0 || (rd & 1) || rd > d || q_pitch < d || (rd > 0 && rope_rows < 1) || num_slots >= (1ll << 31) || block_size < 1 || (whole && G < 1)) return -1;
#define FORGE_NORM_ROPE(T)                                                                                                             \
  return norm_rope<T>({static_cast<const T*>(proj), ld, static_cast<const T*>(q_norm), static_cast<const T*>(k_norm), rope, rope_rows, rd, positions, slots, static_cast<T*>(q),     \
                       static_cast<T*>(k_cache), static_cast<T*>(v_cache), num_slots, H, G, d, dv, q_pitch, block_size, whole, 0, eps, temper, status}, tokens, stream)
  if (fp32) FORGE_NORM_ROPE(float);
  FORGE_NORM_ROPE(bf16);
#undef FORGE_NORM_ROPE
}

}  // namespace forge
