// Grouped-query attention over a sliding window of a paged cache: what stands before it, and the form for any sizes.
//
//   bias_rope_store     q | k | v of a token + biases; q and k rotated (first rd entries of a head, entry i with i + rd / 2); q to
//                       [token][head][q_pitch] (padding columns zero), k and v to the caches [block][kv_head][block_size][dim / vdim]
//   windowed_attend_any softmax attention of a token over itself and the window - 1 tokens before it (or the tokens of its chunk of
//                       the sequence), with the options of attend_options.cuh, bf16 or fp32, any sizes: one warp per query token,
//                       eight tokens of one head per CTA share key and value tiles of 32; pooled blocks (pooled.cuh) come ahead of the window
//
// Scores, weights and sums are fp32.
#include "../include/attend_options.cuh"
#include "../include/launch.cuh"
#include "../include/pooled.cuh"
#include "../include/scalar.cuh"

namespace forge {

template <typename T>
struct QkvArgs {
  const T* proj;            // [tokens][ld]
  long long ld;
  const float* bias;        // [H d + G d + G dv]
  const float* rope;        // [rope_rows][rd]
  int rope_rows, rd;
  const int* positions;
  const int* slots;
  T* q;
  T* k_cache;
  T* v_cache;
  long long num_slots;
  int H, G, d, dv, q_pitch, block_size;
  unsigned* status;
};

// CTA = kTok tokens.  The work of a token is a list of items of N entries: per query and key head the rotated pairs, then the
// entries that pass (and a query's padding); then the values.  A thread keeps its item's bias for all tokens.
template <typename T, int N, int kTok>
__global__ void __launch_bounds__(512) bias_rope_store_kernel(const QkvArgs<T> p, int tokens, uint32_t magic) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = p.rd >> 1, pairs = half / N, rest = (p.d - p.rd) / N, per = pairs + (p.q_pitch - p.rd) / N, heads = p.H + p.G;
  const int vper = p.dv / N, items = heads * per + p.G * vper;
  for (int i = threadIdx.x; i < items; i += blockDim.x) {
    const bool value = i >= heads * per;
    const int h = value ? heads + (i - heads * per) / vper : per == 1 ? i : static_cast<int>(__umulhi(static_cast<uint32_t>(i), magic));
    const int k = value ? (i - heads * per) % vper : i - h * per;
    const bool pair = !value && k < pairs, pad = !value && k >= pairs + rest, query = h < p.H;
    if (pad && !query) continue;
    const int c = value ? k * N : pair ? k * N : p.rd + (k - pairs) * N;
    const size_t at = value ? static_cast<size_t>(heads) * p.d + static_cast<size_t>(h - heads) * p.dv + c : static_cast<size_t>(h) * p.d + c;
    float ab[N], bb[N];
#pragma unroll
    for (int e = 0; e < N; ++e) ab[e] = bb[e] = 0.f;
    if (!pad) load_n<N>(p.bias + at, ab);
    if (pair) load_n<N>(p.bias + at + half, bb);
#pragma unroll
    for (int u = 0; u < kTok; ++u) {
      const int t = blockIdx.x * kTok + u;
      if (t >= tokens) break;
      const T* src = p.proj + static_cast<size_t>(t) * p.ld + at;
      T* dst;
      if (query) {
        dst = p.q + (static_cast<size_t>(t) * p.H + h) * p.q_pitch + c;
      } else {
        const long long slot = p.slots[t];
        if (slot < 0) continue;
        if (slot >= p.num_slots) {
          set_status(p.status, kStatusBadIndex);
          continue;
        }
        const size_t blk = slot / p.block_size, off = slot % p.block_size;
        dst = value ? p.v_cache + ((blk * p.G + (h - heads)) * p.block_size + off) * p.dv + c
                    : p.k_cache + ((blk * p.G + (h - p.H)) * p.block_size + off) * p.d + c;
      }
      float a[N];
#pragma unroll
      for (int e = 0; e < N; ++e) a[e] = 0.f;
      if (!pad) load_n<N>(src, a);
#pragma unroll
      for (int e = 0; e < N; ++e) a[e] += ab[e];
      if (pair) {
        int pos = p.positions[t];
        pos = pos < 0 ? 0 : (pos >= p.rope_rows ? p.rope_rows - 1 : pos);
        const float* cs = p.rope + static_cast<size_t>(pos) * p.rd + c;
        float b[N], co[N], si[N], y[N];
        load_n<N>(src + half, b);
        load_n<N>(cs, co);
        load_n<N>(cs + half, si);
#pragma unroll
        for (int e = 0; e < N; ++e) {
          b[e] += bb[e];
          y[e] = b[e] * co[e] + a[e] * si[e];
          a[e] = a[e] * co[e] - b[e] * si[e];
        }
        store_n<N>(dst + half, y);
      }
      store_n<N>(dst, a);
    }
  }
}

template <typename T, int N>
static int bias_rope_store_n(const QkvArgs<T>& p, int tokens, cudaStream_t stream) {
  const int per = (p.rd >> 1) / N + (p.q_pitch - p.rd) / N, items = (p.H + p.G) * per + p.G * (p.dv / N);
  if (per < 1) return -1;
  const uint32_t magic = per == 1 ? 0u : static_cast<uint32_t>(((1ull << 32) + per - 1) / per);    // exact for the item counts of a token
  const int threads = items >= 512 ? 512 : ((items + 31) / 32) * 32;
  if (static_cast<long long>(items) * per >= (1ll << 32)) return -1;
  if (tokens >= 2048)
    return launch_kernel(bias_rope_store_kernel<T, N, 4>, dim3((tokens + 3) / 4), dim3(threads), 0, stream, 0, p, tokens, magic) == cudaSuccess ? 0 : -2;
  return launch_kernel(bias_rope_store_kernel<T, N, 1>, dim3(tokens), dim3(threads), 0, stream, 0, p, tokens, magic) == cudaSuccess ? 0 : -2;
}

template <typename T>
static int bias_rope_store(const QkvArgs<T>& p, int tokens, cudaStream_t stream) {
  const uintptr_t proj = reinterpret_cast<uintptr_t>(p.proj);
  const int all = (p.rd >> 1) | p.d | p.dv | p.q_pitch | static_cast<int>(p.ld & 7);
  if (sizeof(T) == 2 && (all & 7) == 0 && (proj & 15) == 0) return bias_rope_store_n<T, 8>(p, tokens, stream);
  if ((all & 3) == 0 && (proj & (4 * sizeof(T) - 1)) == 0) return bias_rope_store_n<T, 4>(p, tokens, stream);
  return bias_rope_store_n<T, 1>(p, tokens, stream);
}

extern "C" int forge_bias_rope_store(int fp32, const void* proj, long long ld, int tokens, const float* bias, const float* rope, int rope_rows,
                                     int rd, const int* positions, const int* slots, void* q, int q_pitch, void* k_cache, void* v_cache,
                                     long long num_slots, int block_size, int H, int G, int d, int dv, unsigned* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (rd < 0 || (rd & 1) || rd > d || q_pitch < d) return -1;
  if (fp32)
    return bias_rope_store<float>({static_cast<const float*>(proj), ld, bias, rope, rope_rows, rd, positions, slots, static_cast<float*>(q),
                                   static_cast<float*>(k_cache), static_cast<float*>(v_cache), num_slots, H, G, d, dv, q_pitch, block_size, status}, tokens, stream);
  return bias_rope_store<bf16>({static_cast<const bf16*>(proj), ld, bias, rope, rope_rows, rd, positions, slots, static_cast<bf16*>(q),
                                static_cast<bf16*>(k_cache), static_cast<bf16*>(v_cache), num_slots, H, G, d, dv, q_pitch, block_size, status}, tokens, stream);
}

constexpr int kWTok = 8, kWKeys = 32, kWMaxCols = 16;      // query tokens per CTA, keys per tile, value columns per lane

template <typename T>
struct AttendAny {
  const T* q;               // [tokens][H][q_pitch]
  const T* k_cache;
  const T* v_cache;
  const int* cu;            // [seqs + 1] rows of the sequences' queries
  const int* positions;     // [tokens]
  const int* tables;        // [seqs][width]
  T* out;                   // [tokens][ldo]
  long long ldo;
  int width, num_blocks, block_size, H, G, d, dv, q_pitch, window;
  float scale, out_scale;
  AttendOptions<T> opt;
  PoolCache<T> pool;
  unsigned* status;
};

template <typename T>
__global__ void __launch_bounds__(256) windowed_attend_any_kernel(const AttendAny<T> p) {
  extern __shared__ float sm[];
  const int kp = p.d + 1;
  float* sk = sm;                                  // [32][d + 1]
  float* sv = sk + kWKeys * kp;                    // [32][dv]
  float* sq = sv + kWKeys * p.dv;                  // [8][d]
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y, g = h / (p.H / p.G);
  const int begin = p.cu[s], end = p.cu[s + 1];
  const int t0 = begin + blockIdx.x * kWTok;
  if (t0 >= end) return;                           // uniform for the CTA
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = min(kWTok, end - t0), t = t0 + warp;
  const bool live = warp < n;
  for (int i = threadIdx.x; i < n * p.d; i += blockDim.x)
    sq[i] = load_f(p.q + (static_cast<size_t>(t0 + i / p.d) * p.H + h) * p.q_pitch + i % p.d);
  const int first = p.positions[t0], pos = live ? p.positions[t] : -1;
  const int last = first + n - 1, cap = p.width * p.block_size;
  const int lo = oldest_visible(first, p.window, p.opt.chunked), mine = live ? oldest_visible(pos, p.window, p.opt.chunked) : 0;
  float m = -INFINITY, l = 0.f, acc[kWMaxCols];
#pragma unroll
  for (int c = 0; c < kWMaxCols; ++c) acc[c] = 0.f;
  if (last >= cap) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
  }
  // entries of the pooled blocks that the last token sees, then the tokens of the windows
  const int size = p.pool.size, blocks = size > 0 ? pool_visible(oldest_visible(min(last, cap - 1), p.window, 0), size) : 0;
  const int pooled = (blocks + kWKeys - 1) / kWKeys * kWKeys, j_first = lo / kWKeys * kWKeys - pooled;
  for (int i0 = 0; i0 < pooled || (j_first + i0 <= last && j_first + i0 < cap); i0 += kWKeys) {
    const bool means = i0 < pooled;                // uniform for the CTA
    const int j0 = means ? i0 : j_first + i0, end = means ? blocks : min(last + 1, cap), per = means ? p.pool.rows : p.block_size;
    const T* k_src = means ? p.pool.k : p.k_cache;
    const T* v_src = means ? p.pool.v : p.v_cache;
    __syncthreads();
    for (int r = warp; r < kWKeys; r += 8) {       // one key per warp at a time
      const int j = j0 + r, page = means ? pool_page(j, size, p.block_size) : j / p.block_size;
      int blk = j < end ? p.tables[static_cast<size_t>(s) * p.width + page] : -1;
      if (j < end && (blk < 0 || blk >= p.num_blocks)) {
        if (lane == 0) set_status(p.status, kStatusBadIndex);
        blk = -1;
      }
      const int at = blk < 0 ? 0 : means ? pool_row(j, page, size, p.block_size) : j % p.block_size;
      const size_t row = (static_cast<size_t>(max(blk, 0)) * p.G + g) * per + at;
      for (int c = lane; c < p.d; c += 32) sk[r * kp + c] = blk < 0 ? 0.f : load_f(k_src + row * p.d + c);
      for (int c = lane; c < p.dv; c += 32) sv[r * p.dv + c] = blk < 0 ? 0.f : load_f(v_src + row * p.dv + c);
    }
    __syncthreads();
    if (!live) continue;
    const int j = j0 + lane;
    float x = 0.f;
    for (int c = 0; c < p.d; ++c) x = fmaf(sq[warp * p.d + c], sk[lane * kp + c], x);
    x *= p.scale;
    if (p.opt.softcap > 0.f) x = p.opt.softcap * tanhf(x / p.opt.softcap);
    if (means ? j >= pool_visible(mine, size) : j > pos || j < mine) x = -INFINITY;
    float mt = x;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
    if (mt == -INFINITY) continue;                 // uniform for the warp
    const float m_new = fmaxf(m, mt), alpha = expf(m - m_new), w = expf(x - m_new);
    m = m_new;
    l = l * alpha + warp_sum_f(w);
#pragma unroll
    for (int c = 0; c < kWMaxCols; ++c) acc[c] *= alpha;
    for (int r = 0; r < kWKeys; ++r) {
      const float wr = __shfl_sync(0xffffffffu, w, r);
#pragma unroll
      for (int c = 0; c < kWMaxCols; ++c)
        if (c * 32 < p.dv && c * 32 + lane < p.dv) acc[c] = fmaf(wr, sv[r * p.dv + c * 32 + lane], acc[c]);
    }
  }
  if (!live) return;
  float top = m;
  if (p.opt.sink != nullptr) {                     // one more score, of the denominator alone
    top = fmaxf(m, p.opt.sink[h]);
    l = l * expf(m - top) + expf(p.opt.sink[h] - top);
  }
  const float inv = l > 0.f ? p.out_scale * expf(m - top) / l : 0.f;
  T* dst = p.out + static_cast<size_t>(t) * p.ldo + static_cast<size_t>(h) * p.dv;
#pragma unroll
  for (int c = 0; c < kWMaxCols; ++c)
    if (c * 32 + lane < p.dv) store_f(dst + c * 32 + lane, acc[c] * inv * output_gate(p.opt, t, h, c * 32 + lane));
}

template <typename T>
static int windowed_attend_any(const AttendAny<T>& p, int seqs, int max_q, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(kWKeys * (p.d + 1 + p.dv) + kWTok * p.d) * 4;
  if (smem > 200 * 1024 || p.dv > 32 * kWMaxCols) return -1;
  auto k = windowed_attend_any_kernel<T>;
  FORGE_ENSURE_DYN_SMEM(k, 200 * 1024);
  return launch_kernel(k, dim3((max_q + kWTok - 1) / kWTok, p.H, seqs), dim3(256), smem, stream, 0, p) == cudaSuccess ? 0 : -2;
}

// Sequence s: query rows cu[s] .. cu[s + 1] (consecutive positions), keys by tables[s].  Padding rows: an empty range.
extern "C" int forge_windowed_attend_any(int fp32, const void* q, int q_pitch, const void* k_cache, const void* v_cache, const int* cu, int seqs,
                                         int max_q, const int* positions, const int* tables, int width, int num_blocks, int block_size,
                                         void* out, long long ldo, int H, int G, int d, int dv, int window, float scale, float out_scale,
                                         int chunked, float softcap, const float* sink, const void* gate, long long ldg, int gate_head,
                                         int gate_col, const void* pool_k, const void* pool_v, int pool, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0) return 0;
  if (window < 1 || pool < 0 || (pool > 0 && chunked)) return -1;
  const int rows = pool > 0 ? (block_size + pool - 1) / pool : 0;
  if (seqs > 65535 || H > 65535) return -1;
  if (fp32)
    return windowed_attend_any<float>({static_cast<const float*>(q), static_cast<const float*>(k_cache), static_cast<const float*>(v_cache), cu, positions,
                                       tables, static_cast<float*>(out), ldo, width, num_blocks, block_size, H, G, d, dv, q_pitch, window, scale, out_scale,
                                       {chunked, softcap, sink, static_cast<const float*>(gate), ldg, gate_head, gate_col},
                                       {const_cast<float*>(static_cast<const float*>(pool_k)), const_cast<float*>(static_cast<const float*>(pool_v)), pool, rows}, status},
                                      seqs, max_q, stream);
  return windowed_attend_any<bf16>({static_cast<const bf16*>(q), static_cast<const bf16*>(k_cache), static_cast<const bf16*>(v_cache), cu, positions,
                                    tables, static_cast<bf16*>(out), ldo, width, num_blocks, block_size, H, G, d, dv, q_pitch, window, scale, out_scale,
                                    {chunked, softcap, sink, static_cast<const bf16*>(gate), ldg, gate_head, gate_col},
                                    {const_cast<bf16*>(static_cast<const bf16*>(pool_k)), const_cast<bf16*>(static_cast<const bf16*>(pool_v)), pool, rows}, status},
                                   seqs, max_q, stream);
}

}  // namespace forge
