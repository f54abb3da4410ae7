// Grouped-query attention over a sliding window of a paged cache: what stands before it, and the form for any sizes.
//
//   bias_rope_store     q | k | v of a token + biases; q and k rotated (first rd entries of a head, entry i with i + rd / 2); q to
//                       [token][head][q_pitch] (padding columns zero), k and v to the caches [block][kv_head][block_size][dim / vdim]
//   windowed_attend_any softmax attention of a token over itself and the window - 1 tokens before it, bf16 or fp32, any sizes: one
//                       warp per query token, eight tokens of one head per CTA share key and value tiles of 32
//
// Scores, weights and sums are fp32.
#include "../include/launch.cuh"
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

// CTA = one token.  N entries of a rotated pair half at a time.
template <typename T, int N>
__global__ void __launch_bounds__(256) bias_rope_store_kernel(const QkvArgs<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const T* row = p.proj + static_cast<size_t>(t) * p.ld;
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.rope_rows ? p.rope_rows - 1 : pos);
  const float* cs = p.rope + static_cast<size_t>(pos) * p.rd;
  const long long slot = p.slots[t];
  const bool store = slot >= 0 && slot < p.num_slots;
  if (slot >= p.num_slots && threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
  const int half = p.rd >> 1, heads = p.H + p.G;
  const size_t blk = store ? slot / p.block_size : 0, off = store ? slot % p.block_size : 0;
  auto dest = [&](int h) -> T* {
    if (h < p.H) return p.q + (static_cast<size_t>(t) * p.H + h) * p.q_pitch;
    return p.k_cache + ((blk * p.G + (h - p.H)) * p.block_size + off) * p.d;
  };
  // rotated pairs
  const int pairs = half / N;
  for (int i = threadIdx.x; i < heads * pairs; i += blockDim.x) {
    const int h = i / pairs, c = (i % pairs) * N;
    const size_t at = static_cast<size_t>(h) * p.d + c;
    float a[N], b[N], ab[N], bb[N], co[N], si[N], x[N], y[N];
    load_n<N>(row + at, a);
    load_n<N>(row + at + half, b);
    load_n<N>(p.bias + at, ab);
    load_n<N>(p.bias + at + half, bb);
    load_n<N>(cs + c, co);
    load_n<N>(cs + half + c, si);
#pragma unroll
    for (int e = 0; e < N; ++e) {
      a[e] += ab[e];
      b[e] += bb[e];
      x[e] = a[e] * co[e] - b[e] * si[e];
      y[e] = b[e] * co[e] + a[e] * si[e];
    }
    if (h < p.H || store) {
      T* dst = dest(h) + c;
      store_n<N>(dst, x);
      store_n<N>(dst + half, y);
    }
  }
  // the entries that pass, and the padding of q
  const int rest = p.d - p.rd, per = rest / N;
  for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
    const int h = i / per, c = p.rd + (i % per) * N;
    const size_t at = static_cast<size_t>(h) * p.d + c;
    float a[N], b[N];
    load_n<N>(row + at, a);
    load_n<N>(p.bias + at, b);
#pragma unroll
    for (int e = 0; e < N; ++e) a[e] += b[e];
    if (h < p.H || store) store_n<N>(dest(h) + c, a);
  }
  const int pad = p.q_pitch - p.d;
  for (int i = threadIdx.x; i < p.H * pad; i += blockDim.x) store_f(dest(i / pad) + p.d + i % pad, 0.f);
  // values
  if (!store) return;
  const int vat = heads * p.d, vper = p.dv / N;
  for (int i = threadIdx.x; i < p.G * vper; i += blockDim.x) {
    const int g = i / vper, c = (i % vper) * N;
    float a[N], b[N];
    load_n<N>(row + vat + g * p.dv + c, a);
    load_n<N>(p.bias + vat + g * p.dv + c, b);
#pragma unroll
    for (int e = 0; e < N; ++e) a[e] += b[e];
    store_n<N>(p.v_cache + ((blk * p.G + g) * p.block_size + off) * p.dv + c, a);
  }
}

template <typename T>
static int bias_rope_store(const QkvArgs<T>& p, int tokens, cudaStream_t stream) {
  const bool v4 = ((p.rd >> 1) & 3) == 0 && ((p.d | p.dv | p.q_pitch) & 3) == 0 && (p.ld & 3) == 0 && (reinterpret_cast<uintptr_t>(p.proj) & (4 * sizeof(T) - 1)) == 0;
  return launch_kernel(v4 ? bias_rope_store_kernel<T, 4> : bias_rope_store_kernel<T, 1>, dim3(tokens), dim3(256), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
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
  const int lo = max(first - p.window + 1, 0);
  float m = -INFINITY, l = 0.f, acc[kWMaxCols];
#pragma unroll
  for (int c = 0; c < kWMaxCols; ++c) acc[c] = 0.f;
  if (last >= cap) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
  }
  for (int j0 = lo / kWKeys * kWKeys; j0 <= last && j0 < cap; j0 += kWKeys) {
    __syncthreads();
    for (int r = warp; r < kWKeys; r += 8) {       // one key per warp at a time
      const int j = j0 + r;
      int blk = j <= last && j < cap ? p.tables[static_cast<size_t>(s) * p.width + j / p.block_size] : -1;
      if (j <= last && (blk < 0 || blk >= p.num_blocks)) {
        if (lane == 0) set_status(p.status, kStatusBadIndex);
        blk = -1;
      }
      const size_t row = (static_cast<size_t>(max(blk, 0)) * p.G + g) * p.block_size + j % p.block_size;
      for (int c = lane; c < p.d; c += 32) sk[r * kp + c] = blk < 0 ? 0.f : load_f(p.k_cache + row * p.d + c);
      for (int c = lane; c < p.dv; c += 32) sv[r * p.dv + c] = blk < 0 ? 0.f : load_f(p.v_cache + row * p.dv + c);
    }
    __syncthreads();
    if (!live) continue;
    const int j = j0 + lane;
    float x = 0.f;
    for (int c = 0; c < p.d; ++c) x = fmaf(sq[warp * p.d + c], sk[lane * kp + c], x);
    x = j <= pos && pos - j < p.window ? x * p.scale : -INFINITY;
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
  const float inv = l > 0.f ? p.out_scale / l : 0.f;
  T* dst = p.out + static_cast<size_t>(t) * p.ldo + static_cast<size_t>(h) * p.dv;
#pragma unroll
  for (int c = 0; c < kWMaxCols; ++c)
    if (c * 32 + lane < p.dv) store_f(dst + c * 32 + lane, acc[c] * inv);
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
                                         unsigned* status, cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0) return 0;
  if (seqs > 65535 || H > 65535) return -1;
  if (fp32)
    return windowed_attend_any<float>({static_cast<const float*>(q), static_cast<const float*>(k_cache), static_cast<const float*>(v_cache), cu, positions,
                                       tables, static_cast<float*>(out), ldo, width, num_blocks, block_size, H, G, d, dv, q_pitch, window, scale, out_scale, status},
                                      seqs, max_q, stream);
  return windowed_attend_any<bf16>({static_cast<const bf16*>(q), static_cast<const bf16*>(k_cache), static_cast<const bf16*>(v_cache), cu, positions,
                                    tables, static_cast<bf16*>(out), ldo, width, num_blocks, block_size, H, G, d, dv, q_pitch, window, scale, out_scale, status},
                                   seqs, max_q, stream);
}

}  // namespace forge
