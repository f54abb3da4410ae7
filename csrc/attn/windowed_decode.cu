// Decode attention over a sliding window of the paged cache (bf16): one query token per sequence, grouped queries.
//
// CTA = (key/value head and up to 16 of its query heads, sequence, chunk of the window).  Its four warps are independent: each
// takes every fourth tile of 16 keys, brings it into a ring of its own with 16-byte asynchronous copies, multiplies it with all
// query heads at once (mma.sync: heads on the 16-row side) and keeps its own running maximum, sum and output.  Softmax
// weights are fp32 and enter the second product as bf16 hi + lo halves.  The warps' states are merged through shared memory;
// with more than one chunk, partial outputs go to scratch and a second kernel merges them.  Lengths are read on the device and
// the grid depends on the batch bucket only, so the launch is CUDA-graph safe.  Options: attend_options.cuh.
//
// Pooled blocks behind the window (pooled.cuh) come ahead of it as tiles of 16 entries.  A block that ends with the step's token gets its
// entry here too: no token sees it before a later step.
#include "../include/attend_options.cuh"
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/pooled.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kWDKeys = 16, kWDWarps = 4;

struct WindowedDecode {
  const bf16* q;            // [seqs][H][q_pitch]
  const bf16* k_cache;      // [blocks][G][block_size][d]
  const bf16* v_cache;      // [blocks][G][block_size][dv]
  const int* tables;        // [seqs][width]
  const int* lens;          // [seqs]
  bf16* out;                // [seqs][ldo]
  long long ldo;
  float* part_o;            // [seqs][H][chunks][dv]
  float* part_ml;           // [seqs][H][chunks][2]
  int width, num_blocks, block_size, H, G, d, dv, q_pitch, window, chunk, max_chunks, stages, slices;
  float scale_log2, out_scale, cap_pre, cap_post;
  AttendOptions<bf16> opt;
  PoolCache<bf16> pool;
  int pool_own;             // entries of blocks that end here are made
  unsigned* status;
};

// Row pitch in elements: an odd number of 16-byte units (conflict-free ldmatrix) with room for 16-column reads.
__host__ __device__ __forceinline__ int wd_pitch(int cols) {
  const int u = cols >> 3;
  return ((u & 1) ? u + 2 : u + 1) * 8;
}

struct WindowRange {
  int begin, lo, end;       // first key of the first 16-key tile, first visible key, end of the visible keys
  int blocks, pooled;       // visible pooled blocks; the same in whole tiles
  __device__ int all() const { return pooled + end - begin; }          // places: tiles of pooled blocks, then tiles of keys
};
__device__ __forceinline__ WindowRange window_range(const WindowedDecode& p, int s, unsigned* status) {
  int len = p.lens[s];
  const int cap = p.width * p.block_size;
  if (len > cap) {
    set_status(status, kStatusBadIndex);
    len = cap;
  }
  WindowRange r;
  r.end = max(len, 0);
  r.lo = r.end > 0 ? oldest_visible(r.end - 1, p.window, p.opt.chunked) : 0;
  r.begin = r.lo & ~(kWDKeys - 1);
  r.blocks = p.pool.size > 0 ? pool_visible(r.lo, p.pool.size) : 0;
  r.pooled = (r.blocks + kWDKeys - 1) & ~(kWDKeys - 1);
  return r;
}

// 16 rows of `cols` elements: 2^lanes_log2 lanes to a row, a 16-byte unit each.
__device__ __forceinline__ void wd_load_rows(uint32_t dst, int pitch, const bf16* src, int cols, int lanes_log2, int lane) {
  const int u = lane & ((1 << lanes_log2) - 1), r0 = lane >> lanes_log2, step = 32 >> lanes_log2;
  if (u * 8 >= cols) return;
  dst += (r0 * pitch + u * 8) * 2;
  src += r0 * cols + u * 8;
#pragma unroll 8
  for (int r = r0; r < kWDKeys; r += step, dst += step * pitch * 2, src += step * cols) cp_async16(dst, src, 16);
}
// The same with rows anywhere: lane r < 16 knows row r's place.
__device__ __forceinline__ void wd_load_places(uint32_t dst, int pitch, const bf16* src, int cols, int lanes_log2, int lane, int place) {
  const int u = lane & ((1 << lanes_log2) - 1), r0 = lane >> lanes_log2, step = 32 >> lanes_log2;
  const bool in = u * 8 < cols;
#pragma unroll 8
  for (int r = 0; r < kWDKeys; r += step) {                    // the same for all lanes
    const int at = __shfl_sync(0xffffffffu, place, (r + r0) & (kWDKeys - 1));
    if (in && r + r0 < kWDKeys) cp_async16(dst + ((r + r0) * pitch + u * 8) * 2, src + static_cast<size_t>(at) * cols + u * 8, 16);
  }
}
__device__ __forceinline__ int wd_lanes_log2(int units) { return units <= 1 ? 0 : 32 - __clz(units - 1); }

// Output entry from sums O and L that are relative to the maximum M (base-2 logarithms).
__device__ __forceinline__ float wd_finish(const WindowedDecode& p, int s, int h, int c, float M, float L, float O) {
  if (p.opt.sink != nullptr) {
    const float sink = p.opt.sink[h] * 1.4426950408889634f, top = fmaxf(M, sink), f = exp2f(M - top);
    L = fmaf(L, f, exp2f(sink - top));
    O *= f;
  }
  return L > 0.f ? p.out_scale * O / L * output_gate(p.opt, s, h, c) : 0.f;
}

template <int NV, bool kCap>           // blocks of 8 value columns; bounded scores
__global__ void __launch_bounds__(32 * kWDWarps) windowed_decode_kernel(const WindowedDecode p) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int kp = wd_pitch(p.d), vp = wd_pitch(p.dv);
  const int stage = kWDKeys * (kp + vp);                       // elements per warp and stage
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);                // [16][kp]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, q2 = 2 * (lane & 3);
  bf16* ring = sQ + 16 * kp + static_cast<size_t>(warp) * p.stages * stage;

  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y, g = blockIdx.x / p.slices, slice = blockIdx.x % p.slices, chunk = blockIdx.z;
  const int per = p.H / p.G, h0 = g * per + slice * 16, nh = min(16, per - slice * 16);
  const WindowRange w = window_range(p, s, chunk == 0 ? p.status : nullptr);
  const int c_begin = chunk * p.chunk, c_end = min(c_begin + p.chunk, w.all());       // places of this CTA
  const int n_chunks = (w.all() + p.chunk - 1) / p.chunk;
  if (c_begin >= c_end) {                                      // uniform for the CTA
    if (chunk == 0)                                            // padding row: defined output
      for (int i = threadIdx.x; i < nh * p.dv; i += blockDim.x)
        p.out[static_cast<size_t>(s) * p.ldo + static_cast<size_t>(h0) * p.dv + i] = __float2bfloat16_rn(0.f);
    return;
  }
  const int dpad = (p.d + 15) & ~15, ku = p.d >> 3, qu = dpad >> 3, kl = wd_lanes_log2(ku), vl = wd_lanes_log2(p.dv >> 3);
  for (int i = threadIdx.x; i < 16 * qu; i += blockDim.x) {
    const int r = i / qu, u = i % qu;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < nh && u < ku) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<size_t>(s) * p.H + h0 + r) * p.q_pitch + u * 8);
    *reinterpret_cast<uint4*>(sQ + r * kp + u * 8) = v;
  }
  if (dpad != p.d)                                             // the key columns that complete a 16-column step stay zero
    for (int r = lane; r < p.stages * kWDKeys; r += 32)
      *reinterpret_cast<uint4*>(ring + static_cast<size_t>(r / kWDKeys) * stage + (r % kWDKeys) * kp + p.d) = make_uint4(0, 0, 0, 0);
  __syncthreads();

  const int tiles = (c_end - c_begin + kWDKeys - 1) / kWDKeys;
  const int mine = tiles > warp ? (tiles - warp + kWDWarps - 1) / kWDWarps : 0;
  auto load = [&](int i) {                                     // this warp's tile i
    if (i < mine) {
      const int at = c_begin + (i * kWDWarps + warp) * kWDKeys;
      bf16* sk = ring + static_cast<size_t>(i % p.stages) * stage;
      if (at < w.pooled) {                                     // uniform for the warp
        const int b = min(at + (lane & (kWDKeys - 1)), w.blocks - 1), page = pool_page(b, p.pool.size, p.block_size);
        int blk = p.tables[static_cast<size_t>(s) * p.width + page];
        if (blk < 0 || blk >= p.num_blocks) {
          set_status(p.status, kStatusBadIndex);
          blk = 0;
        }
        const int place = (blk * p.G + g) * p.pool.rows + pool_row(b, page, p.pool.size, p.block_size);
        wd_load_places(smem_u32(sk), kp, p.pool.k, p.d, kl, lane, place);
        wd_load_places(smem_u32(sk + kWDKeys * kp), vp, p.pool.v, p.dv, vl, lane, place);
        cp_async_commit();
        return;
      }
      const int key = w.begin + at - w.pooled;
      int blk = p.tables[static_cast<size_t>(s) * p.width + key / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        if (lane == 0) set_status(p.status, kStatusBadIndex);
        blk = 0;
      }
      const size_t row = (static_cast<size_t>(blk) * p.G + g) * p.block_size + key % p.block_size;   // 16 keys never straddle a block
      wd_load_rows(smem_u32(sk), kp, p.k_cache + row * p.d, p.d, kl, lane);
      wd_load_rows(smem_u32(sk + kWDKeys * kp), vp, p.v_cache + row * p.dv, p.dv, vl, lane);
    }
    cp_async_commit();
  };

  float o[NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int nb = 0; nb < NV; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f;
  for (int i = 0; i + 1 < p.stages; ++i) load(i);
  for (int i = 0; i < mine; ++i) {
    __syncwarp();                                              // every lane has read the stage that is filled next
    load(i + p.stages - 1);
    if (p.stages == 4) cp_async_wait<3>();
    else if (p.stages == 3) cp_async_wait<2>();
    else cp_async_wait<1>();
    __syncwarp();
    const bf16* sk = ring + static_cast<size_t>(i % p.stages) * stage;
    const bf16* sv = sk + kWDKeys * kp;
    float x[2][4] = {};
    for (int k = 0; k < dpad >> 4; ++k) {
      uint32_t a[4], b[4];
      ldsm_x4(smem_u32(sQ + (lane & 15) * kp + k * 16 + (lane >> 4) * 8), a);
      ldsm_x4(smem_u32(sk + ((lane & 7) + (lane >> 4) * 8) * kp + k * 16 + ((lane >> 3) & 1) * 8), b);
      mma16816(x[0], a, b[0], b[1]);
      mma16816(x[1], a, b[2], b[3]);
    }
    const int at = c_begin + (i * kWDWarps + warp) * kWDKeys;
    const bool means = at < w.pooled;
    const int key = means ? at : w.begin + at - w.pooled, lo = means ? 0 : w.lo, end = means ? w.blocks : w.end;     // visible: [lo, end)
    float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = key + n * 8 + q2 + (e & 1);
        const float y = kCap ? softcap_log2(x[n][e], p.cap_pre, p.cap_post) : x[n][e] * p.scale_log2;
        x[n][e] = j >= lo && j < end ? y : -INFINITY;
        mt[e >> 1] = fmaxf(mt[e >> 1], x[n][e]);
      }
    float alpha[2];
    bool moved = false;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 1));
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 2));
      const float m_new = fmaxf(m[r], mt[r]);
      moved |= m_new != m[r];
      alpha[r] = m_new == -INFINITY ? 1.f : ex2_approx(m[r] - m_new);          // nothing visible so far
      m[r] = m_new;
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int nb = 0; nb < NV; ++nb) {
        o[nb][0] *= alpha[0]; o[nb][1] *= alpha[0];
        o[nb][2] *= alpha[1]; o[nb][3] *= alpha[1];
      }
      l[0] *= alpha[0];
      l[1] *= alpha[1];
    }
    uint32_t hi[4], low[4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float ref = m[r] == -INFINITY ? 0.f : m[r];
        const float a = ex2_approx(x[n][2 * r] - ref), b = ex2_approx(x[n][2 * r + 1] - ref);
        l[r] += a + b;
        const uint32_t h = pack_bf16x2(a, b);
        hi[n * 2 + r] = h;
        low[n * 2 + r] = pack_bf16x2(a - bf16_lo(h), b - bf16_hi(h));
      }
    const bf16* vr = sv + ((lane & 7) + ((lane >> 3) & 1) * 8) * vp + (lane >> 4) * 8;
#pragma unroll
    for (int nb = 0; nb < NV; nb += 2) {
      if (nb * 8 < p.dv) {
        uint32_t b[4];
        ldsm_x4_trans(smem_u32(vr + nb * 8), b);
        mma16816(o[nb], hi, b[0], b[1]);
        mma16816(o[nb], low, b[0], b[1]);
        mma16816(o[nb + 1], hi, b[2], b[3]);
        mma16816(o[nb + 1], low, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  cp_async_wait<0>();
  __syncthreads();
  // merge the warps: [4][16][8 NV + 2] floats over the rings
  float* merge = reinterpret_cast<float*>(smem_raw);
  const int mp = NV * 8 + 2;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float* row = merge + (warp * 16 + g4 + r * 8) * mp;
#pragma unroll
    for (int nb = 0; nb < NV; ++nb) {
      row[nb * 8 + q2] = o[nb][2 * r];
      row[nb * 8 + q2 + 1] = o[nb][2 * r + 1];
    }
    if ((lane & 3) == 0) {
      row[NV * 8] = m[r];
      row[NV * 8 + 1] = l[r];
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * p.dv; i += blockDim.x) {
    const int r = i / p.dv, c = i % p.dv;
    float M = -INFINITY;
#pragma unroll
    for (int k = 0; k < kWDWarps; ++k) M = fmaxf(M, merge[(k * 16 + r) * mp + NV * 8]);
    float L = 0.f, O = 0.f;
#pragma unroll
    for (int k = 0; k < kWDWarps; ++k) {
      const float* row = merge + (k * 16 + r) * mp;
      const float f = row[NV * 8] == -INFINITY ? 0.f : exp2f(row[NV * 8] - M);
      L = fmaf(f, row[NV * 8 + 1], L);
      O = fmaf(f, row[c], O);
    }
    if (n_chunks == 1) {
      p.out[static_cast<size_t>(s) * p.ldo + static_cast<size_t>(h0 + r) * p.dv + c] = __float2bfloat16_rn(wd_finish(p, s, h0 + r, c, M, L, O));
    } else {
      const size_t at = (static_cast<size_t>(s) * p.H + h0 + r) * p.max_chunks + chunk;
      p.part_o[at * p.dv + c] = O;
      if (c == 0) {
        p.part_ml[at * 2] = M;
        p.part_ml[at * 2 + 1] = L;
      }
    }
  }
  const int size = p.pool.size;
  if (size > 0 && p.pool_own && chunk == 0 && slice == 0 && w.end % size == 0) {
    const int b = w.end / size - 1, page = pool_page(b, size, p.block_size), ku_all = p.d >> 3, units = ku_all + (p.dv >> 3);
    auto block_of = [&](int i) {
      int blk = p.tables[static_cast<size_t>(s) * p.width + i];
      if (blk < 0 || blk >= p.num_blocks) {
        set_status(p.status, kStatusBadIndex);
        blk = 0;
      }
      return static_cast<size_t>(blk) * p.G + g;
    };
    for (int u = threadIdx.x; u < units; u += blockDim.x) {
      const bool value = u >= ku_all;
      const int cols = value ? p.dv : p.d, c = (value ? u - ku_all : u) * 8;
      const bf16* cache = value ? p.v_cache : p.k_cache;
      float sum[8] = {};
#pragma unroll 8
      for (int t = b * size; t < w.end; ++t) {
        float y[8];
        load_n<8>(cache + (block_of(t / p.block_size) * p.block_size + t % p.block_size) * cols + c, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] += y[e];
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) sum[e] /= static_cast<float>(size);
      store_n<8>((value ? p.pool.v : p.pool.k) + (block_of(page) * p.pool.rows + pool_row(b, page, size, p.block_size)) * cols + c, sum);
    }
  }
}

// CTA = (query head, sequence): merges the chunks of a window that has more than one.
__global__ void __launch_bounds__(128) windowed_merge_kernel(const WindowedDecode p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y;
  const WindowRange w = window_range(p, s, nullptr);
  const int n = (w.all() + p.chunk - 1) / p.chunk;
  if (n <= 1) return;
  const size_t base = (static_cast<size_t>(s) * p.H + h) * p.max_chunks;
  float M = -INFINITY;
  for (int c = 0; c < n; ++c) M = fmaxf(M, p.part_ml[(base + c) * 2]);
  for (int i = threadIdx.x; i < p.dv; i += blockDim.x) {
    float L = 0.f, O = 0.f;
    for (int c = 0; c < n; ++c) {
      const float m = p.part_ml[(base + c) * 2], f = m == -INFINITY ? 0.f : exp2f(m - M);
      L = fmaf(f, p.part_ml[(base + c) * 2 + 1], L);
      O = fmaf(f, p.part_o[(base + c) * p.dv + i], O);
    }
    p.out[static_cast<size_t>(s) * p.ldo + static_cast<size_t>(h) * p.dv + i] = __float2bfloat16_rn(wd_finish(p, s, h, i, M, L, O));
  }
}

static size_t wd_smem(int d, int dv, int nv, int stages) {
  const size_t ring = static_cast<size_t>(16 * wd_pitch(d) + kWDWarps * stages * kWDKeys * (wd_pitch(d) + wd_pitch(dv))) * 2;
  const size_t merge = static_cast<size_t>(kWDWarps) * 16 * (nv * 8 + 2) * 4;
  return ring > merge ? ring : merge;
}

// 1 if the kernel takes these sizes (else: windowed_attend_any).
extern "C" int forge_windowed_decode_ok(int d, int dv, int block_size) {
  return (d & 7) == 0 && (dv & 7) == 0 && d >= 8 && dv >= 8 && d <= 256 && dv <= 256 && block_size % kWDKeys == 0;
}

// q [seqs][H][q_pitch], one token per sequence; out rows of ldo elements.  chunk: a multiple of 16; max_chunks * chunk must cover
// min(window, width * block_size) + 15 keys and, with pooled blocks, width * block_size / pool + 15 entries.  part_o, part_ml: fp32 scratch, needed when max_chunks > 1.
extern "C" int forge_windowed_decode(const void* q, int q_pitch, const void* k_cache, const void* v_cache, const int* tables, const int* lens,
                                     int seqs, int width, int num_blocks, int block_size, void* out, long long ldo, float* part_o, float* part_ml,
                                     int chunk, int max_chunks, int H, int G, int d, int dv, int window, float scale, float out_scale,
                                     int chunked, float softcap, const float* sink, const void* gate, long long ldg, int gate_head, int gate_col,
                                     void* pool_k, void* pool_v, int pool, int pool_own, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (pool < 0 || (pool > 0 && chunked)) return -1;
  const int pool_rows = pool > 0 ? (block_size + pool - 1) / pool : 0;
  if (static_cast<long long>(num_blocks) * G * pool_rows >= (1ll << 31)) return -1;
  if (!forge_windowed_decode_ok(d, dv, block_size) || (q_pitch & 7) || seqs > 65535 || max_chunks > 65535 || chunk % kWDKeys || chunk < kWDKeys || window < 1)
    return -1;
  const long long cap = static_cast<long long>(width) * block_size, span = (window < cap ? window : cap) + kWDKeys - 1 + (pool > 0 ? cap / pool + kWDKeys - 1 : 0);
  if (static_cast<long long>(max_chunks) * chunk < span || (max_chunks > 1 && (part_o == nullptr || part_ml == nullptr))) return -1;
  WindowedDecode p = {static_cast<const bf16*>(q), static_cast<const bf16*>(k_cache), static_cast<const bf16*>(v_cache), tables, lens,
                      static_cast<bf16*>(out), ldo, part_o, part_ml, width, num_blocks, block_size, H, G, d, dv, q_pitch, window, chunk, max_chunks,
                      0, (H / G + 15) / 16, scale * 1.4426950408889634f, out_scale,
                      softcap > 0.f ? 2.f * 1.4426950408889634f * scale / softcap : 0.f, softcap * 1.4426950408889634f,
                      {chunked, softcap, sink, static_cast<const bf16*>(gate), ldg, gate_head, gate_col},
                      {static_cast<bf16*>(pool_k), static_cast<bf16*>(pool_v), pool, pool_rows}, pool_own, status};
  const dim3 grid(G * p.slices, seqs, max_chunks);
#define FORGE_WD(NV)                                                                                                                   \
  {                                                                                                                                    \
    p.stages = 4;                                                                                                                      \
    while (p.stages > 2 && wd_smem(d, dv, NV, p.stages) > 112 * 1024) --p.stages;                                                      \
    const size_t smem = wd_smem(d, dv, NV, p.stages);                                                                                  \
    if (smem > 227 * 1024) return -1;                                                                                                  \
    FORGE_ENSURE_DYN_SMEM((windowed_decode_kernel<NV, false>), 227 * 1024);                                                            \
    FORGE_ENSURE_DYN_SMEM((windowed_decode_kernel<NV, true>), 227 * 1024);                                                             \
    auto k = softcap > 0.f ? windowed_decode_kernel<NV, true> : windowed_decode_kernel<NV, false>;                                     \
    if (launch_kernel(k, grid, dim3(32 * kWDWarps), smem, stream, 0, p) != cudaSuccess) return -2;                                         \
  }
  if (dv <= 64) FORGE_WD(8) else if (dv <= 128) FORGE_WD(16) else if (dv <= 192) FORGE_WD(24) else FORGE_WD(32)
#undef FORGE_WD
  if (max_chunks > 1 && launch_kernel(windowed_merge_kernel, dim3(H, seqs), dim3(128), 0, stream, 0, p) != cudaSuccess) return -2;
  return 0;
}

}  // namespace forge
