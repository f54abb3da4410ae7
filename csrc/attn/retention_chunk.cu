// Retention, and the state-space recurrence (recurrence.cuh), over runs of tokens on the tensor cores, 64 tokens at a time (bf16
// operands, fp32 state).
//
// With g the head's decay and S the state before a chunk of L tokens:
//
//   o_i = g^(i+1) S^T q_i + sum_{j <= i} g^(i-j) (q_i . k_j) v_j            S <- g^L S + sum_j g^(L-1-j) k_j v_j^T
//
// (k_j carries dim^-1/2, applied in fp32 to the weights).  The state-space form (kGated) has a decay per token: with c_i the running
// sum of the logarithms of the decays in the chunk, g^(i-j) becomes exp(c_i - c_j), k_j carries dt_j instead, and D x_i is added.  Everything of the recurrence stays in fp32: the state lives in
// accumulator registers; where it, the decayed scores or the decayed keys are operands of a product they enter as bf16
// hi + lo halves (two products, 16 mantissa bits).  q and k come rotated (retention_rotate, in place).
//
// CTA = (columns of the values, head, sequence x segment).  Two shapes: 16 warps over 128 columns with the next chunk's rows on
// their way while this one is computed (heads up to 128 wide), or 8 warps over 64 columns.  A long run is cut into segments so that a few long
// prompts fill the GPU: the segments' own end states are computed first, a scan over them gives every segment its initial
// state, and then all segments compute their outputs at the same time.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/recurrence.cuh"

namespace forge {

constexpr int kRC = 64, kRPP = kRC + 8;      // tokens per chunk; row pitch of the decayed scores (odd number of 16-byte units)

struct RetentionChunk {
  const bf16* q;            // [tokens][ld] (rotated), head h at (h / share) * dk
  const bf16* k;            // the same
  const bf16* v;            // [tokens][ld], head h at h * dv
  int ld, share;
  const float* decay;       // one per head, or
  const float* cum;         // [heads][ldt]: running sum of log2 of the decays in the token's chunk,
  const float* weight;      // [heads][ldt]: the factor of k_j,
  long long ldt;
  const float* skip;        // [heads]: the factor of v_i in o_i,
  float* seg_decay;         // [seqs][segs][heads]: log2 of a segment's decay
  float* state;             // [slots][heads][dk][dv]
  const int* slots;         // [seqs]
  const int* positions;     // [tokens]
  const int* cu;            // [seqs + 1]
  float* ws;                // [seqs][segs][heads][dk][dv], segs > 1 only
  float* o;                 // [tokens][heads][dv]
  int heads, dk, dv, num_slots, segs, seg_len;
  unsigned* status;
};

// fp32 products of an A fragment with per-column weights, split into hi and lo fragments.
__device__ __forceinline__ void weigh_split(const uint32_t* a, float w0, float w1, float w2, float w3, uint32_t* hi, uint32_t* lo) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float x = bf16_lo(a[i]) * (i < 2 ? w0 : w2), y = bf16_hi(a[i]) * (i < 2 ? w1 : w3);
    hi[i] = pack_bf16x2(x, y);
    lo[i] = pack_bf16x2(x - bf16_lo(hi[i]), y - bf16_hi(hi[i]));
  }
}

// kWide: 16 warps, 128 columns, two stages; else 8 warps, 64 columns, one stage.  MT: 16-row tiles of the state per warp.
template <int MT, bool kStateOnly, bool kWide, bool kGated>
__global__ void __launch_bounds__(kWide ? 512 : 256, kWide || MT == 2 ? 1 : 2) retention_chunk_kernel(const RetentionChunk p) {
  constexpr int kWarps = kWide ? 16 : 8, kQuarters = kWarps / 4, kCols = 32 * kQuarters, kRPitch = kCols + 8, kStages = kWide ? 2 : 1;
  constexpr int kKB = 8 / kQuarters;                                   // 8-key blocks of the scores per warp
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int kp = p.dk + 8;                                             // dk is a multiple of 16: an odd number of units
  const int stage = kRC * (2 * kp + kRPitch);                          // elements: q [64][kp], k [64][kp], v [64][kRPitch]
  bf16* sS = reinterpret_cast<bf16*>(smem_raw) + kStages * stage;      // [hi, lo][dk][kRPitch]
  bf16* sP = sS + 2 * p.dk * kRPitch;                                  // [hi, lo][64][kRPP]
  float* pw = reinterpret_cast<float*>(sP + 2 * kRC * kRPP);           // [65]: g^i; kGated: [stages][c_i, weight][64]

  pdl_launch_dependents();
  pdl_wait();
  const int c0 = blockIdx.x * kCols, h = blockIdx.y;
  const int seq = blockIdx.z / p.segs, seg = blockIdx.z % p.segs;
  const int run = p.cu[seq + 1] - p.cu[seq];
  const int n_segs = p.segs == 1 ? 1 : min((run + p.seg_len - 1) / p.seg_len, p.segs);
  if (run <= 0 || seg >= n_segs || (kStateOnly && seg == n_segs - 1)) return;
  const int t_begin = p.cu[seq] + seg * p.seg_len;
  const int t_end = seg == n_segs - 1 ? p.cu[seq + 1] : t_begin + p.seg_len;
  const int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, q2 = 2 * (lane & 3);
  const float ks = rsqrtf(static_cast<float>(p.dk));
  if (!kGated && threadIdx.x <= kRC) pw[threadIdx.x] = powf(p.decay[h], static_cast<float>(threadIdx.x));
  float total = 0.f;                                                   // log2 of the decay so far (kGated)

  const int steps = p.dk >> 4;
  const bool both = steps > 4;                     // a warp owns two 32-column parts of its state rows, or one
  const size_t head_state = static_cast<size_t>(p.dk) * p.dv;
  float* slot_state = p.state + (static_cast<size_t>(slot) * p.heads + h) * head_state;
  float* seg_state = p.segs == 1 ? nullptr : p.ws + ((static_cast<size_t>(seq) * p.segs + seg) * p.heads + h) * head_state;
  const bool fresh = p.positions[p.cu[seq]] == 0;
  const float* init = kStateOnly ? nullptr : (p.segs > 1 ? seg_state : (fresh ? nullptr : slot_state));

  // state fragments: rows row_tile * 16 + g4 (+ 8), columns col_part * 32 + nb * 8 + q2 (+ 1)
  float st[MT][2][4][4];
  auto row_tile = [&](int m) { return both ? (warp & 7) + 8 * m : (warp & 3); };
  auto col_part = [&](int i) { return both ? (warp >> 3) * 2 + i : (warp >> 2); };
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = row_tile(m) * 16 + g4 + (e >> 1) * 8, c = c0 + col_part(i) * 32 + nb * 8 + q2 + (e & 1);
          st[m][i][nb][e] = (init != nullptr && (both || i == 0) && r < p.dk && c < p.dv) ? init[static_cast<size_t>(r) * p.dv + c] : 0.f;
        }

  const int units = p.dk >> 3;
  auto load_chunk = [&](int t0, int st) {
    bf16* sq = reinterpret_cast<bf16*>(smem_raw) + st * stage;
    bf16* sk = sq + kRC * kp;
    bf16* sv = sk + kRC * kp;
    for (int r = warp; r < kRC; r += kWarps) {
      const bool in = t0 + r < t_end;
      const size_t row = static_cast<size_t>(in ? t0 + r : t0) * p.ld;
      const bf16* qr = p.q + row + (h / p.share) * p.dk;
      const bf16* kr = p.k + row + (h / p.share) * p.dk;
      const bf16* vr = p.v + row + h * p.dv + c0;
      for (int u = lane; u < units; u += 32) {
        if (!kStateOnly) cp_async16(smem_u32(sq + r * kp + u * 8), qr + u * 8, in ? 16 : 0);
        cp_async16(smem_u32(sk + r * kp + u * 8), kr + u * 8, in ? 16 : 0);
      }
      if (lane < kCols / 8) {
        const bool vin = in && c0 + lane * 8 < p.dv;
        cp_async16(smem_u32(sv + r * kRPitch + lane * 8), vin ? vr + lane * 8 : qr, vin ? 16 : 0);
      }
    }
    if (kGated && threadIdx.x < 2 * kRC) {
      const int r = threadIdx.x & (kRC - 1);
      const bool in = t0 + r < t_end;
      const float* src = (threadIdx.x < kRC ? p.cum : p.weight) + h * p.ldt + (in ? t0 + r : t0);
      cp_async4(smem_u32(pw + st * 2 * kRC + threadIdx.x), src, in ? 4 : 0);
    }
  };
  if (kStages == 2) {
    load_chunk(t_begin, 0);
    cp_async_commit();
  }
  int st_now = 0;
  const float skip = kGated ? p.skip[h] : 0.f;
  for (int t0 = t_begin; t0 < t_end; t0 += kRC) {
    const int L = min(kRC, t_end - t0);
    __syncthreads();                                                   // the chunk before is done with shared memory
    if (kStages == 1) load_chunk(t0, 0);
    else if (t0 + kRC < t_end) load_chunk(t0 + kRC, st_now ^ 1);
    cp_async_commit();
    const bf16* sq = reinterpret_cast<bf16*>(smem_raw) + st_now * stage;
    const bf16* sk = sq + kRC * kp;
    const bf16* sv = sk + kRC * kp;
    const float* cum = pw + st_now * 2 * kRC;
    const float* wgt = cum + kRC;
    st_now ^= kStages - 1;
    if (!kStateOnly) {                                                 // the state before this chunk as hi and lo operands
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          if ((!both && i == 1) || row_tile(m) >= steps) continue;
#pragma unroll
          for (int nb = 0; nb < 4; ++nb)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              bf16* dst = sS + (row_tile(m) * 16 + g4 + e * 8) * kRPitch + col_part(i) * 32 + nb * 8 + q2;
              const float x = st[m][i][nb][2 * e], y = st[m][i][nb][2 * e + 1];
              const uint32_t hi = pack_bf16x2(x, y);
              *reinterpret_cast<uint32_t*>(dst) = hi;
              *reinterpret_cast<uint32_t*>(dst + p.dk * kRPitch) = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
            }
        }
    }
    cp_async_wait<kStages - 1>();
    __syncthreads();

    if (!kStateOnly) {
      const int mt = warp & 3, nh = warp >> 2;                         // 16 tokens; 8 kKB keys, then 32 value columns
      float s[kKB][4], o[4][4];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[nb][e] = s[nb % kKB][e] = 0.f;
      const bool any_key = nh * 8 * kKB <= mt * 16 + 15;
      for (int k = 0; k < steps; ++k) {
        uint32_t a[4], b[4];
        ldsm_x4(smem_u32(sq + (mt * 16 + (lane & 15)) * kp + k * 16 + (lane >> 4) * 8), a);
        if (any_key) {
#pragma unroll
          for (int nb = 0; nb < kKB; nb += 2) {
            ldsm_x4(smem_u32(sk + (nh * 8 * kKB + nb * 8 + (lane & 7) + (lane >> 4) * 8) * kp + k * 16 + ((lane >> 3) & 1) * 8), b);
            mma16816(s[nb], a, b[0], b[1]);
            mma16816(s[nb + 1], a, b[2], b[3]);
          }
        }
        const bf16* sr = sS + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kRPitch + nh * 32 + (lane >> 4) * 8;
#pragma unroll
        for (int nb = 0; nb < 4; nb += 2) {
          ldsm_x4_trans(smem_u32(sr + nb * 8), b);
          mma16816(o[nb], a, b[0], b[1]);
          mma16816(o[nb + 1], a, b[2], b[3]);
          ldsm_x4_trans(smem_u32(sr + p.dk * kRPitch + nb * 8), b);
          mma16816(o[nb], a, b[0], b[1]);
          mma16816(o[nb + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = mt * 16 + g4 + e * 8;
#pragma unroll
        for (int nb = 0; nb < kKB; ++nb) {
          const int j = nh * 8 * kKB + nb * 8 + q2;
          float x = 0.f, y = 0.f;
          if (kGated) {
            if (j <= i) x = s[nb][2 * e] * (ex2_approx(cum[i] - cum[j]) * wgt[j]);
            if (j + 1 <= i) y = s[nb][2 * e + 1] * (ex2_approx(cum[i] - cum[j + 1]) * wgt[j + 1]);
          } else {
            if (j <= i) x = s[nb][2 * e] * (pw[i - j] * ks);
            if (j + 1 <= i) y = s[nb][2 * e + 1] * (pw[i - j - 1] * ks);
          }
          const uint32_t hi = pack_bf16x2(x, y);
          bf16* dst = sP + i * kRPP + j;
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + kRC * kRPP) = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
        }
        const float past = kGated ? ex2_approx(cum[i]) : pw[i + 1];
#pragma unroll
        for (int nb = 0; nb < 4; ++nb) {
          o[nb][2 * e] *= past;
          o[nb][2 * e + 1] *= past;
        }
      }
      __syncthreads();
      for (int k = 0; k <= mt; ++k) {                                  // keys up to this warp's last token
        uint32_t ah[4], al[4], b[4];
        const uint32_t at = smem_u32(sP + (mt * 16 + (lane & 15)) * kRPP + k * 16 + (lane >> 4) * 8);
        ldsm_x4(at, ah);
        ldsm_x4(at + kRC * kRPP * 2, al);
        const bf16* vr = sv + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kRPitch + nh * 32 + (lane >> 4) * 8;
#pragma unroll
        for (int nb = 0; nb < 4; nb += 2) {
          ldsm_x4_trans(smem_u32(vr + nb * 8), b);
          mma16816(o[nb], ah, b[0], b[1]);
          mma16816(o[nb + 1], ah, b[2], b[3]);
          mma16816(o[nb], al, b[0], b[1]);
          mma16816(o[nb + 1], al, b[2], b[3]);
        }
      }
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = mt * 16 + g4 + e * 8, c = c0 + nh * 32 + nb * 8 + q2;
          if (kGated) {
            const uint32_t x = *reinterpret_cast<const uint32_t*>(sv + i * kRPitch + nh * 32 + nb * 8 + q2);
            o[nb][2 * e] = fmaf(skip, bf16_lo(x), o[nb][2 * e]);
            o[nb][2 * e + 1] = fmaf(skip, bf16_hi(x), o[nb][2 * e + 1]);
          }
          if (i < L && c < p.dv)
            *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(t0 + i) * p.heads + h) * p.dv + c) = make_float2(o[nb][2 * e], o[nb][2 * e + 1]);
        }
    }

    const float keep = kGated ? ex2_approx(cum[L - 1]) : pw[L];
    if (kGated) total += cum[L - 1];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int nb = 0; nb < 4; ++nb)
#pragma unroll
          for (int e = 0; e < 4; ++e) st[m][i][nb][e] *= keep;
#pragma unroll
    for (int k = 0; k < kRC / 16; ++k) {
      if (k * 16 >= L) continue;
      float w[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = k * 16 + q2 + (e & 1) + (e >> 1) * 8;
        w[e] = j >= L ? 0.f : kGated ? ex2_approx(cum[L - 1] - cum[j]) * wgt[j] : pw[L - 1 - j] * ks;
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        if (row_tile(m) >= steps) continue;
        uint32_t a[4], ah[4], al[4], b[4];
        ldsm_x4_trans(smem_u32(sk + (k * 16 + (lane & 7) + (lane >> 4) * 8) * kp + row_tile(m) * 16 + ((lane >> 3) & 1) * 8), a);
        weigh_split(a, w[0], w[1], w[2], w[3], ah, al);
        const bf16* vr = sv + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kRPitch + (lane >> 4) * 8;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          if (!both && i == 1) continue;
#pragma unroll
          for (int nb = 0; nb < 4; nb += 2) {
            ldsm_x4_trans(smem_u32(vr + col_part(i) * 32 + nb * 8), b);
            mma16816(st[m][i][nb], ah, b[0], b[1]);
            mma16816(st[m][i][nb + 1], ah, b[2], b[3]);
            mma16816(st[m][i][nb], al, b[0], b[1]);
            mma16816(st[m][i][nb + 1], al, b[2], b[3]);
          }
        }
      }
    }
  }

  if (kGated && kStateOnly && blockIdx.x == 0 && threadIdx.x == 0)
    p.seg_decay[(static_cast<size_t>(seq) * p.segs + seg) * p.heads + h] = total;
  float* dst = kStateOnly ? seg_state : (seg == n_segs - 1 ? slot_state : nullptr);
  if (dst == nullptr) return;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = row_tile(m) * 16 + g4 + e * 8, c = c0 + col_part(i) * 32 + nb * 8 + q2;
          if ((both || i == 0) && r < p.dk && c < p.dv)
            *reinterpret_cast<float2*>(dst + static_cast<size_t>(r) * p.dv + c) = make_float2(st[m][i][nb][2 * e], st[m][i][nb][2 * e + 1]);
        }
}

// ws[seq][seg] <- the state before segment `seg`: S_0 = the slot's state (or zero), S_(s+1) = g^seg_len S_s + own end state of s.
__global__ void __launch_bounds__(256) retention_segments_kernel(const RetentionChunk p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z;
  const int run = p.cu[seq + 1] - p.cu[seq];
  const int slot = p.slots[seq];
  if (run <= 0 || slot < 0 || slot >= p.num_slots) return;
  const int n_segs = min((run + p.seg_len - 1) / p.seg_len, p.segs);
  const int n = p.dk * p.dv, i = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= n) return;
  const float g = p.cum != nullptr ? 0.f : powf(p.decay[h], static_cast<float>(p.seg_len));
  float s[4] = {0.f, 0.f, 0.f, 0.f};
  if (p.positions[p.cu[seq]] != 0) load_n<4>(p.state + (static_cast<size_t>(slot) * p.heads + h) * n + i, s);
  for (int seg = 0; seg < n_segs; ++seg) {
    float* w = p.ws + ((static_cast<size_t>(seq) * p.segs + seg) * p.heads + h) * n + i;
    float own[4];
    if (seg + 1 < n_segs) load_n<4>(w, own);
    store_n<4>(w, s);
    if (seg + 1 < n_segs) {
      const float f = p.cum != nullptr ? exp2f(p.seg_decay[(static_cast<size_t>(seq) * p.segs + seg) * p.heads + h]) : g;
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] = fmaf(f, s[e], own[e]);
    }
  }
}

// q and k of the tokens from tok0 on, rotated in place (first rd entries of every head; rd a multiple of 8).
__global__ void __launch_bounds__(128) retention_rotate_kernel(bf16* __restrict__ qkvg, int ld, int tok0, int heads2, int dk, int rd,
                                                               const float* __restrict__ rope, int rope_rows, const int* __restrict__ positions) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = tok0 + blockIdx.x;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= rope_rows ? rope_rows - 1 : pos);
  const float* cs = rope + static_cast<size_t>(pos) * rd;
  bf16* row = qkvg + static_cast<size_t>(t) * ld;
  const int half = rd >> 1, per = half >> 2;
  for (int i = threadIdx.x; i < heads2 * per; i += blockDim.x) {
    bf16* v = row + (i / per) * dk + (i % per) * 4;
    const float* c = cs + (i % per) * 4;
    float a[4], b[4], x[4], y[4];
    load_n<4>(v, a);
    load_n<4>(v + half, b);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[e] = a[e] * c[e] - b[e] * c[half + e];
      y[e] = b[e] * c[e] + a[e] * c[half + e];
    }
    store_n<4>(v, x);
    store_n<4>(v + half, y);
  }
}

static size_t retention_chunk_smem(int dk, bool wide) {
  const int pitch = wide ? 136 : 72;
  return static_cast<size_t>((wide ? 2 : 1) * kRC * (2 * (dk + 8) + pitch) + 2 * dk * pitch + 2 * kRC * kRPP) * 2 + 4 * kRC * 4;
}

// Value columns per CTA for these sizes.
extern "C" int forge_retention_chunk_cols(int dk, int dv) { return dk <= 128 && dv > 64 ? 128 : 64; }

// 1 if the kernels take these sizes (else: retention_scan).
extern "C" int forge_retention_chunk_ok(int heads, int dk, int dv, int rd) {
  return dk % 16 == 0 && dk >= 16 && dk <= 256 && dv % 8 == 0 && rd % 8 == 0 && heads > 0 && (2 * heads * (dk + dv)) % 8 == 0;
}

template <bool kGated>
static int run_chunks(const RetentionChunk& p, int seqs, cudaStream_t stream) {
  const int cols = forge_retention_chunk_cols(p.dk, p.dv);
  const bool wide = cols == 128;
  const dim3 grid((p.dv + cols - 1) / cols, p.heads, seqs * p.segs);
  const size_t smem = retention_chunk_smem(p.dk, wide);
#define FORGE_RC(MT, ONLY, WIDE)                                                                                           \
  {                                                                                                                        \
    auto k = retention_chunk_kernel<MT, ONLY, WIDE, kGated>;                                                               \
    FORGE_ENSURE_DYN_SMEM(k, static_cast<int>(retention_chunk_smem(128 * MT, WIDE)));                                      \
    if (launch_kernel(k, grid, dim3(WIDE ? 512 : 256), smem, stream, 0, p) != cudaSuccess) return -2;                      \
  }
  if (p.segs > 1) {
    if (wide) FORGE_RC(1, true, true) else if (p.dk <= 128) FORGE_RC(1, true, false) else FORGE_RC(2, true, false)
    if (launch_kernel(retention_segments_kernel, dim3((p.dk * p.dv / 4 + 255) / 256, p.heads, seqs), dim3(256), 0, stream, 0, p) != cudaSuccess) return -2;
  }
  if (wide) FORGE_RC(1, false, true) else if (p.dk <= 128) FORGE_RC(1, false, false) else FORGE_RC(2, false, false)
#undef FORGE_RC
  return 0;
}

// Rotates q and k of qkvg in place, then runs sequence s over the step's tokens cu[s] .. cu[s + 1] (cu[0] == tok0, cu[seqs] == tokens).
// segs > 1: every run is cut into segments of seg_len tokens (a multiple of 64), at most `segs` of them; ws holds their states.
extern "C" int forge_retention_chunk(void* qkvg, int ld, const float* decay, float* state, const int* slots, const int* positions,
                                     const float* rope, int rope_rows, int rd, const int* cu, int seqs, int tok0, int tokens, int heads, int dk,
                                     int dv, int num_slots, float* o, float* ws, int segs, int seg_len, unsigned* status,
                                     cudaStream_t stream) {
  if (seqs <= 0 || tokens <= tok0) return 0;
  if (!forge_retention_chunk_ok(heads, dk, dv, rd) || segs < 1 || static_cast<long long>(seqs) * segs > 65535 || (ld & 7) ||
      (reinterpret_cast<uintptr_t>(qkvg) & 15) || (segs > 1 && (ws == nullptr || seg_len < kRC || seg_len % kRC)))
    return -1;
  if (rd > 0 && launch_kernel(retention_rotate_kernel, dim3(tokens - tok0), dim3(128), 0, stream, 0, static_cast<bf16*>(qkvg), ld, tok0, 2 * heads,
                              dk, rd, rope, rope_rows, positions) != cudaSuccess)
    return -2;
  const bf16* rows = static_cast<const bf16*>(qkvg);
  return run_chunks<false>({rows, rows + heads * dk, rows + 2 * heads * dk, ld, 1, decay, nullptr, nullptr, 0, nullptr, nullptr, state, slots, positions,
                            cu, ws, o, heads, dk, dv, num_slots, segs, seg_len, status}, seqs, stream);
}

// The same for the state-space recurrence: q, k [tokens][ld] with head h at (h / share) * dk, v with head h at h * dv; cum, weight
// [heads][ldt] as recurrence_gates leaves them.
extern "C" int forge_state_space_chunk(const void* q, const void* k, const void* v, long long ld, int share, const float* cum, const float* weight,
                                       long long ldt, const float* skip, float* state, const int* slots, const int* positions, const int* cu,
                                       int seqs, int heads, int dk, int dv, int num_slots, float* o, float* ws, float* seg_decay, int segs,
                                       int seg_len, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  const uintptr_t any = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v);
  if (!forge_retention_chunk_ok(heads, dk, dv, 0) || segs < 1 || static_cast<long long>(seqs) * segs > 65535 || (ld & 7) || ld >= (1ll << 31) ||
      (any & 15) || (segs > 1 && (ws == nullptr || seg_decay == nullptr || seg_len < kRC || seg_len % kRC)))
    return -1;
  return run_chunks<true>({static_cast<const bf16*>(q), static_cast<const bf16*>(k), static_cast<const bf16*>(v), static_cast<int>(ld), share, nullptr, cum,
                           weight, ldt, skip, seg_decay, state, slots, positions, cu, ws, o, heads, dk, dv, num_slots, segs, seg_len, status},
                          seqs, stream);
}

// CTA = (64-token chunk of a sequence's run, sequence); a warp takes a head at a time, a lane two tokens.
template <typename T>
__global__ void __launch_bounds__(256) recurrence_gates_kernel(const Recurrence<T> p, const int* __restrict__ cu, float* __restrict__ cum,
                                                               float* __restrict__ weight, long long ldt) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y, t0 = cu[s] + blockIdx.x * kRC, end = min(cu[s + 1], t0 + kRC);
  if (t0 >= end) return;
  const int lane = threadIdx.x & 31, a = t0 + 2 * lane;
  for (int h = threadIdx.x >> 5; h < p.heads; h += blockDim.x >> 5) {
    TokenGates x = {0.f, 0.f}, y = {0.f, 0.f};
    if (a < end) x = token_gates(p, a, h);
    if (a + 1 < end) y = token_gates(p, a + 1, h);
    float sum = x.log_g + y.log_g;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, sum, off);
      if (lane >= off) sum += v;
    }
    const float before = sum - y.log_g;
    if (a < end) {
      cum[h * ldt + a] = before * 1.4426950408889634f;
      weight[h * ldt + a] = x.w;
    }
    if (a + 1 < end) {
      cum[h * ldt + a + 1] = sum * 1.4426950408889634f;
      weight[h * ldt + a + 1] = y.w;
    }
  }
}

// cum, weight [heads][ldt] for the tokens of the runs: the running sum of log2 of the decays within 64-token chunks counted from
// the run's first token, and dt (state-space) or beta (delta).
extern "C" int forge_recurrence_gates(const void* dt, const void* beta, long long ld_raw, const float* A_log, const float* dt_bias, const int* cu,
                                      int seqs, int max_q, int heads, float* cum, float* weight, long long ldt, cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0) return 0;
  if (seqs > 65535) return -1;
  Recurrence<bf16> p = {};
  p.dt = static_cast<const bf16*>(dt);
  p.beta = static_cast<const bf16*>(beta);
  p.ld_raw = ld_raw;
  p.A_log = A_log;
  p.dt_bias = dt_bias;
  p.heads = heads;
  return launch_kernel(recurrence_gates_kernel<bf16>, dim3((max_q + kRC - 1) / kRC, seqs), dim3(256), 0, stream, 0, p, cu, cum, weight, ldt) == cudaSuccess ? 0 : -2;
}

}  // namespace forge
