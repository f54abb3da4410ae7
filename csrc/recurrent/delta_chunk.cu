// The gated delta rule (recurrence.cuh) over runs of tokens on the tensor cores, 64 tokens at a time (bf16 operands, fp32 state).
//
// With c_i the running sum of the logarithms of the decays in a chunk, k and q as they come (r_i and s_i the factors that make
// them unit vectors, s_i with dim^-1/2), S the state before the chunk and u_j what token j writes:
//
//   u_i = beta_i (v_i - e^c_i r_i S^T k_i - sum_{j < i} e^(c_i - c_j) r_i r_j (k_i . k_j) u_j)
//   o_i = e^c_i s_i S^T q_i + sum_{j <= i} e^(c_i - c_j) s_i r_j (q_i . k_j) u_j
//   S <- e^c_L S + sum_j e^(c_L - c_j) r_j k_j u_j^T
//
// The first line is a unit lower triangular system (I + A) u = beta (V - E K S).  delta_prepare, parallel over chunks, inverts it
// and leaves T = (I + A)^-1 diag(beta), the score matrix P of the second line and the factors; delta_chunk walks the chunks of
// a sequence with the state in accumulator registers.  fp32 throughout: fp32 factors that are operands of a product (T, P, S, u)
// enter as bf16 hi + lo halves, k, q and v are bf16 as the convolutions leave them and their factors are applied in fp32.
#include "../include/launch.cuh"
#include "../include/mma_sync.cuh"
#include "../include/recurrence.cuh"

namespace forge {

constexpr int kDC = 64, kDPitch = 72;         // tokens per chunk; row pitch of 64-column operands
constexpr int kDMats = 4 * kDC * kDC;         // elements of a chunk's T hi, T lo, P hi, P lo
constexpr int kDFactors = 3 * kDC + 4;        // e^c r, e^c s, e^(c_L - c) r, then e^c_L

struct DeltaChunk {
  const bf16* q;            // [tokens][ld], head h at (h / share) * dk
  const bf16* k;
  const bf16* v;            // [tokens][ld], head h at h * dv
  long long ld;
  const float* cum;         // [heads][ldt]: see recurrence_gates
  const float* beta;
  long long ldt;
  float* state;             // [slots][heads][dk][dv]
  const int* slots;
  const int* positions;
  const int* cu;
  bf16* mats;               // [chunks][heads][T hi, T lo, P hi, P lo][64][64]
  float* factors;           // [chunks][heads][kDFactors]
  float* o;                 // [tokens][heads][dv]
  int heads, share, dk, dv, num_slots;
  unsigned* status;
};

// Chunks of sequence s start at this index: room for every run's last, partial chunk.
__device__ __forceinline__ int first_chunk(const DeltaChunk& p, int s) { return (p.cu[s] - p.cu[0]) / kDC + s; }

// CTA = (chunk, head, sequence), four warps of 16 rows.
__global__ void __launch_bounds__(128) delta_prepare_kernel(const DeltaChunk p) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int kp = p.dk + 8;
  bf16* sk = reinterpret_cast<bf16*>(smem_raw);              // [64][kp]
  bf16* sq = sk + kDC * kp;                                  // [64][kp]
  float* sA = reinterpret_cast<float*>(sq + kDC * kp);       // [64][68]
  __shared__ __align__(16) float s_r[2][kDC], s_cum[kDC], s_beta[kDC];     // factors of k, of q
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y, t0 = p.cu[s] + blockIdx.x * kDC;
  const int L = min(kDC, p.cu[s + 1] - t0);
  if (L <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, q2 = 2 * (lane & 3);
  const int units = p.dk >> 3;
  const size_t head = static_cast<size_t>(h / p.share) * p.dk;
  for (int u = lane & 15; u < units; u += 16)                // half a warp to a row
    for (int r = warp * 2 + (lane >> 4); r < kDC; r += 8) {
      const size_t at = static_cast<size_t>(t0 + min(r, L - 1)) * p.ld + head + u * 8;
      cp_async16(smem_u32(sk + r * kp + u * 8), p.k + at, r < L ? 16 : 0);
      cp_async16(smem_u32(sq + r * kp + u * 8), p.q + at, r < L ? 16 : 0);
    }
  cp_async_commit();
  if (threadIdx.x < kDC) {
    const bool in = threadIdx.x < L;
    s_cum[threadIdx.x] = in ? p.cum[h * p.ldt + t0 + threadIdx.x] : 0.f;
    s_beta[threadIdx.x] = in ? p.beta[h * p.ldt + t0 + threadIdx.x] : 0.f;
  }
  cp_async_wait<0>();
  __syncthreads();
  {
    const int r = threadIdx.x & (kDC - 1), which = threadIdx.x >> 6;
    const bf16* row = (which ? sq : sk) + r * kp;
    float ss = 0.f;
    for (int u = 0; u < units; ++u) {
      const uint4 a = *reinterpret_cast<const uint4*>(row + u * 8);
      const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) ss += bf16_lo(w[e]) * bf16_lo(w[e]) + bf16_hi(w[e]) * bf16_hi(w[e]);
    }
    s_r[which][r] = rsqrtf(ss + kUnitEps) * (which ? rsqrtf(static_cast<float>(p.dk)) : 1.f);
  }
  __syncthreads();
  const int mt = warp;
  float kk[8][4] = {}, qk[8][4] = {};
  for (int k = 0; k < p.dk >> 4; ++k) {
    uint32_t a[4], c[4], b[4];
    ldsm_x4(smem_u32(sk + (mt * 16 + (lane & 15)) * kp + k * 16 + (lane >> 4) * 8), a);
    ldsm_x4(smem_u32(sq + (mt * 16 + (lane & 15)) * kp + k * 16 + (lane >> 4) * 8), c);
#pragma unroll
    for (int nb = 0; nb < 8; nb += 2) {
      if (nb * 8 > mt * 16 + 15) continue;                   // keys after the warp's last row
      ldsm_x4(smem_u32(sk + (nb * 8 + (lane & 7) + (lane >> 4) * 8) * kp + k * 16 + ((lane >> 3) & 1) * 8), b);
      mma16816(kk[nb], a, b[0], b[1]);
      mma16816(kk[nb + 1], a, b[2], b[3]);
      mma16816(qk[nb], c, b[0], b[1]);
      mma16816(qk[nb + 1], c, b[2], b[3]);
    }
  }
  const size_t chunk = static_cast<size_t>(first_chunk(p, s) + blockIdx.x) * p.heads + h;
  bf16* mats = p.mats + chunk * kDMats;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int i = mt * 16 + g4 + e * 8;
    const float ci = s_cum[i], ka = s_beta[i] * s_r[0][i], qa = s_r[1][i];
#pragma unroll
    for (int nb = 0; nb < 8; ++nb) {
      float x[2], y[2];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int j = nb * 8 + q2 + n;
        const float f = j <= i && i < L ? ex2_approx(ci - s_cum[j]) * s_r[0][j] : 0.f;
        x[n] = j < i ? ka * f * kk[nb][2 * e + n] : 0.f;
        y[n] = qa * f * qk[nb][2 * e + n];
      }
      *reinterpret_cast<float2*>(sA + i * 68 + nb * 8 + q2) = make_float2(x[0], x[1]);
      const uint32_t hi = pack_bf16x2(y[0], y[1]);
      bf16* dst = mats + 2 * kDC * kDC + i * kDC + nb * 8 + q2;
      *reinterpret_cast<uint32_t*>(dst) = hi;
      *reinterpret_cast<uint32_t*>(dst + kDC * kDC) = pack_bf16x2(y[0] - bf16_lo(hi), y[1] - bf16_hi(hi));
    }
  }
  if (threadIdx.x < kDC) {
    const int i = threadIdx.x;
    float* f = p.factors + chunk * kDFactors;
    const float e = ex2_approx(s_cum[i]);
    f[i] = e * s_r[0][i];
    f[kDC + i] = e * s_r[1][i];
    f[2 * kDC + i] = i < L ? ex2_approx(s_cum[L - 1] - s_cum[i]) * s_r[0][i] : 0.f;
    if (i < 4) f[3 * kDC + i] = ex2_approx(s_cum[L - 1]);
  }
  __syncthreads();
  // (I + A)^-1 by halves.  Warps 0 and 1 invert the diagonal 32 x 32 blocks, a column per lane by forward substitution in registers;
  // the lower left block is then -T22 A21 T11 (the upper right quarter of sA holds the product between).
  if (warp < 2) {
    const int b0 = warp * 32;
    float x[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      float a[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
      const float4* row = reinterpret_cast<const float4*>(sA + (b0 + i) * 68 + b0);
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 w = row[j >> 2];                        // zero from the diagonal on
        a[0] = fmaf(-w.x, x[j], a[0]);
        if (j + 1 < i) a[1] = fmaf(-w.y, x[j + 1], a[1]);
        if (j + 2 < i) a[2] = fmaf(-w.z, x[j + 2], a[2]);
        if (j + 3 < i) a[3] = fmaf(-w.w, x[j + 3], a[3]);
      }
      x[i] = (a[0] + a[1]) + (a[2] + a[3]);
    }
    __syncwarp();                                            // every lane has read the block
#pragma unroll
    for (int i = 0; i < 32; ++i) sA[(b0 + i) * 68 + b0 + lane] = x[i];
  }
  __syncthreads();
  const int pi = threadIdx.x >> 3, pj = (threadIdx.x & 7) * 4;        // rows pi and pi + 16, columns pj .. pj + 3 of a 32 x 32 product
  auto product = [&](const float* X, const float* Y, float* Z, float sign) {
    float4 acc[2] = {};
#pragma unroll 4
    for (int k = 0; k < 32; k += 4) {
      const float4 xa = *reinterpret_cast<const float4*>(X + pi * 68 + k), xb = *reinterpret_cast<const float4*>(X + (pi + 16) * 68 + k);
      const float xs[2][4] = {{xa.x, xa.y, xa.z, xa.w}, {xb.x, xb.y, xb.z, xb.w}};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 y = *reinterpret_cast<const float4*>(Y + (k + e) * 68 + pj);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          acc[r].x = fmaf(xs[r][e], y.x, acc[r].x); acc[r].y = fmaf(xs[r][e], y.y, acc[r].y);
          acc[r].z = fmaf(xs[r][e], y.z, acc[r].z); acc[r].w = fmaf(xs[r][e], y.w, acc[r].w);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float4*>(Z + (pi + 16 * r) * 68 + pj) = make_float4(sign * acc[r].x, sign * acc[r].y, sign * acc[r].z, sign * acc[r].w);
  };
  product(sA + 32 * 68, sA, sA + 32, 1.f);                   // A21 T11
  __syncthreads();
  product(sA + 32 * 68 + 32, sA + 32, sA + 32 * 68, -1.f);   // T22 (A21 T11)
  __syncthreads();
  for (int i = threadIdx.x; i < kDC * kDC / 8; i += 128) {
    const int r = i >> 3, c = (i & 7) * 8;
    float y[8], b[8], lo[8];
    load_n<8>(sA + r * 68 + c, y);
    load_n<8>(s_beta + c, b);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      y[e] = c + e > r ? 0.f : y[e] * b[e];
      lo[e] = y[e] - __bfloat162float(__float2bfloat16_rn(y[e]));
    }
    store_n<8>(mats + r * kDC + c, y);
    store_n<8>(mats + kDC * kDC + r * kDC + c, lo);
  }
}

// CTA = (kCols value columns, head, sequence), kCols / 4 warps.  MT: 16-row tiles of the state per warp; two stages: the next
// chunk's operands are on their way while this one is computed.  A warp owns 16 tokens x 16 columns of the products over
// tokens, and 16 rows (MT times) x 32 columns of the state.
template <int MT, int kStages, int kCols>
__global__ void __launch_bounds__(8 * kCols) delta_chunk_kernel(const DeltaChunk p) {
  constexpr int kWarps = kCols / 4, kP = kCols + 8;                    // row pitch of kCols-column operands: an odd number of 16-byte units
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int kp = p.dk + 8;
  const int stage = 2 * kDC * kp + kDC * kP + 4 * kDC * kDPitch;       // elements: q, k [64][kp], v [64][kP], T hi, T lo, P hi, P lo [64][72]
  bf16* base = reinterpret_cast<bf16*>(smem_raw);
  bf16* sS = base + kStages * stage;                                   // [hi, lo][dk][kP]
  bf16* sU = sS;                                                       // [hi, lo][64][kP]: u takes the place of S, which is read before it
  bf16* sR = sS + 2 * max(p.dk, kDC) * kP;                             // [hi, lo][64][kP]
  float* sF = reinterpret_cast<float*>(sR + 2 * kDC * kP);             // [stages][kDFactors]

  pdl_launch_dependents();
  pdl_wait();
  const int c0 = blockIdx.x * kCols, h = blockIdx.y, s = blockIdx.z;
  const int t_begin = p.cu[s], t_end = p.cu[s + 1];
  if (t_begin >= t_end) return;
  const int slot = p.slots[s];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g4 = lane >> 2, q2 = 2 * (lane & 3);
  const int steps = p.dk >> 4, units = p.dk >> 3, chunks = (t_end - t_begin + kDC - 1) / kDC;
  const size_t chunk0 = first_chunk(p, s);
  float* slot_state = p.state + (static_cast<size_t>(slot) * p.heads + h) * p.dk * p.dv;
  const bool fresh = p.positions[t_begin] == 0;

  // state fragments: rows (rt + 8 m) * 16 + g4 (+ 8), columns sc + nb * 8 + q2 (+ 1)
  const int rt = warp & 7, sc = (warp >> 3) * 32;
  float st[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nb = 0; nb < 4; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (rt + 8 * m) * 16 + g4 + (e >> 1) * 8, c = c0 + sc + nb * 8 + q2 + (e & 1);
        st[m][nb][e] = !fresh && r < p.dk && c < p.dv ? slot_state[static_cast<size_t>(r) * p.dv + c] : 0.f;
      }

  auto load_chunk = [&](int n, int at) {
    bf16* sq = base + at * stage;
    bf16* sk = sq + kDC * kp;
    bf16* sv = sk + kDC * kp;
    bf16* sT = sv + kDC * kP;
    const int t0 = t_begin + n * kDC;
    const size_t head = static_cast<size_t>(h / p.share) * p.dk;
    for (int r = warp; r < kDC; r += kWarps) {
      const bool in = t0 + r < t_end;
      const size_t row = static_cast<size_t>(in ? t0 + r : t0) * p.ld;
      for (int u = lane; u < units; u += 32) {
        cp_async16(smem_u32(sq + r * kp + u * 8), p.q + row + head + u * 8, in ? 16 : 0);
        cp_async16(smem_u32(sk + r * kp + u * 8), p.k + row + head + u * 8, in ? 16 : 0);
      }
      if (lane < kCols / 8) {
        const bool vin = in && c0 + lane * 8 < p.dv;
        cp_async16(smem_u32(sv + r * kP + lane * 8), vin ? p.v + row + static_cast<size_t>(h) * p.dv + c0 + lane * 8 : p.q, vin ? 16 : 0);
      }
    }
    const size_t chunk = (chunk0 + n) * p.heads + h;
    const bf16* mats = p.mats + chunk * kDMats;
    for (int i = threadIdx.x; i < kDMats / 8; i += kWarps * 32) cp_async16(smem_u32(sT + (i >> 3) * kDPitch + (i & 7) * 8), mats + i * 8, 16);
    const float* f = p.factors + chunk * kDFactors;
    if (threadIdx.x < kDFactors / 4) cp_async16(smem_u32(sF + at * kDFactors + threadIdx.x * 4), f + threadIdx.x * 4, 16);
  };
  if (kStages == 2) {
    load_chunk(0, 0);
    cp_async_commit();
  }
  const int nh = warp >> 2, mt = nh & 1 ? 3 - (warp & 3) : warp & 3;   // 16 columns, 16 tokens: the triangles even out over the SM's quarters
  const int col = nh * 16 + q2, row = mt * 16 + g4;
  auto split_store = [&](bf16* dst, float x, float y) {                // two neighbours as hi and lo halves
    const uint32_t hi = pack_bf16x2(x, y);
    *reinterpret_cast<uint32_t*>(dst) = hi;
    *reinterpret_cast<uint32_t*>(dst + kDC * kP) = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
  };
  // acc += M B for a lower triangular M [64][64] and B [64][kCols], both as hi and lo halves: this warp's tokens and columns
  auto triangular = [&](const bf16* M, const bf16* B, float (&acc)[2][4]) {
    for (int k = 0; k <= mt; ++k) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      const uint32_t at = smem_u32(M + (mt * 16 + (lane & 15)) * kDPitch + k * 16 + (lane >> 4) * 8);
      const uint32_t bt = smem_u32(B + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kP + nh * 16 + (lane >> 4) * 8);
      ldsm_x4(at, ah);
      ldsm_x4_trans(bt, bh);
      ldsm_x4(at + kDC * kDPitch * 2, al);
      ldsm_x4_trans(bt + kDC * kP * 2, bl);
      mma16816(acc[0], ah, bh[0], bh[1]);
      mma16816(acc[1], ah, bh[2], bh[3]);
      mma16816(acc[0], al, bh[0], bh[1]);
      mma16816(acc[1], al, bh[2], bh[3]);
      mma16816(acc[0], ah, bl[0], bl[1]);
      mma16816(acc[1], ah, bl[2], bl[3]);
    }
  };

  for (int n = 0; n < chunks; ++n) {
    const int now = kStages == 2 ? n & 1 : 0, t0 = t_begin + n * kDC, L = min(kDC, t_end - t0);
    __syncthreads();                                                   // the chunk before is done with shared memory
    if (kStages == 1) load_chunk(n, 0);
    else if (n + 1 < chunks) load_chunk(n + 1, now ^ 1);
    cp_async_commit();
    const bf16* sq = base + now * stage;
    const bf16* sk = sq + kDC * kp;
    const bf16* sv = sk + kDC * kp;
    const bf16* sT = sv + kDC * kP;
    const bf16* sP = sT + 2 * kDC * kDPitch;
    const float* f = sF + now * kDFactors;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (rt + 8 * m >= steps) continue;
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          bf16* dst = sS + ((rt + 8 * m) * 16 + g4 + e * 8) * kP + sc + nb * 8 + q2;
          const float x = st[m][nb][2 * e], y = st[m][nb][2 * e + 1];
          const uint32_t hi = pack_bf16x2(x, y);
          *reinterpret_cast<uint32_t*>(dst) = hi;
          *reinterpret_cast<uint32_t*>(dst + p.dk * kP) = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
        }
    }
    cp_async_wait<kStages - 1>();
    __syncthreads();

    float ks[2][4] = {}, qs[2][4] = {};                                // k and q against the state
#pragma unroll 2
    for (int k = 0; k < steps; ++k) {
      uint32_t a[4], c[4], bh[4], bl[4];
      const uint32_t at = smem_u32(sk + (mt * 16 + (lane & 15)) * kp + k * 16 + (lane >> 4) * 8);
      const uint32_t bt = smem_u32(sS + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kP + nh * 16 + (lane >> 4) * 8);
      ldsm_x4(at, a);
      ldsm_x4(at - kDC * kp * 2, c);
      ldsm_x4_trans(bt, bh);
      ldsm_x4_trans(bt + p.dk * kP * 2, bl);
      mma16816(ks[0], a, bh[0], bh[1]);
      mma16816(ks[1], a, bh[2], bh[3]);
      mma16816(qs[0], c, bh[0], bh[1]);
      mma16816(qs[1], c, bh[2], bh[3]);
      mma16816(ks[0], a, bl[0], bl[1]);
      mma16816(ks[1], a, bl[2], bl[3]);
      mma16816(qs[0], c, bl[0], bl[1]);
      mma16816(qs[1], c, bl[2], bl[3]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = row + e * 8;
      const float ek = f[i], eq = f[kDC + i];
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        const uint32_t v = *reinterpret_cast<const uint32_t*>(sv + i * kP + col + nb * 8);
        split_store(sR + i * kP + col + nb * 8, fmaf(-ek, ks[nb][2 * e], bf16_lo(v)), fmaf(-ek, ks[nb][2 * e + 1], bf16_hi(v)));
        qs[nb][2 * e] *= eq;
        qs[nb][2 * e + 1] *= eq;
      }
    }
    __syncthreads();
    float u[2][4] = {};
    triangular(sT, sR, u);
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) split_store(sU + (row + e * 8) * kP + col + nb * 8, u[nb][2 * e], u[nb][2 * e + 1]);
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 2; ++e) {                                      // nobody reads R any more: u with the factors of the state's update
      const float w = f[2 * kDC + row + e * 8];
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) split_store(sR + (row + e * 8) * kP + col + nb * 8, w * u[nb][2 * e], w * u[nb][2 * e + 1]);
    }
    triangular(sP, sU, qs);
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = row + e * 8, c = c0 + col + nb * 8;
        if (i < L && c < p.dv)
          *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(t0 + i) * p.heads + h) * p.dv + c) = make_float2(qs[nb][2 * e], qs[nb][2 * e + 1]);
      }
    __syncthreads();
    const float keep = f[3 * kDC];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nb = 0; nb < 4; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[m][nb][e] *= keep;
#pragma unroll
    for (int k = 0; k < kDC / 16; ++k) {
      const uint32_t bt = smem_u32(sR + (k * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kP + sc + (lane >> 4) * 8);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        if (rt + 8 * m >= steps) continue;
        uint32_t a[4], b[4];
        ldsm_x4_trans(smem_u32(sk + (k * 16 + (lane & 7) + (lane >> 4) * 8) * kp + (rt + 8 * m) * 16 + ((lane >> 3) & 1) * 8), a);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int nb = 0; nb < 4; nb += 2) {
            ldsm_x4_trans(bt + part * kDC * kP * 2 + nb * 16, b);
            mma16816(st[m][nb], a, b[0], b[1]);
            mma16816(st[m][nb + 1], a, b[2], b[3]);
          }
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nb = 0; nb < 4; ++nb)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = (rt + 8 * m) * 16 + g4 + e * 8, c = c0 + sc + nb * 8 + q2;
        if (r < p.dk && c < p.dv)
          *reinterpret_cast<float2*>(slot_state + static_cast<size_t>(r) * p.dv + c) = make_float2(st[m][nb][2 * e], st[m][nb][2 * e + 1]);
      }
}

static size_t delta_chunk_smem(int dk, int stages, int cols) {
  const size_t pitch = cols + 8;
  return static_cast<size_t>(stages) * ((2 * kDC * (dk + 8) + kDC * pitch + 4 * kDC * kDPitch) * 2 + kDFactors * 4) +
         (2 * (dk > kDC ? dk : kDC) + 2 * kDC) * pitch * 2;
}

// 1 if the kernels take these sizes (else: recurrence, the scan).
extern "C" int forge_delta_chunk_ok(int dk, int dv) { return dk % 16 == 0 && dk >= 16 && dk <= 256 && dv % 8 == 0 && dv >= 8; }

// Elements of scratch for `tokens` tokens in `seqs` runs: mats (which = 0, bf16), factors (which = 1, fp32).
extern "C" long long forge_delta_chunk_scratch(int tokens, int seqs, int heads, int which) {
  const long long chunks = static_cast<long long>(tokens) / kDC + seqs;
  return chunks * heads * (which == 0 ? kDMats : kDFactors);
}

// q, k, v [tokens][ld] (after the convolutions), cum and beta [heads][ldt] from recurrence_gates; sequence s has the step's tokens
// cu[s] .. cu[s + 1]; o fp32 [tokens][heads][dv].  cols: value columns per CTA (32 or 64).
extern "C" int forge_delta_chunk(const void* q, const void* k, const void* v, long long ld, int share, const float* cum, const float* beta,
                                 long long ldt, float* state, const int* slots, const int* positions, const int* cu, int seqs, int max_q, int heads,
                                 int dk, int dv, int num_slots, void* mats, float* factors, float* o, int cols, unsigned* status,
                                 cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0) return 0;
  if (cols != 32 && cols != 64) return -1;
  const uintptr_t any = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(mats) |
                        reinterpret_cast<uintptr_t>(factors);
  if (!forge_delta_chunk_ok(dk, dv) || (ld & 7) || (any & 15) || seqs > 65535 || heads > 65535) return -1;
  const DeltaChunk p = {static_cast<const bf16*>(q), static_cast<const bf16*>(k), static_cast<const bf16*>(v), ld, cum, beta, ldt, state, slots, positions,
                        cu, static_cast<bf16*>(mats), factors, o, heads, share, dk, dv, num_slots, status};
  const size_t prep = static_cast<size_t>(2 * kDC * (dk + 8)) * 2 + kDC * 68 * 4;
  FORGE_ENSURE_DYN_SMEM(delta_prepare_kernel, 100 * 1024);
  if (launch_kernel(delta_prepare_kernel, dim3((max_q + kDC - 1) / kDC, heads, seqs), dim3(128), prep, stream, 0, p) != cudaSuccess) return -2;
  const dim3 grid((dv + cols - 1) / cols, heads, seqs);
#define FORGE_DELTA(MT, STAGES, COLS)                                                                                                     \
  {                                                                                                                                       \
    FORGE_ENSURE_DYN_SMEM((delta_chunk_kernel<MT, STAGES, COLS>), 227 * 1024);                                                            \
    return launch_kernel(delta_chunk_kernel<MT, STAGES, COLS>, grid, dim3(8 * COLS), delta_chunk_smem(dk, STAGES, COLS), stream, 0, p) == \
                   cudaSuccess ? 0 : -2;                                                                                                  \
  }
  if (cols == 64) {
    if (dk <= 128) FORGE_DELTA(1, 2, 64)
    FORGE_DELTA(2, 1, 64)
  }
  if (dk <= 128) FORGE_DELTA(1, 2, 32)
  FORGE_DELTA(2, 1, 32)
#undef FORGE_DELTA
}

}  // namespace forge
