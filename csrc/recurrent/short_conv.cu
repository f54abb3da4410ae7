// A causal convolution over time, per channel (and its silu, if asked), with the last taps - 1 inputs of every sequence kept in its slot.
//
// x [tokens][ldx] are the step's inputs, out [tokens][channels]; state [slots][taps - 1][channels] holds the inputs before
// the step's first token (a sequence at position 0 has zeros before it, whatever its slot holds) and receives the last ones.
// CTA = (tile of tokens of one sequence, block of channels); a thread owns N channels and walks its tile with the taps in
// registers.  The CTA of a sequence's first tile is the only one that reads the old state, and the one that writes the new,
// after reading: no other CTA is involved.
#include "../include/launch.cuh"
#include "../include/scalar.cuh"

namespace forge {

constexpr int kConvMaxTaps = 8, kConvManyTaps = 32, kConvBatch = 4;

template <typename T>
struct ConvArgs {
  const T* x;
  long long ldx;
  const float* taps;        // [channels][taps]
  const float* bias;        // [channels] or null
  T* state;
  const int* slots;         // [seqs]
  const int* positions;     // [tokens]
  const int* cu;            // [seqs + 1]
  T* out;
  int channels, taps_n, num_slots, tile, silu;
  unsigned* status;
};

template <typename T, int N, int K>       // K: taps (0: any up to kConvMaxTaps; -1: up to kConvManyTaps)
__global__ void __launch_bounds__(128) short_conv_kernel(const ConvArgs<T> p) {
  constexpr int kTaps = K > 0 ? K : K == 0 ? kConvMaxTaps : kConvManyTaps;
  const int taps = K > 0 ? K : p.taps_n;
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.y, begin = p.cu[s], end = p.cu[s + 1];
  const int t0 = begin + blockIdx.x * p.tile, t1 = min(t0 + p.tile, end);
  const int c = (blockIdx.z * blockDim.x + threadIdx.x) * N;
  if (t0 >= end || c >= p.channels) return;
  const int slot = taps > 1 ? p.slots[s] : 0;    // one tap: nothing is kept
  const bool bad = taps > 1 && (slot < 0 || slot >= p.num_slots);
  if (bad) {                                     // padding rows have empty ranges: this is a corrupted step
    if (threadIdx.x == 0) set_status(p.status, kStatusBadIndex);
    return;
  }
  float w[kTaps][N], b[N], win[kTaps][N];        // win[i]: the input taps - 1 - i tokens back
#pragma unroll
  for (int e = 0; e < N; ++e) {
    b[e] = p.bias != nullptr ? p.bias[c + e] : 0.f;
#pragma unroll
    for (int i = 0; i < kTaps; ++i) w[i][e] = i < taps ? p.taps[static_cast<size_t>(c + e) * taps + i] : 0.f;
  }
  T* st = p.state + static_cast<size_t>(slot) * (taps - 1) * p.channels + c;
  const bool fresh = p.positions[begin] == 0;
  auto input = [&](int t, float* v) {            // t may lie before the step
    if (t >= begin) {
      load_n<N>(p.x + static_cast<size_t>(t) * p.ldx + c, v);
    } else if (fresh) {
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] = 0.f;
    } else {
      load_n<N>(st + static_cast<size_t>(t - begin + taps - 1) * p.channels, v);
    }
  };
#pragma unroll
  for (int i = 0; i < kTaps - 1; ++i)
    if (i < taps - 1) input(t0 - (taps - 1) + i, win[i]);
  if (blockIdx.x == 0 && taps > 1) {             // the inputs that the next step needs: those of the old state first
    float keep[kTaps][N];
#pragma unroll
    for (int i = 0; i < kTaps - 1; ++i)
      if (i < taps - 1) input(end - (taps - 1) + i, keep[i]);
#pragma unroll
    for (int i = 0; i < kTaps - 1; ++i)
      if (i < taps - 1) store_n<N>(st + static_cast<size_t>(i) * p.channels, keep[i]);
  }
  for (int ta = t0; ta < t1; ta += kConvBatch) {
    float x[kConvBatch][N];                      // loads of several tokens in flight
#pragma unroll
    for (int k = 0; k < kConvBatch; ++k) load_n<N>(p.x + static_cast<size_t>(min(ta + k, t1 - 1)) * p.ldx + c, x[k]);
#pragma unroll
    for (int k = 0; k < kConvBatch; ++k) {
#pragma unroll
      for (int i = 0; i < kTaps; ++i)
        if (i == taps - 1) {
#pragma unroll
          for (int e = 0; e < N; ++e) win[i][e] = x[k][e];
        }
      float y[N];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        float a = b[e];
#pragma unroll
        for (int i = 0; i < kTaps; ++i)
          if (i < taps) a = fmaf(w[i][e], win[i][e], a);
        y[e] = p.silu ? silu_t<T>(a) : a;
      }
      if (ta + k < t1) store_n<N>(p.out + static_cast<size_t>(ta + k) * p.channels + c, y);
#pragma unroll
      for (int i = 0; i + 1 < kTaps; ++i)
        if (i + 1 < taps) {
#pragma unroll
          for (int e = 0; e < N; ++e) win[i][e] = win[i + 1][e];
        }
    }
  }
}

template <typename T>
static int short_conv(const ConvArgs<T>& p, int seqs, int max_q, cudaStream_t stream) {
  const bool v4 = (p.channels & 3) == 0 && (p.ldx & 3) == 0 && (reinterpret_cast<uintptr_t>(p.x) & (4 * sizeof(T) - 1)) == 0;
  const int per = 128 * (v4 ? 4 : 1);
  const dim3 grid((max_q + p.tile - 1) / p.tile, seqs, (p.channels + per - 1) / per);
  if (grid.y > 65535 || grid.z > 65535) return -1;
#define FORGE_CONV(K)                                                                                                                        \
  return launch_kernel(v4 ? short_conv_kernel<T, 4, K> : short_conv_kernel<T, 1, K>, grid, dim3(128), 0, stream, 0, p) == cudaSuccess ? 0 : -2
  if (p.taps_n == 4) FORGE_CONV(4);
  if (p.taps_n == 3) FORGE_CONV(3);
  if (p.taps_n == 2) FORGE_CONV(2);
  if (p.taps_n <= kConvMaxTaps) FORGE_CONV(0);
#undef FORGE_CONV
  return launch_kernel(short_conv_kernel<T, 1, -1>, dim3(grid.x, seqs, (p.channels + 127) / 128), dim3(128), 0, stream, 0, p) == cudaSuccess ? 0 : -2;
}

extern "C" int forge_short_conv(int fp32, const void* x, long long ldx, const float* taps, const float* bias, void* state, const int* slots,
                                const int* positions, const int* cu, int seqs, int max_q, void* out, int channels, int taps_n, int num_slots,
                                int silu, unsigned* status, cudaStream_t stream) {
  if (seqs <= 0 || max_q <= 0) return 0;
  if (taps_n < 1 || taps_n > kConvManyTaps) return -1;
  const int tile = max_q > 64 ? 64 : 32;
  if (fp32)
    return short_conv<float>({static_cast<const float*>(x), ldx, taps, bias, static_cast<float*>(state), slots, positions, cu, static_cast<float*>(out),
                              channels, taps_n, num_slots, tile, silu, status}, seqs, max_q, stream);
  return short_conv<bf16>({static_cast<const bf16*>(x), ldx, taps, bias, static_cast<bf16*>(state), slots, positions, cu, static_cast<bf16*>(out),
                           channels, taps_n, num_slots, tile, silu, status}, seqs, max_q, stream);
}

}  // namespace forge
