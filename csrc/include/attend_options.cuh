// Options of the windowed attention kernels that a decoder may use or not:
//
//   chunked   a query sees the tokens of its own chunk of `window` positions of the sequence instead of the last `window` tokens
//   softcap   scores are bounded, s <- softcap tanh(s / softcap); 0: they are not
//   sink      one more score per query head that only the denominator sees; null: none
//   gate      sigmoid(gate) multiplies the output, entry [token][head * gate_head + column * gate_col]; null: none
#pragma once

#include "scalar.cuh"

namespace forge {

template <typename T>
struct AttendOptions {
  int chunked;
  float softcap;
  const float* sink;        // [heads]
  const T* gate;            // rows of ldg elements
  long long ldg;
  int gate_head, gate_col;
};

__device__ __forceinline__ int oldest_visible(int pos, int window, int chunked) {
  return chunked ? pos - pos % window : max(pos - window + 1, 0);
}

template <typename T>
__device__ __forceinline__ float output_gate(const AttendOptions<T>& o, int token, int head, int col) {
  if (o.gate == nullptr) return 1.f;
  return sigmoid_t<T>(load_f(o.gate + static_cast<size_t>(token) * o.ldg + static_cast<size_t>(head) * o.gate_head + static_cast<size_t>(col) * o.gate_col));
}

// cap tanh(s / cap) log2(e), from tanh(z) = 1 - 2 / (1 + e^2z): pre = 2 log2(e) scale / cap, post = cap log2(e).  The error is a few
// units in the last place of 1, whatever the size of z.
__device__ __forceinline__ float softcap_log2(float raw, float pre, float post) {
  return fmaf(-2.f * post, __fdividef(1.f, 1.f + ex2_approx(raw * pre)), post);
}

}  // namespace forge
