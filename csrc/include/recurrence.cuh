// The operands of a linear recurrence with a decay per token and head, as the state-space mixer and the gated delta rule
// have it, and the quantities of a token that enter it.
//
//   state-space   S <- g S + B (dt x)^T;                                  y = S^T C + D x         key B, query C, value x
//   delta         S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;        o = S^T q               k and q unit vectors
//
// with g = exp(-exp(A_log) softplus(raw + dt_bias)), dt = softplus(raw + dt_bias), beta = sigmoid(raw).  Everything here is fp32.
#pragma once

#include "scalar.cuh"

namespace forge {

template <typename T>
struct Recurrence {
  const T* q;               // [tokens][ld], head h at (h / share) * dk
  const T* k;               // the same
  const T* v;               // [tokens][ld], head h at h * dv
  long long ld;
  const T* dt;              // [tokens][ld_raw], one column per head: the decay's raw projection
  const T* beta;            // the same; null: state-space
  long long ld_raw;
  const float* A_log;
  const float* dt_bias;
  const float* D;           // state-space only
  float* state;             // [slots][heads][dk][dv]
  const int* slots;         // [seqs]
  const int* positions;     // [tokens]
  int heads, share, dk, dv, num_slots;
  unsigned* status;
};

constexpr float kUnitEps = 1e-6f;

struct TokenGates {
  float log_g;              // log of the decay
  float w;                  // dt or beta
};

template <typename T>
__device__ __forceinline__ TokenGates token_gates(const Recurrence<T>& p, size_t t, int h) {
  const float dt = softplus_f(load_f(p.dt + t * p.ld_raw + h) + p.dt_bias[h]);
  TokenGates r;
  r.log_g = -expf(p.A_log[h]) * dt;
  r.w = p.beta != nullptr ? 1.f / (1.f + expf(-load_f(p.beta + t * p.ld_raw + h))) : dt;
  return r;
}

}  // namespace forge
