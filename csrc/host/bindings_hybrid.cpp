// Bindings of the ops of hybrid decoders: windowed attention, short convolutions, recurrences with a decay per token.  Every
// argument is checked here, as in bindings.cpp.
#include "checks.h"

extern "C" {
int forge_bias_rope_store(int fp32, const void* proj, long long ld, int tokens, const float* bias, const float* rope, int rope_rows, int rd,
                          const int* positions, const int* slots, void* q, int q_pitch, void* k_cache, void* v_cache, long long num_slots,
                          int block_size, int H, int G, int d, int dv, unsigned* status, cudaStream_t stream);
int forge_windowed_attend_any(int fp32, const void* q, int q_pitch, const void* k_cache, const void* v_cache, const int* cu, int seqs, int max_q,
                              const int* positions, const int* tables, int width, int num_blocks, int block_size, void* out, long long ldo, int H,
                              int G, int d, int dv, int window, float scale, float out_scale, unsigned* status, cudaStream_t stream);
int forge_short_conv(int fp32, const void* x, long long ldx, const float* taps, const float* bias, void* state, const int* slots,
                     const int* positions, const int* cu, int seqs, int max_q, void* out, int channels, int taps_n, int num_slots,
                     unsigned* status, cudaStream_t stream);
int forge_recurrence_decode_ok(int dk, int dv);
int forge_recurrence(int fp32, const void* q, const void* k, const void* v, long long ld, const void* dt, const void* beta, long long ld_raw,
                     const float* A_log, const float* dt_bias, const float* D, float* state, const int* slots, const int* positions,
                     const int* cu, int seqs, int heads, int share, int dk, int dv, int num_slots, float* o, unsigned* status,
                     cudaStream_t stream);
int forge_gated_norm(int fp32, const float* o, const void* gate, long long ldg, const float* weight, int weight_period, void* out, long long ldo,
                     int tokens, int groups, int n, int gate_first, float factor, float eps, cudaStream_t stream);
}

namespace {

struct Caches {
  int64_t blocks, G, block_size, d, dv;
};
Caches cache_sizes(const Tensor& k_cache, const Tensor& v_cache, at::ScalarType dt) {
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && v_cache.size(0) == k_cache.size(0) && v_cache.size(1) == k_cache.size(1) && v_cache.size(2) == k_cache.size(2),
              "caches: [blocks, kv_heads, block_size, dim] and [.., vdim] expected");
  need(k_cache, dt, 0, "k_cache");
  need(v_cache, dt, 0, "v_cache");
  return {k_cache.size(0), k_cache.size(1), k_cache.size(2), k_cache.size(3), v_cache.size(3)};
}

// proj [tokens, H d + G d + G dv] (a view), q [tokens, H, q_pitch]
void bias_rope_store(const Tensor& proj, const Tensor& bias, const Tensor& rope, const Tensor& positions, const Tensor& slots, Tensor& q,
                     Tensor& k_cache, Tensor& v_cache, const Tensor& status) {
  const int f = elem(proj);
  const auto dt = proj.scalar_type();
  const Caches c = cache_sizes(k_cache, v_cache, dt);
  TORCH_CHECK(q.dim() == 3 && q.size(0) == proj.size(0) && rope.dim() == 2 && rope.size(1) % 2 == 0 && rope.size(1) <= c.d && q.size(2) >= c.d, "bias_rope_store: sizes");
  const int64_t T = proj.size(0), H = q.size(1), rows = (H + c.G) * c.d + c.G * c.dv;
  const c10::cuda::CUDAGuard guard(proj.device());
  check_rc(forge_bias_rope_store(f, view2(proj, dt, T, rows, "proj"), proj.stride(0), i32(T), floats(bias, rows, "bias"), floats(rope, 0, "rope"),
                                 i32(rope.size(0)), i32(rope.size(1)), ints(positions, T, "positions"), ints(slots, T, "slots"), data(q, dt, 0, "q"),
                                 i32(q.size(2)), k_cache.data_ptr(), v_cache.data_ptr(), static_cast<long long>(c.blocks) * c.block_size,
                                 i32(c.block_size), i32(H), i32(c.G), i32(c.d), i32(c.dv), status_word(status), stream_of(proj)),
           "forge_bias_rope_store");
}

struct Attend {
  int64_t T, H;
  Caches c;
};
Attend attend_sizes(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& out, const Tensor& tables, int64_t seqs) {
  const auto dt = q.scalar_type();
  const Caches c = cache_sizes(k_cache, v_cache, dt);
  need(q, dt, 0, "q");
  TORCH_CHECK(q.dim() == 3 && q.size(2) >= c.d && q.size(1) % c.G == 0 && tables.dim() == 2 && tables.size(0) >= seqs, "windowed attention: sizes");
  view2(out, dt, q.size(0), q.size(1) * c.dv, "out");
  return {q.size(0), q.size(1), c};
}

// q [tokens, H, q_pitch], out [tokens, H dv] (a view); sequence s: query rows cu[s] .. cu[s + 1]
void windowed_attend_any(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& cu, int64_t seqs, int64_t max_q,
                         const Tensor& positions, const Tensor& tables, Tensor& out, int64_t window, double scale, double out_scale,
                         const Tensor& status) {
  const int f = elem(q);
  const Attend a = attend_sizes(q, k_cache, v_cache, out, tables, seqs);
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_windowed_attend_any(f, q.data_ptr(), i32(q.size(2)), k_cache.data_ptr(), v_cache.data_ptr(), ints(cu, seqs + 1, "cu"), i32(seqs),
                                     i32(max_q), ints(positions, a.T, "positions"), ints(tables, 0, "tables"), i32(tables.size(1)), i32(a.c.blocks),
                                     i32(a.c.block_size), out.data_ptr(), out.stride(0), i32(a.H), i32(a.c.G), i32(a.c.d), i32(a.c.dv), i32(window),
                                     static_cast<float>(scale), static_cast<float>(out_scale), status_word(status), stream_of(q)),
           "forge_windowed_attend_any");
}

// x [tokens, channels] (a view), taps [channels, n], state [slots, n - 1, channels], out [tokens, channels]
void short_conv(const Tensor& x, const Tensor& taps, const OptTensor& bias, Tensor& state, const Tensor& slots, const Tensor& positions,
                const Tensor& cu, int64_t seqs, int64_t max_q, Tensor& out, const Tensor& status) {
  const int f = elem(x);
  const auto dt = x.scalar_type();
  TORCH_CHECK(taps.dim() == 2 && state.dim() == 3 && state.size(1) == taps.size(1) - 1 && state.size(2) == taps.size(0), "short_conv: sizes");
  const int64_t T = x.size(0), C = taps.size(0);
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_short_conv(f, view2(x, dt, T, C, "x"), x.stride(0), floats(taps, 0, "taps"), bias.has_value() ? floats(*bias, C, "bias") : nullptr,
                            data(state, dt, 0, "state"), ints(slots, seqs, "slots"), ints(positions, T, "positions"), ints(cu, seqs + 1, "cu"),
                            i32(seqs), i32(max_q), data(out, dt, T * C, "out"), i32(C), i32(taps.size(1)), i32(state.size(0)), status_word(status),
                            stream_of(x)),
           "forge_short_conv");
}

struct Rec {
  int64_t T, H, share, dk, dv, slots;
};
// q, k [tokens, heads / share * dk], v [tokens, heads dv]: views of one row stride; dt, beta [tokens, heads]: views of another
Rec recurrence_sizes(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& dt, const OptTensor& beta, const Tensor& state) {
  TORCH_CHECK(state.dim() == 4 && q.dim() == 2, "recurrence: ranks");
  const auto ty = q.scalar_type();
  Rec r{q.size(0), state.size(1), 0, state.size(2), state.size(3), state.size(0)};
  TORCH_CHECK(q.size(1) % r.dk == 0 && q.size(1) > 0 && r.H % (q.size(1) / r.dk) == 0, "recurrence: heads");
  r.share = r.H / (q.size(1) / r.dk);
  view2(q, ty, r.T, q.size(1), "q");
  view2(k, ty, r.T, q.size(1), "k");
  view2(v, ty, r.T, r.H * r.dv, "v");
  view2(dt, ty, r.T, r.H, "dt");
  TORCH_CHECK(k.stride(0) == q.stride(0) && v.stride(0) == q.stride(0), "recurrence: q, k and v share a row stride");
  if (beta.has_value()) {
    view2(*beta, ty, r.T, r.H, "beta");
    TORCH_CHECK(beta->stride(0) == dt.stride(0), "recurrence: dt and beta share a row stride");
  }
  return r;
}

// o fp32 [tokens, heads, dv].  Without cu: one token per sequence, rows 0 .. seqs - 1.
void recurrence(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& dt, const OptTensor& beta, const Tensor& A_log, const Tensor& dt_bias,
                const OptTensor& D, Tensor& state, const Tensor& slots, const Tensor& positions, const OptTensor& cu, int64_t seqs, Tensor& o,
                const Tensor& status) {
  const int f = elem(q);
  const Rec r = recurrence_sizes(q, k, v, dt, beta, state);
  TORCH_CHECK(cu.has_value() || seqs <= r.T, "recurrence: sequences");
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_recurrence(f, q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), dt.data_ptr(), beta.has_value() ? beta->data_ptr() : nullptr,
                            dt.stride(0), floats(A_log, r.H, "A_log"), floats(dt_bias, r.H, "dt_bias"), D.has_value() ? floats(*D, r.H, "D") : nullptr,
                            floats(state, 0, "state"), ints(slots, seqs, "slots"), ints(positions, r.T, "positions"),
                            cu.has_value() ? ints(*cu, seqs + 1, "cu") : nullptr, i32(seqs), i32(r.H), i32(r.share), i32(r.dk), i32(r.dv), i32(r.slots),
                            floats(o, r.T * r.H * r.dv, "o"), status_word(status), stream_of(q)),
           "forge_recurrence");
}

// o fp32 [tokens, groups n], gate and out [tokens, groups n] (views); weight fp32, repeated along the row
void gated_norm(const Tensor& o, const Tensor& gate, const Tensor& weight, Tensor& out, int64_t groups, bool gate_first, double factor, double eps) {
  const int f = elem(gate);
  TORCH_CHECK(gate.dim() == 2 && gate.size(1) % groups == 0 && weight.numel() > 0 && gate.size(1) % weight.numel() == 0, "gated_norm: sizes");
  const int64_t T = gate.size(0), n = gate.size(1);
  const c10::cuda::CUDAGuard guard(gate.device());
  check_rc(forge_gated_norm(f, floats(o, T * n, "o"), view2(gate, gate.scalar_type(), T, n, "gate"), gate.stride(0), floats(weight, 0, "weight"),
                            i32(weight.numel()), view2(out, gate.scalar_type(), T, n, "out"), out.stride(0), i32(T), i32(groups), i32(n / groups),
                            gate_first ? 1 : 0, static_cast<float>(factor), static_cast<float>(eps), stream_of(gate)),
           "forge_gated_norm");
}

}  // namespace

void register_hybrid(pybind11::module& m) {
  m.def("bias_rope_store", &bias_rope_store);
  m.def("windowed_attend_any", &windowed_attend_any);
  m.def("short_conv", &short_conv);
  m.def("recurrence", &recurrence);
  m.def("recurrence_decode_ok", [](int64_t dk, int64_t dv) { return forge_recurrence_decode_ok(i32(dk), i32(dv)) != 0; });
  m.def("gated_norm", &gated_norm);
}
