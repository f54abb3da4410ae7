// Bindings of the ops of hybrid decoders: windowed attention, short convolutions, recurrences with a decay per token.  Every
// argument is checked here, as in bindings.cpp.
#include "checks.h"

extern "C" {
int forge_bias_rope_store(int fp32, const void* proj, long long ld, int tokens, const float* bias, const float* rope, int rope_rows, int rd,
                          const int* positions, const int* slots, void* q, int q_pitch, void* k_cache, void* v_cache, long long num_slots,
                          int block_size, int H, int G, int d, int dv, unsigned* status, cudaStream_t stream);
int forge_windowed_attend_any(int fp32, const void* q, int q_pitch, const void* k_cache, const void* v_cache, const int* cu, int seqs, int max_q,
                              const int* positions, const int* tables, int width, int num_blocks, int block_size, void* out, long long ldo, int H,
                              int G, int d, int dv, int window, float scale, float out_scale, int chunked, float softcap, const float* sink,
                              const void* gate, long long ldg, int gate_head, int gate_col, const void* pool_k, const void* pool_v, int pool,
                              unsigned* status, cudaStream_t stream);
int forge_norm_rope_store(int fp32, const void* proj, long long ld, int tokens, const void* q_norm, const void* k_norm, int whole, float eps,
                          const float* rope, int rope_rows, int rd, const int* positions, const int* slots, void* q, int q_pitch, void* k_cache,
                          void* v_cache, long long num_slots, int block_size, int H, int G, int d, int dv, const float* temper, unsigned* status,
                          cudaStream_t stream);
int forge_pool_blocks(int fp32, const void* k_cache, const void* v_cache, void* pool_k, void* pool_v, int size, int own, const int* cu, const int* lens,
                      const int* tables, int seqs, int max_q, int max_k, const int* offsets, void* gk, void* gv, int bound, int width, int num_blocks,
                      int block_size, int G, int d, int dv, unsigned* status, cudaStream_t stream);
int forge_row_offsets(const int* cu, const int* lens, int seqs, int window, int size, int* out, cudaStream_t stream);
int forge_stream_mix(int fp32, float* x, const void* y, const float* mix, const float* out, const int* ids, const int* prev, const void* embed,
                     int vocab, float scale, const void* pairs, int buckets, long long mul_prev, long long mul_cur, const float* into, const void* w,
                     const void* b, void* h, const int* rows, int out_rows, int n_rows, int W, int S, float eps, cudaStream_t stream);
int forge_short_conv(int fp32, const void* x, long long ldx, const float* taps, const float* bias, void* state, const int* slots,
                     const int* positions, const int* cu, int seqs, int max_q, void* out, int channels, int taps_n, int num_slots,
                     int silu, unsigned* status, cudaStream_t stream);
int forge_recurrence_decode_ok(int dk, int dv);
int forge_recurrence(int fp32, const void* q, const void* k, const void* v, long long ld, const void* dt, const void* beta, long long ld_raw,
                     const float* A_log, const float* dt_bias, const float* D, float* state, const int* slots, const int* positions,
                     const int* cu, int seqs, int heads, int share, int dk, int dv, int num_slots, float* o, unsigned* status,
                     cudaStream_t stream);
int forge_windowed_decode_ok(int d, int dv, int block_size);
int forge_windowed_decode(const void* q, int q_pitch, const void* k_cache, const void* v_cache, const int* tables, const int* lens, int seqs,
                          int width, int num_blocks, int block_size, void* out, long long ldo, float* part_o, float* part_ml, int chunk,
                          int max_chunks, int H, int G, int d, int dv, int window, float scale, float out_scale, int chunked, float softcap,
                          const float* sink, const void* gate, long long ldg, int gate_head, int gate_col, void* pool_k, void* pool_v, int pool,
                          int pool_own, unsigned* status, cudaStream_t stream);
int forge_windowed_prefill_qcols(int d, int dv, int block_size);
int forge_windowed_prefill(const void* q, int tokens, const void* k_cache, const void* v_cache, const int* cu_q, const int* context_lens,
                           const int* tables, int table_width, int num_blocks, int block_size, void* out, long long ldo, int num_seqs, int max_q,
                           int H, int G, int d, int dv, int window, float scale, float out_scale, int chunked, float softcap, const float* sink,
                           const void* gate, long long ldg, int gate_head, int gate_col, const void* pool_k, const void* pool_v, const int* pool_rows,
                           int pool_entries, int pool, unsigned* status, cudaStream_t stream);
int forge_recurrence_gates(const void* dt, const void* beta, long long ld_raw, const float* A_log, const float* dt_bias, const int* cu, int seqs,
                           int max_q, int heads, float* cum, float* weight, long long ldt, cudaStream_t stream);
int forge_retention_chunk_ok(int heads, int dk, int dv, int rd);
int forge_state_space_chunk(const void* q, const void* k, const void* v, long long ld, int share, const float* cum, const float* weight,
                            long long ldt, const float* skip, float* state, const int* slots, const int* positions, const int* cu, int seqs,
                            int heads, int dk, int dv, int num_slots, float* o, float* ws, float* seg_decay, int segs, int seg_len,
                            unsigned* status, cudaStream_t stream);
int forge_delta_chunk_ok(int dk, int dv);
long long forge_delta_chunk_scratch(int tokens, int seqs, int heads, int which);
int forge_delta_chunk(const void* q, const void* k, const void* v, long long ld, int share, const float* cum, const float* beta, long long ldt,
                      float* state, const int* slots, const int* positions, const int* cu, int seqs, int max_q, int heads, int dk, int dv,
                      int num_slots, void* mats, float* factors, float* o, int cols, unsigned* status, cudaStream_t stream);
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

// The same with norms of q and k ahead of the rotation and no biases; norm weights of dim entries (per head) or of all rows.  Without k_norm
// proj is q alone and nothing is stored.  temper fp32 [H]: one more factor of the queries
void norm_rope_store(const Tensor& proj, const Tensor& q_norm, const OptTensor& k_norm, bool whole, double eps, const Tensor& rope, const Tensor& positions,
                     const Tensor& slots, Tensor& q, Tensor& k_cache, Tensor& v_cache, const OptTensor& temper, const Tensor& status) {
  const int f = elem(proj);
  const auto dt = proj.scalar_type();
  Caches c = cache_sizes(k_cache, v_cache, dt);
  if (!k_norm.has_value()) c.G = 0;
  TORCH_CHECK(q.dim() == 3 && q.size(0) == proj.size(0) && rope.dim() == 2 && rope.size(1) % 2 == 0 && rope.size(1) <= c.d && q.size(2) >= c.d, "norm_rope_store: sizes");
  const int64_t T = proj.size(0), H = q.size(1), rows = (H + c.G) * c.d + c.G * c.dv;
  const c10::cuda::CUDAGuard guard(proj.device());
  check_rc(forge_norm_rope_store(f, view2(proj, dt, T, rows, "proj"), proj.stride(0), i32(T), data(q_norm, dt, whole ? H * c.d : c.d, "q_norm"),
                                 k_norm.has_value() ? data(*k_norm, dt, whole ? c.G * c.d : c.d, "k_norm") : nullptr, whole ? 1 : 0, static_cast<float>(eps), floats(rope, 0, "rope"),
                                 i32(rope.size(0)), i32(rope.size(1)), ints(positions, T, "positions"), ints(slots, T, "slots"), data(q, dt, 0, "q"),
                                 i32(q.size(2)), k_cache.data_ptr(), v_cache.data_ptr(), static_cast<long long>(c.blocks) * c.block_size,
                                 i32(c.block_size), i32(H), i32(c.G), i32(c.d), i32(c.dv), temper.has_value() ? floats(*temper, H, "temper") : nullptr,
                                 status_word(status), stream_of(proj)),
           "forge_norm_rope_store");
}

// Means of blocks: caches [blocks, kv_heads, ceil(block_size / size), dim / vdim]
struct Pool {
  void* k = nullptr;
  void* v = nullptr;
};
Pool pool_caches(const OptTensor& pool_k, const OptTensor& pool_v, int64_t size, const Caches& c, at::ScalarType dt) {
  Pool p;
  TORCH_CHECK(size >= 0 && (size == 0) == !pool_k.has_value(), "pooled blocks: size and caches");
  if (size == 0) return p;
  const int64_t rows = (c.block_size + size - 1) / size;
  TORCH_CHECK(pool_v.has_value() && pool_k->dim() == 4 && pool_v->dim() == 4 && pool_k->size(0) == c.blocks && pool_k->size(1) == c.G && pool_k->size(2) == rows &&
                  pool_k->size(3) == c.d && pool_v->size(0) == c.blocks && pool_v->size(1) == c.G && pool_v->size(2) == rows && pool_v->size(3) == c.dv,
              "pooled blocks: caches [blocks, kv_heads, ceil(block_size / size), dim] and [.., vdim] expected");
  p.k = data(*pool_k, dt, 0, "pool_k");
  p.v = data(*pool_v, dt, 0, "pool_v");
  return p;
}

// The entries of the blocks that end in the step's tokens (own), and with offsets all entries gathered to gk, gv [rows, kv_heads, dim / vdim]
void pool_blocks(const Tensor& k_cache, const Tensor& v_cache, const Tensor& pool_k, const Tensor& pool_v, int64_t size, bool own, const Tensor& cu,
                 const Tensor& lens, const Tensor& tables, int64_t seqs, int64_t max_q, int64_t max_k, const OptTensor& offsets, const OptTensor& gk,
                 const OptTensor& gv, const Tensor& status) {
  const int f = elem(k_cache);
  const auto dt = k_cache.scalar_type();
  const Caches c = cache_sizes(k_cache, v_cache, dt);
  TORCH_CHECK(size >= 1 && tables.dim() == 2 && tables.size(0) >= seqs, "pool_blocks: sizes");
  const Pool p = pool_caches(pool_k, pool_v, size, c, dt);
  const int* op = nullptr;
  void *kp = nullptr, *vp = nullptr;
  int64_t bound = 0;
  if (offsets.has_value()) {
    TORCH_CHECK(gk.has_value() && gv.has_value() && gk->dim() == 3 && gv->dim() == 3, "pool_blocks: gather buffers");
    bound = gk->size(0);
    op = ints(*offsets, seqs + 1, "offsets");
    kp = data(*gk, dt, bound * c.G * c.d, "gk");
    vp = data(*gv, dt, bound * c.G * c.dv, "gv");
  }
  const c10::cuda::CUDAGuard guard(k_cache.device());
  check_rc(forge_pool_blocks(f, k_cache.data_ptr(), v_cache.data_ptr(), p.k, p.v, i32(size), own ? 1 : 0, ints(cu, seqs + 1, "cu"), ints(lens, seqs, "lens"),
                             ints(tables, 0, "tables"), i32(seqs), i32(max_q), i32(max_k), op, kp, vp, i32(bound), i32(tables.size(1)), i32(c.blocks),
                             i32(c.block_size), i32(c.G), i32(c.d), i32(c.dv), status_word(status), stream_of(k_cache)),
           "forge_pool_blocks");
}

// out [seqs + 1]: running sums of floor(keys / size) or, with size 0, of min(keys, queries + window - 1)
void row_offsets(const Tensor& cu, const Tensor& lens, int64_t seqs, int64_t window, int64_t size, Tensor& out) {
  TORCH_CHECK(size >= 0 && (size > 0 || window >= 1), "row_offsets: sizes");
  const c10::cuda::CUDAGuard guard(cu.device());
  check_rc(forge_row_offsets(ints(cu, seqs + 1, "cu"), ints(lens, seqs, "lens"), i32(seqs), i32(window), i32(size), const_cast<int*>(ints(out, seqs + 1, "out")),
                             stream_of(cu)),
           "forge_row_offsets");
}

// x fp32 [tokens, streams, width].  With y [tokens, width]: mix [streams, streams], out [streams]; without: the streams begin as embeddings
void stream_mix(Tensor& x, const OptTensor& y, const OptTensor& mix, const OptTensor& out, const OptTensor& ids, const OptTensor& prev,
                const OptTensor& embed, double scale, const OptTensor& pairs, int64_t mul_prev, int64_t mul_cur, const Tensor& into, const OptTensor& w,
                const OptTensor& b, const OptTensor& h, const OptTensor& rows, double eps, bool fp32) {
  TORCH_CHECK(x.dim() == 3, "stream_mix: x [tokens, streams, width] expected");
  const int64_t T = x.size(0), S = x.size(1), W = x.size(2), n = rows.has_value() ? rows->numel() : T;
  const auto dt = fp32 ? at::kFloat : at::kBFloat16;
  const void *yp = nullptr, *ep = nullptr, *pp = nullptr;
  const float *mp = nullptr, *op = nullptr;
  const int *ip = nullptr, *vp = nullptr;
  int64_t vocab = 0, buckets = 0;
  if (y.has_value()) {
    TORCH_CHECK(mix.has_value() && out.has_value(), "stream_mix: y comes with mix and out");
    yp = view2(*y, dt, T, W, "y");
    need(*y, dt, 0, "y");
    mp = floats(*mix, S * S, "mix");
    op = floats(*out, S, "out");
  } else {
    TORCH_CHECK(ids.has_value() && prev.has_value() && embed.has_value() && pairs.has_value(), "stream_mix: y or tokens and tables expected");
    ip = ints(*ids, T, "ids");
    vp = ints(*prev, T, "prev");
    TORCH_CHECK(embed->dim() == 2 && embed->size(1) == W && pairs->dim() == 2 && pairs->size(1) == W && pairs->size(0) >= 2, "stream_mix: tables");
    ep = data(*embed, dt, 0, "embed");
    pp = data(*pairs, dt, 0, "pairs");
    vocab = embed->size(0);
    buckets = pairs->size(0) - 1;
  }
  const bool normed = w.has_value();
  TORCH_CHECK(!normed || (b.has_value() && h.has_value()), "stream_mix: a norm has a bias and a result");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_stream_mix(fp32 ? 1 : 0, floats(x, 0, "x"), yp, mp, op, ip, vp, ep, i32(vocab), static_cast<float>(scale), pp, i32(buckets), mul_prev,
                            mul_cur, floats(into, S, "into"), normed ? data(*w, dt, W, "w") : nullptr, normed ? data(*b, dt, W, "b") : nullptr,
                            normed ? data(*h, dt, n * W, "h") : nullptr, rows.has_value() ? ints(*rows, n, "rows") : nullptr, i32(n), i32(T), i32(W), i32(S),
                            static_cast<float>(eps), stream_of(x)),
           "forge_stream_mix");
}

struct Attend {
  int64_t T, H;
  Caches c;
};

// sink fp32 [heads]; gate [tokens, heads] or [tokens, heads dv] (a view)
struct Options {
  int chunked;
  float softcap;
  const float* sink;
  const void* gate;
  long long ldg;
  int gate_head, gate_col;
};
Options attend_options(bool chunked, double softcap, const OptTensor& sink, const OptTensor& gate, const Attend& a, at::ScalarType dt) {
  TORCH_CHECK(softcap >= 0, "windowed attention: softcap");
  Options o{chunked ? 1 : 0, static_cast<float>(softcap), nullptr, nullptr, 0, 0, 0};
  if (sink.has_value()) o.sink = floats(*sink, a.H, "sink");
  if (gate.has_value()) {
    const bool element = gate->dim() == 2 && gate->size(1) == a.H * a.c.dv;
    o.gate = view2(*gate, dt, a.T, element ? a.H * a.c.dv : a.H, "gate");
    o.ldg = gate->stride(0);
    o.gate_head = element ? i32(a.c.dv) : 1;
    o.gate_col = element ? 1 : 0;
  }
  return o;
}
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
                         bool chunked, double softcap, const OptTensor& sink, const OptTensor& gate, const OptTensor& pool_k, const OptTensor& pool_v,
                         int64_t pool, const Tensor& status) {
  const int f = elem(q);
  const Attend a = attend_sizes(q, k_cache, v_cache, out, tables, seqs);
  const Pool m = pool_caches(pool_k, pool_v, pool, a.c, q.scalar_type());
  const Options x = attend_options(chunked, softcap, sink, gate, a, q.scalar_type());
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_windowed_attend_any(f, q.data_ptr(), i32(q.size(2)), k_cache.data_ptr(), v_cache.data_ptr(), ints(cu, seqs + 1, "cu"), i32(seqs),
                                     i32(max_q), ints(positions, a.T, "positions"), ints(tables, 0, "tables"), i32(tables.size(1)), i32(a.c.blocks),
                                     i32(a.c.block_size), out.data_ptr(), out.stride(0), i32(a.H), i32(a.c.G), i32(a.c.d), i32(a.c.dv), i32(window),
                                     static_cast<float>(scale), static_cast<float>(out_scale), x.chunked, x.softcap, x.sink, x.gate, x.ldg, x.gate_head,
                                     x.gate_col, m.k, m.v, i32(pool), status_word(status), stream_of(q)),
           "forge_windowed_attend_any");
}

constexpr auto kBf16 = at::kBFloat16;

// One token per sequence: rows 0 .. seqs - 1 of q and out.
void windowed_decode(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& tables, const Tensor& lens, int64_t seqs,
                     Tensor& out, const OptTensor& part_o, const OptTensor& part_ml, int64_t chunk, int64_t max_chunks, int64_t window,
                     double scale, double out_scale, bool chunked, double softcap, const OptTensor& sink, const OptTensor& gate, const OptTensor& pool_k,
                     const OptTensor& pool_v, int64_t pool, bool pool_own, const Tensor& status) {
  TORCH_CHECK(q.scalar_type() == kBf16 && seqs <= q.size(0), "windowed_decode: q");
  const Attend a = attend_sizes(q, k_cache, v_cache, out, tables, seqs);
  const Pool m = pool_caches(pool_k, pool_v, pool, a.c, q.scalar_type());
  const Options x = attend_options(chunked, softcap, sink, gate, a, q.scalar_type());
  float *po = nullptr, *pm = nullptr;
  if (max_chunks > 1) {
    TORCH_CHECK(part_o.has_value() && part_ml.has_value(), "windowed_decode: scratch");
    po = floats(*part_o, seqs * a.H * max_chunks * a.c.dv, "part_o");
    pm = floats(*part_ml, seqs * a.H * max_chunks * 2, "part_ml");
  }
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_windowed_decode(q.data_ptr(), i32(q.size(2)), k_cache.data_ptr(), v_cache.data_ptr(), ints(tables, 0, "tables"), ints(lens, seqs, "lens"),
                                 i32(seqs), i32(tables.size(1)), i32(a.c.blocks), i32(a.c.block_size), out.data_ptr(), out.stride(0), po, pm, i32(chunk),
                                 i32(max_chunks), i32(a.H), i32(a.c.G), i32(a.c.d), i32(a.c.dv), i32(window), static_cast<float>(scale),
                                 static_cast<float>(out_scale), x.chunked, x.softcap, x.sink, x.gate, x.ldg, x.gate_head, x.gate_col, m.k, m.v, i32(pool),
                                 pool_own ? 1 : 0, status_word(status), stream_of(q)),
           "forge_windowed_decode");
}

// Sequence s: the rows cu[s] .. cu[s + 1] of q and out, its last ones; context_lens[s] keys.  gk, gv, offsets: entries of pooled blocks as
// pool_blocks gathers them.
void windowed_prefill(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& cu, const Tensor& context_lens, const Tensor& tables,
                      int64_t seqs, int64_t max_q, Tensor& out, int64_t window, double scale, double out_scale, bool chunked, double softcap,
                      const OptTensor& sink, const OptTensor& gate, const OptTensor& gk, const OptTensor& gv, const OptTensor& offsets, int64_t pool,
                      const Tensor& status) {
  TORCH_CHECK(q.scalar_type() == kBf16, "windowed_prefill: q");
  const Attend a = attend_sizes(q, k_cache, v_cache, out, tables, seqs);
  const Options x = attend_options(chunked, softcap, sink, gate, a, q.scalar_type());
  TORCH_CHECK(q.size(2) == forge_windowed_prefill_qcols(i32(a.c.d), i32(a.c.dv), i32(a.c.block_size)), "windowed_prefill: q columns");
  const void *kp = nullptr, *vp = nullptr;
  const int* op = nullptr;
  int64_t entries = 0;
  TORCH_CHECK(pool >= 0 && (pool == 0) == !gk.has_value(), "windowed_prefill: pooled blocks");
  if (pool > 0) {
    TORCH_CHECK(gv.has_value() && offsets.has_value(), "windowed_prefill: pooled blocks");
    entries = gk->size(0);
    kp = data(*gk, kBf16, entries * a.c.G * a.c.d, "gk");
    vp = data(*gv, kBf16, entries * a.c.G * a.c.dv, "gv");
    op = ints(*offsets, seqs + 1, "offsets");
  }
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_windowed_prefill(q.data_ptr(), i32(a.T), k_cache.data_ptr(), v_cache.data_ptr(), ints(cu, seqs + 1, "cu"), ints(context_lens, seqs, "lens"),
                                  ints(tables, 0, "tables"), i32(tables.size(1)), i32(a.c.blocks), i32(a.c.block_size), out.data_ptr(), out.stride(0),
                                  i32(seqs), i32(max_q), i32(a.H), i32(a.c.G), i32(a.c.d), i32(a.c.dv), i32(window), static_cast<float>(scale),
                                  static_cast<float>(out_scale), x.chunked, x.softcap, x.sink, x.gate, x.ldg, x.gate_head, x.gate_col, kp, vp, op,
                                  i32(entries), i32(pool), status_word(status), stream_of(q)),
           "forge_windowed_prefill");
}

// x [tokens, channels] (a view), taps [channels, n], state [slots, n - 1, channels], out [tokens, channels]
void short_conv(const Tensor& x, const Tensor& taps, const OptTensor& bias, Tensor& state, const Tensor& slots, const Tensor& positions,
                const Tensor& cu, int64_t seqs, int64_t max_q, Tensor& out, bool silu, const Tensor& status) {
  const int f = elem(x);
  const auto dt = x.scalar_type();
  TORCH_CHECK(taps.dim() == 2 && state.dim() == 3 && state.size(1) == taps.size(1) - 1 && state.size(2) == taps.size(0), "short_conv: sizes");
  const int64_t T = x.size(0), C = taps.size(0);
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_short_conv(f, view2(x, dt, T, C, "x"), x.stride(0), floats(taps, 0, "taps"), bias.has_value() ? floats(*bias, C, "bias") : nullptr,
                            data(state, dt, 0, "state"), ints(slots, seqs, "slots"), ints(positions, T, "positions"), ints(cu, seqs + 1, "cu"),
                            i32(seqs), i32(max_q), data(out, dt, T * C, "out"), i32(C), i32(taps.size(1)), i32(state.size(0)), silu ? 1 : 0, status_word(status),
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

// cum, weight fp32 [heads, tokens]
void recurrence_gates(const Tensor& dt, const OptTensor& beta, const Tensor& A_log, const Tensor& dt_bias, const Tensor& cu, int64_t seqs, int64_t max_q,
                      Tensor& cum, Tensor& weight) {
  TORCH_CHECK(cum.dim() == 2 && weight.sizes() == cum.sizes(), "recurrence_gates: ranks");
  const int64_t H = cum.size(0), T = cum.size(1);
  view2(dt, kBf16, T, H, "dt");
  if (beta.has_value()) {
    view2(*beta, kBf16, T, H, "beta");
    TORCH_CHECK(beta->stride(0) == dt.stride(0), "recurrence_gates: row strides");
  }
  const c10::cuda::CUDAGuard guard(dt.device());
  check_rc(forge_recurrence_gates(dt.data_ptr(), beta.has_value() ? beta->data_ptr() : nullptr, dt.stride(0), floats(A_log, H, "A_log"),
                                  floats(dt_bias, H, "dt_bias"), ints(cu, seqs + 1, "cu"), i32(seqs), i32(max_q), i32(H), floats(cum, H * T, "cum"),
                                  floats(weight, H * T, "weight"), T, stream_of(dt)),
           "forge_recurrence_gates");
}

// The runs cu[s] .. cu[s + 1]; q, k, v as in recurrence; cum, weight from recurrence_gates; o fp32 [tokens, heads, dv]
void state_space_chunk(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& cum, const Tensor& weight, const Tensor& skip, Tensor& state,
                       const Tensor& slots, const Tensor& positions, const Tensor& cu, int64_t seqs, Tensor& o, const OptTensor& ws,
                       const OptTensor& seg_decay, int64_t segs, int64_t seg_len, const Tensor& status) {
  TORCH_CHECK(q.scalar_type() == kBf16 && state.dim() == 4 && cum.dim() == 2 && cum.size(0) == state.size(1) && cum.size(1) == q.size(0), "state_space_chunk: sizes");
  const Rec r = recurrence_sizes(q, k, v, v.slice(1, 0, state.size(1)), c10::nullopt, state);
  float *wp = nullptr, *sp = nullptr;
  if (segs > 1) {
    TORCH_CHECK(ws.has_value() && seg_decay.has_value(), "state_space_chunk: scratch");
    wp = floats(*ws, seqs * segs * r.H * r.dk * r.dv, "ws");
    sp = floats(*seg_decay, seqs * segs * r.H, "seg_decay");
  }
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_state_space_chunk(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), i32(r.share), floats(cum, r.H * r.T, "cum"),
                                   floats(weight, r.H * r.T, "weight"), r.T, floats(skip, r.H, "skip"), floats(state, 0, "state"),
                                   ints(slots, seqs, "slots"), ints(positions, r.T, "positions"), ints(cu, seqs + 1, "cu"), i32(seqs), i32(r.H),
                                   i32(r.dk), i32(r.dv), i32(r.slots), floats(o, r.T * r.H * r.dv, "o"), wp, sp, i32(segs), i32(seg_len),
                                   status_word(status), stream_of(q)),
           "forge_state_space_chunk");
}

void delta_chunk(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& cum, const Tensor& beta, Tensor& state, const Tensor& slots,
                 const Tensor& positions, const Tensor& cu, int64_t seqs, int64_t max_q, Tensor& mats, Tensor& factors, Tensor& o, int64_t cols,
                 const Tensor& status) {
  TORCH_CHECK(q.scalar_type() == kBf16 && state.dim() == 4 && cum.dim() == 2 && cum.size(0) == state.size(1) && cum.size(1) == q.size(0), "delta_chunk: sizes");
  const Rec r = recurrence_sizes(q, k, v, v.slice(1, 0, state.size(1)), c10::nullopt, state);
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_delta_chunk(q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), i32(r.share), floats(cum, r.H * r.T, "cum"),
                             floats(beta, r.H * r.T, "beta"), r.T, floats(state, 0, "state"), ints(slots, seqs, "slots"),
                             ints(positions, r.T, "positions"), ints(cu, seqs + 1, "cu"), i32(seqs), i32(max_q), i32(r.H), i32(r.dk), i32(r.dv),
                             i32(r.slots), data(mats, kBf16, forge_delta_chunk_scratch(i32(r.T), i32(seqs), i32(r.H), 0), "mats"),
                             floats(factors, forge_delta_chunk_scratch(i32(r.T), i32(seqs), i32(r.H), 1), "factors"),
                             floats(o, r.T * r.H * r.dv, "o"), i32(cols), status_word(status), stream_of(q)),
           "forge_delta_chunk");
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
  m.def("norm_rope_store", &norm_rope_store);
  m.def("stream_mix", &stream_mix);
  m.def("pool_blocks", &pool_blocks);
  m.def("row_offsets", &row_offsets);
  m.def("windowed_attend_any", &windowed_attend_any);
  m.def("windowed_decode", &windowed_decode);
  m.def("windowed_decode_ok", [](int64_t d, int64_t dv, int64_t bs) { return forge_windowed_decode_ok(i32(d), i32(dv), i32(bs)) != 0; });
  m.def("windowed_prefill", &windowed_prefill);
  m.def("windowed_prefill_qcols", [](int64_t d, int64_t dv, int64_t bs) { return forge_windowed_prefill_qcols(i32(d), i32(dv), i32(bs)); });
  m.def("recurrence_gates", &recurrence_gates);
  m.def("state_space_chunk", &state_space_chunk);
  m.def("state_space_chunk_ok", [](int64_t dk, int64_t dv) { return forge_retention_chunk_ok(1, i32(dk), i32(dv), 0) != 0; });
  m.def("delta_chunk", &delta_chunk);
  m.def("delta_chunk_ok", [](int64_t dk, int64_t dv) { return forge_delta_chunk_ok(i32(dk), i32(dv)) != 0; });
  m.def("delta_chunk_scratch", [](int64_t T, int64_t S, int64_t H, int64_t which) { return static_cast<int64_t>(forge_delta_chunk_scratch(i32(T), i32(S), i32(H), i32(which))); });
  m.def("short_conv", &short_conv);
  m.def("recurrence", &recurrence);
  m.def("recurrence_decode_ok", [](int64_t dk, int64_t dv) { return forge_recurrence_decode_ok(i32(dk), i32(dv)) != 0; });
  m.def("gated_norm", &gated_norm);
}
