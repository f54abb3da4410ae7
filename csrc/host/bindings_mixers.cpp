// Bindings of the ops of decoders with an fp32 residual stream, latent attention, retention and expert layers.  As in
// bindings.cpp every argument is checked here (device, dtype, contiguity, shapes), so a malformed call raises in Python
// instead of reaching a kernel.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <algorithm>
#include <cstdint>

#include "checks.h"

extern "C" {
int forge_stream_update(int fp32, float* x, const void* a, const void* b, const int* b_rows, int top, const int* ids, const void* embed,
                        int vocab, const void* vec, const void* w1, const void* w2, void* h1, void* h2, const int* rows, int out_rows,
                        int n_rows, int W, int start, float eps, cudaStream_t stream);
int forge_stream_sandwich(int fp32, float* x, const void* a, const int* a_rows, const float* a_weights, int top, const float* a_bias,
                          const void* post, float mult, float offset, const int* ids, const void* embed, int vocab, const void* w, void* h,
                          const int* rows, int out_rows, int n_rows, int W, int start, float eps, cudaStream_t stream);
int forge_stream_group(int fp32, float* x, const void* a, const int* a_rows, const float* a_weights, int top, const void* post, float mult,
                       float offset, const int* ids, const void* embed, int vocab, const void* w, void* h, const int* rows, int out_rows, int n_rows,
                       int W, int groups, int start, float eps, cudaStream_t stream);
int forge_act_any(int fp32, void* x, long long n, int act, int logits, float scale, float cap, cudaStream_t stream);
int forge_act_mul_any(int fp32, const void* x, void* out, long long rows, int I, int act, float limit, cudaStream_t stream);
int forge_gemm_bf16_act(const void* x, int ldx, const void* w, int ldw, void* out, int ldo, int M, int n_out, int K, int act, float limit,
                        unsigned* status, cudaStream_t stream);
int forge_gemm_simt(int fp32, const void* x, long long ldx, long long x_batch, const void* w, long long ldw, long long w_batch, void* out,
                    long long ldo, long long o_batch, int M, int N, int K, int batch, const int* tile_expert, cudaStream_t stream);
int forge_latent_prepare(int fp32, const void* proj, long long ld, int T, int q_rank, int kv_rank, int rot, const void* qw, const void* kw, float eps,
                         const float* rope, int rope_rows, const int* positions, const int* slots, void* cq, void* cache,
                         long long num_slots, unsigned* status, cudaStream_t stream);
int forge_latent_rotate_q(int fp32, const void* q, long long ld, void* qa, int tokens, int heads, int dim, int rot, int kv_rank, const float* rope,
                          int rope_rows, const int* positions, cudaStream_t stream);
int forge_latent_attend_any(int fp32, const void* qa, const void* cache, void* o, int tok0, int tokens, const int* cu, int num_seqs,
                            const int* positions, const int* block_tables, int table_width, int num_blocks, int block_size, int heads,
                            int kv_rank, int rot, int window, float scale, unsigned* status, cudaStream_t stream);
int forge_retention_decode(int fp32, const void* qkvg, int ld, const float* decay, float* state, const int* slots, const int* positions,
                           const float* rope, int rope_rows, int rd, int seqs, int heads, int dk, int dv, int num_slots, void* y, float eps,
                           unsigned* status, cudaStream_t stream);
int forge_retention_scan(int fp32, const void* qkvg, int ld, const float* decay, float* state, const int* slots, const int* positions,
                         const float* rope, int rope_rows, int rd, const int* cu, int seqs, int heads, int dk, int dv, int num_slots,
                         float* o, unsigned* status, cudaStream_t stream);
int forge_retention_gate(int fp32, const float* o, const void* qkvg, int ld, int gate_at, void* y, int tok0, int tokens, int heads, int dv,
                         float eps, cudaStream_t stream);
int forge_router(int fp32, const void* h, const void* w, int T, int W, int E, int top, int softmax, const float* correction, int groups, int keep,
                 int* experts, float* weights, cudaStream_t stream);
int forge_moe_plan(const int* experts, int n, int E, int tile, int max_tiles, int* pos, int* tile_expert, int* num_tiles, cudaStream_t stream);
int forge_grouped_gemm(const void* x, const void* w, void* out, int experts, int n_out, int K, int gated, int tile, int act, float limit,
                       const int* tile_expert, const int* num_tiles, int max_tiles, unsigned* status, cudaStream_t stream);
int forge_head_linear(const void* x, long long x_tok, long long x_head, const void* w, void* out, long long o_tok, long long o_head, int M,
                      int heads, int N, int K, cudaStream_t stream);
int forge_latent_decode_ok(int R, int rot, int block_size);
long long forge_latent_decode_scratch(int heads, int R, int ctas);
int forge_latent_decode(const void* qa, const void* cache, const int* block_tables, const int* lens, void* o, float* scratch, int ctas,
                        int seqs, int heads, int R, int rot, int table_width, int num_blocks, int block_size, int window, float scale,
                        unsigned* status, cudaStream_t stream);
int forge_latent_prefill_qcols(int dim, int rot, int vdim);
int forge_latent_prefill(const void* q, const void* kv, const void* kr, const int* cu_q, const int* cu_k, void* out, int tokens, int tok0,
                         int keys, int num_seqs, int max_q, int heads, int dim, int rot, int vdim, int window, float scale, unsigned* status,
                         cudaStream_t stream);
int forge_latent_gather(const void* cache, const int* cu_k, const int* lens, int num_seqs, const int* block_tables, int table_width, int num_blocks,
                        int block_size, int R, int rot, int keys, void* c, void* kr, unsigned* status, cudaStream_t stream);
int forge_latent_pack_q(const void* q, long long ld, void* qp, int tokens, int heads, int dim, int rot, const float* rope, int rope_rows,
                        const int* positions, cudaStream_t stream);
int forge_retention_chunk_ok(int heads, int dk, int dv, int rd);
int forge_retention_chunk_cols(int dk, int dv);
int forge_retention_chunk(void* qkvg, int ld, const float* decay, float* state, const int* slots, const int* positions, const float* rope,
                          int rope_rows, int rd, const int* cu, int seqs, int tok0, int tokens, int heads, int dk, int dv, int num_slots,
                          float* o, float* ws, int segs, int seg_len, unsigned* status, cudaStream_t stream);
int forge_moe_scatter(int fp32, const void* h, const int* pos, const float* weights, int n, int top, int W, void* xs, cudaStream_t stream);
}

namespace {

// x fp32 [rows, W]; a, b, embed, vec, w1, w2, h1, h2 of one element type.  b_rows (int32 [rows, top]): b is a buffer of expert
// outputs whose rows b_rows[r, :] are summed.  rows (int32): norms of these rows only, x unchanged.
void stream_update(Tensor& x, const OptTensor& a, const OptTensor& b, const OptTensor& b_rows, const OptTensor& ids, const OptTensor& embed,
                   const OptTensor& vec, const OptTensor& w1, const OptTensor& w2, const OptTensor& h1, const OptTensor& h2,
                   const OptTensor& rows, bool start, double eps, bool fp32) {
  TORCH_CHECK(x.dim() == 2, "stream_update: x must be [rows, width]");
  const int64_t R = x.size(0), W = x.size(1);
  const auto dt = fp32 ? at::kFloat : at::kBFloat16;
  float* xp = floats(x, R * W, "x");
  const void *ap = nullptr, *bp = nullptr, *ep = nullptr, *vp = nullptr, *w1p = nullptr, *w2p = nullptr;
  void *h1p = nullptr, *h2p = nullptr;
  const int *brp = nullptr, *idp = nullptr, *rp = nullptr;
  int64_t top = 0, vocab = 0, out_rows = R;
  if (rows.has_value()) { rp = ints(*rows, 0, "rows"); out_rows = rows->numel(); }
  if (a.has_value()) ap = data(*a, dt, R * W, "a");
  if (b.has_value()) {
    if (b_rows.has_value()) {
      TORCH_CHECK(b_rows->dim() == 2 && b_rows->size(0) == R && b->dim() == 2 && b->size(1) == W, "stream_update: routed b");
      top = b_rows->size(1);
      brp = ints(*b_rows, R * top, "b_rows");
      bp = data(*b, dt, W, "b");
    } else {
      bp = data(*b, dt, R * W, "b");
    }
  }
  if (ids.has_value()) {
    TORCH_CHECK(embed.has_value() && embed->dim() == 2 && embed->size(1) == W, "stream_update: embed");
    idp = ints(*ids, R, "ids");
    vocab = embed->size(0);
    ep = data(*embed, dt, W, "embed");
  }
  if (vec.has_value()) vp = data(*vec, dt, W, "vec");
  if (w1.has_value()) {
    w1p = data(*w1, dt, W, "w1");
    TORCH_CHECK(h1.has_value(), "stream_update: h1");
    h1p = data(*h1, dt, out_rows * W, "h1");
  }
  if (w2.has_value()) {
    TORCH_CHECK(w1.has_value() && h2.has_value(), "stream_update: h2");
    w2p = data(*w2, dt, W, "w2");
    h2p = data(*h2, dt, out_rows * W, "h2");
  }
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_stream_update(fp32, xp, ap, bp, brp, i32(top), idp, ep, i32(vocab), vp, w1p, w2p, h1p, h2p, rp, i32(out_rows), i32(R), i32(W),
                               start ? 1 : 0, static_cast<float>(eps), stream_of(x)),
           "forge_stream_update");
}

// x fp32 [rows, W]; a, post, embed, w, h of one element type.  a_rows (int32 [rows, top]) with a_weights (fp32, or none: 1): a is
// a buffer of expert outputs.  rows (int32): these rows only, x unchanged.
void stream_sandwich(Tensor& x, const OptTensor& a, const OptTensor& a_rows, const OptTensor& a_weights, const OptTensor& a_bias,
                     const OptTensor& post, double mult, double offset, const OptTensor& ids, const OptTensor& embed, const OptTensor& w,
                     const OptTensor& h, const OptTensor& rows, bool start, double eps, bool fp32) {
  TORCH_CHECK(x.dim() == 2, "stream_sandwich: x must be [rows, width]");
  const int64_t R = x.size(0), W = x.size(1);
  const auto dt = fp32 ? at::kFloat : at::kBFloat16;
  float* xp = floats(x, R * W, "x");
  const void *ap = nullptr, *pp = nullptr, *ep = nullptr, *wp = nullptr;
  void* hp = nullptr;
  const int *arp = nullptr, *idp = nullptr, *rp = nullptr;
  const float *awp = nullptr, *abp = nullptr;
  int64_t top = 0, vocab = 0, out_rows = R;
  if (rows.has_value()) { rp = ints(*rows, 0, "rows"); out_rows = rows->numel(); }
  if (a.has_value()) {
    if (a_rows.has_value()) {
      TORCH_CHECK(a_rows->dim() == 2 && a_rows->size(0) == R && a->dim() == 2 && a->size(1) == W, "stream_sandwich: routed a");
      top = a_rows->size(1);
      arp = ints(*a_rows, R * top, "a_rows");
      ap = data(*a, dt, W, "a");
      if (a_weights.has_value()) awp = floats(*a_weights, R * top, "a_weights");
    } else {
      ap = data(*a, dt, R * W, "a");
    }
    if (a_bias.has_value()) abp = floats(*a_bias, W, "a_bias");
  }
  if (post.has_value()) {
    TORCH_CHECK(a.has_value(), "stream_sandwich: post belongs to a");
    pp = data(*post, dt, W, "post");
  }
  if (ids.has_value()) {
    TORCH_CHECK(embed.has_value() && embed->dim() == 2 && embed->size(1) == W, "stream_sandwich: embed");
    idp = ints(*ids, R, "ids");
    vocab = embed->size(0);
    ep = data(*embed, dt, W, "embed");
  }
  if (w.has_value()) {
    TORCH_CHECK(h.has_value(), "stream_sandwich: h");
    wp = data(*w, dt, W, "w");
    hp = data(*h, dt, out_rows * W, "h");
  }
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_stream_sandwich(fp32, xp, ap, arp, awp, i32(top), abp, pp, static_cast<float>(mult), static_cast<float>(offset), idp, ep,
                                 i32(vocab), wp, hp, rp, i32(out_rows), i32(R), i32(W), start ? 1 : 0, static_cast<float>(eps), stream_of(x)),
           "forge_stream_sandwich");
}

// x fp32 [rows, W]; a or embed (with ids), post, w, h of one element type; the rest as in stream_sandwich.  Norms over `groups` equal parts of
// a row; h without w: the row itself.
void stream_group(Tensor& x, const OptTensor& a, const OptTensor& a_rows, const OptTensor& a_weights, const Tensor& post, double mult, double offset,
                  const OptTensor& ids, const OptTensor& embed, const OptTensor& w, const OptTensor& h, const OptTensor& rows, int64_t groups, bool start,
                  double eps, bool fp32) {
  TORCH_CHECK(x.dim() == 2 && a.has_value() != ids.has_value() && groups >= 1 && x.size(1) % groups == 0, "stream_group: sizes and operands");
  const int64_t R = x.size(0), W = x.size(1);
  const auto dt = fp32 ? at::kFloat : at::kBFloat16;
  float* xp = floats(x, R * W, "x");
  const void *ap = nullptr, *ep = nullptr, *wp = nullptr;
  void* hp = nullptr;
  const int *arp = nullptr, *idp = nullptr, *rp = nullptr;
  const float* awp = nullptr;
  int64_t top = 0, vocab = 0, out_rows = R;
  if (rows.has_value()) { rp = ints(*rows, 0, "rows"); out_rows = rows->numel(); }
  if (a.has_value() && a_rows.has_value()) {
    TORCH_CHECK(a_rows->dim() == 2 && a_rows->size(0) == R && a->dim() == 2 && a->size(1) == W, "stream_group: routed a");
    top = a_rows->size(1);
    arp = ints(*a_rows, R * top, "a_rows");
    ap = data(*a, dt, W, "a");
    if (a_weights.has_value()) awp = floats(*a_weights, R * top, "a_weights");
  } else if (a.has_value()) {
    ap = data(*a, dt, R * W, "a");
  } else {
    TORCH_CHECK(embed.has_value() && embed->dim() == 2 && embed->size(1) == W, "stream_group: embed");
    idp = ints(*ids, R, "ids");
    vocab = embed->size(0);
    ep = data(*embed, dt, W, "embed");
  }
  if (w.has_value()) {
    TORCH_CHECK(h.has_value(), "stream_group: h");
    wp = data(*w, dt, W, "w");
  }
  if (h.has_value()) hp = data(*h, dt, out_rows * W, "h");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_stream_group(fp32, xp, ap, arp, awp, i32(top), data(post, dt, W, "post"), static_cast<float>(mult), static_cast<float>(offset), idp, ep,
                              i32(vocab), wp, hp, rp, i32(out_rows), i32(R), i32(W), i32(groups), start ? 1 : 0, static_cast<float>(eps), stream_of(x)),
           "forge_stream_group");
}

// x <- act(x) in place
void act_any(Tensor& x, int64_t act) {
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_act_any(elem(x), data(x, x.scalar_type(), 0, "x"), x.numel(), i32(act), 0, 1.f, 0.f, stream_of(x)), "forge_act_any");
}

// x <- cap tanh(scale x / cap) in place
void bound_logits(Tensor& x, double scale, double cap) {
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_act_any(elem(x), data(x, x.scalar_type(), 0, "x"), x.numel(), 0, 1, static_cast<float>(scale), static_cast<float>(cap), stream_of(x)),
           "forge_act_any");
}

// out = act(x w_gate^T, x w_up^T) for w = gate rows, up rows (bf16, tcgen05)
void gemm_act(const Tensor& x, const Tensor& w, Tensor& out, int64_t act, double limit, const Tensor& status) {
  TORCH_CHECK(x.is_cuda() && w.is_cuda() && out.is_cuda() && x.scalar_type() == at::kBFloat16 && w.scalar_type() == at::kBFloat16 && out.scalar_type() == at::kBFloat16,
              "gemm_act: bf16 CUDA tensors expected");
  TORCH_CHECK(x.dim() == 2 && w.dim() == 2 && out.dim() == 2 && x.stride(1) == 1 && w.stride(1) == 1 && out.stride(1) == 1, "gemm_act: ranks and strides");
  TORCH_CHECK(w.size(1) == x.size(1) && w.size(0) % 2 == 0 && out.size(0) == x.size(0) && out.size(1) == w.size(0) / 2 && act >= 0 && act <= 2, "gemm_act: shapes");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_gemm_bf16_act(x.data_ptr(), i32(x.stride(0)), w.data_ptr(), i32(w.stride(0)), out.data_ptr(), i32(out.stride(0)), i32(x.size(0)),
                               i32(out.size(1)), i32(x.size(1)), i32(act), static_cast<float>(limit), status_word(status), stream_of(x)),
           "forge_gemm_bf16_act");
}

void act_mul_any(const Tensor& x, Tensor& out, int64_t act, double limit) {
  const int f = elem(x);
  TORCH_CHECK(x.dim() == 2 && x.size(1) % 2 == 0, "act_mul_any: x [rows, 2 I]");
  const int64_t rows = x.size(0), I = x.size(1) / 2;
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_act_mul_any(f, data(x, x.scalar_type(), rows * 2 * I, "x"), data(out, x.scalar_type(), rows * I, "out"), rows, i32(I), i32(act),
                             static_cast<float>(limit), stream_of(x)),
           "forge_act_mul_any");
}

// out[b] = x[b] w[b]^T for 3-D views [batch, M, K], [batch, N, K], [batch, M, N] with unit inner strides (2-D: one product).
// tile_expert: w is [experts, N, K] and the 64-row tile i of the 2-D x uses matrix tile_expert[i].
void gemm_simt(const Tensor& x, const Tensor& w, Tensor& out, const OptTensor& tile_expert) {
  const int f = elem(x);
  TORCH_CHECK(x.is_cuda() && w.is_cuda() && out.is_cuda() && w.scalar_type() == x.scalar_type() && out.scalar_type() == x.scalar_type(), "gemm_simt: operands");
  TORCH_CHECK(x.dim() == out.dim() && (x.dim() == 2 || x.dim() == 3), "gemm_simt: ranks");
  const bool three = x.dim() == 3, experts = tile_expert.has_value();
  TORCH_CHECK(w.dim() == (three || experts ? 3 : 2) && !(three && experts), "gemm_simt: rank of w");
  const int64_t batch = three ? x.size(0) : 1, M = x.size(-2), K = x.size(-1), N = w.size(-2);
  TORCH_CHECK(w.size(-1) == K && out.size(-2) == M && out.size(-1) == N && (!three || (w.size(0) == batch && out.size(0) == batch)), "gemm_simt: shapes");
  TORCH_CHECK(x.stride(-1) == 1 && w.stride(-1) == 1 && out.stride(-1) == 1, "gemm_simt: inner strides must be 1");
  const int* te = nullptr;
  if (experts) te = ints(*tile_expert, (M + 63) / 64, "tile_expert");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_gemm_simt(f, x.data_ptr(), x.stride(-2), three ? x.stride(0) : 0, w.data_ptr(), w.stride(-2), w.dim() == 3 ? w.stride(0) : 0,
                           out.data_ptr(), out.stride(-2), three ? out.stride(0) : 0, i32(M), i32(N), i32(K), i32(batch), te, stream_of(x)),
           "forge_gemm_simt");
}

// proj [tokens, >= q_rank + kv_rank + rot]; without qw the first q_rank columns are passed over and there is no cq
void latent_prepare(const Tensor& proj, int64_t q_rank, int64_t kv_rank, const OptTensor& qw, const Tensor& kw, double eps, const Tensor& rope,
                    const Tensor& positions, const Tensor& slots, const OptTensor& cq, Tensor& cache, const Tensor& status) {
  const int f = elem(proj);
  const auto dt = proj.scalar_type();
  TORCH_CHECK(proj.dim() == 2 && cache.dim() == 3 && rope.dim() == 2, "latent_prepare: ranks");
  const int64_t T = proj.size(0), rot = cache.size(2) - kv_rank;
  TORCH_CHECK(q_rank > 0 && kv_rank > 0 && rot >= 0 && proj.size(1) >= q_rank + kv_rank + rot && rope.size(1) == rot && qw.has_value() == cq.has_value(),
              "latent_prepare: sizes");
  const c10::cuda::CUDAGuard guard(proj.device());
  check_rc(forge_latent_prepare(f, data(proj, dt, 0, "proj"), proj.size(1), i32(T), i32(q_rank), i32(kv_rank), i32(rot),
                                qw.has_value() ? data(*qw, dt, q_rank, "qw") : nullptr,
                                data(kw, dt, kv_rank, "kw"), static_cast<float>(eps), floats(rope, 0, "rope"), i32(rope.size(0)),
                                ints(positions, T, "positions"), ints(slots, T, "slots"), cq.has_value() ? data(*cq, dt, T * q_rank, "cq") : nullptr,
                                data(cache, dt, 0, "cache"), static_cast<long long>(cache.size(0)) * cache.size(1), status_word(status),
                                stream_of(proj)),
           "forge_latent_prepare");
}

// q [tokens, heads * (dim + rot)] (a view) -> the rotated parts in qa [tokens, heads, kv_rank + rot]
void latent_rotate_q(const Tensor& q, Tensor& qa, int64_t dim, int64_t kv_rank, const Tensor& rope, const Tensor& positions) {
  const int f = elem(q);
  TORCH_CHECK(q.dim() == 2 && qa.dim() == 3 && rope.dim() == 2, "latent_rotate_q: ranks");
  const int64_t T = q.size(0), H = qa.size(1), rot = rope.size(1);
  TORCH_CHECK(qa.size(0) == T && q.size(1) == H * (dim + rot) && qa.size(2) == kv_rank + rot, "latent_rotate_q: sizes");
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_latent_rotate_q(f, view2(q, q.scalar_type(), T, H * (dim + rot), "q"), q.stride(0), data(qa, q.scalar_type(), 0, "qa"), i32(T), i32(H), i32(dim), i32(rot),
                                 i32(kv_rank), floats(rope, 0, "rope"), i32(rope.size(0)), ints(positions, T, "positions"), stream_of(q)),
           "forge_latent_rotate_q");
}

// qa [tokens, heads, kv_rank + rot] = the step's tokens tok0 .. tok0 + tokens; o [tokens, heads, kv_rank]
void latent_attend_any(const Tensor& qa, const Tensor& cache, Tensor& o, int64_t tok0, const Tensor& cu, int64_t num_seqs,
                       const Tensor& positions, const Tensor& block_tables, int64_t window, double scale, const Tensor& status) {
  const int f = elem(qa);
  TORCH_CHECK(window >= 0, "latent_attend_any: window");
  TORCH_CHECK(qa.dim() == 3 && cache.dim() == 3 && o.dim() == 3 && block_tables.dim() == 2, "latent_attend_any: ranks");
  const int64_t T = qa.size(0), H = qa.size(1), R = o.size(2), D = qa.size(2);
  TORCH_CHECK(o.size(0) == T && o.size(1) == H && cache.size(2) == D && R <= D && block_tables.size(0) >= num_seqs, "latent_attend_any: sizes");
  const c10::cuda::CUDAGuard guard(qa.device());
  check_rc(forge_latent_attend_any(f, data(qa, qa.scalar_type(), 0, "qa"), data(cache, qa.scalar_type(), 0, "cache"),
                                   data(o, qa.scalar_type(), 0, "o"), i32(tok0), i32(T), ints(cu, num_seqs + 1, "cu_seqlens_q"), i32(num_seqs),
                                   ints(positions, tok0 + T, "positions"), ints(block_tables, 0, "block_tables"), i32(block_tables.size(1)),
                                   i32(cache.size(0)), i32(cache.size(1)), i32(H), i32(R), i32(D - R), i32(window),
                                   static_cast<float>(scale), status_word(status), stream_of(qa)),
           "forge_latent_attend_any");
}

struct Ret {
  int64_t T, H, dk, dv, slots;
};
Ret retention_sizes(const Tensor& qkvg, const Tensor& decay, const Tensor& state, const Tensor& rope) {
  TORCH_CHECK(qkvg.dim() == 2 && state.dim() == 4 && rope.dim() == 2, "retention: ranks");
  const Ret r{qkvg.size(0), state.size(1), state.size(2), state.size(3), state.size(0)};
  TORCH_CHECK(qkvg.size(1) == r.H * (2 * r.dk + 2 * r.dv) && decay.numel() == r.H && rope.size(1) <= r.dk && rope.size(1) % 2 == 0, "retention: sizes");
  return r;
}

void retention_decode(const Tensor& qkvg, const Tensor& decay, Tensor& state, const Tensor& slots, const Tensor& positions, const Tensor& rope,
                      int64_t seqs, Tensor& y, double eps, const Tensor& status) {
  const int f = elem(qkvg);
  const Ret r = retention_sizes(qkvg, decay, state, rope);
  TORCH_CHECK(seqs <= r.T, "retention_decode: sequences");
  const c10::cuda::CUDAGuard guard(qkvg.device());
  check_rc(forge_retention_decode(f, data(qkvg, qkvg.scalar_type(), 0, "qkvg"), i32(qkvg.size(1)), floats(decay, r.H, "decay"),
                                  floats(state, 0, "state"), ints(slots, seqs, "slots"), ints(positions, seqs, "positions"),
                                  floats(rope, 0, "rope"), i32(rope.size(0)), i32(rope.size(1)), i32(seqs), i32(r.H), i32(r.dk), i32(r.dv),
                                  i32(r.slots), data(y, qkvg.scalar_type(), seqs * r.H * r.dv, "y"), static_cast<float>(eps),
                                  status_word(status), stream_of(qkvg)),
           "forge_retention_decode");
}

void retention_scan(const Tensor& qkvg, const Tensor& decay, Tensor& state, const Tensor& slots, const Tensor& positions, const Tensor& rope,
                    const Tensor& cu, int64_t seqs, Tensor& o, const Tensor& status) {
  const int f = elem(qkvg);
  const Ret r = retention_sizes(qkvg, decay, state, rope);
  const c10::cuda::CUDAGuard guard(qkvg.device());
  check_rc(forge_retention_scan(f, data(qkvg, qkvg.scalar_type(), 0, "qkvg"), i32(qkvg.size(1)), floats(decay, r.H, "decay"),
                                floats(state, 0, "state"), ints(slots, seqs, "slots"), ints(positions, r.T, "positions"),
                                floats(rope, 0, "rope"), i32(rope.size(0)), i32(rope.size(1)), ints(cu, seqs + 1, "cu"), i32(seqs), i32(r.H),
                                i32(r.dk), i32(r.dv), i32(r.slots), floats(o, r.T * r.H * r.dv, "o"), status_word(status), stream_of(qkvg)),
           "forge_retention_scan");
}

// o fp32 [T, heads * dv] -> y [T, heads * dv] for the tokens from tok0 on
void retention_gate(const Tensor& o, const Tensor& qkvg, Tensor& y, int64_t tok0, int64_t heads, int64_t dv, double eps) {
  const int f = elem(qkvg);
  const int64_t T = qkvg.size(0), ld = qkvg.size(1);
  TORCH_CHECK(qkvg.dim() == 2 && tok0 >= 0 && tok0 <= T && ld >= heads * dv, "retention_gate: sizes");
  const c10::cuda::CUDAGuard guard(qkvg.device());
  check_rc(forge_retention_gate(f, floats(o, T * heads * dv, "o"), data(qkvg, qkvg.scalar_type(), 0, "qkvg"), i32(ld), i32(ld - heads * dv),
                                data(y, qkvg.scalar_type(), T * heads * dv, "y"), i32(tok0), i32(T - tok0), i32(heads), i32(dv),
                                static_cast<float>(eps), stream_of(qkvg)),
           "forge_retention_gate");
}

// correction fp32 [experts]; the experts of the `keep` best of `groups` groups can be chosen
void router(const Tensor& h, const Tensor& w, Tensor& experts, Tensor& weights, bool softmax, const OptTensor& correction, int64_t groups, int64_t keep) {
  const int f = elem(h);
  TORCH_CHECK(h.dim() == 2 && w.dim() == 2 && w.size(1) == h.size(1) && experts.dim() == 2 && experts.size(0) == h.size(0), "router: shapes");
  const int64_t T = h.size(0), W = h.size(1), E = w.size(0), top = experts.size(1);
  const c10::cuda::CUDAGuard guard(h.device());
  check_rc(forge_router(f, data(h, h.scalar_type(), 0, "h"), data(w, h.scalar_type(), 0, "w"), i32(T), i32(W), i32(E), i32(top), softmax ? 1 : 0,
                        correction.has_value() ? floats(*correction, E, "correction") : nullptr, i32(groups), i32(keep), const_cast<int*>(ints(experts, T * top, "experts")), floats(weights, T * top, "weights"), stream_of(h)),
           "forge_router");
}

void moe_plan(const Tensor& experts, int64_t E, int64_t tile, Tensor& pos, Tensor& tile_expert, Tensor& num_tiles) {
  const int64_t n = experts.numel();
  // an expert with c rows takes ceil(c / tile) tiles, at least one row each
  const int64_t worst = std::min(n, n / tile + E);
  const c10::cuda::CUDAGuard guard(experts.device());
  check_rc(forge_moe_plan(ints(experts, n, "experts"), i32(n), i32(E), i32(tile), i32(tile_expert.numel()),
                          const_cast<int*>(ints(pos, n, "pos")), const_cast<int*>(ints(tile_expert, worst, "tile_expert")),
                          const_cast<int*>(ints(num_tiles, 1, "num_tiles")), stream_of(experts)),
           "forge_moe_plan");
}

void moe_scatter(const Tensor& h, const Tensor& pos, const OptTensor& weights, Tensor& xs) {
  const int f = elem(h);
  TORCH_CHECK(h.dim() == 2 && pos.dim() == 2 && pos.size(0) == h.size(0) && xs.dim() == 2 && xs.size(1) == h.size(1), "moe_scatter: shapes");
  const int64_t n = pos.numel();
  const c10::cuda::CUDAGuard guard(h.device());
  check_rc(forge_moe_scatter(f, data(h, h.scalar_type(), 0, "h"), ints(pos, n, "pos"), weights.has_value() ? floats(*weights, n, "weights") : nullptr, i32(n), i32(pos.size(1)),
                             i32(h.size(1)), data(xs, h.scalar_type(), 0, "xs"), stream_of(h)),
           "forge_moe_scatter");
}

// ---- tensor-core kernels (bf16)
constexpr auto kBf16 = at::kBFloat16;

void grouped_gemm(const Tensor& x, const Tensor& w, Tensor& out, bool gated, int64_t tile, const Tensor& tile_expert, const Tensor& num_tiles,
                  int64_t act, double limit, const Tensor& status) {
  TORCH_CHECK(x.dim() == 2 && w.dim() == 3 && out.dim() == 2 && w.size(2) == x.size(1), "grouped_gemm: ranks");
  const int64_t rows = x.size(0), K = x.size(1), N = gated ? w.size(1) / 2 : w.size(1), tiles = tile_expert.numel();
  TORCH_CHECK(rows == tiles * tile && out.size(0) == rows && out.size(1) == N, "grouped_gemm: shapes");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_grouped_gemm(data(x, kBf16, 0, "x"), data(w, kBf16, 0, "w"), data(out, kBf16, 0, "out"), i32(w.size(0)), i32(N), i32(K),
                              gated ? 1 : 0, i32(tile), i32(act), static_cast<float>(limit), ints(tile_expert, 0, "tile_expert"), ints(num_tiles, 1, "num_tiles"), i32(tiles),
                              status_word(status), stream_of(x)),
           "forge_grouped_gemm");
}

// x [tokens, heads, K] and out [tokens, heads, N] may be strided views; w [heads, N, K] contiguous
void head_linear(const Tensor& x, const Tensor& w, Tensor& out) {
  TORCH_CHECK(x.is_cuda() && out.is_cuda() && x.scalar_type() == kBf16 && out.scalar_type() == kBf16, "head_linear: operands");
  TORCH_CHECK(x.dim() == 3 && w.dim() == 3 && out.dim() == 3 && x.stride(2) == 1 && out.stride(2) == 1, "head_linear: ranks");
  TORCH_CHECK(x.size(0) == out.size(0) && x.size(1) == w.size(0) && out.size(1) == w.size(0) && w.size(2) == x.size(2) && w.size(1) == out.size(2),
              "head_linear: shapes");
  const c10::cuda::CUDAGuard guard(x.device());
  check_rc(forge_head_linear(x.data_ptr(), x.stride(0), x.stride(1), data(w, kBf16, 0, "w"), out.data_ptr(), out.stride(0), out.stride(1),
                             i32(x.size(0)), i32(w.size(0)), i32(w.size(1)), i32(w.size(2)), stream_of(x)),
           "forge_head_linear");
}

// scratch: fp32, latent_decode_scratch(heads, R, ctas) elements
void latent_decode(const Tensor& qa, const Tensor& cache, const Tensor& block_tables, const Tensor& lens, Tensor& o, Tensor& scratch, int64_t ctas,
                   int64_t window, double scale, const Tensor& status) {
  TORCH_CHECK(window >= 0, "latent_decode: window");
  TORCH_CHECK(qa.dim() == 3 && cache.dim() == 3 && block_tables.dim() == 2 && o.dim() == 3, "latent_decode: ranks");
  const int64_t B = qa.size(0), H = qa.size(1), D = qa.size(2), R = o.size(2);
  TORCH_CHECK(cache.size(2) == D && R <= D && o.size(0) == B && o.size(1) == H && block_tables.size(0) >= B, "latent_decode: shapes");
  const c10::cuda::CUDAGuard guard(qa.device());
  check_rc(forge_latent_decode(data(qa, kBf16, 0, "qa"), data(cache, kBf16, 0, "cache"), ints(block_tables, 0, "block_tables"), ints(lens, B, "lens"),
                               data(o, kBf16, 0, "o"), floats(scratch, forge_latent_decode_scratch(i32(H), i32(R), i32(ctas)), "scratch"), i32(ctas),
                               i32(B), i32(H), i32(R), i32(D - R), i32(block_tables.size(1)), i32(cache.size(0)), i32(cache.size(1)),
                               i32(window), static_cast<float>(scale), status_word(status), stream_of(qa)),
           "forge_latent_decode");
}

// c [keys, R], kr [keys, rot] <- the cached rows of the sequences, of each the last cu_k[s + 1] - cu_k[s] of lens[s]; zeros after them
void latent_gather(const Tensor& cache, const Tensor& cu_k, const Tensor& lens, int64_t num_seqs, const Tensor& block_tables, Tensor& c, Tensor& kr, const Tensor& status) {
  TORCH_CHECK(cache.dim() == 3 && block_tables.dim() == 2 && c.dim() == 2 && kr.dim() == 2, "latent_gather: ranks");
  const int64_t keys = c.size(0), R = c.size(1), rot = kr.size(1);
  TORCH_CHECK(kr.size(0) == keys && cache.size(2) == R + rot && block_tables.size(0) >= num_seqs, "latent_gather: shapes");
  const c10::cuda::CUDAGuard guard(cache.device());
  check_rc(forge_latent_gather(data(cache, kBf16, 0, "cache"), ints(cu_k, num_seqs + 1, "cu_k"), ints(lens, num_seqs, "lens"), i32(num_seqs), ints(block_tables, 0, "block_tables"),
                               i32(block_tables.size(1)), i32(cache.size(0)), i32(cache.size(1)), i32(R), i32(rot), i32(keys),
                               data(c, kBf16, 0, "c"), data(kr, kBf16, 0, "kr"), status_word(status), stream_of(cache)),
           "forge_latent_gather");
}

void latent_pack_q(const Tensor& q, Tensor& qp, int64_t heads, int64_t dim, const Tensor& rope, const Tensor& positions) {
  TORCH_CHECK(q.dim() == 2 && qp.dim() == 3 && rope.dim() == 2, "latent_pack_q: ranks");
  const int64_t T = q.size(0), rot = rope.size(1);
  TORCH_CHECK(q.size(1) == heads * (dim + rot) && qp.size(0) == T && qp.size(1) == heads && qp.size(2) == 64 * ((dim + 63) / 64 + (rot + 63) / 64),
              "latent_pack_q: shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  check_rc(forge_latent_pack_q(view2(q, kBf16, T, heads * (dim + rot), "q"), q.stride(0), data(qp, kBf16, 0, "qp"), i32(T), i32(heads), i32(dim), i32(rot), floats(rope, 0, "rope"),
                               i32(rope.size(0)), ints(positions, T, "positions"), stream_of(q)),
           "forge_latent_pack_q");
}

// qp [tokens - tok0, heads, qcols], kv [keys, heads * (dim + vdim)], kr [keys, rot], out [tokens, heads * vdim]
void latent_prefill(const Tensor& qp, const Tensor& kv, const Tensor& kr, const Tensor& cu_q, const Tensor& cu_k, Tensor& out, int64_t tok0,
                    int64_t num_seqs, int64_t max_q, int64_t dim, int64_t vdim, int64_t window, double scale, const Tensor& status) {
  TORCH_CHECK(window >= 0, "latent_prefill: window");
  TORCH_CHECK(qp.dim() == 3 && kv.dim() == 2 && kr.dim() == 2 && out.dim() == 2, "latent_prefill: ranks");
  const int64_t H = qp.size(1), T = out.size(0), keys = kv.size(0), rot = kr.size(1);
  TORCH_CHECK(qp.size(0) == T - tok0 && kv.size(1) == H * (dim + vdim) && kr.size(0) == keys && out.size(1) == H * vdim &&
                  qp.size(2) == forge_latent_prefill_qcols(i32(dim), i32(rot), i32(vdim)),
              "latent_prefill: shapes");
  const c10::cuda::CUDAGuard guard(qp.device());
  check_rc(forge_latent_prefill(data(qp, kBf16, 0, "qp"), data(kv, kBf16, 0, "kv"), data(kr, kBf16, 0, "kr"), ints(cu_q, num_seqs + 1, "cu_q"),
                                ints(cu_k, num_seqs + 1, "cu_k"), data(out, kBf16, 0, "out"), i32(T), i32(tok0), i32(keys), i32(num_seqs),
                                i32(max_q), i32(H), i32(dim), i32(rot), i32(vdim), i32(window), static_cast<float>(scale), status_word(status),
                                stream_of(qp)),
           "forge_latent_prefill");
}

// q and k of qkvg are rotated in place (tokens from tok0 on); o fp32 [tokens, heads * dv]
void retention_chunk(Tensor& qkvg, const Tensor& decay, Tensor& state, const Tensor& slots, const Tensor& positions, const Tensor& rope,
                     const Tensor& cu, int64_t seqs, int64_t tok0, Tensor& o, const OptTensor& ws, int64_t segs, int64_t seg_len,
                     const Tensor& status) {
  const Ret r = retention_sizes(qkvg, decay, state, rope);
  float* wp = nullptr;
  if (segs > 1) {
    TORCH_CHECK(ws.has_value(), "retention_chunk: scratch");
    wp = floats(*ws, seqs * segs * r.H * r.dk * r.dv, "ws");
    TORCH_CHECK(segs * seg_len >= r.T - tok0 || seqs > 1, "retention_chunk: segments do not cover the run");
  }
  const c10::cuda::CUDAGuard guard(qkvg.device());
  check_rc(forge_retention_chunk(data(qkvg, kBf16, 0, "qkvg"), i32(qkvg.size(1)), floats(decay, r.H, "decay"), floats(state, 0, "state"),
                                 ints(slots, seqs, "slots"), ints(positions, r.T, "positions"), floats(rope, 0, "rope"), i32(rope.size(0)),
                                 i32(rope.size(1)), ints(cu, seqs + 1, "cu"), i32(seqs), i32(tok0), i32(r.T), i32(r.H), i32(r.dk), i32(r.dv),
                                 i32(r.slots), floats(o, r.T * r.H * r.dv, "o"), wp, i32(segs), i32(seg_len), status_word(status),
                                 stream_of(qkvg)),
           "forge_retention_chunk");
}

}  // namespace

void register_mixers(pybind11::module& m) {
  m.def("stream_update", &stream_update);
  m.def("stream_sandwich", &stream_sandwich);
  m.def("stream_group", &stream_group);
  m.def("act_any", &act_any);
  m.def("bound_logits", &bound_logits);
  m.def("gemm_act", &gemm_act);
  m.def("act_mul_any", &act_mul_any);
  m.def("gemm_simt", &gemm_simt);
  m.def("latent_prepare", &latent_prepare);
  m.def("latent_rotate_q", &latent_rotate_q);
  m.def("latent_attend_any", &latent_attend_any);
  m.def("retention_decode", &retention_decode);
  m.def("retention_scan", &retention_scan);
  m.def("retention_gate", &retention_gate);
  m.def("router", &router);
  m.def("moe_plan", &moe_plan);
  m.def("moe_scatter", &moe_scatter);
  m.def("grouped_gemm", &grouped_gemm);
  m.def("head_linear", &head_linear);
  m.def("latent_decode", &latent_decode);
  m.def("latent_decode_scratch", [](int64_t H, int64_t R, int64_t ctas) { return static_cast<int64_t>(forge_latent_decode_scratch(i32(H), i32(R), i32(ctas))); });
  m.def("latent_decode_ok", [](int64_t R, int64_t rot, int64_t bs) { return forge_latent_decode_ok(i32(R), i32(rot), i32(bs)) != 0; });
  m.def("latent_gather", &latent_gather);
  m.def("latent_pack_q", &latent_pack_q);
  m.def("latent_prefill", &latent_prefill);
  m.def("latent_prefill_qcols", [](int64_t dim, int64_t rot, int64_t vdim) { return forge_latent_prefill_qcols(i32(dim), i32(rot), i32(vdim)); });
  m.def("retention_chunk", &retention_chunk);
  m.def("retention_chunk_cols", [](int64_t dk, int64_t dv) { return forge_retention_chunk_cols(i32(dk), i32(dv)); });
  m.def("retention_chunk_ok", [](int64_t H, int64_t dk, int64_t dv, int64_t rd) { return forge_retention_chunk_ok(i32(H), i32(dk), i32(dv), i32(rd)) != 0; });
}
