"""CUDA ops of decoders built from ``models/blocks.py``: fp32 residual stream, latent attention, retention, experts.

Every op exists for bf16 and for fp32 operands and for any sizes (``*_any`` / ``*_simt`` / ``*_scan`` kernels); the bf16 sizes
of real models go to the tensor-core kernels.  The choice depends on types, sizes and the batch's shape only.
"""
from __future__ import annotations

import torch


class Routed:
    """The output of an expert layer before it is summed: row ``rows[t, j]`` of ``y`` belongs to token t's j-th expert and
    counts ``weights[t, j]`` times (None: once)."""

    def __init__(self, y: torch.Tensor, rows: torch.Tensor, weights: torch.Tensor | None = None):
        self.y, self.rows, self.weights = y, rows, weights


ACTS = {"silu": 0, "gelu_tanh": 1, "clamped_swish": 2}
PLAIN_ACTS = {"gelu": 1}                        # of feed-forwards without gates


class MixerOps:
    """Mixed into ``CudaOps`` (uses its ``C``, ``status``, ``device`` and GEMM methods)."""

    # ------------------------------------------------------------------ residual stream
    def stream_update(self, x, dtype, eps, norms, start=False, a=None, b=None, ids=None, embed=None, vec=None, rows=None,
                      a_bias=None, post=None, mult=1.0, offset=0.0, groups=1):
        n = x.shape[0] if rows is None else rows.shape[0]
        outs = [torch.empty(n, x.shape[1], dtype=dtype, device=x.device) for _ in norms]
        if groups > 1 or None in norms or (a is None and post is not None):
            if b is not None or vec is not None or a_bias is not None or post is None or len(norms) > 1 or (a is not None and ids is not None):
                raise ValueError("stream_update: grouped norms go with one branch, normed on its way in, and one result")
            a_rows = a_weights = None
            if isinstance(a, Routed):
                a, a_rows, a_weights = a.y, a.rows, a.weights
            self.C.stream_group(x, a, a_rows, a_weights, post, mult, offset, ids, embed, norms[0] if norms else None, outs[0] if outs else None, rows,
                                groups, start, eps, dtype == torch.float32)
            return outs
        if post is not None or offset or isinstance(a, Routed):
            if b is not None or vec is not None or len(norms) > 1:
                raise ValueError("stream_update: one branch and one norm where a is normed or norm weights have an offset")
            a_rows = a_weights = None
            if isinstance(a, Routed):
                a, a_rows, a_weights = a.y, a.rows, a.weights
            self.C.stream_sandwich(x, a, a_rows, a_weights, a_bias, post, mult, offset, ids, embed, norms[0] if norms else None,
                                   outs[0] if outs else None, rows, start, eps, dtype == torch.float32)
            return outs
        b_rows = None
        if isinstance(b, Routed):
            if b.weights is not None:
                raise ValueError("stream_update: b is summed without weights")
            b, b_rows = b.y, b.rows
        self.C.stream_update(x, a, b, b_rows, ids, embed, vec, norms[0] if norms else None, norms[1] if len(norms) > 1 else None,
                             outs[0] if outs else None, outs[1] if len(outs) > 1 else None, rows, start, eps, dtype == torch.float32)
        return outs

    def stream_mix(self, x, dtype, eps, into, norm, bias, y=None, mix=None, out=None, ids=None, prev=None, embed=None, scale=1.0, pairs=None,
                   mul_prev=0, mul_cur=0, rows=None):
        h = None
        if norm is not None:
            h = torch.empty(x.shape[0] if rows is None else rows.shape[0], x.shape[2], dtype=dtype, device=x.device)
        self.C.stream_mix(x, y, mix, out, ids, prev, embed, scale, pairs, mul_prev, mul_cur, into, norm, bias, h, rows, eps, dtype == torch.float32)
        return h

    # ------------------------------------------------------------------ products outside the tcgen05 GEMMs' reach
    @staticmethod
    def tma_ok(x: torch.Tensor, w: torch.Tensor) -> bool:
        """bf16, rows of a multiple of 16 bytes."""
        return (x.dtype == torch.bfloat16 and x.shape[-1] % 8 == 0 and x.stride(-2) % 8 == 0 and w.stride(-2) % 8 == 0
                and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)

    def linear_simt(self, x, w):
        out = torch.empty(x.shape[0], w.shape[0], dtype=x.dtype, device=x.device)
        self.C.gemm_simt(x, w, out, None)
        return out

    def act_mul_any(self, x, act="silu", limit=0.0):
        out = torch.empty(x.shape[0], x.shape[1] // 2, dtype=x.dtype, device=x.device)
        self.C.act_mul_any(x, out, ACTS[act], limit)
        return out

    def linear_act_mul(self, x, w_gate_up, act: str, limit: float = 0.0):
        """act(x @ w_gate.T, x @ w_up.T) for w_gate_up = gate rows, up rows."""
        if act == "silu":
            return self.linear_silu_mul(x, w_gate_up)
        if not self.tma_ok(x, w_gate_up):
            return self.act_mul_any(self.linear_simt(x, w_gate_up), act, limit)
        out = torch.empty(x.shape[0], w_gate_up.shape[0] // 2, dtype=x.dtype, device=x.device)
        self.C.gemm_act(x, w_gate_up, out, ACTS[act], limit, self.status)
        return out

    def head_linear(self, x, w, out) -> None:
        """out[:, h] = x[:, h] @ w[h].T for views x [tokens, heads, K], w [heads, N, K], out [tokens, heads, N]."""
        if (x.dtype == torch.bfloat16 and not (x.shape[2] | x.stride(0) | x.stride(1)) % 8 and not (w.shape[1] | out.stride(0) | out.stride(1)) % 2
                and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0):
            self.C.head_linear(x, w, out)
        else:
            self.C.gemm_simt(x.transpose(0, 1), w, out.transpose(0, 1), None)

    # ------------------------------------------------------------------ latent attention
    def latent_prepare(self, proj, q_rank, kv_rank, q_norm, kv_norm, eps, table, positions, slot_mapping, cache):
        cq = None if q_norm is None else torch.empty(proj.shape[0], q_rank, dtype=proj.dtype, device=proj.device)
        self.C.latent_prepare(proj, q_rank, kv_rank, q_norm, kv_norm, eps, table, positions, slot_mapping, cq, cache, self.status)
        return cq

    def latent_attention(self, q, weights, cache, batch, table, spec):
        """Single tokens go through the folded form (queries against the cached latents themselves), runs of tokens through
        the expanded one (keys and values rebuilt per head)."""
        T = q.shape[0]
        out = torch.empty(T, spec.heads * spec.vdim, dtype=q.dtype, device=q.device)
        n1 = T if not batch.is_prefill else batch.num_single
        if T > n1 and not self._latent_expanded(q, weights, cache, batch, table, spec, out, n1):
            n1 = T
        self._latent_folded(q, weights, cache, batch, table, spec, out, n1)
        return out

    def _latent_folded(self, q, weights, cache, batch, table, spec, out, n) -> None:
        """The first n tokens of the step."""
        H, d, r, dv, R = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
        if n <= 0:
            return
        q = q[:n]
        qa = torch.empty(n, H, R + r, dtype=q.dtype, device=q.device)
        self.head_linear(q.view(n, H, d + r)[:, :, :d], weights.uk_t, qa[:, :, :R])
        self.C.latent_rotate_q(q, qa, d, R, table, batch.positions[:n])
        o = torch.empty(n, H, R, dtype=q.dtype, device=q.device)
        singles = n == (batch.num_single if batch.is_prefill else batch.padded_seqs)
        if singles and q.dtype == torch.bfloat16 and n <= 1024 and self.C.latent_decode_ok(R, r, cache.shape[1]):
            scratch = torch.empty(self.C.latent_decode_scratch(H, R, self.num_sms), dtype=torch.float32, device=q.device)
            self.C.latent_decode(qa, cache, batch.block_tables, batch.context_lens, o, scratch, self.num_sms, spec.window, spec.scale, self.status)
        else:
            self.C.latent_attend_any(qa, cache, o, 0, batch.cu_seqlens_q, batch.padded_seqs, batch.positions, batch.block_tables,
                                     spec.window, spec.scale, self.status)
        self.head_linear(o, weights.uv, out[:n].view(n, H, dv))

    def _latent_expanded(self, q, weights, cache, batch, table, spec, out, n1) -> bool:
        """The sequences from ``n1`` on (their tokens start at row n1).  False: these sizes have no kernel, nothing was done."""
        H, d, r, dv, R = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
        qcols = self.C.latent_prefill_qcols(d, r, dv)
        if q.dtype != torch.bfloat16 or qcols == 0 or R % 8 or q.stride(0) % 8 or q.data_ptr() % 16:
            return False
        T, seqs, keys = q.shape[0], batch.num_seqs - n1, batch.kv_rows
        cu_q, cu_k, tables, lens = batch.cu_seqlens_q[n1:], batch.cu_seqlens_k[n1:], batch.block_tables[n1:], batch.context_lens[n1:]
        if spec.window:                              # the keys that some query of the step sees, and no others
            cu_k, keys = self.row_offsets(batch, n1, window=spec.window), min(keys, T - n1 + seqs * (spec.window - 1))
        c = torch.empty(keys, R, dtype=q.dtype, device=q.device)
        kr = torch.empty(keys, r, dtype=q.dtype, device=q.device)
        self.C.latent_gather(cache, cu_k, lens, seqs, tables, c, kr, self.status)
        kv = self.linear(c, weights.ukv)
        qp = torch.empty(T - n1, H, qcols, dtype=q.dtype, device=q.device)
        self.C.latent_pack_q(q[n1:], qp, H, d, table, batch.positions[n1:])
        self.C.latent_prefill(qp, kv, kr, cu_q, cu_k, out, n1, seqs, batch.max_seqlen_q, d, dv, spec.window, spec.scale, self.status)
        return True

    def row_offsets(self, batch, n1: int, window: int = 0, size: int = 0) -> torch.Tensor:
        """Where the rows of the sequences from ``n1`` on begin in a buffer that holds, of each, its last min(keys, queries + window - 1) keys or
        its floor(keys / size) blocks.  The layers of a step share it."""
        known = batch.__dict__.setdefault("_row_offsets", {})
        if (n1, window, size) not in known:
            seqs = batch.padded_seqs - n1
            out = known[n1, window, size] = torch.empty(seqs + 1, dtype=torch.int32, device=self.device)
            self.C.row_offsets(batch.cu_seqlens_q[n1:], batch.context_lens[n1:], seqs, window, size, out)
        return known[n1, window, size]

    # ------------------------------------------------------------------ retention
    def retention(self, qkvg, decay, state, batch, table, spec, eps):
        T = qkvg.shape[0]
        H, dv = spec.heads, spec.vdim
        y = torch.empty(T, H * dv, dtype=qkvg.dtype, device=qkvg.device)
        n1 = batch.padded_seqs if not batch.is_prefill else batch.num_single
        if n1:
            self.C.retention_decode(qkvg, decay, state, batch.state_slots, batch.positions, table, n1, y, eps, self.status)
        rest = batch.num_seqs - n1
        if batch.is_prefill and rest > 0:
            o = torch.empty(T, H * dv, dtype=torch.float32, device=qkvg.device)
            slots, cu = batch.state_slots[n1:], batch.cu_seqlens_q[n1:]
            if qkvg.dtype == torch.bfloat16 and self.C.retention_chunk_ok(H, spec.dim, dv, table.shape[1]):
                segs, seg_len = self.retention_segments(rest, H, spec.dim, dv, batch.max_seqlen_q)
                ws = torch.empty(rest * segs * H * spec.dim * dv, dtype=torch.float32, device=qkvg.device) if segs > 1 else None
                self.C.retention_chunk(qkvg, decay, state, slots, batch.positions, table, cu, rest, n1, o, ws, segs, seg_len, self.status)
            else:
                self.C.retention_scan(qkvg, decay, state, slots, batch.positions, table, cu, rest, o, self.status)
            self.C.retention_gate(o, qkvg, y, n1, H, dv, eps)
        return y

    def retention_segments(self, seqs: int, heads: int, dk: int, dv: int, longest: int) -> tuple[int, int]:
        """(segments per run, tokens per segment): a run is cut when the batch alone leaves half of the CTA places empty."""
        cols = self.C.retention_chunk_cols(dk, dv)
        want = (self.num_sms if cols == 128 or dk > 128 else 2 * self.num_sms) // (seqs * heads * -(-dv // cols))
        segs = max(1, min(want, longest // 256))
        seg_len = -(-longest // segs)
        seg_len = -(-seg_len // 64) * 64
        return max(1, -(-longest // seg_len)), seg_len

    # ------------------------------------------------------------------ experts
    @staticmethod
    def expert_tile(rows: int, experts: int) -> int:
        """Rows per tile of the tensor-core kernel (16 to 128): about what an expert gets."""
        return next((t for t in (16, 32, 64) if rows <= t * experts), 128)

    def moe(self, h, router, up, down, top, score="sigmoid", weigh="input", act="silu", limit=0.0, gated=True, correction=None, groups=1, keep=1):
        T, W = h.shape
        E, n = router.shape[0], T * top
        experts = torch.empty(T, top, dtype=torch.int32, device=h.device)
        weights = torch.empty(T, top, dtype=torch.float32, device=h.device)
        self.C.router(h, router, experts, weights, score == "softmax", correction, groups, keep)
        fast = h.dtype == torch.bfloat16 and W % 8 == 0 and down.shape[2] % 8 == 0
        tile = self.expert_tile(n, E) if fast else 64
        tiles = min(n, n // tile + E)
        rows = torch.empty(T, top, dtype=torch.int32, device=h.device)
        tile_expert = torch.empty(tiles, dtype=torch.int32, device=h.device)
        num_tiles = torch.empty(1, dtype=torch.int32, device=h.device)
        self.C.moe_plan(experts, E, tile, rows, tile_expert, num_tiles)
        xs = torch.empty(tiles * tile, W, dtype=h.dtype, device=h.device)
        self.C.moe_scatter(h, rows, weights if weigh == "input" else None, xs)
        y = torch.empty(tiles * tile, W, dtype=h.dtype, device=h.device)
        if fast:
            g = torch.empty(tiles * tile, down.shape[2], dtype=h.dtype, device=h.device)
            self.C.grouped_gemm(xs, up, g, gated, tile, tile_expert, num_tiles, (ACTS if gated else PLAIN_ACTS)[act], limit, self.status)
            self.C.grouped_gemm(g, down, y, False, tile, tile_expert, num_tiles, 0, 0.0, self.status)
        else:
            g = torch.empty(tiles * tile, up.shape[1], dtype=h.dtype, device=h.device)
            self.C.gemm_simt(xs, up, g, tile_expert)
            if gated:
                g = self.act_mul_any(g, act, limit)
            else:
                self.C.act_any(g, PLAIN_ACTS[act])
            self.C.gemm_simt(g, down, y, tile_expert)
        return Routed(y, rows, weights if weigh == "output" else None)
