"""CUDA ops of decoders built from ``models/blocks.py``: fp32 residual stream, latent attention, retention, experts.

Every op exists for bf16 and for fp32 operands and for any sizes (``*_any`` / ``*_simt`` / ``*_scan`` kernels); the bf16 sizes
of real models go to the tensor-core kernels.  The choice depends on types, sizes and the batch's shape only.
"""
from __future__ import annotations

import torch


class Routed:
    """The output of an expert layer before it is summed: row ``rows[t, j]`` of ``y`` belongs to token t's j-th expert."""

    def __init__(self, y: torch.Tensor, rows: torch.Tensor):
        self.y, self.rows = y, rows


class MixerOps:
    """Mixed into ``CudaOps`` (uses its ``C``, ``status``, ``device`` and GEMM methods)."""

    # ------------------------------------------------------------------ residual stream
    def stream_update(self, x, dtype, eps, norms, start=False, a=None, b=None, ids=None, embed=None, vec=None, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        outs = [torch.empty(n, x.shape[1], dtype=dtype, device=x.device) for _ in norms]
        b_rows = None
        if isinstance(b, Routed):
            b, b_rows = b.y, b.rows
        self.C.stream_update(x, a, b, b_rows, ids, embed, vec, norms[0] if norms else None, norms[1] if len(norms) > 1 else None,
                             outs[0] if outs else None, outs[1] if len(outs) > 1 else None, rows, start, eps, dtype == torch.float32)
        return outs

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

    def silu_mul_any(self, x):
        out = torch.empty(x.shape[0], x.shape[1] // 2, dtype=x.dtype, device=x.device)
        self.C.silu_mul_any(x, out)
        return out

    def head_linear(self, x, w, out) -> None:
        """out[:, h] = x[:, h] @ w[h].T for views x [tokens, heads, K], w [heads, N, K], out [tokens, heads, N]."""
        self.C.gemm_simt(x.transpose(0, 1), w, out.transpose(0, 1), None)

    # ------------------------------------------------------------------ latent attention
    def latent_prepare(self, proj, q_rank, kv_rank, q_norm, kv_norm, eps, table, positions, slot_mapping, cache):
        cq = torch.empty(proj.shape[0], q_rank, dtype=proj.dtype, device=proj.device)
        self.C.latent_prepare(proj, q_rank, kv_rank, q_norm, kv_norm, eps, table, positions, slot_mapping, cq, cache, self.status)
        return cq

    def latent_attention(self, q, weights, cache, batch, table, spec):
        T = q.shape[0]
        out = torch.empty(T, spec.heads * spec.vdim, dtype=q.dtype, device=q.device)
        self._latent_folded(q, weights, cache, batch, table, spec, out, 0, T)
        return out

    def _latent_folded(self, q, weights, cache, batch, table, spec, out, tok0, tok1) -> None:
        """Tokens [tok0, tok1) of the step through the folded form: queries against the cached latents themselves."""
        H, d, r, dv, R = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
        n = tok1 - tok0
        if n <= 0:
            return
        q = q[tok0:tok1]
        qa = torch.empty(n, H, R + r, dtype=q.dtype, device=q.device)
        self.head_linear(q.view(n, H, d + r)[:, :, :d], weights.uk_t, qa[:, :, :R])
        self.C.latent_rotate_q(q, qa, d, R, table, batch.positions[tok0:tok1])
        o = torch.empty(n, H, R, dtype=q.dtype, device=q.device)
        self.C.latent_attend_any(qa, cache, o, tok0, batch.cu_seqlens_q, batch.padded_seqs, batch.positions, batch.block_tables,
                                 spec.scale, self.status)
        self.head_linear(o, weights.uv, out[tok0:tok1].view(n, H, dv))

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
            self.C.retention_scan(qkvg, decay, state, batch.state_slots[n1:], batch.positions, table, batch.cu_seqlens_q[n1:], rest, o,
                                  self.status)
            self.C.retention_gate(o, qkvg, y, n1, H, dv, eps)
        return y

    # ------------------------------------------------------------------ experts
    def moe(self, h, router, gate_up, down, top):
        T, W = h.shape
        E, n = router.shape[0], T * top
        experts = torch.empty(T, top, dtype=torch.int32, device=h.device)
        weights = torch.empty(T, top, dtype=torch.float32, device=h.device)
        self.C.router(h, router, experts, weights)
        tile = 64
        tiles = min(n, n // tile + E)
        rows = torch.empty(T, top, dtype=torch.int32, device=h.device)
        tile_expert = torch.empty(tiles, dtype=torch.int32, device=h.device)
        num_tiles = torch.empty(1, dtype=torch.int32, device=h.device)
        self.C.moe_plan(experts, E, tile, rows, tile_expert, num_tiles)
        xs = torch.empty(tiles * tile, W, dtype=h.dtype, device=h.device)
        self.C.moe_scatter(h, rows, weights, xs)
        gu = torch.empty(tiles * tile, gate_up.shape[1], dtype=h.dtype, device=h.device)
        self.C.gemm_simt(xs, gate_up, gu, tile_expert)
        g = self.silu_mul_any(gu)
        y = torch.empty(tiles * tile, W, dtype=h.dtype, device=h.device)
        self.C.gemm_simt(g, down, y, tile_expert)
        return Routed(y, rows)
