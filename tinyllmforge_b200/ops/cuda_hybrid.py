"""CUDA ops of decoders built from ``models/hybrid_blocks.py``: windowed attention, short convolutions, recurrences with a
decay per token.

Every op exists for bf16 and for fp32 operands and for any sizes (``windowed_attend_any``, ``recurrence``); the bf16 sizes of
real models go to the tensor-core kernels.  The choice depends on types, sizes and the batch's shape only.
"""
from __future__ import annotations

import torch


def _aligned(*views) -> bool:
    """16-byte rows, as the asynchronous copies and TMA want them."""
    return all(v.data_ptr() % 16 == 0 and v.stride(0) % 8 == 0 for v in views)


class HybridOps:
    """Mixed into ``CudaOps`` (uses its ``C``, ``status``, ``device`` and ``num_sms``)."""

    @staticmethod
    def _singles(batch) -> int:
        """Leading sequences of the step with one token each (a decode step's padding rows included)."""
        return batch.num_single if batch.is_prefill else batch.padded_seqs

    # ------------------------------------------------------------------ windowed attention
    def bias_rope_store(self, proj, bias, spec, table, positions, slot_mapping, k_cache, v_cache):
        """q [T, heads, columns]: the columns from ``dim`` on are zero."""
        cols = self.C.windowed_prefill_qcols(spec.dim, spec.vdim, k_cache.shape[2]) if proj.dtype == torch.bfloat16 else 0
        q = torch.empty(proj.shape[0], spec.heads, cols or spec.dim, dtype=proj.dtype, device=proj.device)
        self.C.bias_rope_store(proj, bias, table, positions, slot_mapping, q, k_cache, v_cache, self.status)
        return q

    def norm_rope_store(self, proj, q_norm, k_norm, eps, spec, table, positions, slot_mapping, k_cache, v_cache, temper=None):
        """q [T, heads, columns]: the columns from ``dim`` on are zero.  Without ``k_norm`` proj is q alone."""
        if k_norm is None:
            proj = proj[:, :spec.heads * spec.dim]
        cols = self.C.windowed_prefill_qcols(spec.dim, spec.vdim, k_cache.shape[2]) if proj.dtype == torch.bfloat16 else 0
        q = torch.empty(proj.shape[0], spec.heads, cols or spec.dim, dtype=proj.dtype, device=proj.device)
        self.C.norm_rope_store(proj, q_norm, k_norm, spec.norm == "all", eps, table, positions, slot_mapping, q, k_cache, v_cache, temper, self.status)
        return q

    def windowed_attention(self, q, k_cache, v_cache, batch, spec, out, scale, chunked=False, softcap=0.0, sink=None, gate=None, pool=None) -> None:
        """out (a view [T, heads * vdim]) <- scale * attention over the last ``spec.window`` tokens, or inside chunks of that many.  ``pool`` (a
        ``PooledCache``): with the means of the blocks behind the window; blocks that end in this step get theirs."""
        d, dv, bs = spec.dim, spec.vdim, k_cache.shape[2]
        bf16, seqs = q.dtype == torch.bfloat16, batch.padded_seqs
        options = (spec.window, spec.scale, scale, chunked, softcap, sink, gate)
        size = 0 if pool is None else pool.size
        means = (None, None, 0) if pool is None else (pool.k, pool.v, size)
        n1 = self._singles(batch)
        if n1 and bf16 and self.C.windowed_decode_ok(d, dv, bs):
            chunk, chunks = self.windowed_chunks(n1, spec, batch.table_width * bs, size)
            part_o = part_ml = None
            if chunks > 1:
                part_o = torch.empty(n1 * spec.heads * chunks * dv, dtype=torch.float32, device=q.device)
                part_ml = torch.empty(n1 * spec.heads * chunks * 2, dtype=torch.float32, device=q.device)
            self.C.windowed_decode(q, k_cache, v_cache, batch.block_tables, batch.context_lens, n1, out, part_o, part_ml, chunk, chunks, *options,
                                   *means, pool is not None and pool.own, self.status)
        else:
            n1 = 0
        if seqs == n1:
            return
        cu, tables, lens = batch.cu_seqlens_q[n1:], batch.block_tables[n1:], batch.context_lens[n1:]
        rows = (out,) if gate is None or gate.shape[1] == spec.heads else (out, gate)
        if bf16 and spec.scale > 0 and batch.is_prefill and q.shape[2] == self.C.windowed_prefill_qcols(d, dv, bs) and _aligned(*rows):
            gathered = self.pool_blocks(k_cache, v_cache, pool, batch, n1, cu, lens, tables, spec.window)
            self.C.windowed_prefill(q, k_cache, v_cache, cu, lens, tables, seqs - n1, batch.max_seqlen_q, out, *options, *gathered, self.status)
        else:
            self.pool_blocks(k_cache, v_cache, pool, batch, n1, cu, lens, tables)
            self.C.windowed_attend_any(q, k_cache, v_cache, cu, seqs - n1, batch.max_seqlen_q, batch.positions, tables, out, *options, *means, self.status)

    def pool_blocks(self, k_cache, v_cache, pool, batch, n1, cu, lens, tables, window=None):
        """The means of the blocks that end in the step's tokens, for the sequences from ``n1`` on; with ``window`` all their entries one after
        another for a kernel whose tiles cannot gather them: (keys, values, first rows, size), or nothing where no token sees a block."""
        if pool is None:
            return None, None, None, 0
        seqs = batch.padded_seqs - n1
        entries = (batch.kv_rows if n1 == batch.num_single else seqs * batch.max_seqlen_k) // pool.size
        gather = window is not None and entries > 0 and batch.max_seqlen_k - window >= pool.size
        offsets = gk = gv = None
        if gather:
            offsets = self.row_offsets(batch, n1, size=pool.size)
            gk, gv = (torch.empty(entries, k_cache.shape[1], c.shape[3], dtype=k_cache.dtype, device=k_cache.device) for c in (k_cache, v_cache))
        self.C.pool_blocks(k_cache, v_cache, pool.k, pool.v, pool.size, pool.own, cu, lens, tables, seqs, batch.max_seqlen_q, batch.max_seqlen_k,
                           offsets, gk, gv, self.status)
        return gk, gv, offsets, pool.size if gather else 0

    def windowed_chunks(self, seqs: int, spec, capacity: int, pool: int = 0) -> tuple[int, int]:
        """(keys per chunk, chunks): the window, and the pooled blocks ahead of it, are cut until the two CTAs that an SM holds are busy.
        Depends only on shapes known at graph-capture time."""
        span = min(spec.window, capacity) + 15 + (capacity // pool + 15 if pool else 0)
        ctas = seqs * spec.kv_heads * -(-(spec.heads // spec.kv_heads) // 16)
        parts = max(1, min(2 * self.num_sms // ctas, span // 128))
        chunk = -(-(-(-span // parts)) // 64) * 64
        return chunk, -(-span // chunk)

    # ------------------------------------------------------------------ recurrences
    def short_conv(self, x, taps, bias, state, batch, act="silu"):
        out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
        self.C.short_conv(x, taps, bias, state, batch.state_slots, batch.positions, batch.cu_seqlens_q, batch.padded_seqs, batch.max_seqlen_q,
                          out, act == "silu", self.status)
        return out

    def recur(self, q, k, v, dt, beta, block, state, batch):
        """o fp32 [T, heads, vdim]: single tokens through the decode kernel, runs of tokens through the chunked ones.  With
        ``beta`` the delta rule, without it the state-space recurrence."""
        D = None if beta is not None else block.D
        T, (_, H, dk, dv) = q.shape[0], state.shape
        o = torch.empty(T, H, dv, dtype=torch.float32, device=q.device)
        n1 = self._singles(batch)
        args = (q, k, v, dt, beta, block.A_log, block.dt_bias, D, state)
        if n1 and not self.C.recurrence_decode_ok(dk, dv):
            n1 = 0                                      # the scan takes single tokens too (padding rows have empty ranges)
        if n1:
            self.C.recurrence(*args, batch.state_slots, batch.positions, None, n1, o, self.status)
        seqs = batch.padded_seqs - n1
        if seqs == 0:
            return o
        slots, cu = batch.state_slots[n1:], batch.cu_seqlens_q[n1:]
        chunked = (self.C.state_space_chunk_ok if beta is None else self.C.delta_chunk_ok)(dk, dv)
        if not (chunked and q.dtype == torch.bfloat16 and batch.is_prefill and _aligned(q, k, v)):
            self.C.recurrence(*args, slots, batch.positions, cu, seqs, o, self.status)
            return o
        cum, weight = (torch.empty(H, T, dtype=torch.float32, device=q.device) for _ in range(2))
        self.C.recurrence_gates(dt, beta, block.A_log, block.dt_bias, cu, seqs, batch.max_seqlen_q, cum, weight)
        if beta is None:
            segs, seg_len = self.retention_segments(seqs, H, dk, dv, batch.max_seqlen_q)
            ws = decays = None
            if segs > 1:
                ws = torch.empty(seqs * segs * H * dk * dv, dtype=torch.float32, device=q.device)
                decays = torch.empty(seqs * segs * H, dtype=torch.float32, device=q.device)
            self.C.state_space_chunk(q, k, v, cum, weight, D, state, slots, batch.positions, cu, seqs, o, ws, decays, segs, seg_len, self.status)
        else:
            mats = torch.empty(self.C.delta_chunk_scratch(T, seqs, H, 0), dtype=torch.bfloat16, device=q.device)
            factors = torch.empty(self.C.delta_chunk_scratch(T, seqs, H, 1), dtype=torch.float32, device=q.device)
            self.C.delta_chunk(q, k, v, cum, weight, state, slots, batch.positions, cu, seqs, batch.max_seqlen_q, mats, factors, o,
                               self.delta_columns(seqs, H, dv), self.status)
        return o

    def delta_columns(self, seqs: int, heads: int, dv: int) -> int:
        """Value columns per CTA of the chunked delta rule: narrow slices where wide ones leave half of the SMs idle."""
        return 64 if 2 * seqs * heads * -(-dv // 64) > self.num_sms else 32

    def state_space(self, xbc, z, dt, block, state, batch, out, scale) -> None:
        s = block.spec
        n = s.groups * s.state
        x, B, C = xbc[:, :s.inner], xbc[:, s.inner:s.inner + n], xbc[:, s.inner + n:]
        y = self.recur(C, B, x, dt, None, block, state, batch)
        self.C.gated_norm(y, z, block.norm, out, s.norm_groups, True, scale, block.eps)

    def gated_delta(self, qkv, gate, ba, block, state, batch):
        s = block.spec
        n = s.kv_heads * s.dim
        o = self.recur(qkv[:, :n], qkv[:, n:2 * n], qkv[:, 2 * n:], ba[:, s.heads:], ba[:, :s.heads], block, state, batch)
        y = torch.empty(qkv.shape[0], s.heads * s.vdim, dtype=qkv.dtype, device=qkv.device)
        self.C.gated_norm(o, gate, block.norm, y, s.heads, False, 1.0, block.eps)
        return y
