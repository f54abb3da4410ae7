"""CUDA ops of decoders built from ``models/hybrid_blocks.py``: windowed attention, short convolutions, recurrences with a
decay per token.

Every op exists for bf16 and for fp32 operands and for any sizes; the bf16 sizes of real models go to the tensor-core
kernels.  The choice depends on types, sizes and the batch's shape only.
"""
from __future__ import annotations

import torch


class HybridOps:
    """Mixed into ``CudaOps`` (uses its ``C``, ``status`` and ``device``)."""

    @staticmethod
    def _singles(batch) -> int:
        """Leading sequences of the step with one token each (a decode step's padding rows included)."""
        return batch.num_single if batch.is_prefill else batch.padded_seqs

    # ------------------------------------------------------------------ windowed attention
    def bias_rope_store(self, proj, bias, spec, table, positions, slot_mapping, k_cache, v_cache):
        q = torch.empty(proj.shape[0], spec.heads, spec.dim, dtype=proj.dtype, device=proj.device)
        self.C.bias_rope_store(proj, bias, table, positions, slot_mapping, q, k_cache, v_cache, self.status)
        return q

    def windowed_attention(self, q, k_cache, v_cache, batch, spec, out, scale) -> None:
        """out (a view [T, heads * vdim]) <- scale * attention over the last ``spec.window`` tokens."""
        self.C.windowed_attend_any(q, k_cache, v_cache, batch.cu_seqlens_q, batch.padded_seqs, batch.max_seqlen_q, batch.positions,
                                   batch.block_tables, out, spec.window, spec.scale, scale, self.status)

    # ------------------------------------------------------------------ recurrences
    def short_conv(self, x, taps, bias, state, batch):
        out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
        self.C.short_conv(x, taps, bias, state, batch.state_slots, batch.positions, batch.cu_seqlens_q, batch.padded_seqs, batch.max_seqlen_q,
                          out, self.status)
        return out

    def _recur(self, q, k, v, dt, beta, block, state, batch):
        """o fp32 [T, heads, vdim]: single tokens through the decode kernel, runs of tokens through the others."""
        D = None if beta is not None else block.D
        o = torch.empty(q.shape[0], state.shape[1], state.shape[3], dtype=torch.float32, device=q.device)
        n1 = self._singles(batch)
        args = (q, k, v, dt, beta, block.A_log, block.dt_bias, D, state)
        if n1 and not self.C.recurrence_decode_ok(state.shape[2], state.shape[3]):
            n1 = 0                                      # the scan takes single tokens too (padding rows have empty ranges)
        if n1:
            self.C.recurrence(*args, batch.state_slots, batch.positions, None, n1, o, self.status)
        if batch.padded_seqs > n1:
            self.C.recurrence(*args, batch.state_slots[n1:], batch.positions, batch.cu_seqlens_q[n1:], batch.padded_seqs - n1, o, self.status)
        return o

    def state_space(self, xbc, z, dt, block, state, batch, out, scale) -> None:
        s = block.spec
        n = s.groups * s.state
        x, B, C = xbc[:, :s.inner], xbc[:, s.inner:s.inner + n], xbc[:, s.inner + n:]
        y = self._recur(C, B, x, dt, None, block, state, batch)
        self.C.gated_norm(y, z, block.norm, out, s.norm_groups, True, scale, block.eps)

    def gated_delta(self, qkv, gate, ba, block, state, batch):
        s = block.spec
        n = s.kv_heads * s.dim
        o = self._recur(qkv[:, :n], qkv[:, n:2 * n], qkv[:, 2 * n:], ba[:, s.heads:], ba[:, :s.heads], block, state, batch)
        y = torch.empty(qkv.shape[0], s.heads * s.vdim, dtype=qkv.dtype, device=qkv.device)
        self.C.gated_norm(o, gate, block.norm, y, s.heads, False, 1.0, block.eps)
        return y
