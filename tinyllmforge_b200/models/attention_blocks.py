"""Building blocks of decoders over several residual streams: normed and gated attention, and what joins and splits the streams.

Same interface as ``blocks.py``; projections that read the same input are one matrix, as in ``hybrid_blocks.py``.
"""
from __future__ import annotations

import torch

from .blocks import _empty
from .hybrid_blocks import _f32, _packed


class PooledCache:
    """Means of the keys and values of whole blocks of ``size`` tokens, counted from a sequence's first.  The entry of a block lies in the
    page of the block's last token: a page holds the blocks that end in it, in order.  ``own``: this layer writes the entries (else
    the layer it borrows them from has done so already)."""

    def __init__(self, size: int, k: torch.Tensor, v: torch.Tensor, own: bool = True):
        self.size, self.k, self.v, self.own = size, k, v, own

    @staticmethod
    def rows(block_size: int, size: int) -> int:
        """Entries that a page has room for."""
        return -(-block_size // size)


class NormedAttention:
    """Grouped-query attention whose queries and keys are normed ahead of their rotation, with the options of ``AttentionSpec``: short
    convolutions, chunks or a sliding window, means of the blocks behind it, sinks, capped scores, a factor per head, gated output, keys and
    values of another layer.  Cached per token: rotated keys, and values; per block: their means; kept per sequence: the convolutions' last
    inputs."""

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        s = self.spec = spec
        self.eps = eps
        self.lender = s.kv_from
        self.sizes = (("q", s.heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim))[:3 if s.kv_from is None else 1]
        self.channels = sum(n for _, n in self.sizes)
        self.inp = _packed(self.channels + s.gate_columns, width, dtype, device)
        self.conv = _f32((self.channels, s.conv), device) if s.conv else None
        norms = [torch.ones(s.dim if s.norm == "head" else n, dtype=dtype, device=device) for _, n in self.sizes[:2]]
        self.q_norm, self.k_norm = norms if s.kv_from is None else (norms[0], None)
        self.temper = torch.ones(s.heads, dtype=torch.float32, device=device) if s.temper else None
        self.sink = None if s.sink is None else torch.zeros(s.heads, dtype=torch.float32, device=device)
        self.o = _empty((width, s.heads * s.vdim), dtype, device)
        self.rope = rope(s.rot)

    def named_parameters(self, p):
        at = 0
        for name, n in self.sizes:
            yield p + name, self.inp[at:at + n]
            if self.conv is not None:
                yield f"{p}{name}.conv", self.conv[at:at + n]
            at += n
        yield p + "q.norm", self.q_norm
        if self.k_norm is not None:
            yield p + "k.norm", self.k_norm
        if self.temper is not None:
            yield p + "temp", self.temper
        if self.spec.sink == "learned":
            yield p + "sink", self.sink
        if self.spec.gate is not None:
            yield p + "g", self.inp[at:at + self.spec.gate_columns]
        yield p + "o", self.o

    def finish_loading(self) -> None:
        pass

    def _entry_bytes(self) -> int:
        return self.spec.kv_heads * (self.spec.dim + self.spec.vdim) * self.o.element_size()

    def bytes_per_token(self) -> int:
        return self._entry_bytes() if self.lender is None else 0

    def pool_bytes(self, block_size: int) -> int:
        """Means in a page (a borrower may need its own, of other blocks than its lender's)."""
        return PooledCache.rows(block_size, self.spec.pool) * self._entry_bytes() if self.spec.pool else 0

    def bytes_per_sequence(self) -> int:
        return max(self.spec.conv - 1, 0) * self.channels * self.o.element_size()

    def expansion_bytes(self) -> int:
        return 0

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int, lent=None):
        s, dtype, device = self.spec, self.o.dtype, self.o.device

        def caches(rows):
            return tuple(torch.zeros(num_blocks, s.kv_heads, rows, d, dtype=dtype, device=device) for d in (s.dim, s.vdim))

        k, v, conv_state, pool = (*caches(block_size), None, None) if lent is None else lent
        if s.conv:
            conv_state = torch.zeros(num_slots, s.conv - 1, self.channels, dtype=dtype, device=device)
        if s.pool and pool is not None and pool.size == s.pool:
            pool = PooledCache(s.pool, pool.k, pool.v, own=False)
        else:
            pool = PooledCache(s.pool, *caches(PooledCache.rows(block_size, s.pool))) if s.pool else None
        return k, v, conv_state, pool

    def forward(self, ops, h, memory, batch):
        s, c = self.spec, self.channels
        k_cache, v_cache, conv_state, pool = memory
        proj = ops.linear(h, self.inp)
        qkv, gate = proj[:, :c], proj[:, c:c + s.gate_columns] if s.gate is not None else None
        if self.conv is not None:
            qkv = ops.short_conv(qkv, self.conv, None, conv_state, batch, act="none")
        q = ops.norm_rope_store(qkv, self.q_norm, self.k_norm, self.eps, s, self.rope, batch.positions, batch.slot_mapping, k_cache, v_cache,
                                temper=self.temper)
        out = torch.empty(h.shape[0], self.o.shape[1], dtype=h.dtype, device=h.device)
        ops.windowed_attention(q, k_cache, v_cache, batch, s, out, 1.0, chunked=s.chunked, softcap=s.softcap, sink=self.sink, gate=gate,
                               pool=pool)
        return ops.linear(out, self.o)


class HyperConnection:
    """How a sublayer reads and writes several residual streams: its input is sum_s into[s] x_s; after it
    x_t <- sum_s mix[s, t] x_s + out[t] y."""

    def __init__(self, streams: int, device):
        self.into, self.out = (torch.ones(streams, dtype=torch.float32, device=device) for _ in range(2))
        self.mix = torch.eye(streams, dtype=torch.float32, device=device)

    def named_parameters(self, p):
        yield p + "in", self.into
        yield p + "out", self.out
        yield p + "mix", self.mix
