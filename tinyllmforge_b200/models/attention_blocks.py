"""Building blocks of decoders over several residual streams: normed and gated attention, and what joins and splits the streams.

Same interface as ``blocks.py``; projections that read the same input are one matrix, as in ``hybrid_blocks.py``.
"""
from __future__ import annotations

import torch

from .blocks import _empty
from .hybrid_blocks import _f32, _packed


class NormedAttention:
    """Grouped-query attention whose queries and keys are normed ahead of their rotation, with the options of ``AttentionSpec``: short
    convolutions, chunks or a sliding window, sinks, capped scores, gated output.  Cached per token: rotated keys, and values; kept
    per sequence: the convolutions' last inputs."""

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        s = self.spec = spec
        self.eps = eps
        self.sizes = (("q", s.heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim))
        self.channels = sum(n for _, n in self.sizes)
        self.inp = _packed(self.channels + s.gate_columns, width, dtype, device)
        self.conv = _f32((self.channels, s.conv), device) if s.conv else None
        self.q_norm, self.k_norm = (torch.ones(s.dim if s.norm == "head" else n, dtype=dtype, device=device) for _, n in self.sizes[:2])
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
        yield p + "k.norm", self.k_norm
        if self.spec.sink == "learned":
            yield p + "sink", self.sink
        if self.spec.gate is not None:
            yield p + "g", self.inp[at:at + self.spec.gate_columns]
        yield p + "o", self.o

    def finish_loading(self) -> None:
        pass

    def bytes_per_token(self) -> int:
        return self.spec.kv_heads * (self.spec.dim + self.spec.vdim) * self.o.element_size()

    def bytes_per_sequence(self) -> int:
        return max(self.spec.conv - 1, 0) * self.channels * self.o.element_size()

    def expansion_bytes(self) -> int:
        return 0

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int):
        s, dtype, device = self.spec, self.o.dtype, self.o.device
        caches = tuple(torch.zeros(num_blocks, s.kv_heads, block_size, d, dtype=dtype, device=device) for d in (s.dim, s.vdim))
        return caches + (torch.zeros(num_slots, s.conv - 1, self.channels, dtype=dtype, device=device) if s.conv else None,)

    def forward(self, ops, h, memory, batch):
        s, c = self.spec, self.channels
        k_cache, v_cache, conv_state = memory
        proj = ops.linear(h, self.inp)
        qkv, gate = proj[:, :c], proj[:, c:c + s.gate_columns] if s.gate is not None else None
        if self.conv is not None:
            qkv = ops.short_conv(qkv, self.conv, None, conv_state, batch, act="none")
        q = ops.norm_rope_store(qkv, self.q_norm, self.k_norm, self.eps, s, self.rope, batch.positions, batch.slot_mapping, k_cache, v_cache)
        out = torch.empty(h.shape[0], self.o.shape[1], dtype=h.dtype, device=h.device)
        ops.windowed_attention(q, k_cache, v_cache, batch, s, out, 1.0, chunked=s.chunked, softcap=s.softcap, sink=self.sink, gate=gate)
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
