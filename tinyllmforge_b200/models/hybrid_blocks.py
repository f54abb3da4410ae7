"""Building blocks of hybrid decoders: windowed attention, a state-space mixer, both side by side, and the gated delta rule.

Same interface as ``blocks.py``.  A block packs the projections that read the same input into one matrix (its rows padded to
a multiple of 8, so that every kernel finds 16-byte rows); what follows a projection reads its columns in place.
``out_bias`` (fp32 or None) belongs to the block's result and is added by the op that takes it up.
"""
from __future__ import annotations

import torch

from .blocks import _empty


def _packed(rows: int, width: int, dtype, device):
    """A projection of ``rows`` outputs; the padding rows are zero."""
    return torch.zeros(-(-rows // 8) * 8, width, dtype=dtype, device=device)


def _f32(shape, device):
    return torch.empty(shape, dtype=torch.float32, device=device)


class WindowedAttention:
    """Grouped-query attention over the last ``window`` tokens, with biases.  Cached per token: rotated keys, and values."""

    def __init__(self, spec, device, rope):
        s = self.spec = spec
        self.sizes = (s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim)
        self.rows, self.columns = sum(self.sizes), s.heads * s.vdim
        self.bias = _f32(self.rows, device)
        self.rope = rope(spec.rot)

    def named_parameters(self, p, proj):
        at = 0
        for name, n in zip("qkv", self.sizes):
            yield p + name, proj[at:at + n]
            yield p + name + ".b", self.bias[at:at + n]
            at += n

    def bytes_per_token(self, element: int) -> int:
        return self.spec.kv_heads * (self.spec.dim + self.spec.vdim) * element

    def new_memory(self, num_blocks, block_size, dtype, device):
        s = self.spec
        return tuple(torch.zeros(num_blocks, s.kv_heads, block_size, d, dtype=dtype, device=device) for d in (s.dim, s.vdim))

    def forward(self, ops, proj, memory, batch, out, scale) -> None:
        """proj [tokens, rows] = q | k | v without biases; out (a view) <- scale * the heads' outputs."""
        s = self.spec
        k_cache, v_cache = memory
        q = ops.bias_rope_store(proj, self.bias, s, self.rope, batch.positions, batch.slot_mapping, k_cache, v_cache)
        ops.windowed_attention(q, k_cache, v_cache, batch, s, out, scale)


class StateSpace:
    """A linear recurrence with one decay per head and token, behind a short convolution, with a gated and grouped norm.
    Kept per sequence: one fp32 matrix per head and the convolution's last inputs."""

    def __init__(self, spec, eps, device):
        s = self.spec = spec
        self.eps = eps
        self.rows, self.columns = s.inner + s.channels + s.heads, s.inner
        self.conv, self.conv_bias = _f32((s.channels, s.conv), device), _f32(s.channels, device)
        self.dt_bias, self.A_log, self.D = (_f32(s.heads, device) for _ in range(3))
        self.norm = _f32(s.inner, device)

    def named_parameters(self, p, proj):
        yield p + "in", proj
        yield p + "conv", self.conv
        yield p + "conv.b", self.conv_bias
        for name in ("dt_bias", "A_log", "D", "norm"):
            yield p + name, getattr(self, name)

    def bytes_per_sequence(self, element: int) -> int:
        s = self.spec
        return 4 * s.heads * s.state * s.vdim + (s.conv - 1) * s.channels * element

    def new_memory(self, num_slots, dtype, device):
        s = self.spec
        return (torch.zeros(num_slots, s.conv - 1, s.channels, dtype=dtype, device=device),
                torch.zeros(num_slots, s.heads, s.state, s.vdim, dtype=torch.float32, device=device))

    def forward(self, ops, proj, memory, batch, out, scale) -> None:
        """proj [tokens, rows] = z | x | B | C | dt; out (a view) <- scale * the gated and normed outputs."""
        s = self.spec
        conv_state, state = memory
        xbc = ops.short_conv(proj[:, s.inner:s.inner + s.channels], self.conv, self.conv_bias, conv_state, batch)
        ops.state_space(xbc, proj[:, :s.inner], proj[:, s.inner + s.channels:self.rows], self, state, batch, out, scale)


class ParallelMixer:
    """Windowed attention and a state-space mixer on the same input; the result is the sum of both, each with a factor.  One
    projection feeds both; their outputs, factors applied, lie side by side and go through one output matrix."""

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        self.spec = spec
        self.left, self.right = WindowedAttention(spec.left, device, rope), StateSpace(spec.right, eps, device)
        self.inp = _packed(self.left.rows + self.right.rows, width, dtype, device)
        self.o = _empty((width, self.left.columns + self.right.columns), dtype, device)
        self.o_bias = _f32(width, device)
        self.out_bias = None

    def named_parameters(self, p):
        n, c = self.left.rows, self.left.columns
        yield from self.left.named_parameters(p + "left.", self.inp[:n])
        yield p + "left.o", self.o[:, :c]
        yield p + "left.o.b", self.o_bias
        yield from self.right.named_parameters(p + "right.", self.inp[n:n + self.right.rows])
        yield p + "right.o", self.o[:, c:]

    def finish_loading(self) -> None:
        self.out_bias = self.spec.left_scale * self.o_bias

    def bytes_per_token(self) -> int:
        return self.left.bytes_per_token(self.o.element_size())

    def bytes_per_sequence(self) -> int:
        return self.right.bytes_per_sequence(self.o.element_size())

    def expansion_bytes(self) -> int:
        return 0

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int):
        dtype, device = self.o.dtype, self.o.device
        return self.left.new_memory(num_blocks, block_size, dtype, device), self.right.new_memory(num_slots, dtype, device)

    def forward(self, ops, h, memory, batch):
        n, c = self.left.rows, self.left.columns
        proj = ops.linear(h, self.inp)
        both = torch.empty(h.shape[0], self.o.shape[1], dtype=h.dtype, device=h.device)
        self.left.forward(ops, proj[:, :n], memory[0], batch, both[:, :c], self.spec.left_scale)
        self.right.forward(ops, proj[:, n:n + self.right.rows], memory[1], batch, both[:, c:], self.spec.right_scale)
        return ops.linear(both, self.o)


class GatedDelta:
    """The delta rule with one decay and one write strength per head and token, behind short convolutions.  Kept per sequence:
    one fp32 matrix per head and the convolutions' last inputs."""
    out_bias = None

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        s = self.spec = spec
        self.eps = eps
        self.sizes = (("q", s.kv_heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.heads * s.vdim), ("g", s.heads * s.vdim), ("b", s.heads), ("a", s.heads))
        self.rows = sum(n for _, n in self.sizes)
        self.inp = _packed(self.rows, width, dtype, device)
        self.conv = _f32((s.channels, s.conv), device)
        self.A_log, self.dt_bias, self.norm = _f32(s.heads, device), _f32(s.heads, device), _f32(s.vdim, device)
        self.o = _empty((width, s.heads * s.vdim), dtype, device)

    def named_parameters(self, p):
        at = 0
        for name, n in self.sizes:
            yield p + name, self.inp[at:at + n]
            if name in "qkv":
                yield f"{p}{name}.conv", self.conv[at:at + n]
            at += n
        for name in ("A_log", "dt_bias", "norm", "o"):
            yield p + name, getattr(self, name)

    def finish_loading(self) -> None:
        pass

    def bytes_per_token(self) -> int:
        return 0

    def bytes_per_sequence(self) -> int:
        s = self.spec
        return 4 * s.heads * s.dim * s.vdim + (s.conv - 1) * s.channels * self.o.element_size()

    def expansion_bytes(self) -> int:
        return 0

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int):
        s, device = self.spec, self.o.device
        return (torch.zeros(num_slots, s.conv - 1, s.channels, dtype=self.o.dtype, device=device),
                torch.zeros(num_slots, s.heads, s.dim, s.vdim, dtype=torch.float32, device=device))

    def forward(self, ops, h, memory, batch):
        s = self.spec
        conv_state, state = memory
        proj = ops.linear(h, self.inp)
        qkv = ops.short_conv(proj[:, :s.channels], self.conv, None, conv_state, batch)
        at = s.channels + s.heads * s.vdim
        y = ops.gated_delta(qkv, proj[:, s.channels:at], proj[:, at:at + 2 * s.heads], self, state, batch)
        return ops.linear(y, self.o)
