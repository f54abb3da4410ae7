"""Building blocks of decoders whose layers are listed one by one: mixers and feed-forwards.

A block owns its weights (all sizes and constants come from its spec), names them for the checkpoint loader, says what it
keeps per token (paged cache) or per sequence (recurrent state), and issues its ops.  A model of another design uses the
same blocks with other specs.

    mixer        forward(ops, h, memory, batch) -> [tokens, width]; ``memory`` is what ``new_memory`` returned for this run
    feed-forward forward(ops, h) -> [tokens, width], or the op set's own representation of a sum over experts
"""
from __future__ import annotations

import torch


def _empty(shape, dtype, device):
    return torch.empty(shape, dtype=dtype, device=device)


def _halves_apart(rows: torch.Tensor) -> None:
    """rows [heads, d, width], in place: row 2 i of a head becomes row i, row 2 i + 1 row d / 2 + i."""
    rows.copy_(torch.cat((rows[:, 0::2], rows[:, 1::2]), dim=1))


class LatentAttention:
    """Attention whose keys and values are rebuilt from one low-rank latent per token; a rotated key part is shared by all
    heads.  The queries come from a latent of their own or from the input itself.  Cached per token: the normed latent and the rotated
    part."""
    recurrent = False

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        self.spec, self.eps = spec, eps
        H = spec.heads
        self.q_rows = spec.q_rank or H * (spec.dim + spec.rot_dim)
        rows = self.q_rows + spec.kv_rank + spec.rot_dim
        if spec.q_rank:
            self.a_proj = _empty((rows, width), dtype, device)                                      # dq | dkv
            self.q_norm = _empty(spec.q_rank, dtype, device)
            self.uq = _empty((H * (spec.dim + spec.rot_dim), spec.q_rank), dtype, device)
        else:
            self.a_proj = torch.zeros(-(-rows // 8) * 8, width, dtype=dtype, device=device)         # q | dkv, rows of 16 bytes
            self.q_norm = self.uq = None
        self.kv_norm = _empty(spec.kv_rank, dtype, device)
        self.ukv = _empty((H * (spec.dim + spec.vdim), spec.kv_rank), dtype, device)                # uk | uv
        self.o = _empty((width, H * spec.vdim), dtype, device)
        self.uk_t = None                        # [heads, kv_rank, dim]: see finish_loading
        self.rope = rope(spec.rot)

    def named_parameters(self, p):
        s = self.spec
        if s.q_rank:
            yield p + "dq", self.a_proj[:s.q_rank]
            yield p + "dq.norm", self.q_norm
            yield p + "uq", self.uq
        else:
            yield p + "q", self.a_proj[:self.q_rows]
        yield p + "dkv", self.a_proj[self.q_rows:self.q_rows + s.kv_rank + s.rot_dim]
        yield p + "dkv.norm", self.kv_norm
        yield p + "uk", self.ukv[:s.heads * s.dim]
        yield p + "uv", self.ukv[s.heads * s.dim:]
        yield p + "o", self.o

    def finish_loading(self) -> None:
        """Decode folds the key matrix into the query (q_h . W_h c = (W_h^T q_h) . c): keep each head's matrix transposed too.
        Neighbours that rotate together are moved half a head apart, in queries and keys alike: their products do not change, and the
        kernels know one layout."""
        s = self.spec
        if s.rot.interleaved:
            q = self.a_proj[:self.q_rows] if self.uq is None else self.uq
            _halves_apart(q.view(s.heads, s.dim + s.rot_dim, -1)[:, s.dim:])
            _halves_apart(self.a_proj[None, self.q_rows + s.kv_rank:self.q_rows + s.kv_rank + s.rot_dim])
        self.uk_t = self.ukv[:s.heads * s.dim].view(s.heads, s.dim, s.kv_rank).transpose(1, 2).contiguous()

    @property
    def uv(self):
        s = self.spec
        return self.ukv[s.heads * s.dim:].view(s.heads, s.vdim, s.kv_rank)

    def bytes_per_token(self) -> int:
        return (self.spec.kv_rank + self.spec.rot_dim) * self.o.element_size()

    def bytes_per_sequence(self) -> int:
        return 0

    def expansion_bytes(self) -> int:
        """Workspace per key that a portion of a prompt sees."""
        s = self.spec
        return (s.heads * (s.dim + s.vdim) + s.kv_rank + s.rot_dim) * self.o.element_size()

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int):
        return torch.zeros(num_blocks, block_size, self.spec.kv_rank + self.spec.rot_dim, dtype=self.o.dtype, device=self.o.device)

    def forward(self, ops, h, cache, batch):
        s = self.spec
        proj = ops.linear(h, self.a_proj)
        q = ops.latent_prepare(proj, self.q_rows, s.kv_rank, self.q_norm, self.kv_norm, self.eps, self.rope, batch.positions,
                               batch.slot_mapping, cache)
        q = ops.linear(q, self.uq) if s.q_rank else proj[:, :self.q_rows]
        return ops.linear(ops.latent_attention(q, self, cache, batch, self.rope, s), self.o)


class Retention:
    """Linear attention with a fixed decay per head and no denominator.  Kept per sequence: one fp32 matrix per head."""
    recurrent = True

    def __init__(self, spec, width: int, eps: float, dtype, device, rope):
        self.spec, self.eps = spec, eps
        H = spec.heads
        self.qkvg = _empty((H * (2 * spec.dim + 2 * spec.vdim), width), dtype, device)
        self.o = _empty((width, H * spec.vdim), dtype, device)
        self.decay = torch.tensor(spec.decay, dtype=torch.float32, device=device)
        self.rope = rope(spec.rot)

    def named_parameters(self, p):
        s, at = self.spec, 0
        for name, d in (("q", s.dim), ("k", s.dim), ("v", s.vdim), ("g", s.vdim)):
            yield p + name, self.qkvg[at:at + s.heads * d]
            at += s.heads * d
        yield p + "o", self.o

    def finish_loading(self) -> None:
        pass

    def bytes_per_token(self) -> int:
        return 0

    def expansion_bytes(self) -> int:
        return 0

    def bytes_per_sequence(self) -> int:
        return 4 * self.spec.heads * self.spec.dim * self.spec.vdim

    def new_memory(self, num_blocks: int, block_size: int, num_slots: int):
        s = self.spec
        return torch.zeros(num_slots, s.heads, s.dim, s.vdim, dtype=torch.float32, device=self.o.device)

    def forward(self, ops, h, state, batch):
        y = ops.retention(ops.linear(h, self.qkvg), self.decay, state, batch, self.rope, self.spec, self.eps)
        return ops.linear(y, self.o)


class GatedFeedForward:
    """down(act(gate h) * (up h))"""

    def __init__(self, spec, width: int, dtype, device):
        self.ff, self.act = spec.ff, spec.act
        self.gate_up = _empty((2 * spec.ff, width), dtype, device)
        self.down = _empty((width, spec.ff), dtype, device)

    def named_parameters(self, p):
        yield p + "gate", self.gate_up[:self.ff]
        yield p + "up", self.gate_up[self.ff:]
        yield p + "down", self.down

    def forward(self, ops, h):
        return ops.linear(ops.linear_act_mul(h, self.gate_up, self.act), self.down)


class RoutedFeedForward:
    """Experts chosen per token; how their weights are made and applied is the spec's (see ``MoeSpec``)."""

    def __init__(self, spec, width: int, dtype, device):
        self.spec = spec
        self.router = _empty((spec.experts, width), dtype, device)
        self.correction = torch.zeros(spec.experts, dtype=torch.float32, device=device) if spec.correction else None
        self.up = _empty((spec.experts, (2 if spec.gated else 1) * spec.ff, width), dtype, device)      # gate | up, or up
        self.down = _empty((spec.experts, width, spec.ff), dtype, device)

    def named_parameters(self, p):
        yield p + "router", self.router
        if self.correction is not None:
            yield p + "correction", self.correction
        for e in range(self.spec.experts):
            if self.spec.gated:
                yield f"{p}e{e}.gate", self.up[e, :self.spec.ff]
            yield f"{p}e{e}.up", self.up[e, -self.spec.ff:]
            yield f"{p}e{e}.down", self.down[e]

    def forward(self, ops, h):
        s = self.spec
        return ops.moe(h, self.router, self.up, self.down, s.top, score=s.score, weigh=s.weigh, act=s.act, limit=s.limit, gated=s.gated,
                       correction=self.correction, groups=s.groups, keep=s.keep)
