"""One-kernel cases of hybrid decoders (see ``kernel_case``): windowed attention, short convolution, recurrences with a decay per
token, sandwich norms, attention with its options, several residual streams; sizes of a layer of width 2048.  Bytes and flops are those of the operation, as in ``mixer_cases``: the
recurrences count the token-by-token products of their chunked form (chunks of 64)."""
from __future__ import annotations

import torch

from .mixer_cases import BF, EXPERTS, FF, TOP, WIDTH, Spec, _ints, _rand, _rope

ATTENTION = Spec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, window=1024)
SSD = Spec(heads=32, share=16, dk=128, dv=64)
DELTA = Spec(heads=16, share=2, dk=128, dv=128)


class _Batch:
    def __init__(self, seqs: int, q_len: int, ctx: int, block: int = 256):
        n = -(-ctx // block)
        self.is_prefill, self.num_seqs, self.padded_seqs = q_len > 1, seqs, seqs
        self.num_single = 0 if q_len > 1 else seqs
        self.cu_seqlens_q = _ints([i * q_len for i in range(seqs + 1)])
        self.context_lens = _ints([ctx] * seqs)
        self.block_tables = torch.randperm(seqs * n, dtype=torch.int32).view(seqs, n).cuda()
        self.positions = _ints(list(range(ctx - q_len, ctx)) * seqs)
        self.slot_mapping = _ints(list(range(seqs * q_len)))
        self.state_slots = _ints(list(range(seqs)))
        self.table_width, self.max_seqlen_q, self.num_blocks = n, q_len, seqs * n
        self.max_seqlen_k, self.kv_rows = ctx, seqs * ctx


def _caches(b, s, block=256):
    return _rand(b.num_blocks, s.kv_heads, block, s.dim), _rand(b.num_blocks, s.kv_heads, block, s.vdim)


def _attention(ops, seqs, q_len, ctx, window=None, heads=16, kind=None, pool=0):
    """``kind``: None, "chunked" (chunks, sink, a gate per head) or "capped" (window, sink, bounded scores, a gate per element).  ``pool``:
    blocks of that many tokens behind the window, whose means exist for all but the step's tokens."""
    s = Spec(**{**ATTENTION.__dict__, "heads": heads, "window": window or ATTENTION.window})
    b = _Batch(seqs, q_len, ctx)
    kc, vc = _caches(b, s)
    q, out = _rand(seqs * q_len, s.heads, s.dim), _rand(seqs * q_len, s.heads * s.vdim)
    oldest = (lambda p: p // s.window * s.window) if kind == "chunked" else (lambda p: max(p - s.window + 1, 0))
    keys = sum(p + 1 - oldest(p) for p in range(ctx - q_len, ctx)) * seqs               # (query, key) pairs per head
    cached = seqs * (ctx - oldest(ctx - q_len)) * s.kv_heads * (s.dim + s.vdim) * 2
    options, gates = {}, 0
    if pool:
        from ..models.attention_blocks import PooledCache
        pk, pv = (torch.zeros(b.num_blocks, s.kv_heads, PooledCache.rows(256, pool), c.shape[3], dtype=BF, device="cuda") for c in (kc, vc))
        options = dict(pool=PooledCache(pool, pk, pv))
        keys += sum(oldest(p) // pool for p in range(ctx - q_len, ctx)) * seqs
        cached += seqs * (oldest(ctx - 1) // pool + (q_len // pool if q_len > 1 else 0)) * s.kv_heads * (s.dim + s.vdim) * 2
    if kind is not None:
        gates = {"chunked": s.heads, "capped": s.heads * s.vdim}[kind]
        options = dict(chunked=kind == "chunked", softcap=50.0 if kind == "capped" else 0.0, sink=torch.zeros(s.heads, device="cuda"), gate=_rand(seqs * q_len, gates))
    return (lambda: ops.windowed_attention(q, kc, vc, b, s, out, 0.7, **options), cached + seqs * q_len * (s.heads * (s.dim + s.vdim) + gates) * 2,
            2 * keys * s.heads * (s.dim + s.vdim) if q_len > 1 else 0)


def _bias_rope_store(ops, T):
    s = ATTENTION
    b = _Batch(1, T, T)
    kc, vc = _caches(b, s)
    n = (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim
    proj, bias, table = _rand(T, n), torch.randn(n, device="cuda"), _rope(T, 64)
    return lambda: ops.bias_rope_store(proj, bias, s, table, b.positions, b.slot_mapping, kc, vc), 4 * T * n, 0


def _norm_rope_store(ops, T, whole, rd):
    s = Spec(**{**ATTENTION.__dict__, "norm": "all" if whole else "head"})
    b = _Batch(1, T, T)
    kc, vc = _caches(b, s)
    n = (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim
    proj, table = _rand(T, n), _rope(T, rd)
    qw, kw = (_rand(h * s.dim if whole else s.dim) for h in (s.heads, s.kv_heads))
    return lambda: ops.norm_rope_store(proj, qw, kw, 1e-6, s, table, b.positions, b.slot_mapping, kc, vc), 4 * T * n, 0


def _stream_mix(ops, T, streams):
    x, y, w, W = torch.randn(T, streams, WIDTH, device="cuda"), _rand(T, WIDTH), _rand(WIDTH), WIDTH
    into, mix = torch.ones(streams, device="cuda"), torch.eye(streams, device="cuda")
    return lambda: ops.stream_mix(x, BF, 1e-6, into, w, w, y=y, mix=mix, out=into), (8 * streams + 4) * T * W, 0


def _stream_start(ops, T, streams):
    x, embed, pairs, w, W = torch.empty(T, streams, WIDTH, device="cuda"), _rand(32000, WIDTH), _rand(8192, WIDTH), _rand(WIDTH), WIDTH
    ids, prev = (torch.randint(0, 32000, (T,), dtype=torch.int32, device="cuda") for _ in range(2))
    into = torch.ones(streams, device="cuda")
    return (lambda: ops.stream_mix(x, BF, 1e-6, into, w, w, ids=ids, prev=prev, embed=embed, scale=45.0, pairs=pairs, mul_prev=31, mul_cur=7),
            (4 * streams + 6) * T * W, 0)


def _operands(s, T):
    n = s.heads // s.share * s.dk
    x, raw = torch.nn.functional.silu(_rand(T, 2 * n + s.heads * s.dv)), _rand(T, 2 * s.heads)
    block = Spec(A_log=torch.full((s.heads,), -3.0, device="cuda"), dt_bias=torch.zeros(s.heads, device="cuda"), D=torch.ones(s.heads, device="cuda"))
    return x[:, :n], x[:, n:2 * n], x[:, 2 * n:], raw[:, s.heads:], raw[:, :s.heads], block, n


def _recurrence(ops, s, delta, seqs, q_len):
    T, C = seqs * q_len, 64
    q, k, v, dt, beta, block, n = _operands(s, T)
    state = torch.zeros(seqs, s.heads, s.dk, s.dv, device="cuda")
    b = _Batch(seqs, q_len, q_len if q_len > 1 else 700)
    moved = T * ((2 * n + s.heads * s.dv) * 2 + s.heads * s.dv * 4)
    if q_len == 1:
        return lambda: ops.recur(q, k, v, dt, beta if delta else None, block, state, b), seqs * s.heads * s.dk * s.dv * 8 + moved, 0
    per = 4 * s.dk * s.dv + C * (s.dk + s.dv)                 # state read and update, scores and their sum over half a chunk
    if delta:
        per += 2 * s.dk * s.dv + C * (s.dk + s.dv)            # the same for what the writes see of the state and of each other
    return lambda: ops.recur(q, k, v, dt, beta if delta else None, block, state, b), moved, T * s.heads * per


def _short_conv(ops, seqs, q_len, C=4096, act="silu"):
    T = seqs * q_len
    b = _Batch(seqs, q_len, q_len if q_len > 1 else 700)
    x, taps, state = _rand(T, C), torch.randn(C, 4, device="cuda"), _rand(seqs, 3, C)
    return lambda: ops.short_conv(x, taps, None, state, b, act=act), (4 * T * C if q_len > 1 else seqs * C * (4 + 12)), 0


def _gated_norm(ops, T, groups, first):
    W = 2048
    o, z, w, out = torch.randn(T, W, device="cuda"), _rand(T, W), torch.ones(W // groups, device="cuda"), _rand(T, W)
    return lambda: ops.C.gated_norm(o, z, w, out, groups, first, 1.0, 1e-6), 8 * T * W, 0


def _sandwich(ops, T, routed):
    from ..ops.cuda_mixers import Routed
    x, w, W = torch.randn(T, WIDTH, device="cuda"), _rand(WIDTH), WIDTH
    if not routed:
        y = _rand(T, W)
        return lambda: ops.stream_update(x, BF, 1e-6, [w], a=y, post=w, mult=0.5, offset=1.0), 12 * T * W, 0
    y = Routed(_rand(T * TOP, W), torch.randperm(T * TOP, dtype=torch.int32).view(T, TOP).cuda(), torch.rand(T, TOP, device="cuda"))
    return lambda: ops.stream_update(x, BF, 1e-6, [w], a=y, post=w, mult=0.5, offset=1.0), (10 + 2 * TOP) * T * W, 0


def _pool_blocks(ops, seqs, q_len, pool):
    from ..models.attention_blocks import PooledCache
    s, b = ATTENTION, _Batch(seqs, q_len, q_len)
    kc, vc = _caches(b, s)
    pk, pv = (torch.zeros(b.num_blocks, s.kv_heads, PooledCache.rows(256, pool), c.shape[3], dtype=BF, device="cuda") for c in (kc, vc))
    p, n = PooledCache(pool, pk, pv), s.kv_heads * (s.dim + s.vdim) * 2
    return (lambda: ops.pool_blocks(kc, vc, p, b, 0, b.cu_seqlens_q, b.context_lens, b.block_tables, s.window),
            seqs * (q_len * n + q_len // pool * 2 * n), 0)


def _grouped(ops, T, routed):
    from ..ops.cuda_mixers import Routed
    x, w, W, top = torch.randn(T, WIDTH, device="cuda"), _rand(WIDTH), WIDTH, 8
    y = Routed(_rand(T * top, W), torch.randperm(T * top, dtype=torch.int32).view(T, top).cuda(), torch.rand(T, top, device="cuda")) if routed else _rand(T, W)
    return lambda: ops.stream_update(x, BF, 1e-6, [None], a=y, post=w, groups=4), (10 + 2 * (top if routed else 1)) * T * W, 0


def _gelu_product(ops, M):
    ws = [_rand(6 * WIDTH, WIDTH, scale=0.02) for _ in range(3)]
    x, state = _rand(M, WIDTH), {"i": 0}

    def run():
        state["i"] += 1
        return ops.linear_act_mul(x, ws[state["i"] % 3], "gelu_tanh")
    return run, (6 * WIDTH * WIDTH + M * 4 * WIDTH) * 2, 2 * M * 6 * WIDTH * WIDTH


def _experts(ops, T):
    h, router = _rand(T, WIDTH), _rand(EXPERTS, WIDTH, scale=0.02)
    gu, down = _rand(EXPERTS, 2 * FF, WIDTH, scale=0.02), _rand(EXPERTS, WIDTH, FF, scale=0.02)
    return (lambda: ops.moe(h, router, gu, down, TOP, score="softmax", weigh="output", act="clamped_swish", limit=7.0),
            EXPERTS * 3 * FF * WIDTH * 2, 6 * T * TOP * WIDTH * FF)


CASES = {
    "windowed_decode": lambda ops: _attention(ops, 64, 1, 2048),
    "windowed_decode_b256": lambda ops: _attention(ops, 256, 1, 1500),
    "windowed_decode_b8": lambda ops: _attention(ops, 8, 1, 16384, 8192),
    "windowed_decode_g8": lambda ops: _attention(ops, 64, 1, 2048, heads=32),
    "windowed_prefill": lambda ops: _attention(ops, 8, 2048, 2048),
    "windowed_prefill_long": lambda ops: _attention(ops, 1, 8192, 8192),
    "windowed_prefill_full": lambda ops: _attention(ops, 8, 2048, 2048, 2048),
    "chunked_decode": lambda ops: _attention(ops, 64, 1, 2048, 4096, kind="chunked"),
    "chunked_decode_b8": lambda ops: _attention(ops, 8, 1, 16384, 16384, kind="chunked"),
    "capped_decode": lambda ops: _attention(ops, 64, 1, 2048, kind="capped"),
    "capped_decode_b256": lambda ops: _attention(ops, 256, 1, 1500, kind="capped"),
    "chunked_prefill": lambda ops: _attention(ops, 8, 2048, 2048, 4096, kind="chunked"),
    "chunked_prefill_long": lambda ops: _attention(ops, 1, 8192, 8192, 4096, kind="chunked"),
    "capped_prefill": lambda ops: _attention(ops, 8, 2048, 2048, kind="capped"),
    "capped_prefill_long": lambda ops: _attention(ops, 1, 8192, 8192, kind="capped"),
    "pooled_decode": lambda ops: _attention(ops, 64, 1, 4096, pool=16),
    "pooled_decode_b256": lambda ops: _attention(ops, 256, 1, 3000, pool=16),
    "pooled_decode_b8": lambda ops: _attention(ops, 8, 1, 32768, pool=8),
    "pooled_prefill": lambda ops: _attention(ops, 8, 2048, 2048, pool=16),
    "pooled_prefill_long": lambda ops: _attention(ops, 1, 8192, 8192, pool=16),
    "pool_blocks": lambda ops: _pool_blocks(ops, 8, 16384, 16),
    "grouped_norm": lambda ops: _grouped(ops, 16384, False),
    "grouped_norm_routed": lambda ops: _grouped(ops, 16384, True),
    "norm_rope_heads": lambda ops: _norm_rope_store(ops, 16384, False, 128),
    "norm_rope_whole": lambda ops: _norm_rope_store(ops, 16384, True, 64),
    "stream_mix2": lambda ops: _stream_mix(ops, 16384, 2),
    "stream_mix4": lambda ops: _stream_mix(ops, 16384, 4),
    "stream_start2": lambda ops: _stream_start(ops, 16384, 2),
    "short_conv_plain": lambda ops: _short_conv(ops, 8, 2048, 3072, "none"),
    "bias_rope_store": lambda ops: _bias_rope_store(ops, 16384),
    "state_space_prefill": lambda ops: _recurrence(ops, SSD, False, 8, 2048),
    "state_space_prefill_long": lambda ops: _recurrence(ops, SSD, False, 1, 16384),
    "state_space_decode": lambda ops: _recurrence(ops, SSD, False, 128, 1),
    "delta_prefill": lambda ops: _recurrence(ops, DELTA, True, 8, 2048),
    "delta_prefill_long": lambda ops: _recurrence(ops, DELTA, True, 1, 16384),
    "delta_decode": lambda ops: _recurrence(ops, DELTA, True, 128, 1),
    "short_conv": lambda ops: _short_conv(ops, 8, 2048),
    "short_conv_decode": lambda ops: _short_conv(ops, 256, 1),
    "gated_norm_heads": lambda ops: _gated_norm(ops, 16384, 16, False),
    "gated_norm_groups": lambda ops: _gated_norm(ops, 16384, 2, True),
    "sandwich_norm": lambda ops: _sandwich(ops, 16384, False),
    "sandwich_norm_routed": lambda ops: _sandwich(ops, 16384, True),
    "gelu_product": lambda ops: _gelu_product(ops, 8192),
    "gelu_product_decode": lambda ops: _gelu_product(ops, 64),
    "clamped_experts": lambda ops: _experts(ops, 8192),
    "clamped_experts_decode": lambda ops: _experts(ops, 64),
}
