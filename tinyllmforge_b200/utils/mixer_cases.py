"""One-kernel cases of the mixers and the expert layers (see ``kernel_case``): sizes of a layer of width 2048.

Every entry returns (callable, bytes, flops): what the operation has to move and to multiply, whatever the kernel does on top
(hi + lo halves, padding, re-reads), so that the fraction printed is of the operation's own roofline.
"""
from __future__ import annotations

import torch

BF = torch.bfloat16


class Spec:
    def __init__(self, **kw):
        self.__dict__.update(kw)


LATENT = Spec(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512, scale=192 ** -0.5, window=0)
RETENTION = Spec(heads=8, dim=128, vdim=256)
WIDTH, EXPERTS, TOP, FF = 2048, 32, 4, 1536


def _rand(*shape, scale=1.0):
    return torch.randn(*shape, device="cuda", dtype=BF) * scale


def _rope(n, d):
    from ..ops.ref import rope_table
    return rope_table(n, d, 1e6, "cuda", torch.float64)


def _ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _latent_decode(ops, heads, B=64, ctx=2048, window=0):
    R, r, bs = LATENT.kv_rank, LATENT.rot_dim, 256
    cache = _rand(B * ctx // bs, bs, R + r)
    bt = torch.randperm(B * ctx // bs, dtype=torch.int32).view(B, -1).cuda()
    lens = _ints([ctx] * B)
    qa, o = _rand(B, heads, R + r), _rand(B, heads, R)
    scratch = torch.empty(ops.C.latent_decode_scratch(heads, R, ops.num_sms), device="cuda")
    keys = min(ctx, window or ctx)
    return (lambda: ops.C.latent_decode(qa, cache, bt, lens, o, scratch, ops.num_sms, window, LATENT.scale, ops.status),
            B * keys * (R + r) * 2 + B * heads * (2 * R + r) * 2, 2 * B * heads * keys * (2 * R + r))


def _latent_prefill(ops, S, n, window=0):
    s = LATENT
    T = S * n
    qp, kv, kr = _rand(T, s.heads, 192), _rand(T, s.heads * (s.dim + s.vdim)), _rand(T, s.rot_dim)
    cu = _ints([i * n for i in range(S + 1)])
    out = _rand(T, s.heads * s.vdim)
    seen = sum(min(i + 1, window or n) for i in range(n))
    return (lambda: ops.C.latent_prefill(qp, kv, kr, cu, cu, out, 0, S, n, s.dim, s.vdim, window, s.scale, ops.status),
            T * s.heads * (192 + s.dim + 2 * s.vdim) * 2, 2 * S * s.heads * seen * (s.dim + s.rot_dim + s.vdim))


def _retention_prefill(ops, S, n):
    s = RETENTION
    T, C = S * n, 64
    x = _rand(T, s.heads * 2 * (s.dim + s.vdim))
    state = torch.zeros(S, s.heads, s.dim, s.vdim, device="cuda")
    decay = torch.linspace(0.9, 0.9999, s.heads, device="cuda")
    cu, slots, pos = _ints([i * n for i in range(S + 1)]), _ints(list(range(S))), _ints(list(range(n)) * S)
    o = torch.empty(T, s.heads * s.vdim, device="cuda")
    segs, seg_len = ops.retention_segments(S, s.heads, s.dim, s.vdim, n)
    ws = torch.empty(S * segs * s.heads * s.dim * s.vdim, device="cuda")
    table = _rope(n, 128)
    flops = T * s.heads * (4 * s.dim * s.vdim + C * (s.dim + s.vdim))
    return (lambda: ops.C.retention_chunk(x, decay, state, slots, pos, table, cu, S, 0, o, ws, segs, seg_len, ops.status),
            T * s.heads * ((2 * s.dim + s.vdim) * 2 + s.vdim * 4), flops)


def _retention_decode(ops, B):
    s = RETENTION
    x = _rand(B, s.heads * 2 * (s.dim + s.vdim))
    state = torch.zeros(B, s.heads, s.dim, s.vdim, device="cuda")
    decay = torch.linspace(0.9, 0.9999, s.heads, device="cuda")
    slots, pos, y, table = _ints(list(range(B))), _ints([700] * B), _rand(B, s.heads * s.vdim), _rope(1024, 128)
    return (lambda: ops.C.retention_decode(x, decay, state, slots, pos, table, B, y, 1e-6, ops.status),
            B * s.heads * s.dim * s.vdim * 8 + B * x.shape[1] * 2, 0)


def _ungated(ops, T, part):
    """Eight of 32 experts without gates, chosen within four of eight groups."""
    E, top, ff = 32, 8, 9 * WIDTH // 16
    h, router, corr = _rand(T, WIDTH), _rand(E, WIDTH, scale=0.02), torch.zeros(E, device="cuda")
    experts, weights = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    choose = lambda: ops.C.router(h, router, experts, weights, False, corr, 8, 4)
    if part == "router":
        return choose, T * WIDTH * 2, 2 * T * WIDTH * E
    choose()
    n = T * top
    tile = ops.expert_tile(n, E)
    tiles = min(n, n // tile + E)
    rows = torch.empty(T, top, dtype=torch.int32, device="cuda")
    te, nt = torch.empty(tiles, dtype=torch.int32, device="cuda"), torch.empty(1, dtype=torch.int32, device="cuda")
    ops.C.moe_plan(experts, E, tile, rows, te, nt)
    used = int((torch.bincount(experts.view(-1).long(), minlength=E) > 0).sum())
    xs, g, y = _rand(tiles * tile, WIDTH), _rand(tiles * tile, ff), _rand(tiles * tile, WIDTH)
    up, down = _rand(E, ff, WIDTH, scale=0.02), _rand(E, WIDTH, ff, scale=0.02)
    moved, flops = (used * ff * WIDTH + n * (WIDTH + ff)) * 2, 2 * n * WIDTH * ff
    if part == "up":
        return lambda: ops.C.grouped_gemm(xs, up, g, False, tile, te, nt, 1, 0.0, ops.status), moved, flops
    return lambda: ops.C.grouped_gemm(g, down, y, False, tile, te, nt, 0, 0.0, ops.status), moved, flops


def _experts(ops, T, part):
    h, router = _rand(T, WIDTH), _rand(EXPERTS, WIDTH, scale=0.02)
    experts = torch.empty(T, TOP, dtype=torch.int32, device="cuda")
    weights = torch.empty(T, TOP, device="cuda")
    if part == "router":
        return lambda: ops.C.router(h, router, experts, weights, False, None, 1, 1), T * WIDTH * 2, 2 * T * WIDTH * EXPERTS
    ops.C.router(h, router, experts, weights, False, None, 1, 1)
    n = T * TOP
    tile = ops.expert_tile(n, EXPERTS)
    tiles = min(n, n // tile + EXPERTS)
    rows = torch.empty(T, TOP, dtype=torch.int32, device="cuda")
    te, nt = torch.empty(tiles, dtype=torch.int32, device="cuda"), torch.empty(1, dtype=torch.int32, device="cuda")
    if part == "plan":
        return lambda: ops.C.moe_plan(experts, EXPERTS, tile, rows, te, nt), 3 * n * 4, 0
    ops.C.moe_plan(experts, EXPERTS, tile, rows, te, nt)
    xs = torch.zeros(tiles * tile, WIDTH, device="cuda", dtype=BF)
    if part == "scatter":
        return lambda: ops.C.moe_scatter(h, rows, weights, xs), (T + n) * WIDTH * 2, 0
    used = int((torch.bincount(experts.view(-1).long(), minlength=EXPERTS) > 0).sum())
    if part == "gate_up":
        w, out = _rand(EXPERTS, 2 * FF, WIDTH, scale=0.02), _rand(tiles * tile, FF)
        return (lambda: ops.C.grouped_gemm(xs, w, out, True, tile, te, nt, 0, 0.0, ops.status),
                (used * 2 * FF * WIDTH + n * (WIDTH + FF)) * 2, 4 * n * WIDTH * FF)
    g, w, out = _rand(tiles * tile, FF), _rand(EXPERTS, WIDTH, FF, scale=0.02), _rand(tiles * tile, WIDTH)
    return (lambda: ops.C.grouped_gemm(g, w, out, False, tile, te, nt, 0, 0.0, ops.status), (used * FF * WIDTH + n * (WIDTH + FF)) * 2, 2 * n * WIDTH * FF)


def _stream(ops, T, W=WIDTH):
    x = torch.randn(T, W, device="cuda")
    a, b, w = _rand(T, W), _rand(T, W), _rand(W)
    return lambda: ops.stream_update(x, BF, 1e-6, [w, w], a=a, b=b), 16 * T * W, 0


def _latent_small(ops, which, T):
    s = LATENT
    D = s.q_rank + s.kv_rank + s.rot_dim
    pos = _ints(list(range(T)))
    table = _rope(T, s.rot_dim)
    cache = _rand(-(-T // 256), 256, s.kv_rank + s.rot_dim)
    if which == "prepare_direct":                     # queries come from the input itself
        cols = s.heads * (s.dim + s.rot_dim)
        proj, kw = _rand(T, cols + s.kv_rank + s.rot_dim), _rand(s.kv_rank)
        return (lambda: ops.C.latent_prepare(proj, cols, s.kv_rank, None, kw, 1e-6, table, pos, pos, None, cache, ops.status)), 4 * T * (s.kv_rank + s.rot_dim), 0
    if which == "prepare":
        proj, qw, kw, cq = _rand(T, D), _rand(s.q_rank), _rand(s.kv_rank), _rand(T, s.q_rank)
        return (lambda: ops.C.latent_prepare(proj, s.q_rank, s.kv_rank, qw, kw, 1e-6, table, pos, pos, cq, cache, ops.status)), 4 * T * D, 0
    if which == "pack_q":
        q, qp = _rand(T, s.heads * 192), _rand(T, s.heads, 192)
        return (lambda: ops.C.latent_pack_q(q, qp, s.heads, s.dim, table, pos)), 4 * T * s.heads * 192, 0
    cu, bt, lens = _ints([0, T]), _ints([list(range(-(-T // 256)))]), _ints([T])
    c, kr = _rand(T, s.kv_rank), _rand(T, s.rot_dim)
    return (lambda: ops.C.latent_gather(cache, cu, lens, 1, bt, c, kr, ops.status)), 4 * T * (s.kv_rank + s.rot_dim), 0


def _retention_small(ops, T):
    s = RETENTION
    x, y = _rand(T, s.heads * 2 * (s.dim + s.vdim)), _rand(T, s.heads * s.vdim)
    o = torch.randn(T, s.heads * s.vdim, device="cuda")
    return lambda: ops.C.retention_gate(o, x, y, 0, s.heads, s.vdim, 1e-6), T * s.heads * s.vdim * 8, 0


CASES = {
    "latent_decode": lambda ops: _latent_decode(ops, 16),
    "latent_decode_h32": lambda ops: _latent_decode(ops, 32),
    "latent_decode_b8": lambda ops: _latent_decode(ops, 16, 8, 16384),
    "latent_prefill": lambda ops: _latent_prefill(ops, 8, 2048),
    "latent_prefill_long": lambda ops: _latent_prefill(ops, 1, 8192),
    "latent_decode_b8_short": lambda ops: _latent_decode(ops, 16, 8, 4096),
    "latent_decode_window": lambda ops: _latent_decode(ops, 16, 64, 4096, 2048),
    "latent_decode_window_b8": lambda ops: _latent_decode(ops, 16, 8, 16384, 4096),
    "latent_prefill_window": lambda ops: _latent_prefill(ops, 1, 8192, 4096),
    "latent_prefill_window_short": lambda ops: _latent_prefill(ops, 8, 2048, 512),
    "latent_prepare_direct": lambda ops: _latent_small(ops, "prepare_direct", 65536),
    "latent_prepare": lambda ops: _latent_small(ops, "prepare", 65536),
    "latent_pack_q": lambda ops: _latent_small(ops, "pack_q", 16384),
    "latent_gather": lambda ops: _latent_small(ops, "gather", 131072),
    "retention_prefill": lambda ops: _retention_prefill(ops, 8, 2048),
    "retention_prefill_long": lambda ops: _retention_prefill(ops, 1, 16384),
    "retention_decode": lambda ops: _retention_decode(ops, 128),
    "retention_gate": lambda ops: _retention_small(ops, 16384),
    "router": lambda ops: _experts(ops, 32768, "router"),
    "router_decode": lambda ops: _experts(ops, 64, "router"),
    "moe_plan": lambda ops: _experts(ops, 8192, "plan"),
    "moe_scatter": lambda ops: _experts(ops, 16384, "scatter"),
    "expert_gate_up": lambda ops: _experts(ops, 8192, "gate_up"),
    "expert_down": lambda ops: _experts(ops, 8192, "down"),
    "expert_gate_up_decode": lambda ops: _experts(ops, 64, "gate_up"),
    "expert_down_decode": lambda ops: _experts(ops, 64, "down"),
    "grouped_router": lambda ops: _ungated(ops, 32768, "router"),
    "ungated_up": lambda ops: _ungated(ops, 8192, "up"),
    "ungated_down": lambda ops: _ungated(ops, 8192, "down"),
    "ungated_up_decode": lambda ops: _ungated(ops, 64, "up"),
    "ungated_down_decode": lambda ops: _ungated(ops, 64, "down"),
    "stream_update": lambda ops: _stream(ops, 16384),
}
