"""Galupel on the CUDA op set: every kernel against the plain oracle's mechanism, and whole models (fp32 and bf16) against the oracle with
prompts, portions, mixed batches, reused pages, long decoding, and generation with CUDA graphs."""
import numpy as np
import pytest
import torch

import galupel_cases as lc
import goselix_cases as gc
import oracle_galupel as oracle
from kernel_helpers import Batch, Spec, close, rnd
from tinyllmforge_b200.models.attention_blocks import PooledCache
from tinyllmforge_b200.ops.ref_hybrid import pool_place

pytestmark = pytest.mark.gpu

F32, BF = torch.float32, torch.bfloat16


@pytest.fixture(scope="module")
def ops():
    from tinyllmforge_b200.ops.cuda import CudaOps
    return CudaOps()


# ------------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("W,groups", [(64, 4), (50, 5), (50, 1), (2048, 4), (2040, 3), (4096, 1), (4096, 32), (6144, 6), (96, 12), (1030, 2), (8192, 8)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_grouped_stream(ops, W, groups, dtype):
    from tinyllmforge_b200.ops.cuda_mixers import Routed
    T, top = 9, 3
    x, y = rnd(T, W, seed=1), rnd(T, W, seed=2, dtype=dtype)
    y[:, :W // groups] *= 30                            # one group far larger than the others
    post, w = (1 + 0.3 * rnd(W, seed=3)).to(dtype), (1 + 0.3 * rnd(W, seed=4)).to(dtype)
    tol = 2e-5 if dtype == F32 else 6e-3
    want = x.double() + oracle.grouped_rms(y.double(), post.double(), groups, 1e-3)
    xc = x.cuda()
    rows = torch.tensor([7, 0, 7], dtype=torch.int32, device="cuda")
    only = ops.stream_update(xc, dtype, 1e-3, [w.cuda()], a=y.cuda(), post=post.cuda(), groups=groups, rows=rows)[0]
    assert torch.equal(xc.cpu(), x)                     # x is left alone when rows are picked
    close(only, oracle.grouped_rms(want, w.double(), groups, 1e-3)[[7, 0, 7]], tol)
    h = ops.stream_update(xc, dtype, 1e-3, [None], a=y.cuda(), post=post.cuda(), groups=groups)[0]
    close(xc, want, 3e-6)
    assert torch.equal(h, xc.to(dtype))
    # a weighted sum over a buffer of rows, nothing emitted
    buf, pick, by = rnd(40, W, seed=5, dtype=dtype), torch.randint(0, 40, (T, top), generator=torch.Generator().manual_seed(6)), rnd(T, top, seed=7)
    mix = torch.einsum("tj,tjw->tw", by.double(), buf.double()[pick])
    want = x.double() + oracle.grouped_rms(mix, post.double(), groups, 1e-3)
    xc = x.cuda()
    assert ops.stream_update(xc, dtype, 1e-3, [], a=Routed(buf.cuda(), pick.int().cuda(), by.cuda()), post=post.cuda(), groups=groups) == []
    close(xc, want, 3e-6)
    # the start of the stream
    ids = torch.tensor([3, 0, 39, 3, 1, 2, 5, 8, 13], dtype=torch.int32)
    xc = torch.full((T, W), 9.0, device="cuda")
    h = ops.stream_update(xc, dtype, 1e-3, [w.cuda()], start=True, ids=ids.cuda(), embed=buf.cuda(), post=post.cuda(), groups=groups)[0]
    want = oracle.grouped_rms(buf.double()[ids.long()], post.double(), groups, 1e-3)
    close(xc, want, 3e-6)
    close(h, oracle.grouped_rms(want, w.double(), groups, 1e-3), tol)


# ------------------------------------------------------------------------------------------------ ahead of the attention
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("tokens", [9, 2100])
@pytest.mark.parametrize("heads,kv_heads,d,dv", [(16, 4, 128, 128), (6, 2, 40, 72), (5, 1, 9, 7)])
def test_normed_queries_with_a_factor_per_head(ops, heads, kv_heads, d, dv, tokens, dtype):
    s = Spec(heads=heads, kv_heads=kv_heads, dim=d, vdim=dv, norm="head")
    b = Batch([(0, 5), (14, 18)] if tokens == 9 else [(3, 1103), (0, 1000)], 64, seed=6, pad=2)
    rows = (heads + kv_heads) * d + kv_heads * dv
    proj, temper = rnd(tokens + 2, rows + 8, seed=1, dtype=dtype), rnd(heads, seed=2)
    qw, kw = ((1.0 + 0.3 * rnd(d, seed=n)).to(dtype) for n in (3, 4))
    kc, vc = (torch.zeros(b.num_blocks, kv_heads, 64, n, dtype=dtype, device="cuda") for n in (d, dv))
    table = torch.zeros(1, 0, device="cuda")
    x = proj[:tokens].double()
    want = oracle.unit_rms(x[:, :heads * d].reshape(tokens, heads, d), 1e-3) * qw.double() * temper.double()[:, None]
    tol = 5e-6 if dtype == F32 else 6e-3
    q = ops.norm_rope_store(proj.cuda(), qw.cuda(), None, 1e-3, s, table, b.positions, b.slot_mapping, kc, vc, temper=temper.cuda())
    close(q[:tokens, :, :d], want, tol)
    assert not q[:, :, d:].any() and not kc.any() and not vc.any()                   # queries alone
    q = ops.norm_rope_store(proj.cuda()[:, :rows], qw.cuda(), kw.cuda(), 1e-3, s, table, b.positions, b.slot_mapping, kc, vc, temper=temper.cuda())
    ops.check_status()
    close(q[:tokens, :, :d], want, tol)
    at = b.slot_mapping[:tokens].long()
    close(kc[at // 64, :, at % 64], oracle.unit_rms(x[:, heads * d:(heads + kv_heads) * d].reshape(tokens, kv_heads, d), 1e-3) * kw.double(), tol)


# ------------------------------------------------------------------------------------------------ windows and blocks
ATTENTION = {
    "real": Spec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, window=100),
    "values": Spec(heads=6, kv_heads=2, dim=64, vdim=256, scale=0.1, window=64),
    "deep": Spec(heads=4, kv_heads=4, dim=256, vdim=256, scale=0.06, window=65),
    "groups": Spec(heads=40, kv_heads=2, dim=40, vdim=72, scale=0.2, window=63),
    "one": Spec(heads=3, kv_heads=3, dim=24, vdim=40, scale=0.2, window=1),
    "odd": Spec(heads=5, kv_heads=1, dim=9, vdim=7, scale=0.3, window=17),
}


def attention_case(ops, s, pool, ranges, page, dtype, seed=0, decode=False, pad=0, needle=None, own=True, **options):
    """Random keys and values of whole sequences in shuffled pages, queries for the ranges; what the oracle gives for the ranges.  Means of the
    blocks that ended before a range are in place, the others are not.  ``needle(position) -> key or ~block``: the query of that position points at
    that key, or at that block's mean."""
    b = Batch(ranges, page, decode=decode, pad=pad, seed=seed)
    H, G, d, dv, T = s.heads, s.kv_heads, s.dim, s.vdim, sum(hi - lo for lo, hi in ranges)
    kc, vc = (torch.full((b.num_blocks, G, page, n), 7.0, dtype=dtype, device="cuda") for n in (d, dv))
    rows = PooledCache.rows(page, pool)
    pk, pv = (torch.full((b.num_blocks, G, rows, n), -9.0, dtype=dtype, device="cuda") for n in (d, dv))
    cols = ops.C.windowed_prefill_qcols(d, dv, page) if dtype == BF else 0
    q_all = torch.zeros(T + pad, H, cols or d, dtype=dtype)
    wants, at, places = [], 0, []
    for i, (lo, hi) in enumerate(ranges):
        k, v = rnd(hi, G, d, seed=100 * seed + i + 5, dtype=dtype), rnd(hi, G, dv, seed=100 * seed + i + 6, dtype=dtype)
        mk, mv = oracle.pooled(k.double(), pool), oracle.pooled(v.double(), pool)
        q = rnd(hi, H, d, seed=100 * seed + i + 7)
        if needle is not None:
            for n in range(lo, hi):
                j = needle(n)
                t = (k[j].float() if j >= 0 else mk[~j].float()).repeat_interleave(H // G, 0)
                q[n] = 12 / s.scale * t / (t * t).sum(-1, keepdim=True)
        q = q.to(dtype)
        slots = torch.tensor([int(b.tables[i][p // page]) * page + p % page for p in range(hi)], device="cuda")
        kc[slots // page, :, slots % page], vc[slots // page, :, slots % page] = k.cuda(), v.cuda()
        blocks = torch.arange(hi // pool)
        p, r = pool_place(blocks, pool, page)
        p = b.tables[i][p]
        done = hi // pool if not own else lo // pool
        pk[p[:done], :, r[:done]], pv[p[:done], :, r[:done]] = mk[:done].to(dtype).cuda(), mv[:done].to(dtype).cuda()
        places.append((p, r, mk, mv))
        wants.append(0.8 * oracle.pooled_window_attention(q.double(), k.double(), v.double(), s.scale, s.window, pool)[lo:].reshape(hi - lo, -1))
        q_all[at:at + hi - lo, :, :d] = q[lo:]
        at += hi - lo
    out = torch.full((T + pad, H * dv + 8), 3.0, dtype=dtype, device="cuda")
    ops.windowed_attention(q_all.cuda(), kc, vc, b, s, out[:, :H * dv], 0.8, pool=PooledCache(pool, pk, pv, own), **options)
    ops.check_status()
    assert (out[:, H * dv:] == 3.0).all()
    for p, r, mk, mv in places:                            # every whole block has its means, and nothing else has been written
        if len(mk):
            close(pk[p, :, r], mk, 2e-6 if dtype == F32 else 4e-3)
            close(pv[p, :, r], mv, 2e-6 if dtype == F32 else 4e-3)
    assert int((pk == -9.0).all(-1).sum()) == pk.shape[0] * G * rows - G * sum(len(m[2]) for m in places)
    return out[:T, :H * dv], torch.cat(wants)


POOLS = (1, 3, 8, 16, 100)


@pytest.mark.parametrize("dtype,page", [(F32, 16), (BF, 16), (BF, 64), (BF, 256)])
@pytest.mark.parametrize("pool", POOLS)
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_prompts(ops, name, pool, dtype, page):
    ranges = [(0, 130), (0, 2), (60, 64), (127, 300), (5, 69), (400, 529), (64, 65)]
    if dtype == F32:
        ranges = [(0, 70), (30, 33), (15, 18), (64, 65), (90, 121)]
    got, want = attention_case(ops, ATTENTION[name], pool, ranges, page, dtype, seed=1)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)
    ranges = [(8, 9), (699, 700), (95, 96)] + ranges      # single tokens ahead of portions
    got, want = attention_case(ops, ATTENTION[name], pool, ranges, page, dtype, seed=2, own=page != 64)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype,page", [(F32, 16), (BF, 16), (BF, 64)])
@pytest.mark.parametrize("pool", POOLS)
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_decode(ops, name, pool, dtype, page):
    lens = (1, 2, 63, 64, 65, 66, 100, 101, 127, 128, 129, 256, 400, 17)
    got, want = attention_case(ops, ATTENTION[name], pool, [(n - 1, n) for n in lens], page, dtype, seed=2, decode=True, pad=3)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)
    for own in (True, False):
        got, want = attention_case(ops, ATTENTION[name], pool, [(n - 1, n) for n in (1500, 3)], page, dtype, seed=3, decode=True, own=own)
        close(got, want, 1e-5 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("name,pool", [("real", 8), ("real", 5), ("values", 16), ("groups", 3), ("odd", 4), ("one", 2)])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("kind", ["oldest key", "key before", "newest block", "block after", "first block"])
def test_attention_edges(ops, name, pool, decode, kind):
    """Every query points at one key or one block: the oldest key of its window, the one before it, the newest block that it sees, the one after that, or the
    first of the sequence."""
    s = ATTENTION[name]

    def needle(p):
        oldest = max(p - s.window + 1, 0)
        blocks = oldest // pool
        if kind == "oldest key":
            return oldest
        if kind == "key before":
            return max(oldest - 1, 0)
        b = {"newest block": blocks - 1, "block after": blocks, "first block": 0}[kind]
        return ~b if 0 <= b < (p + 1) // pool else p
    ranges = [(n - 1, n) for n in (301, 302, 303, 304, 65, 64, 63, 17, 128, 129, 130, 100, 101, 66, 107, 108)] if decode else [(0, 313), (280, 320), (130, 132)]
    for dtype in (BF, F32):
        got, want = attention_case(ops, s, pool, ranges, 64, dtype, seed=4, decode=decode, needle=needle)
        close(got, want, 2e-2 if dtype == BF else 2e-5)


@pytest.mark.parametrize("ranges", [[(499, 500), (0, 2)], [(499, 500), (0, 7), (3, 5)], [(40, 41), (0, 17)]])
def test_portions_without_a_whole_block_beside_long_requests(ops, ranges):
    for dtype in (BF, F32):
        got, want = attention_case(ops, ATTENTION["real"], 16, ranges, 64, dtype, seed=8)
        close(got, want, 1e-5 if dtype == F32 else 8e-3)


def test_blocks_go_with_the_other_options(ops):
    s = ATTENTION["real"]
    for ranges, decode in (([(0, 300), (290, 300)], False), ([(299, 300), (511, 512)], True)):
        for dtype in (BF, F32):
            plain, want = attention_case(ops, s, 8, ranges, 64, dtype, seed=7, decode=decode)
            capped, _ = attention_case(ops, s, 8, ranges, 64, dtype, seed=7, decode=decode, softcap=1e4, sink=torch.full((16,), -200.0, device="cuda"),
                                       gate=torch.full((want.shape[0], 16), 30.0, dtype=dtype, device="cuda"))
            close(capped, plain, 1e-4 if dtype == F32 else 8e-3)


# ------------------------------------------------------------------------------------------------ latent attention over a window
LATENT = {
    "real": Spec(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, window=100),
    "groups": Spec(heads=20, dim=40, rot_dim=32, vdim=72, kv_rank=112, scale=0.13, window=64),
    "small": Spec(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, scale=0.2, window=1),
    "wide": Spec(heads=40, dim=64, rot_dim=64, vdim=64, kv_rank=256, scale=0.1, window=65),
    "odd": Spec(heads=5, dim=9, rot_dim=6, vdim=7, kv_rank=13, scale=0.3, window=17),
}


def latent_case(ops, s, ranges, page, dtype, seed=0, decode=False, pad=0, needle=None):
    """Keys are made with the rotation left out (the same angle for all), so that a query can point at a key."""
    b = Batch(ranges, page, decode=decode, pad=pad, seed=seed)
    R, r, H, d, dv = s.kv_rank, s.rot_dim, s.heads, s.dim, s.vdim
    wkv = rnd(H * (d + dv), R, seed=seed + 1, scale=R ** -0.5, dtype=dtype)
    cache = torch.full((b.num_blocks, page, R + r), 7.0, dtype=dtype)
    cols, wants, qs = H * (d + r), [], []
    for i, (lo, hi) in enumerate(ranges):
        row = rnd(hi, R + r, seed=100 * seed + i + 5, dtype=dtype)
        for p in range(hi):
            cache[b.tables[i][p // page], p % page] = row[p]
        c, kr = row[:, :R].double(), row[:, R:].double()
        k = torch.cat([(c @ wkv[:H * d].double().T).view(hi, H, d), kr[:, None].expand(hi, H, r)], -1)
        v = (c @ wkv[H * d:].double().T).view(hi, H, dv)
        q = rnd(hi, H, d + r, seed=100 * seed + i + 7).double()
        if needle is not None:
            for n in range(lo, hi):
                t = k[needle(n)]
                q[n] = 12 / s.scale * t / (t * t).sum(-1, keepdim=True)
        q = q.to(dtype)
        wants.append(oracle.softmax_attention(q.double(), k, v, s.scale, oracle.sliding(hi, s.window))[lo:].reshape(hi - lo, -1))
        qs.append(q[lo:].reshape(hi - lo, -1))
    q = torch.zeros(b.positions.shape[0], -(-cols // 8) * 8 + 16, dtype=dtype)               # a view of wider rows
    q[:sum(x.shape[0] for x in qs), :cols] = torch.cat(qs)
    w = Spec(ukv=wkv.cuda(), uk_t=wkv[:H * d].view(H, d, R).transpose(1, 2).contiguous().cuda(), uv=wkv[H * d:].view(H, dv, R).cuda())
    still = torch.cat([torch.ones(2000, r // 2), torch.zeros(2000, r // 2)], -1).cuda()
    got = ops.latent_attention(q.cuda()[:, :cols], w, cache.cuda(), b, still, s)
    ops.check_status()
    return got[:got.shape[0] - pad], torch.cat(wants)


@pytest.mark.parametrize("dtype,page", [(F32, 16), (BF, 16), (BF, 64)])
@pytest.mark.parametrize("name", list(LATENT))
def test_latent_windows(ops, name, dtype, page):
    ranges = [(0, 130), (0, 2), (60, 64), (127, 300), (5, 69), (400, 529), (64, 65)] if dtype == BF else [(0, 70), (30, 33), (15, 18), (90, 121)]
    tol = 1e-5 if dtype == F32 else 1.5e-2
    for window in (LATENT[name].window, 5000):
        s = Spec(**{**LATENT[name].__dict__, "window": window})
        close(*latent_case(ops, s, ranges, page, dtype, seed=1), tol)
        close(*latent_case(ops, s, [(8, 9), (499, 500), (95, 96)] + ranges, page, dtype, seed=2), tol)
        lens = (1, 2, 63, 64, 65, 66, 100, 101, 127, 128, 129, 256, 400, 17)
        close(*latent_case(ops, s, [(n - 1, n) for n in lens], page, dtype, seed=3, decode=True, pad=3), tol)
        close(*latent_case(ops, s, [(n - 1, n) for n in (1500, 3)], page, dtype, seed=4, decode=True), tol)


@pytest.mark.parametrize("name", list(LATENT))
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("out", [0, 1])
def test_latent_edges(ops, name, decode, out):
    """Every query points at the oldest key of its window (0) or at the one before it, which must not be seen (1)."""
    s = LATENT[name]
    ranges = [(n - 1, n) for n in (301, 302, 303, 65, 64, 63, 17, 128, 129, 130, 100, 101, 66, 127)] if decode else [(0, 213), (180, 220), (130, 132)]
    for dtype in (BF, F32):
        got, want = latent_case(ops, s, ranges, 64, dtype, seed=5, decode=decode, needle=lambda p: max(p - s.window + 1 - out, 0))
        close(got, want, 4e-2 if dtype == BF else 2e-5)


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("T", [1, 100, 300, 2100])
@pytest.mark.parametrize("W,E,top,count,keep", [(64, 8, 3, 2, 1), (128, 64, 8, 8, 4), (96, 100, 6, 10, 3), (50, 6, 2, 3, 3), (64, 5, 5, 1, 1), (64, 12, 4, 12, 4), (64, 256, 8, 8, 4)])
def test_router_within_groups(ops, W, E, top, count, keep, T, dtype):
    h, w, corr = rnd(T, W, seed=1, dtype=dtype), rnd(E, W, seed=2, scale=W ** -0.5, dtype=dtype), 0.6 * rnd(E, seed=3) - 0.8
    e, by = torch.full((T, top), -1, dtype=torch.int32, device="cuda"), torch.zeros(T, top, device="cuda")
    ops.C.router(h.cuda(), w.cuda(), e, by, False, corr.cuda(), count, keep)
    s = torch.sigmoid(h.double() @ w.double().T)
    assert (by.cpu() - s.gather(1, e.cpu().long())).abs().max() < 2e-5                      # weights without the correction
    same = torch.tensor([oracle.choose(s[t], corr, top, count, keep) == e[t].tolist() for t in range(T)])
    assert same.float().mean() > 0.97                                                       # up to close calls
    assert all(len(set(row)) == top for row in e.tolist())
    groups = torch.div(e.cpu(), E // count, rounding_mode="floor")
    assert max(len(set(row)) for row in groups.tolist()) <= keep


def test_router_survives_scores_that_are_not_numbers(ops):
    """Every place is filled with an expert that exists."""
    for T in (5, 300):
        h = torch.full((T, 64), float("nan"), dtype=BF, device="cuda")
        w = torch.ones(16, 64, dtype=BF, device="cuda")
        e, by = torch.full((T, 4), -1, dtype=torch.int32, device="cuda"), torch.zeros(T, 4, device="cuda")
        ops.C.router(h, w, e, by, False, torch.zeros(16, device="cuda"), 4, 2)
        assert e.min() >= 0 and e.max() < 16 and all(len(set(row)) == 4 for row in e.tolist())


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("T,W,E,top,ff,count,keep", [(3, 64, 4, 2, 40, 2, 1), (200, 256, 8, 3, 320, 2, 1), (700, 128, 6, 4, 136, 3, 2), (40, 50, 5, 2, 11, 1, 1), (2000, 256, 4, 2, 512, 2, 2)])
def test_experts_without_gates(ops, T, W, E, top, ff, count, keep, dtype):
    h, router, corr = rnd(T, W, seed=1, dtype=dtype), rnd(E, W, seed=2, scale=3 * W ** -0.5, dtype=dtype), 0.3 * rnd(E, seed=3)
    up, down = rnd(E, ff, W, seed=4, scale=2 * W ** -0.5, dtype=dtype), rnd(E, W, ff, seed=5, scale=ff ** -0.5, dtype=dtype)
    y = ops.moe(h.cuda(), router.cuda(), up.cuda(), down.cuda(), top, weigh="output", act="gelu", gated=False, correction=corr.cuda(), groups=count, keep=keep)
    ops.check_status()
    got = (y.y.double()[y.rows.long()] * y.weights.double()[:, :, None]).sum(1).cpu()
    n = min(T, 120)
    w = {"router": router.double(), "correction": corr.double()}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = up[e].double(), down[e].double()
    want = oracle.experts(h[:n].double(), w, "", {"router": {"top": top, "groups": {"count": count, "keep": keep}}})
    err = (got[:n] - want).abs().amax(-1) / want.abs().max()
    assert err.median() < (1e-5 if dtype == F32 else 1e-2) and (err < (1e-4 if dtype == F32 else 2e-2)).float().mean() > 0.95


@pytest.mark.parametrize("dtype", [F32, BF])
def test_gelu_of_an_expert(ops, dtype):
    """One expert with unit matrices: the activation alone, also far out on the negative side."""
    n, W = 640, 64
    h = torch.zeros(n, W)
    h[:, :32] = torch.linspace(-9, 9, n)[:, None]
    h = h.to(dtype)
    eye = torch.eye(W, dtype=dtype, device="cuda")[None].contiguous()
    y = ops.moe(h.cuda(), torch.zeros(1, W, dtype=dtype, device="cuda"), eye, eye, 1, weigh="output", act="gelu", gated=False)
    got, want = y.y[y.rows[:, 0].long()].double().cpu(), oracle.gelu(h.double())
    if dtype == BF:
        want = want.bfloat16().double()
    assert ((got - want).abs() <= (2e-7 if dtype == F32 else 5e-7) + (1e-6 if dtype == F32 else 2.0 ** -7) * want.abs()).all()


# ------------------------------------------------------------------------------------------------ logits
def test_bounded_logits(ops):
    for dtype, tol in ((F32, 1e-6), (BF, 4e-3)):
        x = torch.linspace(-300, 300, 4001).to(dtype)
        for scale, cap in ((0.3, 12.0), (1.0, 50.0), (0.5, 0.0)):
            z = x.double() * scale
            close(ops.bound_logits(x.cuda(), scale, cap), cap * torch.tanh(z / cap) if cap else z, tol)


def test_bounded_logits_in_the_lm_head(ops):
    """Sampling in the head's epilogue gives the tokens of logits, bound and sampler as three kernels."""
    rows, vocab, K = 40, 80000, 64
    x, w = rnd(rows, K, seed=1, dtype=BF).cuda(), rnd(vocab, K, seed=2, dtype=BF).cuda()
    temps = torch.tensor([0.0, 0.7, 1.5, 3.0] * 10, device="cuda")
    header = torch.zeros(16, dtype=torch.int32, device="cuda")
    header[9:12] = torch.tensor([5, 77, 3])
    assert ops.can_sample_in_lm_head(rows, w)
    for scale, cap in ((0.5, 4.0), (0.25, 30.0)):
        ids, _ = ops.lm_head_sample_shard(x, w, temps, header, 0, scale, cap)
        logits = ops.bound_logits(ops.linear(x, w), scale, cap)
        assert float(logits.abs().max()) <= cap
        want, _ = ops.sample_shard(logits, temps, header, 0)
        ops.check_status()
        assert torch.equal(ids, want)
        free, _ = ops.lm_head_sample_shard(x, w, temps, header, 0)
        assert not torch.equal(free, ids)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = lc.Case(name, tmp_path_factory.mktemp(name), "cuda")
        return made[name]
    return get


def agree(err, dtype):
    """fp32: every position.  bf16: sharp scores, and close calls of routers that go the other way, so nine positions in ten."""
    if dtype == "float32":
        assert err.max() < 1e-4, err.max()
    else:
        assert np.quantile(err, 0.9) < 0.25 and np.median(err) < 0.1, np.quantile(err, [0.5, 0.9, 1.0])


@pytest.mark.parametrize("dtype,block", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64)])
@pytest.mark.parametrize("name", list(lc.CONFIGS))
def test_model(cases, name, dtype, block):
    c = cases(name)
    toks = gc.tokens(c.cfg, 150, 1)
    p = c.player(dtype, block=block)
    for sched in ([[("a", toks)]], [[("a", toks[:100])]] + [[("a", [t])] for t in toks[100:]],
                  [[("a", part)] for part in gc.portions(toks, [2, 15, 1, 33, 17, 16, 3])]):
        agree(c.error(gc.run(p, sched)["a"], toks, slice(None)), dtype)
    p.engine.exit()


@pytest.mark.parametrize("dtype,block,blocks", [("float32", 16, 18), ("bfloat16", 16, 18), ("bfloat16", 64, 8)])
@pytest.mark.parametrize("name", ["varied", "wide", "odd"])
def test_model_mixed_batches(cases, name, dtype, block, blocks):
    c = cases(name)
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 30 + i) for i, n in enumerate((1, 65, 50, 2, 100, 48, 130, 17))}
    p = c.player(dtype, block=block, blocks=blocks, slots=3)
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 1, 2, 3, 19, 40], live=3))
    agree(np.concatenate([c.error(got[n], t, slice(None)) for n, t in reqs.items()]), dtype)
    assert p.pool.num_free == blocks
    if dtype == "float32":                                # the same requests, each alone: nothing depends on the company
        for n, t in list(reqs.items())[:4]:
            alone = gc.run(p, [[(n, t)]])[n]
            assert np.abs(alone - got[n]).max() < 1e-3
    p.engine.exit()


def test_long_decoding(cases):
    """Windows pass over decoded tokens alone several times, and blocks of decoded tokens come into view."""
    c = cases("varied")
    toks = gc.tokens(c.cfg, 260, 8)
    for dtype in ("float32", "bfloat16"):
        p = c.player(dtype)
        agree(c.error(gc.run(p, [[("a", toks[:10])]] + [[("a", [t])] for t in toks[10:]])["a"], toks, slice(None)), dtype)
        p.engine.exit()


def test_generation_with_graphs(cases):
    from tinyllmforge_b200 import LLM, SamplingParams
    c = cases("short")
    prompts = [gc.tokens(c.cfg, n, 20 + n) for n in (1, 5, 16, 23, 40, 64)]

    def outputs(**kw):
        base = dict(dtype="float32", kvcache_block_size=16, num_kvcache_blocks=64, max_model_len=128, max_num_batched_tokens=128, max_num_seqs=4,
                    skip_tokenizer_init=True)
        llm = LLM(c.path, **{**base, **kw})
        outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True), use_tqdm=False)
        llm.worker.ops.check_status()
        llm.exit()
        return [o["token_ids"] for o in outs]

    got = outputs()
    for prompt, out in zip(prompts, got):
        logits = c.want(prompt + out)[len(prompt) - 1:-1]
        best = logits.max(-1).values
        picked = logits[torch.arange(len(out)), torch.tensor(out)]
        assert ((best - picked) < 1e-3 * logits.std()).all()         # greedy up to a tie
    assert outputs(enforce_eager=True) == got
    assert outputs(chunked_prefill=True, max_num_batched_tokens=16, extra={"pipeline": False}) == got
    low = outputs(dtype="bfloat16")
    assert np.mean([a == b for s, t in zip(low, got) for a, b in zip(s, t)]) > 0.4
