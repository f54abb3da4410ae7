"""Tonapel on the CUDA op set: every kernel against the plain oracle's mechanism, and whole models (fp32 and bf16) against the
oracle with prompts, portions, mixed batches, reused blocks and slots, and generation with CUDA graphs."""
import numpy as np
import pytest
import torch

import goselix_cases as gc
import oracle_tonapel as oracle
import tonapel_cases as tc
from kernel_helpers import Batch, Spec, close, rnd, rope

pytestmark = pytest.mark.gpu

F32, BF = torch.float32, torch.bfloat16


@pytest.fixture(scope="module")
def ops():
    from tinyllmforge_b200.ops.cuda import CudaOps
    return CudaOps()


# ------------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("W", [64, 50, 2048, 4100])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_sandwich_norm(ops, W, dtype):
    from tinyllmforge_b200.ops.cuda_mixers import Routed
    T, top, V = 9, 3, 11
    x = rnd(T, W, seed=1)
    a, y, emb = (rnd(*s, seed=i, dtype=dtype) for i, s in enumerate([(T, W), (40, W), (V, W)], 2))
    post, pre, bias, weights = rnd(W, seed=8, dtype=dtype), rnd(W, seed=9, dtype=dtype), rnd(W, seed=10), rnd(T, top, seed=11)
    rows = torch.randint(0, 40, (T, top), generator=torch.Generator().manual_seed(3), dtype=torch.int32)
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(4), dtype=torch.int32)
    tol = 3e-6 if dtype == F32 else 6e-3
    routed = Routed(y.cuda(), rows.cuda(), weights.cuda())
    for branch, value in ((a.cuda(), a.double() + bias.double()), (routed, (weights.double()[..., None] * y.double()[rows.long()]).sum(1) + bias.double())):
        kw = dict(a=branch, a_bias=bias.cuda(), post=post.cuda(), mult=0.3, offset=1.0)
        want = x.double() + 0.3 * oracle.shifted_norm(value, post.double(), 1e-5)
        xc = x.cuda()
        only, = ops.stream_update(xc, dtype, 1e-5, [pre.cuda()], rows=torch.tensor([7, 0, 7], dtype=torch.int32, device="cuda"), **kw)
        assert torch.equal(xc.cpu(), x)                              # x is left alone when rows are picked
        h, = ops.stream_update(xc, dtype, 1e-5, [pre.cuda()], **kw)
        close(xc, want, 3e-6)
        close(h, oracle.shifted_norm(want, pre.double(), 1e-5), tol)
        close(only, oracle.shifted_norm(want, pre.double(), 1e-5)[[7, 0, 7]], tol)
    h, = ops.stream_update(xc, dtype, 1e-5, [pre.cuda()], start=True, ids=ids.cuda(), embed=emb.cuda(), offset=1.0)
    close(xc, emb.double()[ids.long()], 1e-7)
    close(h, oracle.shifted_norm(emb.double()[ids.long()], pre.double(), 1e-5), tol)


# ------------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype,M,F,K", [(F32, 20, 37, 50), (BF, 20, 37, 50), (BF, 1, 96, 64), (BF, 40, 256, 128), (BF, 200, 384, 512), (BF, 700, 320, 256),
                                         (BF, 100, 2048, 4096)])
@pytest.mark.parametrize("act", ["gelu_tanh", "clamped_swish"])
def test_gated_products(ops, dtype, M, F, K, act):
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(2 * F, K, seed=2, scale=2 * K ** -0.5, dtype=dtype)
    g, u = x.double() @ w[:F].double().T, x.double() @ w[F:].double().T
    want = oracle.gelu_tanh(g) * u if act == "gelu_tanh" else oracle.clamped_expert(x.double(), w[:F].double(), w[F:].double(), torch.eye(F).double(), 0.9)
    close(ops.linear_act_mul(x.cuda(), w.cuda(), act, 0.9), want, 5e-6 if dtype == F32 else 8e-3)
    ops.check_status()


@pytest.mark.parametrize("dtype,T,E,top,W,F", [(F32, 33, 5, 2, 50, 11), (BF, 33, 5, 2, 50, 11), (BF, 1, 8, 1, 64, 32), (BF, 70, 16, 2, 512, 200),
                                               (BF, 500, 9, 4, 192, 136), (BF, 1100, 20, 5, 96, 48), (BF, 2100, 100, 2, 64, 16), (BF, 20, 300, 2, 64, 16)])
def test_experts(ops, dtype, T, E, top, W, F):
    h = rnd(T, W, seed=1, dtype=dtype)
    w = {"router": rnd(E, W, seed=2, scale=2 * W ** -0.5, dtype=dtype)}
    for e in range(E):
        w.update({f"e{e}.gate": rnd(F, W, seed=3 * e + 10, scale=W ** -0.5, dtype=dtype), f"e{e}.up": rnd(F, W, seed=3 * e + 11, scale=W ** -0.5, dtype=dtype),
                  f"e{e}.down": rnd(W, F, seed=3 * e + 12, scale=F ** -0.5, dtype=dtype)})
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).cuda()
    down = torch.stack([w[f"e{e}.down"] for e in range(E)]).cuda()
    out = ops.moe(h.cuda(), w["router"].cuda(), gu, down, top, score="softmax", weigh="output", act="clamped_swish", limit=1.1)
    ops.check_status()
    got = (out.y.float()[out.rows.long()] * out.weights[..., None]).sum(1)
    wd = {k: v.double() for k, v in w.items()}
    z = (h.double() @ wd["router"].T).sort(-1, descending=True).values
    ok = z[:, top - 1] - z[:, top] > 1e-4 if top < E else torch.ones(T, dtype=torch.bool)     # leave out close calls
    assert ok.float().mean() > 0.9
    _, weights = oracle.route(h.double(), wd["router"], top)
    close(out.weights[ok.cuda()], weights[ok], 1e-5)
    n = min(T, 200)
    want = oracle.mixture(h[:n].double(), wd, "", {"router": {"top": top}, "expert": {"limit": 1.1}})
    close(got[:n][ok[:n].cuda()], want[ok[:n]], 1e-5 if dtype == F32 else 2e-2)


# ------------------------------------------------------------------------------------------------ windowed attention
ATTENTION = {
    "real": Spec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, window=100, rd=64),
    "values": Spec(heads=6, kv_heads=2, dim=64, vdim=256, scale=0.1, window=64, rd=64),
    "deep": Spec(heads=4, kv_heads=4, dim=256, vdim=256, scale=0.06, window=65, rd=32),
    "groups": Spec(heads=40, kv_heads=2, dim=40, vdim=72, scale=0.2, window=63, rd=16),
    "one": Spec(heads=3, kv_heads=3, dim=24, vdim=40, scale=0.2, window=1, rd=24),
    "long": Spec(heads=8, kv_heads=1, dim=96, vdim=192, scale=0.1, window=5000, rd=96),
    "odd": Spec(heads=5, kv_heads=1, dim=9, vdim=7, scale=0.3, window=17, rd=6),
}


def attention_setup(ops, s, ranges, block, dtype, seed=0, decode=False, pad=0, needle=None, factor=0.8, stale=7.0):
    """Whole sequences' keys and values through bias_rope_store, queries for the ranges; what the oracle gives for the ranges.
    ``needle(position) -> key``: the query of that position points at that key."""
    b = Batch(ranges, block, decode=decode, pad=pad, seed=seed)
    H, G, d, dv = s.heads, s.kv_heads, s.dim, s.vdim
    table = rope(4096, s.rd)
    kc, vc = (torch.full((b.num_blocks, G, block, n), stale, dtype=dtype, device="cuda") for n in (d, dv))
    rows = (H + G) * d + G * dv
    bias = rnd(rows, seed=seed + 1, scale=0.5)
    full = Batch([(0, e) for _, e in ranges], block, seed=seed)             # the same tables, all tokens
    assert torch.equal(full.tables, b.tables)
    projs, wants, queries = [], [], []
    for i, (lo, hi) in enumerate(ranges):
        proj = rnd(hi, rows + 5, seed=100 * seed + i + 5).to(dtype)
        x = proj[:, :rows].double() + bias.double()
        q, k, v = x[:, :H * d].reshape(hi, H, d), x[:, H * d:(H + G) * d].reshape(hi, G, d), x[:, (H + G) * d:].reshape(hi, G, dv)
        kr = oracle.rotate(k, 10000.0, s.rd)
        if needle is not None:
            for n in range(lo, hi):
                t = kr[needle(n)].repeat_interleave(H // G, 0)
                back = oracle.rotate((12 / s.scale * t / (t * t).sum(-1, keepdim=True))[None], 10000.0, s.rd, -n)[0]
                proj[n, :H * d] = (back.reshape(-1) - bias[:H * d].double()).to(dtype)
            q = (proj[:, :H * d].double() + bias[:H * d].double()).reshape(hi, H, d)
        wants.append(factor * oracle.windowed_attention(oracle.rotate(q, 10000.0, s.rd), kr, v, s.scale, s.window)[lo:].reshape(hi - lo, -1))
        projs.append(proj)
        queries.append(proj[lo:])
    allp = torch.cat(projs).cuda()
    ops.bias_rope_store(allp[:, :rows], bias.cuda(), s, table, full.positions, full.slot_mapping, kc, vc)
    mine = torch.cat(queries + [torch.zeros(pad, rows + 5, dtype=dtype)]).cuda()
    q = ops.bias_rope_store(mine[:, :rows], bias.cuda(), s, table, b.positions, b.slot_mapping, kc, vc)
    out = torch.full((q.shape[0], H * dv + 8), 3.0, dtype=dtype, device="cuda")
    ops.windowed_attention(q, kc, vc, b, s, out[:, :H * dv], factor)
    ops.check_status()
    assert (out[:, H * dv:] == 3.0).all()
    return out[:out.shape[0] - pad, :H * dv], torch.cat(wants)


@pytest.mark.parametrize("dtype,block", [(F32, 16), (BF, 16), (BF, 64), (BF, 256)])
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_prompts(ops, name, dtype, block):
    ranges = [(0, 130), (0, 2), (60, 64), (127, 300), (5, 69), (700, 829), (64, 65)]
    if dtype == F32:
        ranges = [(0, 70), (30, 33), (15, 18), (64, 65)]
    got, want = attention_setup(ops, ATTENTION[name], ranges, block, dtype, seed=1)
    close(got, want, 1e-5 if dtype == F32 else 1.5e-2)


@pytest.mark.parametrize("dtype,block", [(F32, 16), (BF, 16), (BF, 64), (BF, 256)])
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_decode(ops, name, dtype, block):
    lens = (1, 2, 63, 64, 65, 100, 101, 127, 128, 129, 256, 700, 17)
    got, want = attention_setup(ops, ATTENTION[name], [(n - 1, n) for n in lens], block, dtype, seed=2, decode=True, pad=3)
    close(got, want, 1e-5 if dtype == F32 else 1.5e-2)
    got, want = attention_setup(ops, ATTENTION[name], [(n - 1, n) for n in (1500, 3)], block, dtype, seed=3, decode=True)
    close(got, want, 1e-5 if dtype == F32 else 1.5e-2)


@pytest.mark.parametrize("name", ["real", "values", "groups", "deep", "odd"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("out", [0, 1, 2])
def test_attention_window_edges(ops, name, decode, out):
    """Every query points at one key: the oldest in its window (0), the one before it, which must not be seen (1), or keys at the
    borders of blocks and tiles and its own (2)."""
    s = ATTENTION[name]
    near = [0, 15, 16, 63, 64, 127, 128, 255, 256]
    if out < 2:
        needle = lambda p: max(p - s.window + 1 - out, 0)
    else:
        needle = lambda p: max((t for t in near if p - s.window < t <= p), default=p)
    ranges = [(n - 1, n) for n in (301, 302, 303, 65, 64, 63, 17, 128, 129, 130, 100, 101, 66)] if decode else [(0, 313), (280, 320), (130, 132)]
    got, want = attention_setup(ops, s, ranges, 64, BF, seed=4, decode=decode, needle=needle)
    close(got, want, 2.5e-2)


def test_attention_with_large_scores_and_an_empty_first_tile(ops):
    """Rows whose first visible key comes after the first tiles of their CTA, with scores far above and below zero."""
    s = Spec(**{**ATTENTION["real"].__dict__, "scale": 2.0, "window": 64})
    got, want = attention_setup(ops, s, [(0, 400), (100, 300)], 64, F32, seed=6)
    close(got, want, 1e-3)
    got, want = attention_setup(ops, s, [(0, 400), (100, 300)], 64, BF, seed=6, needle=lambda p: max(p - 40, 0))
    close(got, want, 4e-2)


def test_bias_rope_store(ops):
    for dtype, s in ((F32, ATTENTION["odd"]), (BF, ATTENTION["odd"]), (BF, ATTENTION["real"]), (BF, ATTENTION["groups"])):
        b = Batch([(0, 5), (14, 18)], 64, seed=6, pad=2)
        H, G, d, dv, T = s.heads, s.kv_heads, s.dim, s.vdim, 9
        rows = (H + G) * d + G * dv
        proj, bias = rnd(T + 2, rows, seed=1, dtype=dtype), rnd(rows, seed=2)
        kc, vc = (torch.zeros(b.num_blocks, G, 64, n, dtype=dtype, device="cuda") for n in (d, dv))
        q = ops.bias_rope_store(proj.cuda(), bias.cuda(), s, rope(64, s.rd), b.positions, b.slot_mapping, kc, vc)
        x = (proj.double() + bias.double())[:T]
        turn = lambda m: torch.cat([oracle.rotate(m[:5], 10000.0, s.rd), oracle.rotate(m[5:], 10000.0, s.rd, 14)])
        tol = 2e-6 if dtype == F32 else 6e-3
        close(q[:T, :, :d], turn(x[:, :H * d].reshape(T, H, d)), tol)
        assert not q[:, :, d:].any()
        at = b.slot_mapping[:T].long()
        close(kc[at // 64, :, at % 64], turn(x[:, H * d:(H + G) * d].reshape(T, G, d)), tol)
        close(vc[at // 64, :, at % 64], x[:, (H + G) * d:].reshape(T, G, dv), tol)
        assert int((kc.abs().sum((1, 3)) > 0).sum()) == T and int((vc.abs().sum((1, 3)) > 0).sum()) == T
        ops.check_status()


# ------------------------------------------------------------------------------------------------ short convolution
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("C,taps", [(64, 4), (200, 3), (50, 2), (7, 5), (36, 1), (1000, 8)])
def test_short_conv(ops, dtype, C, taps):
    ranges = [(9, 10), (0, 1), (1, 2), (0, 100), (3, 5), (33, 97), (2, 4), (0, 2), (40, 73)]
    slots = [4, 0, 9, 2, 7, 1, 3, 8, 6]
    b = Batch(ranges, 64, slots=slots, seed=1)
    w, bias = rnd(C, taps, seed=2), rnd(C, seed=3)
    state = rnd(11, taps - 1, C, seed=4, dtype=dtype)
    for use in (bias, None):
        xs, wants, left = [], [], state.clone()
        for i, (lo, hi) in enumerate(ranges):
            x = rnd(hi, C, seed=20 + i, dtype=dtype)
            if lo > 0:                                                  # what an earlier step left, shorter than the taps or not
                tail = torch.zeros(taps - 1, C, dtype=dtype)
                n = min(lo, taps - 1)
                if n:
                    tail[taps - 1 - n:] = x[lo - n:lo]
                left[slots[i]] = tail
            y = oracle.silu(oracle.causal_conv(x.double(), w.double(), None if use is None else use.double()))
            wants.append(y[lo:])
            xs.append(x[lo:])
        st = left.clone().cuda()
        x = torch.cat(xs)
        wide = torch.zeros(x.shape[0], C + 16, dtype=dtype)
        wide[:, 8:8 + C] = x
        out = ops.short_conv(wide.cuda()[:, 8:8 + C], w.cuda(), None if use is None else use.cuda(), st, b)
        ops.check_status()
        close(out, torch.cat(wants), 3e-6 if dtype == F32 else 6e-3)
        for i, (lo, hi) in enumerate(ranges):
            full = torch.cat([torch.zeros(taps - 1, C, dtype=dtype), rnd(hi, C, seed=20 + i, dtype=dtype)])
            assert torch.equal(st[slots[i]].cpu(), full[hi:])
        untouched = [i for i in range(11) if i not in slots]
        assert torch.equal(st[untouched].cpu(), left[untouched])


# ------------------------------------------------------------------------------------------------ recurrences
RECURRENCE = {
    "real": Spec(heads=4, share=2, dk=128, dv=128),
    "ssd": Spec(heads=6, share=3, dk=128, dv=64),
    "small": Spec(heads=4, share=1, dk=32, dv=64),
    "part": Spec(heads=6, share=2, dk=48, dv=24),
    "deep": Spec(heads=2, share=2, dk=256, dv=136),
    "large": Spec(heads=1, share=1, dk=256, dv=256),
    "odd": Spec(heads=6, share=3, dk=9, dv=7),
    "sliver": Spec(heads=1, share=1, dk=16, dv=8),
}


def recurrence_check(ops, s, delta, dtype, ranges, decode=False, pad=0, seed=0, strong=False):
    """Random operands of whole sequences; the state of what lies before a range is the oracle's."""
    slots = np.random.default_rng(seed).permutation(len(ranges) + 2)[:len(ranges)].tolist()
    b = Batch(ranges, 64, slots=slots, decode=decode, pad=pad, seed=seed)
    H, G, dk, dv = s.heads, s.heads // s.share, s.dk, s.dv
    A, bias, D = rnd(H, seed=seed + 1, scale=1.2) + (1.5 if strong else -3.0), rnd(H, seed=seed + 2), rnd(H, seed=seed + 3)
    state = rnd(len(ranges) + 2, H, dk, dv, seed=seed + 4)                       # fresh sequences must not see it
    xs, raws, outs, ends = [], [], [], {}
    for i, (lo, hi) in enumerate(ranges):
        x = oracle.silu(rnd(hi, 2 * G * dk + H * dv, seed=50 * seed + i + 9)).to(dtype)
        raw = rnd(hi, 2 * H, seed=50 * seed + i + 10).to(dtype)
        q, k, v = x[:, :G * dk].double().view(hi, G, dk), x[:, G * dk:2 * G * dk].double().view(hi, G, dk), x[:, 2 * G * dk:].double().view(hi, H, dv)
        dt = oracle.softplus(raw[:, H:].double() + bias.double())
        if delta:
            beta, g = oracle.sigmoid(raw[:, :H].double()), torch.exp(-torch.exp(A.double()) * dt)
            q, k = oracle.unit_vectors(q) * dk ** -0.5, oracle.unit_vectors(k)
            q, k = q.repeat_interleave(s.share, 1), k.repeat_interleave(s.share, 1)
            go = lambda a, z, S: oracle.delta_scan(q[a:z], k[a:z], v[a:z], g[a:z], beta[a:z], S)
        else:
            go = lambda a, z, S: oracle.ssd_scan(v[a:z], k[a:z], q[a:z], dt[a:z], A.double(), D.double(), S)
        S = None
        if lo:
            _, S = go(0, lo, None)
            state[slots[i]] = S.float()
            S = S.float().double()
        o, S = go(lo, hi, S)
        outs.append(o)
        ends[slots[i]] = S
        xs.append(x[lo:])
        raws.append(raw[lo:])
    x, raw = (torch.cat(z + [torch.zeros(pad, z[0].shape[1], dtype=dtype)]).cuda() for z in (xs, raws))
    st = state.clone().cuda()
    n = G * dk
    o = ops.recur(x[:, :n], x[:, n:2 * n], x[:, 2 * n:], raw[:, H:], raw[:, :H] if delta else None, Spec(A_log=A.cuda(), dt_bias=bias.cuda(), D=D.cuda()), st, b)
    ops.check_status()
    tol = 2e-5 if dtype == F32 else 1e-3
    close(o[:o.shape[0] - pad], torch.cat(outs), tol)
    if pad:
        assert not o[o.shape[0] - pad:].any() or s.dv % 4
    for i, S in ends.items():
        close(st[i], S, tol)
    untouched = [i for i in range(len(state)) if i not in ends]
    assert torch.equal(st[untouched].cpu(), state[untouched])


@pytest.mark.parametrize("delta", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(RECURRENCE))
def test_recurrence_decode(ops, name, dtype, delta):
    recurrence_check(ops, RECURRENCE[name], delta, dtype, [(0, 1), (5, 6), (130, 131), (64, 65)], decode=True, pad=2, seed=2)


@pytest.mark.parametrize("delta", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(RECURRENCE))
def test_recurrence_prompts(ops, name, dtype, delta):
    recurrence_check(ops, RECURRENCE[name], delta, dtype, [(8, 9), (0, 1), (0, 200), (3, 5), (0, 64), (64, 129), (60, 124), (0, 2), (7, 70)], seed=3)
    recurrence_check(ops, RECURRENCE[name], delta, dtype, [(0, 65), (0, 63), (100, 101)], seed=4, strong=True)


@pytest.mark.parametrize("name", ["real", "ssd", "small"])
def test_state_space_segments(ops, name):
    """One long run is cut into segments; the state crosses them.  The token scan of the oracle has no segments."""
    s = RECURRENCE[name]
    assert ops.retention_segments(1, s.heads, s.dk, s.dv, 1500)[0] > 1
    recurrence_check(ops, s, False, BF, [(0, 1500)], seed=5)
    recurrence_check(ops, s, False, BF, [(0, 1100), (64, 75), (2, 770)], seed=6)


def test_delta_long_run(ops):
    recurrence_check(ops, RECURRENCE["real"], True, BF, [(0, 1100), (3, 770)], seed=7)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("groups,n,period", [(3, 40, 120), (1, 100, 100), (5, 7, 7), (4, 128, 128), (2, 384, 768)])
def test_gated_norm(ops, dtype, groups, n, period):
    T, W = 13, groups * n
    o, z, w = rnd(T, W, seed=1), rnd(T, W + 8, seed=2, dtype=dtype), rnd(period, seed=3)
    for first in (True, False):
        out = torch.zeros(T, W + 16, dtype=dtype, device="cuda")
        ops.C.gated_norm(o.cuda(), z.cuda()[:, :W], w.cuda(), out[:, 8:8 + W], groups, first, 0.7, 1e-5)
        gate, weight = z[:, :W].double(), w.double().repeat(W // period)
        if first:
            want = 0.7 * oracle.grouped_gate_norm(o.double(), gate, weight, groups, 1e-5)
        else:
            want = 0.7 * oracle.unit_rms(o.double().view(T, groups, n), 1e-5).reshape(T, W) * weight * oracle.silu(gate)
        close(out[:, 8:8 + W], want, 3e-6 if dtype == F32 else 6e-3)
        assert not out[:, :8].any() and not out[:, 8 + W:].any()


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = tc.Case(name, tmp_path_factory.mktemp(name), "cuda")
        return made[name]
    return get


def agree(err, dtype):
    """fp32: every position.  bf16: a close call of a router may go the other way for a token, so nine positions in ten."""
    if dtype == "float32":
        assert err.max() < 1e-4, err.max()
    else:
        assert np.quantile(err, 0.9) < 0.12, np.quantile(err, [0.5, 0.9, 1.0])
        assert np.median(err) < 0.05


@pytest.mark.parametrize("dtype,block", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64)])
@pytest.mark.parametrize("name", list(tc.CONFIGS))
def test_model(cases, name, dtype, block):
    c = cases(name)
    toks = gc.tokens(c.cfg, 150, 1)
    p = c.player(dtype, block=block)
    for sched in ([[("a", toks)]], [[("a", toks[:100])]] + [[("a", [t])] for t in toks[100:]],
                  [[("a", part)] for part in gc.portions(toks, [2, 15, 1, 33, 17, 16, 3])]):
        agree(c.error(gc.run(p, sched)["a"], toks, slice(None)), dtype)
    p.engine.exit()


@pytest.mark.parametrize("dtype,block,blocks", [("float32", 16, 18), ("bfloat16", 16, 18), ("bfloat16", 64, 8)])
@pytest.mark.parametrize("name", ["varied", "wide"])
def test_model_mixed_batches(cases, name, dtype, block, blocks):
    c = cases(name)
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 30 + i) for i, n in enumerate((1, 65, 50, 2, 100, 48, 130, 17))}
    p = c.player(dtype, block=block, blocks=blocks, slots=3)
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 1, 2, 3, 19, 40], live=3))
    agree(np.concatenate([c.error(got[n], t, slice(None)) for n, t in reqs.items()]), dtype)
    assert p.pool.num_free == blocks and len(p.pool.state_slots.free) == 3
    if dtype == "float32":                                # the same requests, each alone: nothing depends on the company
        for n, t in list(reqs.items())[:4]:
            alone = gc.run(p, [[(n, t)]])[n]
            assert np.abs(alone - got[n]).max() < 1e-3
    p.engine.exit()


def test_long_decoding(cases):
    """The window passes over decoded tokens alone several times."""
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
