"""Mezapel on the CUDA op set: every kernel against the plain oracle's mechanism, and whole models (fp32 and bf16) against the oracle with
prompts, portions, mixed batches, reused blocks and slots, long decoding, and generation with CUDA graphs."""
import numpy as np
import pytest
import torch

import goselix_cases as gc
import mezapel_cases as mc
import oracle_mezapel as oracle
from kernel_helpers import Batch, Spec, close, rnd

pytestmark = pytest.mark.gpu

F32, BF = torch.float32, torch.bfloat16


@pytest.fixture(scope="module")
def ops():
    from tinyllmforge_b200.ops.cuda import CudaOps
    return CudaOps()


# ------------------------------------------------------------------------------------------------ residual streams
@pytest.mark.parametrize("W", [64, 50, 2048, 2056, 4100])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_streams(ops, W, streams, dtype):
    T = 9
    x, y = rnd(T, streams, W, seed=1) + 2.0, rnd(T, W, seed=2, dtype=dtype)            # a mean that is not zero
    into, out, mix = rnd(streams, seed=3), rnd(streams, seed=4), rnd(streams, streams, seed=5)
    w, b = rnd(W, seed=6, dtype=dtype), rnd(W, seed=7, dtype=dtype)
    xs = oracle.spread_streams([x[:, s].double() for s in range(streams)], y.double(), mix.double(), out.double())
    want = oracle.layer_norm(oracle.gather_streams(xs, into.double()), w.double(), b.double(), 1e-3)
    dev = dict(y=y.cuda(), mix=mix.cuda(), out=out.cuda())
    args = (dtype, 1e-3, into.cuda(), w.cuda(), b.cuda())
    tol = 2e-5 if dtype == F32 else 6e-3
    xc = x.cuda()
    only = ops.stream_mix(xc, *args, rows=torch.tensor([7, 0, 7], dtype=torch.int32, device="cuda"), **dev)
    assert torch.equal(xc.cpu(), x)                                  # x is left alone when rows are picked
    close(only, want[[7, 0, 7]], tol)
    h = ops.stream_mix(xc, *args, **dev)
    close(xc, torch.stack(xs, 1), 3e-6)
    close(h, want, tol)
    xc = x.cuda()
    assert ops.stream_mix(xc, dtype, 1e-3, into.cuda(), None, None, **dev) is None
    close(xc, torch.stack(xs, 1), 3e-6)


@pytest.mark.parametrize("W,streams", [(64, 2), (50, 3), (4096, 4), (256, 6)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_pair_embedding(ops, W, streams, dtype):
    V, T = 20000, 40
    g = torch.Generator().manual_seed(1)
    embed, w, b, into = rnd(V, W, seed=1, dtype=dtype), rnd(W, seed=3, dtype=dtype), rnd(W, seed=4, dtype=dtype), rnd(streams, seed=5)
    toks = torch.randint(0, V, (T,), generator=g).tolist()
    toks[5] = toks[4] = V - 1
    prev = torch.tensor([-1] + toks[:-1], dtype=torch.int32)
    for buckets, mul_prev, mul_cur in ((1, 3, 5), (977, 1000003, 999983), (64, 0, 1)):     # products beyond 32 bits
        pairs = rnd(buckets + 1, W, seed=2, dtype=dtype)
        want = oracle.embedding(toks, {"embed": embed.double(), "bigram": pairs.double()},
                                {"scale": 1.7, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}})
        x = torch.full((T, streams, W), 9.0, device="cuda")
        h = ops.stream_mix(x, dtype, 1e-5, into.cuda(), w.cuda(), b.cuda(), ids=torch.tensor(toks, dtype=torch.int32, device="cuda"), prev=prev.cuda(),
                           embed=embed.cuda(), scale=1.7, pairs=pairs.cuda(), mul_prev=mul_prev, mul_cur=mul_cur)
        close(x, want[:, None].expand(T, streams, W), 1e-6)
        close(h, oracle.layer_norm(want * into.double().sum(), w.double(), b.double(), 1e-5), 2e-5 if dtype == F32 else 6e-3)


# ------------------------------------------------------------------------------------------------ attention
ATTENTION = {
    "real": Spec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, window=100),
    "values": Spec(heads=6, kv_heads=2, dim=64, vdim=256, scale=0.1, window=64),
    "deep": Spec(heads=4, kv_heads=4, dim=256, vdim=256, scale=0.06, window=65),
    "groups": Spec(heads=40, kv_heads=2, dim=40, vdim=72, scale=0.2, window=63),
    "one": Spec(heads=3, kv_heads=3, dim=24, vdim=40, scale=0.2, window=1),
    "long": Spec(heads=8, kv_heads=1, dim=96, vdim=192, scale=0.1, window=5000),
    "odd": Spec(heads=5, kv_heads=1, dim=9, vdim=7, scale=0.3, window=17),
}
OPTIONS = {                       # chunked, softcap, sink, gate
    "chunks": (True, 0.0, "zero", "head"),
    "capped": (False, 5.0, "learned", "element"),
    "all": (True, 3.0, "learned", "head"),
    "bare": (True, 0.0, None, None),
}


def attention_case(ops, s, options, ranges, block, dtype, seed=0, decode=False, pad=0, needle=None, sharp=1.0):
    """Random keys and values of whole sequences in shuffled blocks, queries for the ranges; what the oracle gives for the ranges.
    ``needle(position) -> key``: the query of that position points at that key."""
    chunked, cap, sink, gate = options
    b = Batch(ranges, block, decode=decode, pad=pad, seed=seed)
    H, G, d, dv, T = s.heads, s.kv_heads, s.dim, s.vdim, sum(hi - lo for lo, hi in ranges)
    kc, vc = (torch.full((b.num_blocks, G, block, n), 7.0, dtype=dtype, device="cuda") for n in (d, dv))
    cols = ops.C.windowed_prefill_qcols(d, dv, block) if dtype == BF else 0
    q_all = torch.zeros(T + pad, H, cols or d, dtype=dtype)
    sinks = None if sink is None else torch.zeros(H) if sink == "zero" else 1.0 + rnd(H, seed=seed + 1)
    gates = None if gate is None else rnd(T + pad, (H if gate == "head" else H * dv) + 8, seed=seed + 2, dtype=dtype)
    wants, at = [], 0
    for i, (lo, hi) in enumerate(ranges):
        k, v = rnd(hi, G, d, seed=100 * seed + i + 5, dtype=dtype), rnd(hi, G, dv, seed=100 * seed + i + 6, dtype=dtype)
        q = rnd(hi, H, d, seed=100 * seed + i + 7, scale=sharp)
        if needle is not None:
            for n in range(lo, hi):
                t = k[needle(n)].float().repeat_interleave(H // G, 0)
                q[n] = 12 / s.scale * t / (t * t).sum(-1, keepdim=True)
        q = q.to(dtype)
        slots = [int(b.tables[i][p // block]) * block + p % block for p in range(hi)]
        slots = torch.tensor(slots, device="cuda")
        kc[slots // block, :, slots % block], vc[slots // block, :, slots % block] = k.cuda(), v.cuda()
        visible = (oracle.chunked if chunked else oracle.sliding)(hi, s.window)
        none = torch.full((H,), -1e9).double()
        o = oracle.sink_attention(q.double(), k.double(), v.double(), s.scale, visible, none if sinks is None else sinks.double(), cap or None)[lo:]
        n = hi - lo
        if gate is not None:
            o = o * oracle.sigmoid(gates[at:at + n, :H if gate == "head" else H * dv].double()).view(n, H, -1)
        wants.append(0.8 * o.reshape(n, -1))
        q_all[at:at + n, :, :d] = q[lo:]
        at += n
    out = torch.full((T + pad, H * dv + 8), 3.0, dtype=dtype, device="cuda")
    gv = None if gate is None else gates.cuda()[:, :H if gate == "head" else H * dv]
    ops.windowed_attention(q_all.cuda(), kc, vc, b, s, out[:, :H * dv], 0.8, chunked=chunked, softcap=cap, sink=None if sinks is None else sinks.cuda(), gate=gv)
    ops.check_status()
    assert (out[:, H * dv:] == 3.0).all()
    return out[:T, :H * dv], torch.cat(wants)


@pytest.mark.parametrize("dtype,block", [(F32, 16), (BF, 16), (BF, 64), (BF, 256)])
@pytest.mark.parametrize("options", list(OPTIONS))
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_prompts(ops, name, options, dtype, block):
    ranges = [(0, 130), (0, 2), (60, 64), (127, 300), (5, 69), (400, 529), (64, 65)]
    if dtype == F32:
        ranges = [(0, 70), (30, 33), (15, 18), (64, 65)]
    got, want = attention_case(ops, ATTENTION[name], OPTIONS[options], ranges, block, dtype, seed=1)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype,block", [(F32, 16), (BF, 16), (BF, 64)])
@pytest.mark.parametrize("options", list(OPTIONS))
@pytest.mark.parametrize("name", list(ATTENTION))
def test_attention_decode(ops, name, options, dtype, block):
    lens = (1, 2, 63, 64, 65, 66, 100, 101, 127, 128, 129, 256, 400, 17)
    got, want = attention_case(ops, ATTENTION[name], OPTIONS[options], [(n - 1, n) for n in lens], block, dtype, seed=2, decode=True, pad=3)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)
    got, want = attention_case(ops, ATTENTION[name], OPTIONS[options], [(n - 1, n) for n in (900, 3)], block, dtype, seed=3, decode=True)
    close(got, want, 1e-5 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("name", ["real", "values", "groups", "deep", "odd"])
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("out", [0, 1, 2])
def test_attention_edges(ops, name, decode, chunked, out):
    """Every query points at one key: the oldest of its window or chunk (0), the one before it, which must not be seen (1), or keys at
    the borders of blocks and tiles and its own (2)."""
    s = ATTENTION[name]
    near = [0, 15, 16, 63, 64, 127, 128, 255, 256]
    oldest = (lambda p: p // s.window * s.window) if chunked else (lambda p: max(p - s.window + 1, 0))
    if out < 2:
        needle = lambda p: max(oldest(p) - out, 0)
    else:
        needle = lambda p: max((t for t in near if oldest(p) <= t <= p), default=p)
    ranges = [(n - 1, n) for n in (301, 302, 303, 65, 64, 63, 17, 128, 129, 130, 100, 101, 66, 127)] if decode else [(0, 313), (280, 320), (130, 132)]
    for cap in (0.0, 20.0):
        got, want = attention_case(ops, s, (chunked, cap, "zero", None), ranges, 64, BF, seed=4, decode=decode, needle=needle)
        close(got, want, 2e-2)


@pytest.mark.parametrize("decode", [False, True])
def test_scores_beyond_the_bound(ops, decode):
    """Scores far larger and far smaller than the bound, and tiles in which only a few are: the exact form beside the polynomial one."""
    s = Spec(**{**ATTENTION["real"].__dict__, "window": 150})
    ranges = [(n - 1, n) for n in (200, 77, 300)] if decode else [(0, 200), (60, 300)]
    for sharp in (0.05, 0.8, 1.5, 30.0):
        got, want = attention_case(ops, s, (False, 2.0, "learned", "element"), ranges, 64, BF, seed=5, decode=decode, sharp=sharp)
        close(got, want, 8e-3)
    got, want = attention_case(ops, s, (False, 2.0, "learned", None), ranges, 64, F32, seed=5, decode=decode, sharp=3.0)
    close(got, want, 1e-5)


def test_sinks_far_above_and_below_the_scores(ops):
    for ranges, decode in (([(0, 100), (90, 200)], False), ([(99, 100), (0, 1), (299, 300)], True)):
        for dtype in (BF, F32):
            for level in (-200.0, 30.0):
                s = ATTENTION["real"]
                b = Batch(ranges, 64, decode=decode, seed=8)
                T = sum(hi - lo for lo, hi in ranges)
                kc, vc = (rnd(b.num_blocks, s.kv_heads, 64, n, seed=n, dtype=dtype).cuda() for n in (s.dim, s.vdim))
                q, outs = rnd(T, s.heads, s.dim, seed=3, dtype=dtype).cuda(), []
                for sink in (None, torch.full((s.heads,), level, device="cuda")):
                    outs.append(torch.zeros(T, s.heads * s.vdim, dtype=dtype, device="cuda"))
                    ops.windowed_attention(q, kc, vc, b, s, outs[-1], 1.0, sink=sink)
                ops.check_status()
                if level < 0:
                    close(outs[1], outs[0], 1e-6)
                else:
                    assert torch.isfinite(outs[1]).all() and outs[1].abs().max() < 1e-6


# ------------------------------------------------------------------------------------------------ ahead of the attention
NORM_ROPE = {
    "real": (Spec(heads=16, kv_heads=4, dim=128, vdim=128), 128),
    "partial": (Spec(heads=6, kv_heads=2, dim=64, vdim=48), 16),
    "passing": (Spec(heads=3, kv_heads=1, dim=48, vdim=40), 0),
    "padded": (Spec(heads=40, kv_heads=2, dim=40, vdim=72), 24),
    "many": (Spec(heads=72, kv_heads=8, dim=256, vdim=32), 64),
    "odd": (Spec(heads=5, kv_heads=1, dim=9, vdim=7), 6),
    "wide": (Spec(heads=4, kv_heads=4, dim=100, vdim=20), 50),
}


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("norm", ["head", "all"])
@pytest.mark.parametrize("tokens", [9, 2100])
@pytest.mark.parametrize("name", list(NORM_ROPE))
def test_norm_rope_store(ops, name, tokens, norm, dtype):
    from tinyllmforge_b200.ops.ref import rotation_table
    base, rd = NORM_ROPE[name]
    s = Spec(**base.__dict__, norm=norm)
    H, G, d, dv = s.heads, s.kv_heads, s.dim, s.vdim
    ranges = [(0, 5), (14, 18)] if tokens == 9 else [(3, 1103), (0, 1000)]
    b = Batch(ranges, 64, seed=6, pad=2)
    rows = (H + G) * d + G * dv
    proj = rnd(tokens + 2, rows + 8, seed=1, dtype=dtype)
    qw, kw = (1.0 + 0.3 * rnd(d if norm == "head" else n * d, seed=n) for n in (H, G))
    qw, kw = qw.to(dtype), kw.to(dtype)
    f = [10.0 ** (-2.0 * i / max(rd, 1)) for i in range(rd // 2)]
    kc, vc = (torch.zeros(b.num_blocks, G, 64, n, dtype=dtype, device="cuda") for n in (d, dv))
    q = ops.norm_rope_store(proj.cuda()[:, :rows], qw.cuda(), kw.cuda(), 1e-3, s, rotation_table(1200, f, 1.3, "cuda"), b.positions, b.slot_mapping, kc, vc)
    ops.check_status()
    x = proj[:tokens, :rows].double()

    def normed(m, w, heads):
        m = oracle.unit_rms(m.reshape(tokens, heads, d) if norm == "head" else m, 1e-3) * w.double()
        m, n0 = m.reshape(tokens, heads, d), ranges[0][1] - ranges[0][0]
        return torch.cat([oracle.rotate(m[:n0], f, 1.3, ranges[0][0]), oracle.rotate(m[n0:], f, 1.3, ranges[1][0])])

    tol = 5e-6 if dtype == F32 else 6e-3
    close(q[:tokens, :, :d], normed(x[:, :H * d], qw, H), tol)
    assert not q[:, :, d:].any()
    at = b.slot_mapping[:tokens].long()
    close(kc[at // 64, :, at % 64], normed(x[:, H * d:(H + G) * d], kw, G), tol)
    close(vc[at // 64, :, at % 64], x[:, (H + G) * d:].reshape(tokens, G, dv), tol)
    assert int((kc.abs().sum((1, 3)) > 0).sum()) == tokens and int((vc.abs().sum((1, 3)) > 0).sum()) == tokens


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("C,taps", [(64, 4), (50, 2), (7, 5), (36, 1), (200, 9), (24, 32)])
def test_plain_short_conv(ops, dtype, C, taps):
    """Without an activation; more taps than fit the usual instances; with one tap no slot is needed."""
    ranges = [(9, 10), (0, 1), (1, 2), (0, 100), (3, 5), (33, 97), (0, 2), (40, 73)]
    slots = [-1] * 8 if taps == 1 else [4, 0, 9, 2, 7, 1, 8, 6]
    b = Batch(ranges, 64, slots=slots, seed=1)
    w = rnd(C, taps, seed=2)
    left = rnd(0 if taps == 1 else 11, taps - 1, C, seed=4, dtype=dtype)
    xs, wants = [], []
    for i, (lo, hi) in enumerate(ranges):
        x = rnd(hi, C, seed=20 + i, dtype=dtype)
        if lo > 0 and taps > 1:
            tail = torch.zeros(taps - 1, C, dtype=dtype)
            n = min(lo, taps - 1)
            tail[taps - 1 - n:] = x[lo - n:lo]
            left[slots[i]] = tail
        wants.append(oracle.causal_conv(x.double(), w.double())[lo:])
        xs.append(x[lo:])
    st = left.clone().cuda()
    out = ops.short_conv(torch.cat(xs).cuda(), w.cuda(), None, st, b, act="none")
    ops.check_status()
    close(out, torch.cat(wants), 3e-6 if dtype == F32 else 6e-3)
    for i, (lo, hi) in enumerate(ranges):
        if taps > 1:
            full = torch.cat([torch.zeros(taps - 1, C, dtype=dtype), rnd(hi, C, seed=20 + i, dtype=dtype)])
            assert torch.equal(st[slots[i]].cpu(), full[hi:])


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = mc.Case(name, tmp_path_factory.mktemp(name), "cuda")
        return made[name]
    return get


def agree(err, dtype):
    assert err.max() < (1e-4 if dtype == "float32" else 0.15) and np.median(err) < (1e-4 if dtype == "float32" else 0.05), np.quantile(err, [0.5, 0.9, 1.0])


@pytest.mark.parametrize("dtype,block", [("float32", 16), ("bfloat16", 16), ("bfloat16", 64)])
@pytest.mark.parametrize("name", list(mc.CONFIGS))
def test_model(cases, name, dtype, block):
    c = cases(name)
    toks = gc.tokens(c.cfg, 150, 1)
    p = c.player(dtype, block=block)
    for sched in ([[("a", toks)]], [[("a", toks[:100])]] + [[("a", [t])] for t in toks[100:]],
                  [[("a", part)] for part in gc.portions(toks, [2, 15, 1, 33, 17, 16, 3])]):
        agree(c.error(gc.run(p, sched)["a"], toks, slice(None)), dtype)
    p.engine.exit()


@pytest.mark.parametrize("dtype,block,blocks", [("float32", 16, 18), ("bfloat16", 16, 18), ("bfloat16", 64, 8)])
@pytest.mark.parametrize("name", ["varied", "wide", "chunks"])
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
    """Windows and chunks pass over decoded tokens alone several times."""
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
