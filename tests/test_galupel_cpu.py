"""Galupel on the PyTorch op set against the plain oracle: configuration, every mechanism, the model through the engine with portions,
batches, the edges of windows and blocks, pages used again, generation through ``LLM`` with its scheduler."""
import copy
import io
import json
import math
import warnings

import numpy as np
import pytest
import torch

import galupel_cases as lc
import goselix_cases as gc
import oracle_galupel as oracle
from tinyllmforge_b200 import LLM, SamplingParams
from tinyllmforge_b200.engine.request import Request
from tinyllmforge_b200.engine.step_batch import build_prefill
from tinyllmforge_b200.models import registry
from tinyllmforge_b200.models.galupel import GalupelForCausalLM
from tinyllmforge_b200.models.galupel_config import GalupelConfig, example_dict
from tinyllmforge_b200.ops.ref import RefOps, choose_experts
from tinyllmforge_b200.ops.ref_hybrid import pool_place

TOL = 6e-5


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = lc.Case(name, tmp_path_factory.mktemp(name), "cpu")
        return made[name]
    return get


def changed(d, path, value):
    """A copy of ``d`` with the entry at ``path`` replaced, or removed (value: None)."""
    d = copy.deepcopy(d)
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return d


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


ATT, LAT, ROUTER = ("layers", 0, "mixer"), ("layers", 1, "mixer"), ("layers", 0, "mlp", "router")         # of "varied"


# ------------------------------------------------------------------------------------------------ configuration and registry
def test_registry_chooses_by_architecture():
    cfg = registry.config_from_dict(lc.CONFIGS["varied"])
    assert isinstance(cfg, GalupelConfig) and registry.model_class(cfg) is GalupelForCausalLM
    assert cfg.prefix_cacheable and cfg.num_recurrent_runs == 0
    assert [getattr(l.mixer, "kv_from", None) for l in cfg.layers] == [None, None, 0, None, None, 0]
    example = GalupelConfig.from_dict(example_dict(1024))
    assert [getattr(l.mixer, "kv_from", None) for l in example.layers] == [None, None, None, 1]


def test_config_errors():
    d = lc.CONFIGS["varied"]
    for path, value in ((("layers", 0, "type"), "attention_2"), (ATT + ("kv_heads",), 4), (ATT + ("mask", "size"), 0), (ATT + ("mask", "pool"), 0), (ATT + ("dim",), 0),
                        (LAT + ("mask", "size"), 0), (LAT + ("rot", "dims"), 8), (LAT + ("rot_dim",), 15), (("norm", "groups"), 5), (("norm", "groups"), 0),
                        (("layers", 0, "mlp", "kind"), "dense"), (ROUTER + ("top",), 5), (ROUTER + ("groups", "count"), 3), (ROUTER + ("groups", "keep"), 5),
                        (ROUTER + ("top",), 0), (("logit_softcap",), 0.0), (("layers", 2, "mixer", "kv_from"), 1), (("layers", 2, "mixer", "kv_from"), 2),
                        (("layers", 5, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "heads"), 4), (("layers", 2, "mixer", "kv_from"), 5)):
        with pytest.raises(ValueError):
            GalupelConfig.from_dict(changed(d, path, value))
    for path in (("logit_scale",), ("norm", "groups"), ATT + ("scale",), ATT + ("mask",), LAT + ("rot", "base"), LAT + ("mask", "size"), ROUTER + ("groups",)):
        with pytest.raises(ValueError, match=path[-1]):
            GalupelConfig.from_dict(changed(d, path, None))
    with warnings.catch_warnings(record=True) as w:
        warnings.simplefilter("always")
        GalupelConfig.from_dict(changed(d, ATT + ("bias",), True))
    assert any("bias" in str(x.message) for x in w)


def test_unsupported_engine_options(cases):
    path = cases("short").path
    with pytest.raises(ValueError, match="one GPU"):
        LLM(path, device="cpu", tensor_parallel_size=2, kvcache_block_size=16)
    with pytest.raises(ValueError, match="quantization"):
        LLM(path, device="cpu", quantization="fp8_block", kvcache_block_size=16)


def test_checkpoint_errors(tmp_path, cases):
    c = cases("short")
    for change, match in ((lambda w: w.pop("l0.mlp.correction"), "l0.mlp.correction"), (lambda w: w.update({"l2.mix.k": w["l0.mix.k"].clone()}), "l2.mix.k"),
                          (lambda w: w.update(head=w["embed"].clone()), "head")):
        w = dict(c.weights)
        change(w)
        path = lc.write_model(tmp_path / match, c.cfg, w)
        with pytest.raises(KeyError, match=match):
            LLM(path, device="cpu", kvcache_block_size=16, skip_tokenizer_init=True)


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("groups", [1, 2, 5])
def test_grouped_norms(groups):
    x, a, w, u = rnd(7, 20, seed=1), 3.0 * rnd(7, 20, seed=2), rnd(20, seed=3), rnd(20, seed=4)
    a[:, :4] *= 100.0                                   # one group far larger than the others
    want = x.double() + oracle.grouped_rms(a.double(), w.double(), groups, 1e-3)
    got = x.clone()
    picked = RefOps.stream_update(got, torch.float32, 1e-3, [u], a=a, post=w, groups=groups, rows=torch.tensor([5, 0]))[0]
    assert torch.equal(got, x)
    assert (picked - oracle.grouped_rms(want, u.double(), groups, 1e-3)[[5, 0]]).abs().max() < 1e-5
    h = RefOps.stream_update(got, torch.float32, 1e-3, [None], a=a, post=w, groups=groups)[0]
    assert (got - want).abs().max() < 1e-5 and torch.equal(h, got)
    ids, table = torch.tensor([3, 0, 3], dtype=torch.int32), rnd(4, 20, seed=5)
    got = torch.full((3, 20), 9.0)
    RefOps.stream_update(got, torch.float32, 1e-3, [None], start=True, ids=ids, embed=table, post=w, groups=groups)
    assert (got - oracle.grouped_rms(table.double(), w.double(), groups, 1e-3)[ids.long()]).abs().max() < 1e-5


def test_norm_of_groups_by_hand():
    x = torch.tensor([[3.0, 4.0, 0.0, 0.0, 1.0, -1.0]]).double()
    got = oracle.grouped_rms(x, torch.tensor([1.0, 2.0, 1.0, 1.0, 1.0, 0.5]).double(), 3, 1e-30)
    r = math.sqrt(12.5)
    assert torch.allclose(got, torch.tensor([[3 / r, 8 / r, 0.0, 0.0, 1.0, -0.5]]).double())


@pytest.mark.parametrize("base,d", [(10000.0, 8), (300.0, 2), (2e5, 12)])
def test_rotation_of_neighbours(base, d):
    x = rnd(30, 2, d, seed=1).double()
    got = oracle.rotate_neighbours(x, base, 5)
    z = torch.view_as_complex(x.view(30, 2, d // 2, 2))
    angle = torch.arange(5, 35).double()[:, None, None] * torch.tensor([base ** (-2 * i / d) for i in range(d // 2)]).double()
    assert torch.allclose(got, torch.view_as_real(z * torch.exp(1j * angle)).reshape(x.shape), atol=1e-5)


def test_windows_and_blocks():
    """By the definition, token by token: a window's tokens, the blocks that end before it, nothing else."""
    for size in (1, 3, 8, 16, 17):
        for pool in (1, 2, 5, 8, 40):
            n = 50
            tokens, blocks = oracle.sliding(n, size), oracle.blocks_behind(n, size, pool)
            for i in range(n):
                assert [j for j in range(n) if tokens[i, j]] == [j for j in range(n) if 0 <= i - j < size]
                assert [b for b in range(n // pool) if blocks[i, b]] == [b for b in range(n // pool) if all(i - j >= size for j in range(b * pool, b * pool + pool))]


def test_places_of_blocks():
    """Every block has a place of its own in the page of its last token."""
    for page in (8, 16, 64):
        for pool in (1, 2, 3, 5, 7, 8, 13, 16, 19, 64, 100):
            blocks = torch.arange(1000)
            at, row = pool_place(blocks, pool, page)
            assert torch.equal(at, (blocks * pool + pool - 1) // page) and row.min() >= 0 and row.max() < -(-page // pool)
            assert len(set(zip(at.tolist(), row.tolist()))) == 1000


@pytest.mark.parametrize("size,pool", [(1, 1), (4, 2), (7, 3), (16, 8), (5, 11)])
def test_edges_of_windows_and_blocks(size, pool):
    """Every query points at one block's mean: the newest that it sees is found, the one after it is not."""
    n, d = 60, 64
    k, v = rnd(n, 1, d, seed=1).double(), rnd(n, 1, 5, seed=2).double()
    k = k / k.norm(dim=-1, keepdim=True)
    means = oracle.pooled(k, pool)
    for i in range(size, n):
        blocks = max(i - size + 1, 0) // pool              # visible
        for b in (blocks - 1, blocks):
            if not 0 <= b < n // pool:
                continue
            q = torch.zeros(n, 1, d).double()
            q[i] = 80.0 * means[b] / (means[b] ** 2).sum()
            got = oracle.pooled_window_attention(q, k, v, 1.0, size, pool)[i, 0]
            target = v[b * pool:(b + 1) * pool].mean(dim=0)[0]
            near = (k[max(i - size + 1, 0):i + 1, 0] @ q[i, 0]).max() > 60 or (pool > 1 and (means[:blocks, 0] @ q[i, 0] > 60).sum() > 1)
            if not near:
                assert ((got - target).norm() < 1e-3 * target.norm()) == (b < blocks), (i, b)


def test_choice_within_groups():
    """Groups are compared by their two best, corrections choose but do not weigh, negative sums beat experts of other groups."""
    s = torch.tensor([0.9, 0.1, 0.6, 0.5, 0.3, 0.2])
    none = torch.zeros(6)
    assert oracle.choose(s, none, 2, 3, 1) == [2, 3] and oracle.choose(s, none, 2, 1, 1) == [0, 2] and oracle.choose(s, none, 3, 3, 2) == [0, 2, 3]
    low = torch.tensor([-2.0, -2.0, -3.0, -3.0, -4.0, -4.0])
    assert oracle.choose(s, low, 2, 3, 1) == [0, 1] and oracle.choose(s, low, 4, 3, 2) == [0, 1, 2, 3]
    assert oracle.choose(s, torch.tensor([0.0, 0.0, 0.0, 0.0, 1.0, 1.0]), 2, 3, 1) == [4, 5]
    for count, keep, top in ((1, 1, 5), (2, 1, 4), (4, 2, 6), (6, 5, 3), (12, 4, 4)):
        scores, corr = torch.sigmoid(rnd(40, 12, seed=count)), 0.8 * rnd(12, seed=keep) - 0.9
        got = choose_experts(scores, corr, count, keep)[:, :top]
        assert got.tolist() == [oracle.choose(t, corr, top, count, keep) for t in scores]


@pytest.mark.parametrize("E,top,ff,count,keep", [(4, 2, 8, 2, 1), (6, 6, 5, 1, 1), (9, 2, 12, 3, 2), (4, 1, 3, 4, 4)])
def test_experts(E, top, ff, count, keep):
    h, router, corr = rnd(30, 16, seed=1), rnd(E, 16, seed=2), rnd(E, seed=3) - 1.0
    up, down = rnd(E, ff, 16, seed=4), rnd(E, 16, ff, seed=5)
    w = {"router": router.double(), "correction": corr.double()}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = up[e].double(), down[e].double()
    want = oracle.experts(h.double(), w, "", {"router": {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}})
    got = RefOps.moe(h, router, up, down, top, weigh="output", act="gelu", gated=False, correction=corr, groups=count, keep=keep)
    assert (got - want).abs().max() < 1e-4


def test_gelu_and_bounded_logits():
    z = torch.linspace(-6, 6, 101).double()
    assert torch.allclose(oracle.gelu(z), torch.tensor([0.5 * x * math.erfc(-x / math.sqrt(2)) for x in z.tolist()]).double())
    assert (RefOps.bound_logits(z.float() * 40, 0.3, 7.0) - 7 * torch.tanh(z * 12 / 7)).abs().max() < 1e-5


# ------------------------------------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("name", list(lc.CONFIGS))
def test_whole_prompt_and_token_by_token(cases, name):
    c = cases(name)
    toks = gc.tokens(c.cfg, 80, 1)
    p = c.player()
    whole = gc.run(p, [[("a", toks)]])["a"]
    assert c.error(whole, toks, slice(None)).max() < TOL
    single = gc.run(p, [[("b", [t])] for t in toks])["b"]
    assert c.error(single, toks, slice(None)).max() < TOL
    p.engine.exit()


@pytest.mark.parametrize("sizes", [[2], [3, 2], [16], [17, 15, 1], [5, 1, 1, 30]])
def test_portions(cases, sizes):
    for name in ("varied", "odd"):
        c = cases(name)
        toks = gc.tokens(c.cfg, 67, 2)
        p = c.player()
        got = gc.run(p, [[("a", part)] for part in gc.portions(toks, sizes)])["a"]
        assert c.error(got, toks, slice(None)).max() < TOL
        p.engine.exit()


@pytest.mark.parametrize("name", ["varied", "odd", "bare"])
def test_mixed_batches_reuse_blocks(cases, name):
    c = cases(name)
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 10 + i) for i, n in enumerate((1, 33, 50, 2, 16, 48, 65, 17))}
    p = c.player(blocks=10, slots=3)                      # far fewer than all requests together need
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 2, 3, 14], live=3))
    for r, toks in reqs.items():
        assert c.error(got[r], toks, slice(None)).max() < TOL, r
    p.pool.check_invariants()
    assert p.pool.num_free == 10 and p.pool.state_slots is None
    p.engine.exit()


def test_observed_residual_stream(cases):
    c = cases("varied")
    toks = gc.tokens(c.cfg, 20, 3)
    p = c.player()
    r = Request(toks)
    p.pool.extend(r)
    want, got = [], []
    oracle.forward(c.cfg, c.weights, toks, trace=want)
    with torch.inference_mode():
        w = p.engine.worker
        w.model.forward(w._stage(build_prefill([r], 16)), observe=lambda x: got.append(x.clone()))
    assert len(got) == len(want) == 6
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()
    p.engine.exit()


def test_borrowed_caches(cases):
    """A borrower has no keys and values of its own; means of blocks are shared where both layers have the same blocks."""
    p = cases("varied").player()
    m = p.engine.worker.model
    k, v, _, pool = m.memory[0]
    assert m.memory[2][0] is k and m.memory[5][1] is v
    assert m.memory[2][3].own and m.memory[2][3].k is not pool.k and m.memory[2][3].size == 5
    assert not m.memory[5][3].own and m.memory[5][3].k is pool.k
    assert m.layers[2].mix.bytes_per_token() == 0 and m.kv_block_bytes(16) > 16 * sum(l.mix.bytes_per_token() for l in m.layers)
    assert not any(n.startswith(("l2.mix.k", "l2.mix.v", "head")) for n, *_ in m.named_parameters())
    p.engine.exit()


def test_constants_reach_the_logits(cases):
    """A small change of each constant moves the logits by far more than the agreement above allows."""
    c = cases("varied")
    toks = gc.tokens(c.cfg, 60, 4)
    base = oracle.forward(c.cfg, c.weights, toks)
    third = ("layers", 2, "mixer")
    for path, value in ((("norm", "eps"), 1e-2), (("norm", "groups"), 2), (("logit_scale",), 0.71), (("logit_softcap",), 9.2), (ATT + ("mask", "size"), 19), (ATT + ("mask", "size"), 21),
                        (ATT + ("mask", "pool"), 3), (ATT + ("scale",), 0.31), (LAT + ("mask", "size"), 23), (LAT + ("mask", "size"), 25), (LAT + ("scale",), 0.26),
                        (LAT + ("rot", "base"), 9000.0), (third + ("mask", "size"), 32), (third + ("mask", "size"), 34), (third + ("mask", "pool"), 4),
                        (ROUTER + ("top",), 2), (ROUTER + ("groups", "keep"), 3), (ROUTER + ("groups", "count"), 2)):
        moved = (oracle.forward(changed(c.cfg, path, value), c.weights, toks) - base).pow(2).mean(-1).sqrt() / base.std()
        assert moved.max() > 10 * TOL, (path, moved.max())


def test_every_tensor_reaches_the_logits(cases):
    c = cases("varied")
    toks = gc.tokens(c.cfg, 40, 4)
    base = oracle.forward(c.cfg, c.weights, toks)
    for name, t in c.weights.items():
        if name == "l3.mlp.correction" or ".e" in name and ".mlp." in name:      # all are chosen there; a single expert may be chosen by nobody
            continue
        step = 0.05 if "correction" not in name else 0.4 * torch.arange(t.numel())
        moved = (oracle.forward(c.cfg, {**c.weights, name: t + step}, toks) - base).pow(2).mean(-1).sqrt() / base.std()
        assert moved.max() > 10 * TOL, name


# ------------------------------------------------------------------------------------------------ generation
def greedy(c, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(c.cfg, c.weights, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"extra": {"pipeline": False}}, {"chunked_prefill": True, "max_num_batched_tokens": 16}])
def test_greedy_generation(cases, kw):
    c = cases("short")
    prompts = [gc.tokens(c.cfg, n, 20 + n) for n in (1, 5, 16, 23, 40)]
    want = [greedy(c, p, 12) for p in prompts]
    base = dict(dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=32, max_model_len=96, max_num_batched_tokens=96,
                max_num_seqs=3, skip_tokenizer_init=True)
    llm = LLM(c.path, **{**base, **kw})
    for order in (1, -1):                                 # the second time on used blocks
        outs = llm.generate(prompts[::order], SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), use_tqdm=False)
        assert [o["token_ids"] for o in outs] == want[::order]
    llm.exit()


def test_generation_with_preemption(cases):
    c = cases("short")
    prompts = [gc.tokens(c.cfg, n, 40 + n) for n in (14, 15, 16)]
    want = [greedy(c, p, 24) for p in prompts]
    llm = LLM(c.path, dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=5, max_model_len=64, max_num_batched_tokens=64,
              max_num_seqs=3, skip_tokenizer_init=True)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True), use_tqdm=False)
    assert [o["token_ids"] for o in outs] == want
    assert llm.stats.to_dict()["preemptions"] > 0
    llm.exit()


@pytest.mark.parametrize("page", [8, 16])
def test_cached_prefixes(cases, page):
    """Cached pages bring the means of the blocks that end in them; a block that began in one of them and ends behind it is made anew."""
    c = cases("varied")
    shared = gc.tokens(c.cfg, 43, 50)
    prompts = [shared + gc.tokens(c.cfg, n, 60 + n) for n in (3, 9, 30)]
    want = [greedy(c, p, 10) for p in prompts]
    llm = LLM(c.path, dtype="float32", device="cpu", kvcache_block_size=page, num_kvcache_blocks=80, max_model_len=96, max_num_batched_tokens=96,
              max_num_seqs=2, skip_tokenizer_init=True)
    for p, w in zip(prompts, want):
        assert llm.generate([p], SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True), use_tqdm=False)[0]["token_ids"] == w
    assert llm.stats.to_dict()["prefix_cached_tokens"] == 2 * (43 // page * page)
    llm.exit()


def test_replay_program(cases, tmp_path):
    from tinyllmforge_b200.engine.replay import replay
    c = cases("odd")
    toks = gc.tokens(c.cfg, 30, 5)
    lines = [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [3, 19]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "x", "tokens": toks[20:21], "want": []}], "end": []}),
             json.dumps({"step": 2, "entries": [{"id": "x", "tokens": toks[21:], "want": [0]}], "end": ["x"]})]
    echo = io.StringIO()
    replay(c.path, str(tmp_path), 64, "float32", "cpu", lines=lines, echo=echo)
    assert echo.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    got = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)
    assert c.error(got, toks, [3, 19]).max() < TOL
    assert not (tmp_path / "1.f32").exists()
    assert c.error(np.fromfile(tmp_path / "2.f32", "<f4").reshape(1, -1), toks, [21]).max() < TOL
