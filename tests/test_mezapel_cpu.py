"""Mezapel on the PyTorch op set against the plain oracle: configuration, every mechanism, the model through the engine with portions,
batches, window and chunk edges, blocks and state slots used again, generation through ``LLM`` with its scheduler."""
import copy
import io
import json
import math
import warnings

import numpy as np
import pytest
import torch

import goselix_cases as gc
import mezapel_cases as mc
import oracle_mezapel as oracle
from tinyllmforge_b200 import LLM, SamplingParams
from tinyllmforge_b200.engine.request import Request
from tinyllmforge_b200.engine.step_batch import DecodeBuilder, build_decode, build_prefill
from tinyllmforge_b200.models import registry
from tinyllmforge_b200.models.mezapel import MezapelForCausalLM
from tinyllmforge_b200.models.mezapel_config import MezapelConfig, example_dict
from tinyllmforge_b200.models.specs import BandScaling, RampScaling, Rotation
from tinyllmforge_b200.ops.ref import RefOps, rotation_table

TOL = 6e-5


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = mc.Case(name, tmp_path_factory.mktemp(name), "cpu")
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


FIRST, SECOND = ("layers", 1, "mixer"), ("layers", 0, "mixer")         # of "varied": chunks, window


# ------------------------------------------------------------------------------------------------ configuration and registry
def test_registry_chooses_by_architecture():
    cfg = registry.config_from_dict(mc.CONFIGS["varied"])
    assert isinstance(cfg, MezapelConfig) and registry.model_class(cfg) is MezapelForCausalLM
    assert [i for i, _ in cfg.layer_runs()] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert cfg.num_recurrent_runs == 4 and not cfg.prefix_cacheable
    only_chunks = registry.config_from_dict(mc.CONFIGS["chunks"])
    assert only_chunks.num_recurrent_runs == 0 and only_chunks.prefix_cacheable
    assert len(MezapelConfig.from_dict(example_dict(1024)).layers) == 4


def test_config_errors():
    d = mc.CONFIGS["varied"]
    for path, value in ((("layers", 0, "type"), "attention_3"), (FIRST + ("kv_heads",), 3), (FIRST + ("rot", "dims"), 18), (FIRST + ("rot", "dims"), 5),
                        (FIRST + ("mask", "size"), 0), (SECOND + ("conv",), 0), (SECOND + ("softcap",), 0.0), (SECOND + ("vdim",), 0), (("streams",), 0),
                        (("streams",), 17), (("loop", "stop"), 9), (("layers", 0, "mlp", "kind"), "moe"), (("embedding", "bigram", "buckets"), 0)):
        with pytest.raises(ValueError):
            MezapelConfig.from_dict(changed(d, path, value))
    for path in (("streams",), ("embedding", "scale"), ("embedding", "bigram", "mul_prev"), FIRST + ("scale",), SECOND + ("softcap",),
                 FIRST + ("rot", "scaling", "fast"), SECOND + ("rot", "scaling", "low")):
        with pytest.raises(ValueError, match=path[-1]):
            MezapelConfig.from_dict(changed(d, path, None))
    with warnings.catch_warnings(record=True) as w:
        warnings.simplefilter("always")
        MezapelConfig.from_dict(changed(d, FIRST + ("bias",), True))
    assert any("bias" in str(x.message) for x in w)


def test_unsupported_engine_options(cases):
    path = cases("short").path
    with pytest.raises(ValueError, match="one GPU"):
        LLM(path, device="cpu", tensor_parallel_size=2, kvcache_block_size=16)
    with pytest.raises(ValueError, match="quantization"):
        LLM(path, device="cpu", quantization="fp8_block", kvcache_block_size=16)


def test_checkpoint_errors(tmp_path, cases):
    c = cases("short")
    for change, match in ((lambda w: w.pop("l0.hc2.mix"), "l0.hc2.mix"), (lambda w: w.update(extra=torch.zeros(3)), "extra")):
        w = dict(c.weights)
        change(w)
        path = mc.write_model(tmp_path / match, c.cfg, w)
        with pytest.raises(KeyError, match=match):
            LLM(path, device="cpu", kvcache_block_size=16, skip_tokenizer_init=True)


# ------------------------------------------------------------------------------------------------ mechanisms
def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


@pytest.mark.parametrize("base,dims,factor,original,fast,slow", [(10000.0, 16, 4.0, 64, 4.0, 0.25), (3e4, 32, 6.0, 300, 24.0, 1.5), (100.0, 8, 2.0, 4096, 1000.0, 999.0),
                                                                (1e4, 2, 16.0, 128, 8.0, 1.0), (1e4, 64, 1.0, 256, 16.0, 2.0), (50.0, 12, 3.0, 8, 100.0, 50.0)])
def test_ramped_frequencies(base, dims, factor, original, fast, slow):
    c = dict(factor=factor, original=original, fast=fast, slow=slow)
    rot = Rotation.from_dict({"base": base, "dims": dims, "scaling": c}, RampScaling)
    want = oracle.yarn_frequencies(base, dims, c)
    assert np.allclose(rot.frequencies, want, rtol=1e-13) and math.isclose(rot.amplitude, oracle.yarn_amplitude(c))
    plain = oracle.plain_frequencies(base, dims)
    assert all(p / factor * (1 - 1e-12) <= f <= p * (1 + 1e-12) for f, p in zip(want, plain))
    turns = [original * p / (2 * math.pi) for p in plain]              # within the original length
    spacing = base ** (2.0 / dims)                                     # of neighbouring pairs' turns
    for f, p, t in zip(want, plain, turns):
        if t > fast * spacing * 1.001 and fast > slow * spacing:
            assert math.isclose(f, p)
    table = rotation_table(40, rot.frequencies, rot.amplitude)
    x = rnd(40, 2, dims + 3, seed=1)
    from tinyllmforge_b200.ops.ref import apply_partial_rope
    got = apply_partial_rope(x, torch.arange(40), table)
    assert (got - oracle.rotate(x.double(), want, oracle.yarn_amplitude(c))).abs().max() < 1e-5


@pytest.mark.parametrize("base,dims,factor,original,low,high", [(10000.0, 16, 4.0, 64, 1.0, 4.0), (2e5, 40, 5.0, 700, 2.0, 6.0), (500.0, 6, 2.0, 32, 0.5, 8.0)])
def test_banded_frequencies(base, dims, factor, original, low, high):
    c = dict(factor=factor, original=original, low=low, high=high)
    rot = Rotation.from_dict({"base": base, "dims": dims, "scaling": c}, BandScaling)
    want = oracle.banded_frequencies(base, dims, c)
    assert np.allclose(rot.frequencies, want, rtol=1e-13) and rot.amplitude == 1.0
    kinds = set()
    for f, p in zip(want, oracle.plain_frequencies(base, dims)):
        turns = original * p / (2 * math.pi)
        kinds.add("kept" if turns > high else "stretched" if turns < low else "blended")
        assert math.isclose(f, p if turns > high else p / factor) if not low <= turns <= high else p / factor <= f <= p
    assert len(kinds) >= 2


def test_pair_rows_and_embedding():
    assert oracle.bigram_rows([4, 9, 9, 0], 7, 5, 3) == [7, (4 * 5 + 9 * 3) % 7, (9 * 5 + 9 * 3) % 7, 45 % 7]
    toks = torch.tensor([4, 9, 9, 0, 11, 2])
    w = {"embed": rnd(12, 10, seed=1), "bigram": rnd(8, 10, seed=2)}
    want = oracle.embedding(toks.tolist(), w, {"scale": 2.5, "bigram": {"buckets": 7, "mul_prev": 5, "mul_cur": 3}})
    x = torch.empty(6, 3, 10)
    prev = torch.cat([torch.tensor([-1]), toks[:-1]]).int()
    h = RefOps.stream_mix(x, torch.float32, 1e-4, torch.tensor([0.5, 1.0, -0.2]), torch.ones(10), torch.zeros(10), ids=toks.int(), prev=prev,
                          embed=w["embed"], scale=2.5, pairs=w["bigram"], mul_prev=5, mul_cur=3)
    assert (x - want[:, None]).abs().max() < 1e-6
    assert (h - oracle.layer_norm(1.3 * want, 1.0, 0.0, 1e-4)).abs().max() < 1e-5


@pytest.mark.parametrize("streams", [1, 2, 5])
def test_streams(streams):
    x, y = rnd(9, streams, 20, seed=1), rnd(9, 20, seed=2)
    into, out, mix, w, b = rnd(streams, seed=3), rnd(streams, seed=4), rnd(streams, streams, seed=5), rnd(20, seed=6), rnd(20, seed=7)
    xs = oracle.spread_streams([x[:, s].double() for s in range(streams)], y.double(), mix.double(), out.double())
    want = oracle.layer_norm(oracle.gather_streams(xs, into.double()), w.double(), b.double(), 1e-3)
    got = x.clone()
    rows = RefOps.stream_mix(got, torch.float32, 1e-3, into, w, b, y=y, mix=mix, out=out, rows=torch.tensor([7, 0]))
    assert torch.equal(got, x) and (rows - want[[7, 0]]).abs().max() < 1e-5
    h = RefOps.stream_mix(got, torch.float32, 1e-3, into, w, b, y=y, mix=mix, out=out)
    assert (got - torch.stack(xs, 1)).abs().max() < 1e-5 and (h - want).abs().max() < 1e-5


@pytest.mark.parametrize("mask", ["sliding", "chunked"])
@pytest.mark.parametrize("size", [1, 3, 16, 17])
def test_edges_of_the_masks(mask, size):
    """Every query points at one key: the oldest that its window or chunk holds is found, the one before it is not."""
    n, d = 50, 24
    k, v = rnd(n, 1, d, seed=1).double(), rnd(n, 1, 5, seed=2).double()
    visible = getattr(oracle, mask)(n, size)
    oldest = [i // size * size if mask == "chunked" else max(i - size + 1, 0) for i in range(n)]
    assert [int(visible[i].nonzero()[0]) for i in range(n)] == oldest and all(visible[i, oldest[i]:i + 1].all() and not visible[i, i + 1:].any() for i in range(n))
    for before in (0, 1):
        at = [max(o - before, 0) for o in oldest]
        q = torch.stack([60.0 * k[a] / k[a].norm() ** 2 for a in at])
        got = oracle.sink_attention(q, k, v, 1.0, visible, torch.zeros(1).double())
        for i in range(n):
            if (k[oldest[i]:i + 1, 0] @ k[at[i], 0] / k[at[i]].norm() ** 2 > 0.7).sum() == (at[i] >= oldest[i]):         # nothing else comes near
                assert ((got[i, 0] - v[at[i], 0]).norm() < 1e-2 * v[at[i], 0].norm()) == (at[i] >= oldest[i]), (size, i)


def test_sinks_and_capped_scores():
    q, k, v = (rnd(9, 2, 6, seed=s).double() for s in (1, 2, 3))
    visible, sink = oracle.sliding(9, 4), torch.tensor([0.5, -30.0]).double()
    got = oracle.sink_attention(q, k, v, 0.7, visible, sink, 1.5)
    for i in range(9):
        for h in range(2):
            js = [j for j in range(9) if 0 <= i - j < 4]
            e = [math.exp(1.5 * math.tanh(0.7 * float(q[i, h] @ k[j, h]) / 1.5)) for j in js]
            want = sum(x * v[j, h] for x, j in zip(e, js)) / (sum(e) + math.exp(float(sink[h])))
            assert (got[i, h] - want).abs().max() < 1e-12


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_causal_convolution_of_the_oracle(taps):
    x, w = rnd(12, 3, seed=1).double(), rnd(3, taps, seed=2).double()
    y = oracle.causal_conv(x, w)
    for t in range(12):
        want = sum(w[:, taps - 1 - back] * x[t - back] for back in range(taps) if t >= back)
        assert torch.allclose(y[t], want)


# ------------------------------------------------------------------------------------------------ step buffer
def test_previous_tokens_in_the_step_buffer():
    reqs = [Request([5, 6, 7, 8]), Request([9]), Request([1, 2, 3])]
    for i, (r, start) in enumerate(zip(reqs, (2, 0, 0))):
        r.block_table, r.num_computed_tokens, r.prefill_end = [i], start, len(r)
    sb = build_prefill(reqs, 16)
    assert sb.prev_ids.tolist() == [6, 7, -1, -1, 1, 2]
    assert build_decode(reqs, 16, pad_to=5).prev_ids.tolist() == [7, -1, 2, -1, -1]
    b = DecodeBuilder(16)
    b.build(reqs, 0, 0, None, None)
    for r in reqs:
        r.append_token(40 + len(r))
    assert b.build(reqs, 1, 0, None, None).prev_ids.tolist() == [8, 9, 3]


# ------------------------------------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("name", list(mc.CONFIGS))
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
    c = cases("varied")
    toks = gc.tokens(c.cfg, 67, 2)
    p = c.player()
    got = gc.run(p, [[("a", part)] for part in gc.portions(toks, sizes)])["a"]
    assert c.error(got, toks, slice(None)).max() < TOL
    p.engine.exit()


@pytest.mark.parametrize("name", ["varied", "odd", "chunks"])
def test_mixed_batches_reuse_blocks_and_slots(cases, name):
    c = cases(name)
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 10 + i) for i, n in enumerate((1, 33, 50, 2, 16, 48, 65, 17))}
    p = c.player(blocks=10, slots=3)                      # far fewer than all requests together need
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 2, 3, 14], live=3))
    for r, toks in reqs.items():
        assert c.error(got[r], toks, slice(None)).max() < TOL, r
    p.pool.check_invariants()
    assert p.pool.num_free == 10 and (p.pool.state_slots is None) == (name == "chunks")
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
    assert len(got) == len(want) == 8
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()
    p.engine.exit()


def test_constants_reach_the_logits(cases):
    """A small change of each constant moves the logits by far more than the agreement above allows."""
    c = cases("varied")
    toks = gc.tokens(c.cfg, 60, 4)
    base = oracle.forward(c.cfg, c.weights, toks)
    rot1, rot2 = FIRST + ("rot",), SECOND + ("rot",)
    for path, value in ((("norm", "eps"), 1e-2), (("embedding", "scale"), 3.1), (("embedding", "bigram", "mul_prev"), 6), (("embedding", "bigram", "mul_cur"), 4),
                        (("loop", "times"), 2), (FIRST + ("mask", "size"), 23), (FIRST + ("mask", "size"), 25), (FIRST + ("scale",), 0.26), (rot1 + ("base",), 9000.0),
                        (rot1 + ("dims",), 6), (rot1 + ("scaling", "factor"), 3.9), (rot1 + ("scaling", "original"), 1000), (rot1 + ("scaling", "fast"), 1.0),
                        (rot1 + ("scaling", "slow"), 2.0), (SECOND + ("mask", "size"), 19), (SECOND + ("mask", "size"), 21), (SECOND + ("scale",), 0.21),
                        (SECOND + ("softcap",), 5.5), (rot2 + ("base",), 9000.0), (rot2 + ("scaling", "factor"), 3.5), (rot2 + ("scaling", "original"), 70),
                        (rot2 + ("scaling", "low"), 0.5), (rot2 + ("scaling", "high"), 5.0)):
        moved = (oracle.forward(changed(c.cfg, path, value), c.weights, toks) - base).pow(2).mean(-1).sqrt() / base.std()
        assert moved.max() > 10 * TOL, (path, moved.max())


def test_every_tensor_reaches_the_logits(cases):
    c = cases("varied")
    toks = gc.tokens(c.cfg, 40, 4)
    base = oracle.forward(c.cfg, c.weights, toks)
    for name, t in c.weights.items():
        if name == "l0.hc1.in":                           # all streams are equal there, and the norm takes their common factor out
            continue
        moved = (oracle.forward(c.cfg, {**c.weights, name: t + 0.05}, toks) - base).pow(2).mean(-1).sqrt() / base.std()
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
    for order in (1, -1):                                 # the second time on used blocks and slots
        outs = llm.generate(prompts[::order], SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), use_tqdm=False)
        assert [o["token_ids"] for o in outs] == want[::order]
    assert llm.stats.to_dict()["prefix_cached_tokens"] == 0
    llm.exit()


def test_generation_with_preemption(cases):
    c = cases("short")
    prompts = [gc.tokens(c.cfg, n, 40 + n) for n in (14, 15, 16)]
    want = [greedy(c, p, 24) for p in prompts]
    llm = LLM(c.path, dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=5, max_model_len=64, max_num_batched_tokens=64,
              max_num_seqs=3, skip_tokenizer_init=True)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True), use_tqdm=False)
    assert [o["token_ids"] for o in outs] == want
    assert llm.stats.to_dict()["preemptions"] > 0          # the convolutions' inputs were rebuilt from the tokens so far
    llm.exit()


def test_cached_prefixes(cases):
    """A model without convolutions picks up cached blocks; the first token after them still pairs with the last one in them."""
    c = cases("chunks")
    shared = gc.tokens(c.cfg, 40, 50)
    prompts = [shared + gc.tokens(c.cfg, n, 60 + n) for n in (3, 9, 30)]
    want = [greedy(c, p, 10) for p in prompts]
    llm = LLM(c.path, dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=40, max_model_len=96, max_num_batched_tokens=96,
              max_num_seqs=2, skip_tokenizer_init=True)
    for p, w in zip(prompts, want):
        assert llm.generate([p], SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True), use_tqdm=False)[0]["token_ids"] == w
    assert llm.stats.to_dict()["prefix_cached_tokens"] == 64
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
