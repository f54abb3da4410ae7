"""Tonapel on the PyTorch op set against the plain oracle: configuration, every mechanism through the engine, portions, batches,
window edges, blocks and state slots used again, generation through ``LLM`` with its scheduler."""
import copy
import io
import json
import warnings

import numpy as np
import pytest
import torch

import goselix_cases as gc
import oracle_tonapel as oracle
import tonapel_cases as tc
from tinyllmforge_b200 import LLM, SamplingParams
from tinyllmforge_b200.engine.request import Request
from tinyllmforge_b200.engine.step_batch import build_prefill
from tinyllmforge_b200.models import registry
from tinyllmforge_b200.models.tonapel import TonapelForCausalLM
from tinyllmforge_b200.models.tonapel_config import TonapelConfig, example_dict
from tinyllmforge_b200.ops.ref import RefOps

TOL = 6e-5


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = tc.Case(name, tmp_path_factory.mktemp(name), "cpu")
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


# ------------------------------------------------------------------------------------------------ configuration and registry
def test_registry_chooses_by_architecture():
    cfg = registry.config_from_dict(tc.CONFIGS["varied"])
    assert isinstance(cfg, TonapelConfig) and registry.model_class(cfg) is TonapelForCausalLM
    assert cfg.num_recurrent_runs == 4 and not cfg.prefix_cacheable
    assert len(TonapelConfig.from_dict(example_dict(1024)).layers) == 4


def test_config_errors():
    d = tc.CONFIGS["varied"]
    left, right = ("layers", 0, "mixer", "left"), ("layers", 0, "mixer", "right")
    for path, value in ((("layers", 0, "type"), "retention"), (left + ("kv_heads",), 4), (left + ("rot", "dims"), 26), (left + ("rot", "dims"), 3),
                        (left + ("mask", "size"), 0), (right + ("groups",), 3), (right + ("norm_groups",), 5), (("layers", 1, "mixer", "kv_heads"), 4),
                        (("layers", 1, "mlp", "kind"), "sparse"), (("layers", 0, "mlp", "router", "top"), 6), (("layers", 1, "mixer", "conv"), 0)):
        with pytest.raises(ValueError):
            TonapelConfig.from_dict(changed(d, path, value))
    for path in (("residual_mult",), ("layers", 0, "mixer", "left_scale"), left + ("scale",), ("layers", 0, "mlp", "expert", "limit")):
        with pytest.raises(ValueError, match=path[-1]):
            TonapelConfig.from_dict(changed(d, path, None))
    with warnings.catch_warnings(record=True) as w:
        warnings.simplefilter("always")
        TonapelConfig.from_dict(changed(d, left + ("sinks",), 4))
    assert any("sinks" in str(x.message) for x in w)


def test_unsupported_engine_options(cases):
    path = cases("short").path
    with pytest.raises(ValueError, match="one GPU"):
        LLM(path, device="cpu", tensor_parallel_size=2, kvcache_block_size=16)
    with pytest.raises(ValueError, match="quantization"):
        LLM(path, device="cpu", quantization="fp8_block", kvcache_block_size=16)


def test_checkpoint_errors(tmp_path, cases):
    c = cases("short")
    for change, match in ((lambda w: w.pop("l0.mix.q.conv"), "l0.mix.q.conv"), (lambda w: w.update(extra=torch.zeros(3)), "extra")):
        w = dict(c.weights)
        change(w)
        path = tc.write_model(tmp_path / match, c.cfg, w)
        with pytest.raises(KeyError, match=match):
            LLM(path, device="cpu", kvcache_block_size=16, skip_tokenizer_init=True)


# ------------------------------------------------------------------------------------------------ mechanisms
def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


@pytest.mark.parametrize("act", ["gelu_tanh", "clamped_swish"])
def test_gated_activations(act):
    h, w = rnd(20, 24, seed=1), rnd(2 * 18, 24, seed=2)
    got = RefOps.linear_act_mul(h, w, act, 0.7)
    g, u = h.double() @ w[:18].double().T, h.double() @ w[18:].double().T
    if act == "gelu_tanh":
        want = oracle.gelu_tanh(g) * u
    else:
        want = oracle.clamped_expert(h.double(), w[:18].double(), w[18:].double(), torch.eye(18).double(), 0.7)
    assert (got - want).abs().max() < 1e-4 and (g > 0.7).any() and (u < -0.7).any() and (u > 0.7).any()


def test_routing_weights_are_a_softmax_over_the_chosen():
    h, router = rnd(30, 16, seed=1), rnd(7, 16, seed=2)
    _, weights = oracle.route(h.double(), router.double(), 3)
    assert torch.allclose(weights.sum(-1), torch.ones(30).double())
    gu, down = rnd(7, 2 * 10, 16, seed=3), rnd(7, 16, 10, seed=4)
    w = {"router": router.double()}
    for e in range(7):
        w.update({f"e{e}.gate": gu[e, :10].double(), f"e{e}.up": gu[e, 10:].double(), f"e{e}.down": down[e].double()})
    want = oracle.mixture(h.double(), w, "", {"router": {"top": 3}, "expert": {"limit": 1.1}})
    got = RefOps.moe(h, router, gu, down, 3, score="softmax", weigh="output", act="clamped_swish", limit=1.1)
    assert (got - want).abs().max() < 1e-4 * want.abs().max()


def test_sandwich_norm():
    x, a, bias, post, pre = rnd(9, 20, seed=1), rnd(9, 20, seed=2), rnd(20, seed=3), rnd(20, seed=4), rnd(20, seed=5)
    want = x.double() + 0.3 * oracle.shifted_norm((a + bias).double(), post.double(), 1e-4)
    got = x.clone()
    h, = RefOps.stream_update(got, torch.float32, 1e-4, [pre], a=a, a_bias=bias, post=post, mult=0.3, offset=1.0)
    assert (got - want).abs().max() < 1e-5
    assert (h - oracle.shifted_norm(want, pre.double(), 1e-4)).abs().max() < 1e-5


@pytest.mark.parametrize("window", [1, 3, 16, 17, 40])
def test_window_edges_of_the_oracle(window):
    """Every query points at one key: the oldest that its window holds is found, the one before it is not."""
    n, d = 50, 24
    k, v = rnd(n, 1, d, seed=1), rnd(n, 1, 5, seed=2)
    for back in (window - 1, window):
        q = torch.stack([60.0 * k[max(i - back, 0)] / k[max(i - back, 0)].norm() ** 2 for i in range(n)])
        got = oracle.windowed_attention(q.double(), k.double(), v.double(), 1.0, window)
        for i in range(back, n):
            seen = k[max(0, i - window + 1):i + 1, 0] @ k[i - back, 0] / k[i - back, 0].norm() ** 2
            if (seen > 0.7).sum() == (back < window):              # nothing else comes near
                near = (got[i, 0] - v[i - back, 0].double()).norm() < 1e-2 * v[i - back, 0].norm()
                assert near == (back < window), (window, i)


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_causal_convolution_of_the_oracle(taps):
    x, w = rnd(12, 3, seed=1).double(), rnd(3, taps, seed=2).double()
    y = oracle.causal_conv(x, w)
    for t in range(12):
        want = sum(w[:, taps - 1 - back] * x[t - back] for back in range(taps) if t >= back)
        assert torch.allclose(y[t], want)


# ------------------------------------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("name", list(tc.CONFIGS))
def test_whole_prompt_and_token_by_token(cases, name):
    c = cases(name)
    toks = gc.tokens(c.cfg, 40 if name == "wide" else 70, 1)
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


@pytest.mark.parametrize("name", ["varied", "odd"])
def test_mixed_batches_reuse_blocks_and_slots(cases, name):
    c = cases(name)
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 10 + i) for i, n in enumerate((1, 33, 50, 2, 16, 48, 65, 17))}
    p = c.player(blocks=10, slots=3)                      # far fewer than all requests together need
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 2, 3, 14], live=3))
    for r, toks in reqs.items():
        assert c.error(got[r], toks, slice(None)).max() < TOL, r
    p.pool.check_invariants()
    assert p.pool.num_free == 10 and len(p.pool.state_slots.free) == 3
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
    assert len(got) == len(want) == 4
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()
    p.engine.exit()


def test_constants_reach_the_logits(cases):
    """A small change of each constant moves the logits by far more than the agreement above allows."""
    c = cases("varied")
    toks = gc.tokens(c.cfg, 30, 4)
    base = oracle.forward(c.cfg, c.weights, toks)
    left, right = ("layers", 0, "mixer", "left"), ("layers", 0, "mixer", "right")
    for path, value in ((("residual_mult",), 0.6), (("norm", "eps"), 0.1), (left + ("mask", "size"), 19), (left + ("mask", "size"), 21), (left + ("scale",), 0.31),
                        (left + ("rot", "base"), 9000.0), (left + ("rot", "dims"), 14), (("layers", 0, "mixer", "left_scale"), 0.8),
                        (("layers", 0, "mixer", "right_scale"), 0.5), (right + ("norm_groups",), 2), (("layers", 0, "mlp", "expert", "limit"), 0.7),
                        (("layers", 0, "mlp", "router", "top"), 3)):
        moved = (oracle.forward(changed(c.cfg, path, value), c.weights, toks) - base).pow(2).mean(-1).sqrt() / base.std()
        assert moved.max() > 10 * TOL, path


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
    assert llm.stats.to_dict()["preemptions"] > 0          # states and convolution inputs were rebuilt from the tokens so far
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
