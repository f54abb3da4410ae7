"""Goselix on the PyTorch op set against the plain oracle: configuration, every mechanism through the engine, portions, batches,
blocks and state slots used again, generation through ``LLM`` with its scheduler."""
import copy
import warnings

import numpy as np
import pytest
import torch

import goselix_cases as gc
import oracle_goselix as oracle
from tinyllmforge_b200 import LLM, SamplingParams
from tinyllmforge_b200.engine.kv_blocks import KVBlockPool
from tinyllmforge_b200.engine.request import Request
from tinyllmforge_b200.engine.step_batch import build_decode, build_prefill
from tinyllmforge_b200.models import registry
from tinyllmforge_b200.models.goselix import GoselixForCausalLM
from tinyllmforge_b200.models.goselix_config import GoselixConfig

TOL = 2e-5


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = gc.Case(name, tmp_path_factory.mktemp(name), "cpu")
        return made[name]
    return get


# ------------------------------------------------------------------------------------------------ configuration and registry
def test_registry_chooses_by_architecture():
    cfg = registry.config_from_dict(gc.CONFIGS["varied"])
    assert isinstance(cfg, GoselixConfig) and registry.model_class(cfg) is GoselixForCausalLM
    assert registry.model_class(registry.config_from_dict({"model_type": "qwen3"})).__name__ == "Qwen3ForCausalLM"
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.config_from_dict({"architecture": "Nonesuch"})


def test_config_errors():
    d = copy.deepcopy(gc.CONFIGS["varied"])
    for path, value in ((("layers", 0, "type"), "convolution"), (("layers", 0, "mixer", "decay"), [0.5]), (("layers", 1, "mixer", "rot", "dims"), 8),
                        (("layers", 0, "mlp", "kind"), "sparse"), (("loop", "stop"), 9), (("layers", 0, "mlp", "router", "top"), 6)):
        bad = copy.deepcopy(d)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            GoselixConfig.from_dict(bad)
    missing = copy.deepcopy(d)
    del missing["layers"][1]["mixer"]["scale"]
    with pytest.raises(ValueError, match="scale"):
        GoselixConfig.from_dict(missing)
    extra = copy.deepcopy(d)
    extra["layers"][1]["mixer"]["window"] = 4
    with warnings.catch_warnings(record=True) as w:
        warnings.simplefilter("always")
        GoselixConfig.from_dict(extra)
    assert any("window" in str(x.message) for x in w)


def test_layer_runs_match_oracle():
    for d in gc.CONFIGS.values():
        cfg = GoselixConfig.from_dict(d)
        assert cfg.layer_runs() == oracle.layer_runs(d)
        assert cfg.num_recurrent_runs == sum(d["layers"][i]["type"] == "retention" for i, _ in oracle.layer_runs(d))


def test_unsupported_engine_options(cases):
    path = cases("looped").path
    with pytest.raises(ValueError, match="one GPU"):
        LLM(path, device="cpu", tensor_parallel_size=2, kvcache_block_size=16)
    with pytest.raises(ValueError, match="quantization"):
        LLM(path, device="cpu", quantization="fp8_block", kvcache_block_size=16)


def test_checkpoint_errors(tmp_path, cases):
    c = cases("looped")
    w = dict(c.weights)
    del w["l0.mix.g"]
    path = gc.write_model(tmp_path / "missing", c.cfg, w)
    with pytest.raises(KeyError, match="l0.mix.g"):
        LLM(path, device="cpu", kvcache_block_size=16, skip_tokenizer_init=True)
    w = dict(c.weights, extra=torch.zeros(3))
    path = gc.write_model(tmp_path / "extra", c.cfg, w)
    with pytest.raises(KeyError, match="extra"):
        LLM(path, device="cpu", kvcache_block_size=16, skip_tokenizer_init=True)


# ------------------------------------------------------------------------------------------------ pool and step buffer
def test_state_slots_follow_the_blocks():
    pool = KVBlockPool(8, 4, prefix_caching=False, num_state_slots=2)
    a, b, c = Request([1] * 5), Request([1] * 5), Request([1] * 5)
    pool.admit(a)
    pool.admit(b)
    assert {a.state_slot, b.state_slot} == {0, 1} and b.num_cached_tokens == 0       # equal prompts share nothing
    assert not pool.can_admit(c)                                                     # blocks are left, slots are not
    slot = a.state_slot
    pool.release(a)
    assert a.state_slot == -1 and pool.can_admit(c)
    pool.admit(c)
    assert c.state_slot == slot
    pool.check_invariants()
    c.token_ids += [2] * 6
    pool.extend(c)
    assert len(c.block_table) == 3
    with pytest.raises(RuntimeError, match="free blocks"):
        c.token_ids += [2] * 40
        pool.extend(c)


def test_mixed_step_buffer():
    reqs = []
    for n, start, slot in ((9, 8, 2), (4, 3, 0), (7, 2, 3), (6, 5, 1)):
        r = Request([n] * n)
        r.block_table, r.state_slot = [n, n + 10], slot
        r.num_computed_tokens, r.prefill_end = start, n
        reqs.append(r)
    sb = build_prefill(reqs, 8)
    assert sb.num_single == 2                            # the single token after the first longer portion is not a leading one
    assert sb.cu_seqlens_k.tolist() == [0, 0, 0, 7, 13] and sb.kv_rows == 13
    assert sb.state_slots.tolist() == [2, 0, 3, 1] and sb.cu_seqlens_q.tolist() == [0, 1, 2, 7, 8]
    d = build_decode(reqs[:2], 8, pad_to=4, table_width=3)
    assert d.num_single == 2 and d.state_slots.tolist() == [2, 0, -1, -1]


# ------------------------------------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("name", list(gc.CONFIGS))
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


def test_mixed_batches_reuse_blocks_and_slots(cases):
    c = cases("varied")
    reqs = {f"r{i}": gc.tokens(c.cfg, n, 10 + i) for i, n in enumerate((1, 33, 50, 2, 16, 48, 65, 17))}
    p = c.player(blocks=10, slots=3)                      # far fewer than all requests together need
    got = gc.run(p, gc.mixed_schedule(reqs, [1, 1, 2, 3, 14], live=3))
    for name, toks in reqs.items():
        assert c.error(got[name], toks, slice(None)).max() < TOL, name
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
    assert len(got) == len(want)
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()
    p.engine.exit()


# ------------------------------------------------------------------------------------------------ generation
def greedy(c, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(c.cfg, c.weights, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"extra": {"pipeline": False}}, {"chunked_prefill": True, "max_num_batched_tokens": 16}])
def test_greedy_generation(cases, kw):
    c = cases("looped")
    prompts = [gc.tokens(c.cfg, n, 20 + n) for n in (1, 5, 16, 23, 40)]
    want = [greedy(c, p, 12) for p in prompts]
    base = dict(dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=32, max_model_len=96, max_num_batched_tokens=96,
                max_num_seqs=3, skip_tokenizer_init=True)
    llm = LLM(c.path, **{**base, **kw})
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), use_tqdm=False)
    assert [o["token_ids"] for o in outs] == want
    assert llm.stats.to_dict()["prefix_cached_tokens"] == 0
    again = llm.generate(prompts[::-1], SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), use_tqdm=False)
    assert [o["token_ids"] for o in again] == want[::-1]
    llm.exit()


def test_generation_with_preemption(cases):
    c = cases("looped")
    prompts = [gc.tokens(c.cfg, n, 40 + n) for n in (14, 15, 16)]
    want = [greedy(c, p, 24) for p in prompts]
    llm = LLM(c.path, dtype="float32", device="cpu", kvcache_block_size=16, num_kvcache_blocks=5, max_model_len=64, max_num_batched_tokens=64,
              max_num_seqs=3, skip_tokenizer_init=True)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True), use_tqdm=False)
    assert [o["token_ids"] for o in outs] == want
    assert llm.stats.to_dict()["preemptions"] > 0          # the state was rebuilt from the prompt and the tokens so far
    llm.exit()


def test_replay_program(cases, tmp_path):
    import io
    import json
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
