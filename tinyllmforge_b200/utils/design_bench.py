"""Prefill and decode throughput of a design beside others at equal width, head size, feed-forward work and number of layers:
Goselix beside Qwen3, Tonapel beside Goselix and Qwen3, Mezapel beside Tonapel and Qwen3, Galupel beside Goselix, Mezapel and Qwen3.

    python bench.py --design goselix|tonapel|mezapel|galupel [--steps K] [--warmup W]

A few layers of each (random weights, bf16), through the engine's own step: packed step buffer, model, sampling, CUDA graph for
decode steps.  Device time per step (CUDA events); ahead of every timed step a buffer larger than L2 is written.  One JSON line
per model, size and workload.
"""
from __future__ import annotations

import json

import torch

SIZES = (1024, 2048, 4096)
LAYERS, VOCAB = 4, 32000
WORKLOADS = [("prefill", 8, 1024), ("prefill", 1, 8192), ("decode", 64, 1024), ("decode", 16, 4096), ("decode", 1, 4096)]


def _configs(design: str, width: int):
    from ..config import ModelConfig
    from ..models import galupel_config, goselix_config, mezapel_config, tonapel_config
    heads = max(8, width // 128)
    qwen = ModelConfig(hidden_size=width, num_hidden_layers=LAYERS, num_attention_heads=heads, num_key_value_heads=max(2, heads // 2) if width < 4096 else 8,
                       head_dim=128, intermediate_size=3 * width, vocab_size=VOCAB, tie_word_embeddings=False)
    known = {"goselix": (goselix_config.GoselixConfig, goselix_config.example_dict), "tonapel": (tonapel_config.TonapelConfig, tonapel_config.example_dict),
             "mezapel": (mezapel_config.MezapelConfig, mezapel_config.example_dict), "galupel": (galupel_config.GalupelConfig, galupel_config.example_dict)}
    order = {"goselix": ["goselix"], "tonapel": ["tonapel", "goselix"], "mezapel": ["mezapel", "tonapel"], "galupel": ["galupel", "goselix", "mezapel"]}[design]
    return [(name, known[name][0].from_dict(known[name][1](width, LAYERS, VOCAB))) for name in order] + [("qwen3", qwen)]


def _requests(worker, seqs: int, tokens: int):
    from ..engine.request import Request
    bs = worker.block_size
    per = -(-(tokens + 1) // bs)
    out = []
    for i in range(seqs):
        r = Request([(17 * i + 31 * j) % VOCAB for j in range(tokens)])
        r.block_table = list(range(i * per, (i + 1) * per))
        r.state_slot = i if worker.num_slots else -1
        out.append(r)
    return out


def run(design: str, steps: int, warmup: int, clock_sampler=None) -> None:
    from .. import LLM
    from ..engine.step_batch import build_decode, build_prefill
    flush = torch.empty(1 << 30, dtype=torch.uint8, device="cuda")
    for width in SIZES:
        for name, cfg in _configs(design, width):
            llm = LLM(name, hf_config=cfg, load_format="dummy", skip_tokenizer_init=True, max_model_len=8448, max_num_batched_tokens=8448,
                      max_num_seqs=64, num_kvcache_blocks=5 * 64 + 64, extra={"device_timing": True})
            w = llm.worker
            for kind, seqs, tokens in WORKLOADS:
                reqs = _requests(w, seqs, tokens)
                times = []
                sampler = clock_sampler(torch.cuda.current_device()) if clock_sampler else None
                if sampler:
                    sampler.start()
                launches = 0
                for i in range(max(3, warmup) + steps):
                    if kind == "prefill":
                        sb = build_prefill(reqs, w.block_size, i)
                    else:
                        pad, table = w.decode_padding(seqs)
                        sb = build_decode(reqs, w.block_size, i, pad_to=pad, table_width=table)
                    flush.fill_(i & 1)
                    before = w.kernel_launches
                    w.run(sb)
                    launches = w.kernel_launches - before
                    if i >= max(3, warmup):
                        times.append(w.last_step_ms)
                clocks = sampler.stop() if sampler else None
                ms = sum(times) / len(times)
                n = seqs * tokens if kind == "prefill" else seqs
                print(json.dumps({"metric": f"{kind}_tokens_per_second", "value": n / ms * 1e3, "unit": "tok/s", "model": name, "width": width,
                                  "layers": LAYERS, "sequences": seqs, "context": tokens, "ms_per_step": round(ms, 4), "steps": steps,
                                  "launches_per_step": launches, "weights": "random-init", "dtype": "bf16", "n_gpus": 1,
                                  "parameter_bytes": w.model.num_parameter_bytes(), "l2": "flushed before every step", "clocks": clocks}), flush=True)
            llm.exit()
            del llm, w
            torch.cuda.empty_cache()
