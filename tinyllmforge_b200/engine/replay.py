"""Replay of recorded steps: given token ids instead of sampled ones, logits instead of tokens.

    python -m tinyllmforge_b200.engine.replay --model DIR --out DIR --max-tokens N [--dtype bfloat16|float32]

Each line of standard input is one step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry carries the next tokens of a request and the places among them whose logits are wanted; ``end`` names the
requests that are finished after the step.  All entries run as one batch through the engine's block pool, step builder and
worker, portions of prompts beside single decoded tokens.  Wanted logits go to ``<out>/<step>.f32`` (little-endian fp32, in
the order of the entries); ``done <step>`` is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from .engine import LLMEngine
from .request import Request
from .step_batch import build_decode, build_prefill

BLOCK = 64
MAX_LIVE = 4


class Replayer:
    """Feeds chosen tokens of several requests through an engine, step by step."""

    def __init__(self, engine: LLMEngine):
        self.engine = engine
        self.pool = engine.scheduler.pool
        self.live: dict = {}

    def step(self, entries: list, end: list = ()) -> np.ndarray:
        """One batch.  Returns the wanted logits, [wanted, vocab] fp32, in the order of the entries."""
        batch = []
        for e in entries:
            req = self.live.get(e["id"])
            tokens = list(e["tokens"])
            if not tokens:
                raise ValueError(f"request {e['id']!r} brings no tokens")
            if req is None:
                req = self.live[e["id"]] = Request(tokens)
                start = 0
            else:
                start = len(req)
                req.token_ids += tokens
            self.pool.extend(req)
            req.num_computed_tokens, req.prefill_end = start, len(req)
            batch.append((req, e.get("want", ())))
        logits = self._run(batch) if batch else np.zeros((0, self.engine.config.hf_config.vocab_size), np.float32)
        for name in end:
            self.pool.release(self.live.pop(name))
        return logits

    def _run(self, batch) -> np.ndarray:
        cfg, worker = self.engine.config, self.engine.worker
        single = [r.prefill_end - r.num_computed_tokens == 1 for r, _ in batch]
        order = sorted(range(len(batch)), key=lambda i: not single[i])         # decoded tokens first (stable)
        reqs = [batch[i][0] for i in order]
        first, at = {}, 0                                                      # entry -> row of its first token
        for i, r in zip(order, reqs):
            first[i] = at
            at += r.prefill_end - r.num_computed_tokens
        build = build_decode if all(single) else build_prefill
        sb = build(reqs, cfg.kvcache_block_size, self.engine.step_index, cfg.seed)
        self.engine.step_index += 1
        rows = [first[i] + w for i, (_, want) in enumerate(batch) for w in want]
        if not rows:
            worker.run(sb)
            return np.zeros((0, cfg.hf_config.vocab_size), np.float32)
        return worker.logits(sb, rows).numpy()


def replay(model: str, out: str, max_tokens: int, dtype: str = "bfloat16", device: str = "auto", lines=sys.stdin, echo=sys.stdout) -> None:
    blocks = (max_tokens + BLOCK - 1) // BLOCK
    longest = blocks * BLOCK
    engine = LLMEngine(model, dtype=dtype, device=device, kvcache_block_size=BLOCK, num_kvcache_blocks=blocks, max_model_len=longest,
                       max_num_batched_tokens=longest, max_num_seqs=MAX_LIVE, enforce_eager=True, skip_tokenizer_init=True)
    try:
        player = Replayer(engine)
        for line in lines:
            if not line.strip():
                continue
            rec = json.loads(line)
            logits = player.step(rec["entries"], rec.get("end", ()))
            if logits.shape[0]:
                logits.astype("<f4").tofile(os.path.join(out, f"{rec['step']}.f32"))
            echo.write(f"done {rec['step']}\n")
            echo.flush()
    finally:
        engine.exit()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="Replay recorded steps through the engine and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time (the cache pool's size)")
    ap.add_argument("--device", default="cuda", choices=("cuda", "cpu"))
    a = ap.parse_args(argv)
    replay(a.model, a.out, a.max_tokens, a.dtype, a.device)
    return 0


if __name__ == "__main__":
    sys.exit(main())
