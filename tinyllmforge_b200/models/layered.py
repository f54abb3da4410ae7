"""What decoders whose layers are listed one by one have in common: embedding and head, memory per layer run, sampling.

A design derives from ``LayeredDecoder``, fills ``layers`` (each with ``mix``, a block of ``blocks.py``,
``hybrid_blocks.py`` or ``attention_blocks.py``) and ``runs`` (the layer runs in order of computation), and states its residual stream in ``forward``.
"""
from __future__ import annotations

import torch

from ..ops import ref as ref_ops
from ..parallel.comm import TPGroup
from ..parallel.tp_layers import ParallelLMHead, VocabParallelEmbedding


class LayeredDecoder:
    tied, logit_scale, logit_softcap = False, 1.0, 0.0      # the embedding table is the head; logits <- bounded by softcap (scale * logits)

    def __init__(self, cfg, tp: TPGroup | None = None, dtype=None, device="cpu", ops=None, max_positions: int | None = None):
        self.cfg = cfg
        self.tp = tp or TPGroup()
        cfg.validate_tp(self.tp.size)
        self.dtype = dtype or cfg.dtype
        self.device = torch.device(device)
        self.ops = ops or ref_ops.RefOps
        self.eps = cfg.rms_norm_eps
        positions = max_positions or cfg.max_position_embeddings
        tables: dict = {}

        def rope(rot):                           # layers with the same rotation share one table
            if rot not in tables:
                tables[rot] = ref_ops.rotation_table(positions, rot.frequencies, rot.amplitude, self.device)
            return tables[rot]

        self.rope = rope
        self.embed = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, self.tp, self.dtype, self.device)
        self.final_norm = torch.ones(cfg.hidden_size, dtype=self.dtype, device=self.device)
        self.head = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, self.tp, self.dtype, self.device, tied=self.embed if self.tied else None,
                                   scale=self.logit_scale, softcap=self.logit_softcap)
        self.layers: list = []
        self.runs: list = []                     # index into ``layers`` of every layer run
        self.memory: list = []                   # per layer run: paged cache, recurrent state, or both

    # ------------------------------------------------------------------ parameters by checkpoint name
    def layer_parameters(self, i: int):
        """(name, tensor) of layer ``i``."""
        raise NotImplementedError

    def extra_parameters(self):
        return ()

    def named_parameters(self):
        yield "embed", self.embed.weight, self.embed, None
        for name, t in self.extra_parameters():
            yield name, t, None, None
        for i in range(len(self.layers)):
            for name, t in self.layer_parameters(i):
                yield name, t, None, None
        yield "final.norm", self.final_norm, None, None
        if not self.tied:
            yield "head", self.head.weight, self.head, None

    def num_parameter_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for _, t, _, _ in self.named_parameters())

    def finish_loading(self, config=None) -> None:
        for l in self.layers:
            l.mix.finish_loading()

    # ------------------------------------------------------------------ cache and state
    def kv_block_bytes(self, block_size: int) -> int:
        return sum(block_size * m.bytes_per_token() + (m.pool_bytes(block_size) if hasattr(m, "pool_bytes") else 0)
                   for m in (self.layers[i].mix for i in self.runs))

    def state_bytes(self) -> int:
        """Recurrent state of one sequence."""
        return sum(self.layers[i].mix.bytes_per_sequence() for i in self.runs)

    def expansion_bytes(self, tokens: int) -> int:
        """Largest workspace that ``tokens`` cached keys take when a portion of a prompt sees them."""
        return tokens * max((l.mix.expansion_bytes() for l in self.layers), default=0)

    def bind_cache(self, num_blocks: int, block_size: int, num_slots: int) -> None:
        """Every layer run has a cache or state of its own, or borrows an earlier layer's; all share block and slot numbers."""
        self.memory, latest = [], {}
        for i in self.runs:
            mix = self.layers[i].mix
            lender = getattr(mix, "lender", None)
            latest[i] = mix.new_memory(num_blocks, block_size, num_slots, **({} if lender is None else {"lent": latest[lender]}))
            self.memory.append(latest[i])

    def drop_cache(self) -> None:
        self.memory = []

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        """Hidden states after the final norm, of all tokens or of the tokens ``rows`` (an index tensor).  ``observe(x)`` is
        called with the residual stream after every layer run."""
        raise NotImplementedError

    def logits_at(self, batch, rows: torch.Tensor) -> torch.Tensor:
        """Logits ``[rows, vocab]`` of the batch's tokens ``rows``."""
        return self.head.forward(self.ops, self.forward(batch, rows))

    def compute_logits(self, hidden: torch.Tensor, batch) -> torch.Tensor:
        return self.head.forward(self.ops, self.ops.select_rows(hidden, batch.last_index))

    def step(self, batch) -> torch.Tensor:
        """forward + logits + sampling: token ids for the first ``batch.num_seqs`` rows.  Only the last token of every sequence
        goes through the final norm and the head."""
        hidden = self.forward(batch, batch.last_index)
        ops, head = self.ops, self.head
        if hasattr(ops, "can_sample_in_lm_head") and ops.can_sample_in_lm_head(hidden.shape[0], head.weight):
            ids, best = ops.lm_head_sample_shard(hidden, head.weight, batch.temperatures, batch.header, 0, head.scale, head.softcap)
            return ops.merge_ranks(ids, best, self.tp)
        return ops.sample(head.forward(ops, hidden), batch, 0, self.tp)
