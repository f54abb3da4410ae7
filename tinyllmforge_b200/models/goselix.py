"""Goselix: a decoder with parallel layers (mixer and feed-forward read the same residual stream), two kinds of mixers
(latent attention over a paged cache, retention over a per-sequence state) and a range of layers that may run several
times with the same weights, every pass with a cache or state of its own.

The residual stream is fp32 in every precision.  Between two layers one op adds both branches of the layer before to it
(and, ahead of a pass of the loop, the pass's vector and the embedding) and emits both norms of the layer after:

    [add + inject + norm1, norm2] -> mixer(norm1) ; feed-forward(norm2) -> [add + ...]
"""
from __future__ import annotations

import torch

from ..ops import ref as ref_ops
from ..parallel.comm import TPGroup
from ..parallel.tp_layers import ParallelLMHead, VocabParallelEmbedding
from .blocks import GatedFeedForward, LatentAttention, Retention, RoutedFeedForward
from .goselix_config import DenseSpec, GoselixConfig

MIXERS = {"latent_attention": LatentAttention, "retention": Retention}


class GoselixLayer:
    def __init__(self, spec, cfg: GoselixConfig, dtype, device, rope):
        W = cfg.hidden_size
        self.mix = MIXERS[spec.type](spec.mixer, W, cfg.rms_norm_eps, dtype, device, rope)
        self.norm1 = torch.ones(W, dtype=dtype, device=device)
        self.mlp = self.norm2 = None
        if spec.mlp is not None:
            self.mlp = (GatedFeedForward if isinstance(spec.mlp, DenseSpec) else RoutedFeedForward)(spec.mlp, W, dtype, device)
            self.norm2 = torch.ones(W, dtype=dtype, device=device)

    @property
    def norms(self):
        return [self.norm1] if self.mlp is None else [self.norm1, self.norm2]


class GoselixForCausalLM:
    def __init__(self, cfg: GoselixConfig, tp: TPGroup | None = None, dtype=None, device="cpu", ops=None,
                 max_positions: int | None = None):
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
                tables[rot] = ref_ops.rope_table(positions, rot.dims, rot.base, self.device, torch.float64)
            return tables[rot]

        self.embed = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, self.tp, self.dtype, self.device)
        self.layers = [GoselixLayer(s, cfg, self.dtype, self.device, rope) for s in cfg.layers]
        self.step_vectors = None if cfg.loop is None else torch.zeros(cfg.loop.times, cfg.hidden_size, dtype=self.dtype, device=self.device)
        self.final_norm = torch.ones(cfg.hidden_size, dtype=self.dtype, device=self.device)
        self.head = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, self.tp, self.dtype, self.device)
        self.runs = cfg.layer_runs()
        self.memory: list = []                   # per layer run: the paged latent cache or the recurrent state

    # ------------------------------------------------------------------ parameters by checkpoint name
    def named_parameters(self):
        yield "embed", self.embed.weight, self.embed, None
        if self.step_vectors is not None:
            yield "loop.step", self.step_vectors, None, None
        for i, l in enumerate(self.layers):
            yield f"l{i}.norm1", l.norm1, None, None
            for name, t in l.mix.named_parameters(f"l{i}.mix."):
                yield name, t, None, None
            if l.mlp is not None:
                yield f"l{i}.norm2", l.norm2, None, None
                for name, t in l.mlp.named_parameters(f"l{i}.mlp."):
                    yield name, t, None, None
        yield "final.norm", self.final_norm, None, None
        yield "head", self.head.weight, self.head, None

    def num_parameter_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for _, t, _, _ in self.named_parameters())

    def finish_loading(self, config=None) -> None:
        for l in self.layers:
            l.mix.finish_loading()

    # ------------------------------------------------------------------ cache and state
    def kv_block_bytes(self, block_size: int) -> int:
        return block_size * sum(self.layers[i].mix.bytes_per_token() for i, _ in self.runs)

    def state_bytes(self) -> int:
        """Recurrent state of one sequence."""
        return sum(self.layers[i].mix.bytes_per_sequence() for i, _ in self.runs)

    def expansion_bytes(self, tokens: int) -> int:
        """Largest workspace that ``tokens`` cached keys take when a portion of a prompt sees them (keys and values rebuilt per head)."""
        return tokens * max((l.mix.expansion_bytes() for l in self.layers), default=0)

    def bind_cache(self, num_blocks: int, block_size: int, num_slots: int) -> None:
        """Every layer run (each pass of a looped layer) has a cache or state of its own; all share block and slot numbers."""
        self.memory = [self.layers[i].mix.new_memory(num_blocks, block_size, num_slots) for i, _ in self.runs]

    def drop_cache(self) -> None:
        self.memory = []

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        """Hidden states after the final norm, of all tokens or of the tokens ``rows`` (an index tensor).  ``observe(x)`` is
        called with the residual stream after every layer run."""
        ops, dtype, eps = self.ops, self.dtype, self.eps
        loop = self.cfg.loop
        x = torch.empty(batch.padded_tokens, self.cfg.hidden_size, dtype=torch.float32, device=self.device)
        a = b = None
        for run, (i, t) in enumerate(self.runs):
            layer = self.layers[i]
            inject = {}
            if run == 0 or (t is not None and t > 0 and i == loop.start):          # x starts as the embedding; later passes add it
                inject.update(ids=batch.input_ids, embed=self.embed.weight)
            if t is not None and i == loop.start:
                inject.update(vec=self.step_vectors[t])
            h = ops.stream_update(x, dtype, eps, layer.norms, start=run == 0, a=a, b=b, **inject)
            a = layer.mix.forward(ops, h[0], self.memory[run], batch)
            b = layer.mlp.forward(ops, h[1]) if layer.mlp is not None else None
            if observe is not None:
                probe = x.clone()
                ops.stream_update(probe, dtype, eps, [], a=a, b=b)
                observe(probe)
        return ops.stream_update(x, dtype, eps, [self.final_norm], a=a, b=b, rows=rows)[0]

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
            ids, best = ops.lm_head_sample_shard(hidden, head.weight, batch.temperatures, batch.header, 0)
            return ops.merge_ranks(ids, best, self.tp)
        return ops.sample(head.forward(ops, hidden), batch, 0, self.tp)
