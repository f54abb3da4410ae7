"""Goselix: a decoder with parallel layers (mixer and feed-forward read the same residual stream), two kinds of mixers
(latent attention over a paged cache, retention over a per-sequence state) and a range of layers that may run several
times with the same weights, every pass with a cache or state of its own.

The residual stream is fp32 in every precision.  Between two layers one op adds both branches of the layer before to it
(and, ahead of a pass of the loop, the pass's vector and the embedding) and emits both norms of the layer after:

    [add + inject + norm1, norm2] -> mixer(norm1) ; feed-forward(norm2) -> [add + ...]
"""
from __future__ import annotations

import torch

from .blocks import GatedFeedForward, LatentAttention, Retention, RoutedFeedForward
from .goselix_config import GoselixConfig
from .layered import LayeredDecoder
from .specs import DenseSpec

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


class GoselixForCausalLM(LayeredDecoder):
    def __init__(self, cfg: GoselixConfig, tp=None, dtype=None, device="cpu", ops=None, max_positions: int | None = None):
        super().__init__(cfg, tp, dtype, device, ops, max_positions)
        self.layers = [GoselixLayer(s, cfg, self.dtype, self.device, self.rope) for s in cfg.layers]
        self.step_vectors = None if cfg.loop is None else torch.zeros(cfg.loop.times, cfg.hidden_size, dtype=self.dtype, device=self.device)
        self.passes = cfg.layer_runs()
        self.runs = [i for i, _ in self.passes]

    # ------------------------------------------------------------------ parameters by checkpoint name
    def extra_parameters(self):
        if self.step_vectors is not None:
            yield "loop.step", self.step_vectors

    def layer_parameters(self, i: int):
        l = self.layers[i]
        yield f"l{i}.norm1", l.norm1
        yield from l.mix.named_parameters(f"l{i}.mix.")
        if l.mlp is not None:
            yield f"l{i}.norm2", l.norm2
            yield from l.mlp.named_parameters(f"l{i}.mlp.")

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        ops, dtype, eps = self.ops, self.dtype, self.eps
        loop = self.cfg.loop
        x = torch.empty(batch.padded_tokens, self.cfg.hidden_size, dtype=torch.float32, device=self.device)
        a = b = None
        for run, (i, t) in enumerate(self.passes):
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
