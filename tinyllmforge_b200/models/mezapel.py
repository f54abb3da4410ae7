"""Mezapel: a decoder over several residual streams with two kinds of attention (inside chunks, and over a sliding window behind short
convolutions), an embedding that reads pairs of tokens, and a range of layers that may run several times with the same weights,
every pass with a cache and state of its own.

The streams are fp32 in every precision.  Between two sublayers one op takes up the result of the one before into all streams and
emits the normed input of the one after, which is a weighted sum of the streams.
"""
from __future__ import annotations

import torch

from .attention_blocks import HyperConnection, NormedAttention
from .blocks import GatedFeedForward
from .layered import LayeredDecoder
from .mezapel_config import MezapelConfig


class LayerNorm:
    def __init__(self, width: int, dtype, device):
        self.weight, self.bias = torch.ones(width, dtype=dtype, device=device), torch.zeros(width, dtype=dtype, device=device)

    def named_parameters(self, p):
        yield p, self.weight
        yield p + ".b", self.bias


class MezapelLayer:
    def __init__(self, spec, cfg: MezapelConfig, dtype, device, rope):
        W = cfg.hidden_size
        self.mix = NormedAttention(spec.mixer, W, cfg.rms_norm_eps, dtype, device, rope)
        self.norm1, self.hc1 = LayerNorm(W, dtype, device), HyperConnection(cfg.streams, device)
        self.mlp = None
        if spec.mlp is not None:
            self.mlp = GatedFeedForward(spec.mlp, W, dtype, device)
            self.norm2, self.hc2 = LayerNorm(W, dtype, device), HyperConnection(cfg.streams, device)


class MezapelForCausalLM(LayeredDecoder):
    def __init__(self, cfg: MezapelConfig, tp=None, dtype=None, device="cpu", ops=None, max_positions: int | None = None):
        super().__init__(cfg, tp, dtype, device, ops, max_positions)
        W = cfg.hidden_size
        self.pairs = torch.empty(cfg.bigram.buckets + 1, W, dtype=self.dtype, device=self.device)
        self.final_bias = torch.zeros(W, dtype=self.dtype, device=self.device)
        self.layers = [MezapelLayer(s, cfg, self.dtype, self.device, self.rope) for s in cfg.layers]
        self.runs = [i for i, _ in cfg.layer_runs()]
        self.all_streams = torch.ones(cfg.streams, dtype=torch.float32, device=self.device)

    # ------------------------------------------------------------------ parameters by checkpoint name
    def extra_parameters(self):
        yield "bigram", self.pairs
        yield "final.norm.b", self.final_bias

    def layer_parameters(self, i: int):
        l = self.layers[i]
        yield from l.norm1.named_parameters(f"l{i}.norm1")
        yield from l.hc1.named_parameters(f"l{i}.hc1.")
        yield from l.mix.named_parameters(f"l{i}.mix.")
        if l.mlp is not None:
            yield from l.norm2.named_parameters(f"l{i}.norm2")
            yield from l.hc2.named_parameters(f"l{i}.hc2.")
            yield from l.mlp.named_parameters(f"l{i}.mlp.")

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        ops, dtype, eps, cfg = self.ops, self.dtype, self.eps, self.cfg
        x = torch.empty(batch.padded_tokens, cfg.streams, cfg.hidden_size, dtype=torch.float32, device=self.device)
        taken = dict(ids=batch.input_ids, prev=batch.prev_ids, embed=self.embed.weight, scale=cfg.embed_scale, pairs=self.pairs,
                     mul_prev=cfg.bigram.mul_prev, mul_cur=cfg.bigram.mul_cur)           # what the streams take up next
        for i, memory in zip(self.runs, self.memory):
            l = self.layers[i]
            h = ops.stream_mix(x, dtype, eps, l.hc1.into, l.norm1.weight, l.norm1.bias, **taken)
            taken = dict(y=l.mix.forward(ops, h, memory, batch), mix=l.hc1.mix, out=l.hc1.out)
            if l.mlp is not None:
                h = ops.stream_mix(x, dtype, eps, l.hc2.into, l.norm2.weight, l.norm2.bias, **taken)
                taken = dict(y=l.mlp.forward(ops, h), mix=l.hc2.mix, out=l.hc2.out)
            if observe is not None:
                probe = x.clone()
                ops.stream_mix(probe, dtype, eps, self.all_streams, None, None, **taken)
                observe(probe.sum(dim=1))
        return ops.stream_mix(x, dtype, eps, self.all_streams, self.final_norm, self.final_bias, rows=rows, **taken)
