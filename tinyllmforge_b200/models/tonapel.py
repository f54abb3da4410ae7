"""Tonapel: a decoder of two kinds of layers (windowed attention beside a state-space mixer, and the gated delta rule) whose
sublayers are normed on their way in and on their way out.

    x <- x + mult * norm_b(sublayer(norm(x)))          norm weights are stored around zero

The residual stream is fp32 in every precision.  Between two sublayers one op takes up the result of the one before (bias,
norm, factor, sum) and emits the normed input of the one after.
"""
from __future__ import annotations

import torch

from .blocks import GatedFeedForward, RoutedFeedForward
from .hybrid_blocks import GatedDelta, ParallelMixer
from .layered import LayeredDecoder
from .specs import DenseSpec
from .tonapel_config import TonapelConfig

MIXERS = {"parallel": ParallelMixer, "delta": GatedDelta}


class TonapelLayer:
    def __init__(self, spec, cfg: TonapelConfig, dtype, device, rope):
        W = cfg.hidden_size
        self.mix = MIXERS[spec.type](spec.mixer, W, cfg.rms_norm_eps, dtype, device, rope)
        self.mlp = None
        if spec.mlp is not None:
            self.mlp = (GatedFeedForward if isinstance(spec.mlp, DenseSpec) else RoutedFeedForward)(spec.mlp, W, dtype, device)
        self.norms = {name: torch.zeros(W, dtype=dtype, device=device)
                      for name in ("norm1", "norm1b") + (() if self.mlp is None else ("norm2", "norm2b"))}


class TonapelForCausalLM(LayeredDecoder):
    def __init__(self, cfg: TonapelConfig, tp=None, dtype=None, device="cpu", ops=None, max_positions: int | None = None):
        super().__init__(cfg, tp, dtype, device, ops, max_positions)
        self.layers = [TonapelLayer(s, cfg, self.dtype, self.device, self.rope) for s in cfg.layers]
        self.runs = list(range(len(self.layers)))

    def layer_parameters(self, i: int):
        l = self.layers[i]
        for name, t in l.norms.items():
            yield f"l{i}.{name}", t
        yield from l.mix.named_parameters(f"l{i}.mix.")
        if l.mlp is not None:
            yield from l.mlp.named_parameters(f"l{i}.mlp.")

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        ops, dtype, eps, mult = self.ops, self.dtype, self.eps, self.cfg.residual_mult
        x = torch.empty(batch.padded_tokens, self.cfg.hidden_size, dtype=torch.float32, device=self.device)
        taken = dict(start=True, ids=batch.input_ids, embed=self.embed.weight)       # what x takes up next

        def advance(norm, rows=None):
            return ops.stream_update(x, dtype, eps, [norm], rows=rows, offset=1.0, **taken)[0]

        for layer, memory in zip(self.layers, self.memory):
            n = layer.norms
            y = layer.mix.forward(ops, advance(n["norm1"]), memory, batch)
            taken = dict(a=y, a_bias=layer.mix.out_bias, post=n["norm1b"], mult=mult)
            if layer.mlp is not None:
                y = layer.mlp.forward(ops, advance(n["norm2"]))
                taken = dict(a=y, post=n["norm2b"], mult=mult)
            if observe is not None:
                probe = x.clone()
                ops.stream_update(probe, dtype, eps, [], offset=1.0, **taken)
                observe(probe)
        return advance(self.final_norm, rows)
