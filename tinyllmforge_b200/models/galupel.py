"""Galupel: a decoder whose sublayers read the residual stream itself and are normed, in groups of columns, on their way out.

    x <- x + norm1(mixer(x)),  x <- x + norm2(experts(x))

Two kinds of mixers take turns as the configuration lists them: attention over a window and means of the blocks behind it (some layers on
the keys and values of an earlier one), and latent attention over a window.  The embedding is normed, its table is the head, and the
logits are bounded.  The residual stream is fp32 in every precision.  Between two sublayers one op takes up the result of the one before
(sum over a token's experts, norm, sum) and emits the input of the one after, which is the stream rounded once.
"""
from __future__ import annotations

import torch

from .attention_blocks import NormedAttention
from .blocks import LatentAttention, RoutedFeedForward
from .galupel_config import GalupelConfig
from .layered import LayeredDecoder

MIXERS = {"attention": NormedAttention, "latent_attention": LatentAttention}


class GalupelLayer:
    def __init__(self, spec, cfg: GalupelConfig, dtype, device, rope):
        W = cfg.hidden_size
        self.mix = MIXERS[spec.type](spec.mixer, W, cfg.rms_norm_eps, dtype, device, rope)
        self.norm1 = torch.ones(W, dtype=dtype, device=device)
        self.mlp = self.norm2 = None
        if spec.mlp is not None:
            self.mlp = RoutedFeedForward(spec.mlp, W, dtype, device)
            self.norm2 = torch.ones(W, dtype=dtype, device=device)


class GalupelForCausalLM(LayeredDecoder):
    tied = True

    def __init__(self, cfg: GalupelConfig, tp=None, dtype=None, device="cpu", ops=None, max_positions: int | None = None):
        self.logit_scale, self.logit_softcap = cfg.logit_scale, cfg.logit_softcap
        super().__init__(cfg, tp, dtype, device, ops, max_positions)
        self.embed_norm = torch.ones(cfg.hidden_size, dtype=self.dtype, device=self.device)
        self.layers = [GalupelLayer(s, cfg, self.dtype, self.device, self.rope) for s in cfg.layers]
        self.runs = list(range(len(self.layers)))

    # ------------------------------------------------------------------ parameters by checkpoint name
    def extra_parameters(self):
        yield "embed.norm", self.embed_norm

    def layer_parameters(self, i: int):
        l = self.layers[i]
        yield f"l{i}.norm1", l.norm1
        yield from l.mix.named_parameters(f"l{i}.mix.")
        if l.mlp is not None:
            yield f"l{i}.norm2", l.norm2
            yield from l.mlp.named_parameters(f"l{i}.mlp.")

    # ------------------------------------------------------------------ forward
    def forward(self, batch, rows=None, observe=None) -> torch.Tensor:
        ops, dtype, eps, groups = self.ops, self.dtype, self.eps, self.cfg.norm_groups
        x = torch.empty(batch.padded_tokens, self.cfg.hidden_size, dtype=torch.float32, device=self.device)
        taken = dict(start=True, ids=batch.input_ids, embed=self.embed.weight, post=self.embed_norm)       # what x takes up next

        def advance(norm=None, rows=None):
            return ops.stream_update(x, dtype, eps, [norm], rows=rows, groups=groups, **taken)[0]

        for layer, memory in zip(self.layers, self.memory):
            taken = dict(a=layer.mix.forward(ops, advance(), memory, batch), post=layer.norm1)
            if layer.mlp is not None:
                taken = dict(a=layer.mlp.forward(ops, advance()), post=layer.norm2)
            if observe is not None:
                probe = x.clone()
                ops.stream_update(probe, dtype, eps, [], groups=groups, **taken)
                observe(probe)
        return advance(self.final_norm, rows)
