"""Configuration of Galupel, a decoder whose layers are listed one by one and normed on their way out, in groups.

``config.json`` gives, for every layer, the type and the sizes of its mixer ("attention": a sliding window of tokens and means of the
blocks behind it, with keys and values of its own or of an earlier layer; "latent_attention": over a sliding window, with queries
made from the input itself) and its feed-forward (experts chosen within groups, or none), and the model's vocabulary, width, norm
constants, and what is done to the logits.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..config import parse_dtype
from .specs import NO_ROTATION, AttentionSpec, LatentAttentionSpec, MoeSpec, Rotation, take


def _attention(d: dict) -> AttentionSpec:
    keys = {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float,
            "mask": lambda m: take(m, "attention.mask", {"size": int, **({"pool": int} if m.get("pool") is not None else {})})}
    if "kv_from" in d:
        keys["kv_from"] = lambda j: None if j is None else int(j)
    t = take(d, "attention", keys)
    mask = t.pop("mask")
    if mask.get("pool", 1) < 1:
        raise ValueError("attention: mask.pool: blocks of at least one token")
    return AttentionSpec(rot=NO_ROTATION, window=mask["size"], pool=mask.get("pool", 0), temper=True, **t)


def _latent_attention(d: dict) -> LatentAttentionSpec:
    t = take(d, "latent_attention", {"heads": int, "dim": int, "rot_dim": int, "vdim": int, "kv_rank": int, "scale": float,
                                     "rot": lambda r: Rotation.from_dict(r, interleaved=True),
                                     "mask": lambda m: take(m, "latent_attention.mask", {"size": int})["size"]})
    if t["mask"] < 1:
        raise ValueError("latent_attention: mask.size: a token sees at least itself")
    return LatentAttentionSpec(window=t.pop("mask"), **t)


MIXER_SPECS = {"attention": _attention, "latent_attention": _latent_attention}


def _mlp_from_dict(d):
    if d is None:
        return None
    if d.get("kind") != "moe":
        raise ValueError(f"unknown feed-forward kind {d.get('kind')!r}; known: moe")
    r = take(d["router"], "mlp.router", {"experts": int, "top": int, "groups": lambda g: take(g, "mlp.router.groups", {"count": int, "keep": int})})
    return MoeSpec(r["experts"], r["top"], take(d["expert"], "mlp.expert", {"ff": int})["ff"], act="gelu", weigh="output", gated=False, correction=True,
                   groups=r["groups"]["count"], keep=r["groups"]["keep"])


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: object

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d.get("type") not in MIXER_SPECS:
            raise ValueError(f"unknown layer type {d.get('type')!r}; known: {sorted(MIXER_SPECS)}")
        return cls(d["type"], MIXER_SPECS[d["type"]](d["mixer"]), _mlp_from_dict(d.get("mlp")))


def _check_lenders(layers: tuple) -> None:
    for i, l in enumerate(layers):
        j = getattr(l.mixer, "kv_from", None)
        if j is None:
            continue
        if not 0 <= j < i or layers[j].type != "attention" or layers[j].mixer.kv_from is not None:
            raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own")
        a, b = l.mixer, layers[j].mixer
        if (a.heads, a.kv_heads, a.dim, a.vdim) != (b.heads, b.kv_heads, b.dim, b.vdim):
            raise ValueError(f"layer {i}: kv_from: the heads of both layers must be alike")


@dataclass
class GalupelConfig:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    norm_groups: int
    logit_scale: float
    logit_softcap: float
    layers: tuple
    torch_dtype: str = "bfloat16"
    eos_token_id: int = -1
    max_position_embeddings: int = 1 << 20      # the design names no limit; rotary tables are built for max_model_len

    quantizable = False
    num_recurrent_runs = 0
    prefix_cacheable = True                     # means of blocks lie in the page of the block's last token

    @classmethod
    def from_dict(cls, d: dict) -> "GalupelConfig":
        for key in ("vocab", "width", "norm", "logit_scale", "logit_softcap", "layers"):
            if key not in d:
                raise ValueError(f"Galupel config: missing {key!r}")
        if not d["layers"]:
            raise ValueError("Galupel config: no layers")
        norm = take(d["norm"], "norm", {"eps": float, "groups": int})
        layers = tuple(LayerSpec.from_dict(l) for l in d["layers"])
        _check_lenders(layers)
        cfg = cls(int(d["vocab"]), int(d["width"]), norm["eps"], norm["groups"], float(d["logit_scale"]), float(d["logit_softcap"]), layers,
                  torch_dtype=str(d.get("torch_dtype") or d.get("dtype") or "bfloat16").replace("torch.", ""))
        if cfg.norm_groups < 1 or cfg.hidden_size % cfg.norm_groups:
            raise ValueError("Galupel config: norm.groups must divide width")
        if not cfg.logit_softcap > 0:
            raise ValueError("Galupel config: logit_softcap must be positive")
        if d.get("eos_token_id") is not None:
            eos = d["eos_token_id"]
            cfg.eos_token_id = int(eos[0] if isinstance(eos, (list, tuple)) else eos)
        if d.get("max_position_embeddings"):
            cfg.max_position_embeddings = int(d["max_position_embeddings"])
        return cfg

    def validate_tp(self, size: int) -> None:
        if size != 1:
            raise ValueError("Galupel runs on one GPU (tensor_parallel_size=1)")

    @property
    def dtype(self):
        return parse_dtype(self.torch_dtype)


def example_dict(width: int, layers: int = 4, vocab: int = 32000) -> dict:
    """A configuration with the proportions of a real model of this width: heads of 128 (four query heads per key/value head) over a window
    of 1024 and means of 16 tokens behind it, latents of 512 over a window of 4096, 32 experts of which eight (out of four groups of
    eight) take the work of a feed-forward of three times the width; both mixers in turn, the last attention layer on the keys and values of the
    first where there are two."""
    heads = max(8, width // 128)
    attend = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 1024, "pool": 16}}
    latent = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "mask": {"size": 4096},
              "rot": {"base": 1e6, "dims": 64}}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 8, "groups": {"count": 8, "keep": 4}}, "expert": {"ff": 9 * width // 16}}
    kinds = [("latent_attention", latent), ("attention", attend)]
    last = max((i for i in range(layers) if i % 2), default=1)
    return {"architecture": "Galupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6, "groups": 4}, "logit_scale": 0.5, "logit_softcap": 30.0,
            "layers": [{"type": kinds[i % 2][0], "mixer": {**kinds[i % 2][1], **({"kv_from": 1} if i == last > 1 else {})}, "mlp": moe}
                       for i in range(layers)]}
