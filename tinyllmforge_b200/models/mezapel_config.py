"""Configuration of Mezapel, a decoder whose layers are listed one by one over several residual streams.

``config.json`` gives, for every layer, the type and the sizes of its mixer ("attention": inside chunks, with a fixed sink;
"attention_2": over a sliding window behind short convolutions, with learned sinks and capped scores) and its feed-forward
(dense or none), optionally a range of layers that runs several times with the same weights (``loop``), and the model's
vocabulary, width, norm constant, number of streams and embedding constants.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..config import parse_dtype
from .specs import AttentionSpec, BandScaling, DenseSpec, LoopSpec, RampScaling, Rotation, layer_runs, take

MAX_STREAMS = 16                                # of the residual-stream kernels


def _mask_size(d: dict) -> int:
    return take(d, "mask", {"size": int})["size"]


def _chunk_attention(d: dict) -> AttentionSpec:
    t = take(d, "attention", {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float,
                              "rot": lambda r: Rotation.from_dict(r, RampScaling), "mask": _mask_size})
    return AttentionSpec(window=t.pop("mask"), chunked=True, norm="all", sink="zero", gate="head", **t)


def _window_attention(d: dict) -> AttentionSpec:
    t = take(d, "attention_2", {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float, "conv": int, "softcap": float,
                                "rot": lambda r: Rotation.from_dict(r, BandScaling), "mask": _mask_size})
    if t["conv"] < 1:
        raise ValueError("attention_2: a convolution has at least one tap")
    if not t["softcap"] > 0:
        raise ValueError("attention_2: softcap must be positive")
    return AttentionSpec(window=t.pop("mask"), norm="head", sink="learned", gate="element", **t)


MIXER_SPECS = {"attention": _chunk_attention, "attention_2": _window_attention}


def _mlp_from_dict(d):
    if d is None:
        return None
    if d.get("kind") != "dense":
        raise ValueError(f"unknown feed-forward kind {d.get('kind')!r}; known: dense")
    return DenseSpec(int(d["ff"]))


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: AttentionSpec
    mlp: object

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d.get("type") not in MIXER_SPECS:
            raise ValueError(f"unknown layer type {d.get('type')!r}; known: {sorted(MIXER_SPECS)}")
        return cls(d["type"], MIXER_SPECS[d["type"]](d["mixer"]), _mlp_from_dict(d.get("mlp")))


@dataclass(frozen=True)
class BigramSpec:
    """A token's row of the pair table is (previous token * mul_prev + token * mul_cur) mod buckets, or row ``buckets`` for a
    sequence's first token."""
    buckets: int
    mul_prev: int
    mul_cur: int

    @classmethod
    def from_dict(cls, d: dict) -> "BigramSpec":
        s = cls(**take(d, "embedding.bigram", {"buckets": int, "mul_prev": int, "mul_cur": int}))
        if s.buckets < 1:
            raise ValueError("embedding.bigram: at least one bucket")
        return s


@dataclass
class MezapelConfig:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    streams: int
    embed_scale: float
    bigram: BigramSpec
    layers: tuple
    loop: object = None
    torch_dtype: str = "bfloat16"
    eos_token_id: int = -1
    max_position_embeddings: int = 1 << 20      # the design names no limit; rotary tables are built for max_model_len

    quantizable = False

    @classmethod
    def from_dict(cls, d: dict) -> "MezapelConfig":
        for key in ("vocab", "width", "norm", "streams", "embedding", "layers"):
            if key not in d:
                raise ValueError(f"Mezapel config: missing {key!r}")
        if not d["layers"]:
            raise ValueError("Mezapel config: no layers")
        emb = take(d["embedding"], "embedding", {"scale": float, "bigram": BigramSpec.from_dict})
        layers = tuple(LayerSpec.from_dict(l) for l in d["layers"])
        cfg = cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), int(d["streams"]), emb["scale"], emb["bigram"], layers,
                  LoopSpec.from_dict(d["loop"], len(layers)) if d.get("loop") else None,
                  torch_dtype=str(d.get("torch_dtype") or d.get("dtype") or "bfloat16").replace("torch.", ""))
        if not 1 <= cfg.streams <= MAX_STREAMS:
            raise ValueError(f"Mezapel config: streams must lie between 1 and {MAX_STREAMS}")
        if d.get("eos_token_id") is not None:
            eos = d["eos_token_id"]
            cfg.eos_token_id = int(eos[0] if isinstance(eos, (list, tuple)) else eos)
        if d.get("max_position_embeddings"):
            cfg.max_position_embeddings = int(d["max_position_embeddings"])
        return cfg

    def validate_tp(self, size: int) -> None:
        if size != 1:
            raise ValueError("Mezapel runs on one GPU (tensor_parallel_size=1)")

    def layer_runs(self) -> list:
        return layer_runs(len(self.layers), self.loop)

    @property
    def dtype(self):
        return parse_dtype(self.torch_dtype)

    @property
    def num_recurrent_runs(self) -> int:
        """Layer runs that keep the last inputs of a convolution."""
        return sum(self.layers[i].mixer.conv > 1 for i, _ in self.layer_runs())

    @property
    def prefix_cacheable(self) -> bool:
        return self.num_recurrent_runs == 0


def example_dict(width: int, layers: int = 4, vocab: int = 32000) -> dict:
    """A configuration with the proportions of a real model of this width: heads of 128, four query heads per key/value head, a
    window of 1024 and chunks of 4096, a feed-forward of three times the width, two streams; both mixers in turn."""
    heads = max(8, width // 128)
    sizes = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    first = {**sizes, "rot": {"base": 5e5, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}, "mask": {"size": 4096}}
    second = {**sizes, "conv": 4, "softcap": 50.0, "mask": {"size": 1024},
              "rot": {"base": 1e6, "dims": 128, "scaling": {"factor": 8.0, "original": 4096, "low": 1.0, "high": 4.0}}}
    kinds = [("attention_2", second), ("attention", first)]
    return {"architecture": "Mezapel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "streams": 2,
            "embedding": {"scale": width ** 0.5, "bigram": {"buckets": 8191, "mul_prev": 31, "mul_cur": 7}},
            "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": {"kind": "dense", "ff": 3 * width}} for i in range(layers)]}
