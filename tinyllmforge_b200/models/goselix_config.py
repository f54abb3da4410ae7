"""Configuration of Goselix, a decoder whose layers are listed one by one.

``config.json`` gives, for every layer, the type and the sizes of its mixer (latent attention or retention) and its
feed-forward (dense, mixture of experts, or none), optionally a range of layers that runs several times with the same
weights (``loop``), and the model's vocabulary, width and norm constant.  Nothing here has a default taken from one
checkpoint: a missing size is an error, an unknown key a warning.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..config import parse_dtype
from .specs import DenseSpec, LatentAttentionSpec, LoopSpec, MoeSpec, Rotation, layer_runs, take


def _latent_attention(d: dict) -> LatentAttentionSpec:
    s = LatentAttentionSpec(**take(d, "latent_attention", {"heads": int, "dim": int, "rot_dim": int, "vdim": int, "q_rank": int, "kv_rank": int,
                                                           "scale": float, "rot": Rotation.from_dict}))
    if s.q_rank < 1:
        raise ValueError("latent_attention: sizes must be positive")
    return s


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: Rotation

    @classmethod
    def from_dict(cls, d: dict) -> "RetentionSpec":
        s = cls(**take(d, "retention", {"heads": int, "dim": int, "vdim": int, "decay": lambda v: tuple(float(x) for x in v),
                                         "rot": Rotation.from_dict}))
        if len(s.decay) != s.heads:
            raise ValueError("retention: one decay per head")
        if not all(0.0 <= g <= 1.0 for g in s.decay):
            raise ValueError("retention: decays lie between 0 and 1")
        if s.rot.dims > s.dim:
            raise ValueError("retention: rot.dims cannot exceed dim")
        return s


def _mlp_from_dict(d):
    if d is None:
        return None
    kind = d.get("kind")
    if kind == "dense":
        return DenseSpec(int(d["ff"]))
    if kind == "moe":
        router = take(d["router"], "mlp.router", {"experts": int, "top": int})
        return MoeSpec(router["experts"], router["top"], int(d["expert"]["ff"]))
    raise ValueError(f"unknown feed-forward kind {kind!r}; known: dense, moe")


MIXER_SPECS = {"latent_attention": _latent_attention, "retention": RetentionSpec.from_dict}


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


@dataclass
class GoselixConfig:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    layers: tuple
    loop: object = None
    torch_dtype: str = "bfloat16"
    eos_token_id: int = -1
    max_position_embeddings: int = 1 << 20      # the design names no limit; rotary tables are built for max_model_len

    quantizable = False

    @classmethod
    def from_dict(cls, d: dict) -> "GoselixConfig":
        for key in ("vocab", "width", "norm", "layers"):
            if key not in d:
                raise ValueError(f"Goselix config: missing {key!r}")
        cfg = cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), tuple(LayerSpec.from_dict(l) for l in d["layers"]),
                  LoopSpec.from_dict(d["loop"], len(d["layers"])) if d.get("loop") else None,
                  torch_dtype=str(d.get("torch_dtype") or d.get("dtype") or "bfloat16").replace("torch.", ""))
        if d.get("eos_token_id") is not None:
            eos = d["eos_token_id"]
            cfg.eos_token_id = int(eos[0] if isinstance(eos, (list, tuple)) else eos)
        if d.get("max_position_embeddings"):
            cfg.max_position_embeddings = int(d["max_position_embeddings"])
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("Goselix config: no layers")

    def validate_tp(self, size: int) -> None:
        if size != 1:
            raise ValueError("Goselix runs on one GPU (tensor_parallel_size=1)")

    def layer_runs(self) -> list:
        """[(layer, pass)] in the order of computation; pass is None for a layer outside the loop."""
        return layer_runs(len(self.layers), self.loop)

    @property
    def dtype(self):
        return parse_dtype(self.torch_dtype)

    @property
    def num_recurrent_runs(self) -> int:
        return sum(self.layers[i].type == "retention" for i, _ in self.layer_runs())

    @property
    def prefix_cacheable(self) -> bool:
        """A recurrent state cannot be picked up in the middle of a prompt from cached blocks alone."""
        return self.num_recurrent_runs == 0


def example_dict(width: int, layers: int = 4, vocab: int = 32000) -> dict:
    """A configuration with the proportions of a real model of this width (16 heads of 128 per 2048 columns, latents of 512, feed-forwards of
    three times the width, 32 experts of which four take the dense one's work together): latent attention and retention in
    turn, dense and expert layers in turn two by two."""
    heads = max(8, width // 128)
    latent = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 3 * width // 8, "kv_rank": 512, "scale": 192 ** -0.5,
              "rot": {"base": 1e6, "dims": 64}}
    n = max(4, width // 256)
    retention = {"heads": n, "dim": 128, "vdim": 256, "decay": [1.0 - 2.0 ** (-4 - 6.0 * h / n) for h in range(n)], "rot": {"base": 1e4, "dims": 128}}
    dense = {"kind": "dense", "ff": 3 * width}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": 3 * width // 4}}
    kinds = [("latent_attention", latent, dense), ("retention", retention, moe), ("latent_attention", latent, moe), ("retention", retention, dense)]
    return {"architecture": "Goselix", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
            "layers": [dict(zip(("type", "mixer", "mlp"), kinds[i % 4])) for i in range(layers)]}
