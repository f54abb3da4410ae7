"""Configuration of Tonapel, a decoder whose layers are listed one by one.

``config.json`` gives, for every layer, the type and the sizes of its mixer ("parallel": windowed attention beside a
state-space mixer, or "delta": the gated delta rule) and its feed-forward (dense, mixture of experts, or none), and the
model's vocabulary, width, norm constant and residual factor.
"""
from __future__ import annotations

from dataclasses import dataclass

from ..config import parse_dtype
from .specs import DenseSpec, MoeSpec, Rotation, take


def _positive(what: str, *sizes) -> None:
    if any(n < 1 for n in sizes):
        raise ValueError(f"{what}: sizes must be positive")


def _window(d: dict) -> int:
    size = take(d, "mask", {"size": int})["size"]
    if size < 1:
        raise ValueError("mask.size: a token sees at least itself")
    return size


@dataclass(frozen=True)
class WindowedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    window: int

    @classmethod
    def from_dict(cls, d: dict) -> "WindowedAttentionSpec":
        t = take(d, "left", {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float, "rot": Rotation.from_dict, "mask": _window})
        s = cls(window=t.pop("mask"), **t)
        _positive("left", s.heads, s.kv_heads, s.dim, s.vdim)
        if s.heads % s.kv_heads:
            raise ValueError("left: kv_heads must divide heads")
        if s.rot.dims > s.dim:
            raise ValueError("left: rot.dims cannot exceed dim")
        return s


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: dict) -> "StateSpaceSpec":
        s = cls(**take(d, "right", {k: int for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}))
        _positive("right", s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups)
        if s.heads % s.groups:
            raise ValueError("right: groups must divide heads")
        if s.inner % s.norm_groups:
            raise ValueError("right: norm_groups must divide heads * vdim")
        return s

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Of the short convolution: x | B | C."""
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class ParallelSpec:
    left: WindowedAttentionSpec
    right: StateSpaceSpec
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "ParallelSpec":
        return cls(**take(d, "parallel", {"left": WindowedAttentionSpec.from_dict, "right": StateSpaceSpec.from_dict,
                                          "left_scale": float, "right_scale": float}))


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, d: dict) -> "DeltaSpec":
        s = cls(**take(d, "delta", {k: int for k in ("heads", "kv_heads", "dim", "vdim", "conv")}))
        _positive("delta", s.heads, s.kv_heads, s.dim, s.vdim, s.conv)
        if s.heads % s.kv_heads:
            raise ValueError("delta: kv_heads must divide heads")
        return s

    @property
    def channels(self) -> int:
        """Of the short convolutions: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


def _mlp_from_dict(d):
    if d is None:
        return None
    kind = d.get("kind")
    if kind == "dense":
        return DenseSpec(int(d["ff"]), act="gelu_tanh")
    if kind == "moe":
        router = take(d["router"], "mlp.router", {"experts": int, "top": int})
        expert = take(d["expert"], "mlp.expert", {"ff": int, "limit": float})
        return MoeSpec(router["experts"], router["top"], expert["ff"], act="clamped_swish", limit=expert["limit"], score="softmax", weigh="output")
    raise ValueError(f"unknown feed-forward kind {kind!r}; known: dense, moe")


MIXER_SPECS = {"parallel": ParallelSpec, "delta": DeltaSpec}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: object

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d.get("type") not in MIXER_SPECS:
            raise ValueError(f"unknown layer type {d.get('type')!r}; known: {sorted(MIXER_SPECS)}")
        return cls(d["type"], MIXER_SPECS[d["type"]].from_dict(d["mixer"]), _mlp_from_dict(d.get("mlp")))


@dataclass
class TonapelConfig:
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    residual_mult: float
    layers: tuple
    torch_dtype: str = "bfloat16"
    eos_token_id: int = -1
    max_position_embeddings: int = 1 << 20      # the design names no limit; rotary tables are built for max_model_len

    quantizable = False
    prefix_cacheable = False                    # every layer has a recurrent state, which cached blocks do not hold

    @classmethod
    def from_dict(cls, d: dict) -> "TonapelConfig":
        for key in ("vocab", "width", "norm", "residual_mult", "layers"):
            if key not in d:
                raise ValueError(f"Tonapel config: missing {key!r}")
        if not d["layers"]:
            raise ValueError("Tonapel config: no layers")
        cfg = cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["residual_mult"]),
                  tuple(LayerSpec.from_dict(l) for l in d["layers"]),
                  torch_dtype=str(d.get("torch_dtype") or d.get("dtype") or "bfloat16").replace("torch.", ""))
        if d.get("eos_token_id") is not None:
            eos = d["eos_token_id"]
            cfg.eos_token_id = int(eos[0] if isinstance(eos, (list, tuple)) else eos)
        if d.get("max_position_embeddings"):
            cfg.max_position_embeddings = int(d["max_position_embeddings"])
        return cfg

    def validate_tp(self, size: int) -> None:
        if size != 1:
            raise ValueError("Tonapel runs on one GPU (tensor_parallel_size=1)")

    @property
    def dtype(self):
        return parse_dtype(self.torch_dtype)

    @property
    def num_recurrent_runs(self) -> int:
        return len(self.layers)


def example_dict(width: int, layers: int = 4, vocab: int = 32000) -> dict:
    """A configuration with the proportions of a real model of this width: heads of 128, four query heads per key/value head,
    a window of 1024, state-space heads of 64 with a state of 128, a feed-forward of three times the width, 32 experts of which
    four take the dense one's work together; parallel and delta layers in turn, dense and expert layers in turn two by two."""
    heads = max(8, width // 128)
    left = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 64},
            "mask": {"size": 1024}}
    right = {"heads": width // 64, "vdim": 64, "state": 128, "groups": max(1, width // 1024), "conv": 4, "norm_groups": max(1, width // 1024)}
    parallel = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.7}
    delta = {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}
    dense = {"kind": "dense", "ff": 3 * width}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": 3 * width // 4, "limit": 7.0}}
    kinds = [("parallel", parallel, dense), ("delta", delta, moe), ("parallel", parallel, moe), ("delta", delta, dense)]
    return {"architecture": "Tonapel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "layers": [dict(zip(("type", "mixer", "mlp"), kinds[i % 4])) for i in range(layers)]}
