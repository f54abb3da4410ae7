"""Specifications shared by designs whose layers are listed one by one: what a ``config.json`` says about one mechanism,
as a frozen dataclass.  A missing size is an error, an unknown key a warning; nothing has a default taken from one checkpoint."""
from __future__ import annotations

import warnings
from dataclasses import dataclass


def take(d: dict, what: str, keys: dict) -> dict:
    """The values of ``keys`` (name -> converter) in ``d``."""
    missing = [k for k in keys if k not in d]
    if missing:
        raise ValueError(f"{what}: missing {missing}")
    extra = sorted(set(d) - set(keys))
    if extra:
        warnings.warn(f"{what}: keys not used by this model: {extra}")
    return {k: conv(d[k]) for k, conv in keys.items()}


@dataclass(frozen=True)
class Rotation:
    """Pairs (i, i + dims / 2) of the first ``dims`` entries of a head, angle = position * base ** (-2 i / dims)."""
    base: float
    dims: int

    @classmethod
    def from_dict(cls, d: dict) -> "Rotation":
        r = cls(**take(d, "rot", {"base": float, "dims": int}))
        if r.dims < 0 or r.dims % 2:
            raise ValueError("rot.dims must be even")
        return r


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "silu"           # of the gate: see ops.ref.ACTIVATIONS


@dataclass(frozen=True)
class MoeSpec:
    """``score``: "sigmoid" (each logit on its own) or "softmax" (over the chosen logits only).  ``weigh``: whether the weight
    multiplies an expert's "input" or its "output".  ``limit`` belongs to the activations that clamp."""
    experts: int
    top: int
    ff: int
    act: str = "silu"
    limit: float = 0.0
    score: str = "sigmoid"
    weigh: str = "input"

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError("mlp.router: top must lie between 1 and experts")
