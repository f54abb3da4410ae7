"""Specifications shared by designs whose layers are listed one by one: what a ``config.json`` says about one mechanism,
as a frozen dataclass.  A missing size is an error, an unknown key a warning; nothing has a default taken from one checkpoint."""
from __future__ import annotations

import math
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
class RampScaling:
    """YaRN: pairs that turn more than ``fast`` times within ``original`` positions keep their frequency, pairs that turn less than
    ``slow`` times have it divided by ``factor``, with a linear ramp over the pair's index between; cos and sin grow a little."""
    factor: float
    original: float
    fast: float
    slow: float

    @classmethod
    def from_dict(cls, d: dict) -> "RampScaling":
        return cls(**take(d, "rot.scaling", {k: float for k in ("factor", "original", "fast", "slow")}))

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def apply(self, freqs: list, base: float, dims: int) -> list:
        def pair_with(turns):
            return dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(base))

        lo = max(math.floor(pair_with(self.fast)), 0)
        hi = min(math.ceil(pair_with(self.slow)), dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(freqs))]
        return [f / self.factor * r + f * (1.0 - r) for f, r in zip(freqs, ramp)]


@dataclass(frozen=True)
class BandScaling:
    """Llama 3.1: wavelengths below ``original / high`` are kept, those above ``original / low`` stretched by ``factor``, blended between."""
    factor: float
    original: float
    low: float
    high: float
    amplitude = 1.0

    @classmethod
    def from_dict(cls, d: dict) -> "BandScaling":
        return cls(**take(d, "rot.scaling", {k: float for k in ("factor", "original", "low", "high")}))

    def apply(self, freqs: list, base: float, dims: int) -> list:
        def scaled(f):
            wave = 2 * math.pi / f
            if wave < self.original / self.high:
                return f
            if wave > self.original / self.low:
                return f / self.factor
            keep = (self.original / wave - self.low) / (self.high - self.low)
            return (1.0 - keep) * f / self.factor + keep * f

        return [scaled(f) for f in freqs]


@dataclass(frozen=True)
class Rotation:
    """Pairs (i, i + dims / 2) of the first ``dims`` entries of a head, or neighbours (2 i, 2 i + 1) if ``interleaved``; angle =
    position * base ** (-2 i / dims), with the frequencies changed by ``scaling`` if there is one."""
    base: float
    dims: int
    scaling: object = None
    interleaved: bool = False

    @classmethod
    def from_dict(cls, d: dict, scaling=None, interleaved: bool = False) -> "Rotation":
        """``scaling``: the class that reads ``rot.scaling`` in this design, None if it knows none."""
        keys = {"base": float, "dims": int}
        if scaling is not None and d.get("scaling") is not None:
            keys["scaling"] = scaling.from_dict
        r = cls(**take(d, "rot", keys), interleaved=interleaved)
        if r.dims < 0 or r.dims % 2:
            raise ValueError("rot.dims must be even")
        return r

    @property
    def frequencies(self) -> list:
        freqs = [self.base ** (-2 * i / self.dims) for i in range(self.dims // 2)]
        return freqs if self.scaling is None else self.scaling.apply(freqs, self.base, self.dims)

    @property
    def amplitude(self) -> float:
        """Factor of cos and sin."""
        return 1.0 if self.scaling is None else self.scaling.amplitude


NO_ROTATION = Rotation(1.0, 0)


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run ``times`` times in a row before the rest follow."""
    start: int
    stop: int
    times: int

    @classmethod
    def from_dict(cls, d: dict, layers: int) -> "LoopSpec":
        loop = cls(**take(d, "loop", {"start": int, "stop": int, "times": int}))
        if not (0 <= loop.start < loop.stop <= layers and loop.times >= 1):
            raise ValueError("loop must name a range of layers and at least one pass")
        return loop


def layer_runs(layers: int, loop: LoopSpec | None) -> list:
    """[(layer, pass)] in the order of computation; pass is None for a layer outside the loop."""
    if loop is None:
        return [(i, None) for i in range(layers)]
    return ([(i, None) for i in range(loop.start)]
            + [(i, t) for t in range(loop.times) for i in range(loop.start, loop.stop)]
            + [(i, None) for i in range(loop.stop, layers)])


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention with normed queries and keys.  A query at position i sees the keys j <= i of its own chunk of ``window``
    positions (``chunked``) or the last ``window`` tokens.  ``conv``: taps of the short convolutions ahead of the norms (0: none).
    ``norm``: over each "head" or over "all" rows of a projection at once.  ``sink``: a score that only the denominator
    sees, "learned" per head, "zero", or None.  ``softcap``: bound of the scores (0: none).  ``gate``: one sigmoid per "head" or per
    "element" of the output, or None.  ``pool``: behind the window, one key and value (the means) for every whole block of that many
    tokens of the sequence that lies before the window (0: none).  ``temper``: a learned factor of the scores per head.  ``kv_from``: the
    layer whose keys and values are used instead of own ones."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    window: int
    chunked: bool = False
    conv: int = 0
    norm: str = "head"
    sink: str | None = None
    softcap: float = 0.0
    gate: str | None = None
    pool: int = 0
    temper: bool = False
    kv_from: int | None = None

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1:
            raise ValueError("attention: sizes must be positive")
        if self.heads % self.kv_heads:
            raise ValueError("attention: kv_heads must divide heads")
        if self.rot.dims > self.dim:
            raise ValueError("attention: rot.dims cannot exceed dim")
        if self.window < 1:
            raise ValueError("attention: mask.size: a token sees at least itself")
        if self.pool < 0 or (self.pool and self.chunked):
            raise ValueError("attention: mask.pool: blocks of at least one token behind a sliding window")
        if self.kv_from is not None and (self.conv or self.norm != "head"):
            raise ValueError("attention: kv_from goes with norms per head and no convolutions")

    @property
    def gate_columns(self) -> int:
        return {None: 0, "head": self.heads, "element": self.heads * self.vdim}[self.gate]


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention over one latent of ``kv_rank`` entries per token, from which keys and values of every head are made, and one rotated key
    part of ``rot_dim`` entries for all heads.  ``q_rank``: size of a latent of the queries (0: queries come from the input itself).
    ``window``: a token sees the last ``window`` tokens (0: all)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation
    q_rank: int = 0
    window: int = 0

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.kv_rank) < 1 or self.q_rank < 0:
            raise ValueError("latent_attention: sizes must be positive")
        if self.rot.dims != self.rot_dim:
            raise ValueError("latent_attention: the whole rotated part is rotated (rot.dims == rot_dim)")
        if self.window < 0:
            raise ValueError("latent_attention: mask.size: a token sees at least itself")


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "silu"           # of the gate: see ops.ref.ACTIVATIONS


@dataclass(frozen=True)
class MoeSpec:
    """``score``: "sigmoid" (each logit on its own) or "softmax" (over the chosen logits only).  ``weigh``: whether the weight
    multiplies an expert's "input" or its "output".  ``limit`` belongs to the activations that clamp.  ``gated``: an expert is
    down(act(gate h, up h)), else down(act(up h)).  ``correction``: a learned number per expert is added to the scores that choose, not to those
    that weigh.  ``groups``: experts form that many groups of neighbours, and only those of the ``keep`` groups whose two best experts are
    best together can be chosen."""
    experts: int
    top: int
    ff: int
    act: str = "silu"
    limit: float = 0.0
    score: str = "sigmoid"
    weigh: str = "input"
    gated: bool = True
    correction: bool = False
    groups: int = 1
    keep: int = 1

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError("mlp.router: top must lie between 1 and experts")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError("mlp.router: groups.count must divide experts, groups.keep lie between 1 and groups.count")
        if self.top > self.keep * (self.experts // self.groups):
            raise ValueError("mlp.router: the groups kept must hold at least top experts")
        if self.score == "softmax" and (self.correction or self.groups > 1):
            raise ValueError("mlp.router: corrections and groups go with sigmoid scores")
