"""Small Mezapel models with random weights, and what the CPU and the GPU tests share."""
import copy

import torch

import oracle_mezapel as oracle
from goselix_cases import Case as BaseCase
from goselix_cases import write_model


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _chunk(heads, kv_heads, dim, vdim, size, scale, rot, mlp, base=10000.0, factor=4.0, original=64, fast=4.0, slow=0.25):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
                      "rot": {"base": base, "dims": rot, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}}


def _window(heads, kv_heads, dim, vdim, size, scale, rot, conv, cap, mlp, base=10000.0, factor=4.0, original=64, low=1.0, high=4.0):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "softcap": cap, "mask": {"size": size},
                      "rot": {"base": base, "dims": rot, "scaling": {"factor": factor, "original": original, "low": low, "high": high}}}}


def _model(vocab, width, streams, layers, loop=None, eps=1e-5, scale=3.0, buckets=31, mul_prev=5, mul_cur=3):
    d = {"architecture": "Mezapel", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers,
         "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # layers of different sizes, windows and chunks shorter and longer than a block, shared and unshared keys, a layer without feed-forward,
    # a loop in the middle
    "varied": _model(257, 96, 3, [
        _window(6, 2, 24, 16, 20, 0.2, 16, 4, 5.0, _dense(136)),
        _chunk(4, 4, 16, 24, 24, 0.25, 8, _dense(72)),
        _window(3, 3, 16, 8, 7, 0.3, 16, 2, 2.0, None, 300.0, 2.0, 32),
        _chunk(6, 1, 24, 40, 50, 0.2, 24, _dense(64), 500.0, 8.0, 128, 8.0, 1.0)], (1, 3, 3)),
    # no size is a multiple of 8: the kernels that check every bound; a convolution of one tap, a window and chunks of one token
    "odd": _model(101, 50, 5, [
        _chunk(5, 1, 9, 7, 33, 0.3, 6, _dense(27)),
        _window(6, 2, 9, 11, 5, 0.3, 4, 5, 9.0, None),
        _window(4, 4, 5, 13, 1, 0.4, 2, 1, 1.0, _dense(11)),
        _chunk(2, 2, 7, 3, 1, 0.4, 2, None)], eps=1e-3, buckets=1, mul_prev=7, mul_cur=11),
    # short, for generation; everything looped
    "short": _model(130, 64, 2, [
        _window(2, 1, 32, 16, 5, 0.2, 32, 4, 8.0, _dense(64)),
        _chunk(2, 2, 16, 32, 12, 0.3, 16, _dense(48))], (0, 2, 2), buckets=1009, mul_prev=141, mul_cur=19),
    # one stream, one kind of attention, nothing looped: no state per sequence, so cached prefixes are found again
    "chunks": _model(90, 48, 1, [
        _chunk(3, 1, 16, 16, 32, 0.3, 16, _dense(40)),
        _chunk(4, 2, 24, 8, 20, 0.2, 0, _dense(56))], scale=1.0),
    # sizes of the tensor-core kernels: several head groups, boxes and value slices
    "wide": _model(300, 256, 4, [
        _window(8, 2, 128, 72, 70, 0.09, 64, 4, 6.0, _dense(320)),
        _chunk(20, 1, 40, 192, 129, 0.15, 32, _dense(72)),
        _window(4, 4, 64, 64, 64, 0.125, 64, 3, 30.0, None),
        _chunk(4, 2, 256, 256, 64, 0.06, 96, _dense(128))], (1, 2, 2)),
}


def tensor_shapes(cfg):
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    out = {"embed": (V, W), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W), "final.norm": (W,), "final.norm.b": (W,), "head": (V, W)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for k in ("1",) if l["mlp"] is None else ("1", "2"):
            out.update({f"{p}norm{k}": (W,), f"{p}norm{k}.b": (W,), f"{p}hc{k}.in": (S,), f"{p}hc{k}.out": (S,), f"{p}hc{k}.mix": (S, S)})
        q = p + "mix."
        for name, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
            out[q + name] = (n, W)
            if l["type"] == "attention_2":
                out[q + name + ".conv"] = (n, m["conv"])
        per_head = l["type"] == "attention_2"
        out.update({q + "q.norm": (d if per_head else H * d,), q + "k.norm": (d if per_head else G * d,), q + "g": (H * dv if per_head else H, W), q + "o": (W, H * dv)})
        if per_head:
            out[q + "sink"] = (H,)
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors.  The norms of queries and keys are scaled up, so that single keys stand out and one that is lost, a window or a
    chunk that is one token off, or a sink left out shows."""
    g = torch.Generator().manual_seed(seed)
    S = cfg["streams"]
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.split(".")[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = 1.7 * (1.0 + 0.3 * t)
        elif last == "b":
            t = 0.3 * t
        elif last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.4 * t
        elif last == "in":
            t = 1.0 / S + 0.3 * t
        elif last == "out":
            t = 1.0 + 0.4 * t
        elif last == "mix":
            t = 0.9 * torch.eye(S) + 0.25 * t / S ** 0.5
        elif last == "conv":
            t = t * shape[1] ** -0.5
        elif last == "sink":
            t = 1.0 + t
        elif last == "g":
            t = 2.0 * t / shape[1] ** 0.5
        elif name not in ("embed", "bigram"):
            t = t / shape[1] ** 0.5
        out[name] = t.bfloat16().contiguous()
    return out


class Case(BaseCase):
    def __init__(self, name, path, device, seed=0):
        self.cfg = copy.deepcopy(CONFIGS[name])
        self.weights = random_weights(self.cfg, seed)
        self.path = write_model(path, self.cfg, self.weights)
        self.device = device
        self._want = {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self._want:
            self._want[key] = oracle.forward(self.cfg, self.weights, toks)
        return self._want[key]
