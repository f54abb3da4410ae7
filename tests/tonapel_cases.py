"""Small Tonapel models with random weights, and what the CPU and the GPU tests share."""
import copy

import torch

import oracle_tonapel as oracle
from goselix_cases import Case as BaseCase
from goselix_cases import write_model


def _left(heads, kv_heads, dim, vdim, window, scale, rot, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}, "mask": {"size": window}}


def _right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _parallel(left, right, left_scale, right_scale, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def _delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def _model(vocab, width, mult, layers, eps=1e-5):
    return {"architecture": "Tonapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


CONFIGS = {
    # layers of different sizes, windows shorter and longer than a block, shared and unshared keys, a layer without feed-forward
    "varied": _model(257, 96, 0.7, [
        _parallel(_left(6, 2, 24, 40, 20, 0.3, 16), _right(4, 24, 16, 2, 4, 4), 0.9, 0.4, _moe(5, 2, 40, 0.8)),
        _delta(6, 3, 24, 16, 2, _dense(136)),
        _parallel(_left(3, 3, 16, 8, 7, 0.5, 16, 300.0), _right(3, 16, 24, 1, 3, 1), 0.3, 1.1, None),
        _delta(2, 2, 16, 40, 4, _moe(3, 3, 24, 2.5))]),
    # no size is a multiple of 8: the kernels that check every bound
    "odd": _model(101, 50, 1.0, [
        _delta(6, 2, 9, 7, 5, _moe(4, 1, 11, 0.4)),
        _parallel(_left(5, 1, 9, 7, 1, 0.4, 6), _right(3, 5, 11, 3, 2, 5), 1.0, 1.0, _dense(27)),
        _parallel(_left(4, 4, 5, 13, 33, 0.6, 2), _right(2, 6, 3, 1, 1, 2), 0.5, 0.6, None)], eps=1e-3),
    # short, for generation; a convolution of one tap, one head
    "short": _model(130, 64, 0.5, [
        _delta(1, 1, 32, 16, 1, _dense(64)),
        _parallel(_left(2, 1, 32, 16, 5, 0.35, 32), _right(1, 32, 16, 1, 4, 2), 0.8, 0.8, _moe(6, 2, 32, 1.5))]),
    # sizes of the tensor-core kernels: several column slices, head groups, boxes and feature tiles
    "wide": _model(300, 256, 0.4, [
        _parallel(_left(8, 2, 128, 72, 70, 0.09, 64), _right(6, 64, 128, 2, 4, 3), 0.7, 0.9, _moe(9, 3, 160, 1.2)),
        _delta(4, 2, 128, 136, 4, _dense(320)),
        _parallel(_left(20, 1, 40, 192, 129, 0.2, 40), _right(2, 136, 48, 1, 3, 2), 0.6, 0.5, _dense(72)),
        _delta(3, 3, 160, 64, 3, _moe(16, 4, 64, 0.9)),
        _parallel(_left(4, 4, 256, 256, 64, 0.0625, 96), _right(2, 80, 192, 2, 2, 1), 0.5, 0.5, None)]),
}


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if l["type"] == "delta":
            q, v = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, n in (("q", q), ("k", q), ("v", v)):
                out.update({f"{p}mix.{name}": (n, W), f"{p}mix.{name}.conv": (n, m["conv"])})
            out.update({p + "mix.g": (v, W), p + "mix.b": (m["heads"], W), p + "mix.a": (m["heads"], W), p + "mix.A_log": (m["heads"],),
                        p + "mix.dt_bias": (m["heads"],), p + "mix.norm": (m["vdim"],), p + "mix.o": (W, v)})
        else:
            a, r, q = m["left"], m["right"], p + "mix.left."
            for name, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out.update({q + name: (n, W), q + name + ".b": (n,)})
            out.update({q + "o": (W, a["heads"] * a["vdim"]), q + "o.b": (W,)})
            inner, channels, q = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"], p + "mix.right."
            out.update({q + "in": (inner + channels + r["heads"], W), q + "conv": (channels, r["conv"]), q + "conv.b": (channels,),
                        q + "dt_bias": (r["heads"],), q + "A_log": (r["heads"],), q + "D": (r["heads"],), q + "norm": (inner,), q + "o": (W, inner)})
        mlp = l["mlp"]
        if mlp is None:
            continue
        out.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if mlp["kind"] == "dense":
            out.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
        else:
            out[p + "mlp.router"] = (mlp["router"]["experts"], W)
            F = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors.  Query and key matrices of the attention are scaled up, so that single keys stand out and one that is lost
    or a window that is one token off shows; decays keep a token alive for some tens of tokens."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.split(".")[-1]
        if last == "A_log":
            t = -3.0 + 1.2 * t
        elif last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":
            t = 0.4 * t
        elif last == "norm":
            t = 1.0 + 0.4 * t
        elif last == "conv":
            t = t * shape[1] ** -0.5
        elif len(shape) == 2 and name != "embed":
            gain = 2.0 if name.endswith(("left.q", "left.k")) else 3.0 if last == "router" else 1.0
            t = t * gain / shape[1] ** 0.5
        elif len(shape) == 1:
            t = 0.5 * t
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
