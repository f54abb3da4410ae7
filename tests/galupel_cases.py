"""Small Galupel models with random weights, and what the CPU and the GPU tests share."""
import copy

import torch

import oracle_galupel as oracle
from goselix_cases import Case as BaseCase
from goselix_cases import write_model


def _moe(experts, top, ff, count=1, keep=1):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}, "expert": {"ff": ff}}


def _attend(heads, kv_heads, dim, vdim, size, pool, scale, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size, "pool": pool}}
    return {"type": "attention", "mixer": m if kv_from is None else {**m, "kv_from": kv_from}, "mlp": mlp}


def _latent(heads, dim, rot, vdim, rank, size, scale, mlp, base=10000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": size},
                      "rot": {"base": base, "dims": rot}}}


def _model(vocab, width, groups, layers, eps=1e-5, scale=0.7, cap=9.0):
    return {"architecture": "Galupel", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "layers": layers, "logit_scale": scale,
            "logit_softcap": cap}


CONFIGS = {
    # layers of different sizes, windows shorter and longer than a page, blocks that divide a page and blocks that do not, keys and values of another
    # layer under another window with the same and with other blocks, a layer without feed-forward
    "varied": _model(257, 96, 3, [
        _attend(6, 2, 24, 16, 20, 4, 0.3, _moe(8, 3, 40, 4, 2)),
        _latent(3, 24, 16, 40, 48, 24, 0.25, _moe(6, 2, 24, 2, 1)),
        _attend(6, 2, 24, 16, 33, 5, 0.35, None, 0),
        _attend(4, 4, 16, 24, 7, 7, 0.3, _moe(5, 5, 16)),
        _latent(5, 16, 8, 8, 32, 9, 0.4, _moe(9, 2, 32, 3, 2), 300.0),
        _attend(6, 2, 24, 16, 11, 4, 0.25, _moe(4, 1, 72, 2, 2), 0)]),
    # no size is a multiple of 8: the kernels that check every bound; a window of one token, blocks of one token and longer than a page, every group
    # of columns odd, one expert to a group
    "odd": _model(101, 50, 2, [
        _latent(5, 9, 6, 7, 13, 33, 0.3, _moe(4, 2, 11, 4, 3)),
        _attend(6, 2, 9, 11, 5, 3, 0.5, None),
        _latent(1, 5, 2, 3, 5, 1, 0.5, _moe(3, 3, 7)),
        _attend(4, 4, 5, 13, 1, 1, 0.6, _moe(6, 2, 9, 2, 1)),
        _attend(6, 2, 9, 11, 3, 19, 0.5, _moe(6, 1, 9, 3, 1), 1)], eps=1e-3),
    # short, for generation
    "short": _model(130, 64, 4, [
        _attend(2, 1, 32, 16, 6, 4, 0.3, _moe(4, 2, 32, 2, 1)),
        _latent(2, 16, 16, 32, 40, 12, 0.3, _moe(4, 2, 24, 2, 2)),
        _attend(2, 1, 32, 16, 10, 4, 0.3, _moe(3, 1, 24), 0)], scale=1.5, cap=20.0),
    # sizes of the tensor-core kernels: several head groups, boxes, value slices and tiles of blocks
    "wide": _model(300, 256, 4, [
        _attend(8, 2, 128, 72, 70, 3, 0.12, _moe(16, 4, 160, 4, 2)),
        _latent(20, 128, 64, 128, 256, 65, 0.1, _moe(9, 3, 64, 3, 3)),
        _attend(20, 1, 40, 192, 129, 16, 0.2, _moe(80, 6, 24, 8, 4)),
        _latent(3, 40, 32, 72, 112, 200, 0.15, None),
        _attend(8, 2, 128, 72, 64, 2, 0.1, _moe(40, 4, 32, 1, 1), 0)]),
    # one group, no experts at all, logits nearly unbounded
    "bare": _model(64, 40, 1, [_attend(5, 5, 8, 8, 16, 8, 0.4, None), _latent(2, 8, 8, 8, 16, 40, 0.4, None)], scale=1.0, cap=1000.0),
}


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
        H, d, dv, q = m["heads"], m["dim"], m["vdim"], f"l{i}.mix."
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            out.update({q + "q": (H * d, W), q + "q.norm": (d,), q + "temp": (H,), q + "o": (W, H * dv)})
            if m.get("kv_from") is None:
                out.update({q + "k": (m["kv_heads"] * d, W), q + "v": (m["kv_heads"] * dv, W), q + "k.norm": (d,)})
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            out.update({q + "q": (H * (d + r), W), q + "dkv": (R + r, W), q + "dkv.norm": (R,), q + "uk": (H * d, R), q + "uv": (H * dv, R), q + "o": (W, H * dv)})
        if mlp is not None:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors.  What makes queries and keys is scaled up, so that single keys stand out and one that is lost, or a window or a block that
    is one token off, shows; corrections are as large as scores, and some sums are negative."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.split(".")[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = 1.3 * (1.0 + 0.3 * t)
        elif last in ("norm", "norm1"):
            t = 1.0 + 0.4 * t
        elif last == "norm2":                   # small: where a rounded router's close call goes the other way, the rest still agrees
            t = 0.25 * (1.0 + 0.4 * t)
        elif last == "temp":
            t = 1.0 + 0.3 * t
        elif last == "correction":
            t = 0.5 * t - 0.3
        elif name != "embed":
            t = t * (2.0 if name.endswith((".uk", "mix.q")) else 1.5 if last == "router" else 1.0) / shape[1] ** 0.5
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
