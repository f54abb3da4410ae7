"""Small Goselix models with random weights, and the checks that the CPU and the GPU tests share."""
import copy
import json
import os

import numpy as np
import torch
from safetensors.torch import save_file

import oracle_goselix as oracle


def _latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot}}


def _retention(dim, vdim, decay, rot_dims, base=10000.0):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def _model(vocab, width, layers, loop=None, eps=1e-5):
    d = {"architecture": "Goselix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = loop
    return d


CONFIGS = {
    # layers of different sizes, several experts per token, a layer without feed-forward, a loop in the middle, half-rotated heads
    "varied": _model(257, 96, [
        _layer("retention", _retention(24, 40, [0.9, 0.0, 1.0], 16), _moe(5, 2, 40)),
        _layer("latent_attention", _latent(3, 24, 16, 40, 56, 48, 0.17), _dense(136)),
        _layer("retention", _retention(48, 24, [0.99, 0.5], 32, 500.0), None),
        _layer("latent_attention", _latent(5, 16, 8, 8, 24, 32, 0.3, 300.0), _moe(3, 3, 24))], {"start": 1, "stop": 3, "times": 3}),
    # no size is a multiple of 8: the kernels that check every bound
    "odd": _model(101, 50, [
        _layer("latent_attention", _latent(5, 9, 6, 7, 11, 13, 0.31), _moe(4, 1, 11)),
        _layer("retention", _retention(10, 9, [0.97, 0.8, 0.999], 4), _dense(27)),
        _layer("latent_attention", _latent(1, 5, 2, 3, 7, 5, 0.5), None)], eps=1e-3),
    # everything looped, one pass more than twice; one head
    "looped": _model(130, 64, [
        _layer("retention", _retention(16, 8, [0.95], 16), _dense(64)),
        _layer("latent_attention", _latent(1, 32, 8, 16, 32, 16, 0.2), _dense(48))], {"start": 0, "stop": 2, "times": 4}),
    # sizes of the tensor-core kernels: several head groups, value slices and feature tiles
    "wide": _model(300, 256, [
        _layer("latent_attention", _latent(20, 128, 64, 128, 128, 256, 0.08), _moe(9, 4, 160)),
        _layer("retention", _retention(128, 200, [0.99, 0.9995, 0.7], 128), _dense(320)),
        _layer("retention", _retention(256, 64, [0.998], 64), None),
        _layer("latent_attention", _latent(3, 40, 32, 72, 64, 112, 0.12), _moe(16, 3, 64))], {"start": 0, "stop": 1, "times": 2}),
}


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H = m["heads"]
        out[p + "norm1"] = (W,)
        if l["type"] == "latent_attention":
            out.update({p + "mix.dq": (m["q_rank"], W), p + "mix.dq.norm": (m["q_rank"],), p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], W), p + "mix.dkv.norm": (m["kv_rank"],),
                        p + "mix.uk": (H * m["dim"], m["kv_rank"]), p + "mix.uv": (H * m["vdim"], m["kv_rank"]), p + "mix.o": (W, H * m["vdim"])})
        else:
            out.update({p + "mix.q": (H * m["dim"], W), p + "mix.k": (H * m["dim"], W), p + "mix.v": (H * m["vdim"], W),
                        p + "mix.g": (H * m["vdim"], W), p + "mix.o": (W, H * m["vdim"])})
        mlp = l["mlp"]
        if mlp is None:
            continue
        out[p + "norm2"] = (W,)
        if mlp["kind"] == "dense":
            out.update({p + "mlp.gate": (mlp["ff"], W), p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"])})
        else:
            out[p + "mlp.router"] = (mlp["router"]["experts"], W)
            F = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                out.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors.  Norm weights vary (a norm applied with the wrong weight shows); the query and key matrices of latent
    attention are scaled up, so that single keys stand out among hundreds and a lost or a wrong one shows."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if len(shape) == 1:
            t = 1.0 + 0.4 * t
        elif name == "loop.step":
            t = 0.5 * t
        elif name == "embed":
            pass
        else:
            gain = 2.0 if name.endswith((".uq", ".uk")) else 3.0 if name.endswith("router") else 1.0
            t = t * gain / shape[1] ** 0.5
        out[name] = t.bfloat16().contiguous()
    return out


def write_model(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


class Case:
    """A model on disk, its oracle logits per prompt (computed once), and engines over it."""

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

    def player(self, dtype="float32", block=16, blocks=64, slots=4, max_len=512):
        from tinyllmforge_b200.engine.engine import LLMEngine
        from tinyllmforge_b200.engine.replay import Replayer
        eng = LLMEngine(self.path, dtype=dtype, device=self.device, kvcache_block_size=block, num_kvcache_blocks=blocks, max_model_len=max_len,
                        max_num_batched_tokens=max(max_len, 512), max_num_seqs=slots, enforce_eager=True, skip_tokenizer_init=True)
        return Replayer(eng)

    def error(self, got, toks, positions):
        """RMS logit error per position, relative to the logits' spread."""
        want = self.want(toks)
        return ((torch.from_numpy(np.asarray(got)).double() - want[positions]).pow(2).mean(-1).sqrt() / want.std()).numpy()


def run(player, schedule):
    """schedule: [[(id, tokens of this step), ...], ...]; a request ends with the step that is its last.
    Returns {id: logits of all its tokens}."""
    last = {}
    for n, step in enumerate(schedule):
        for name, _ in step:
            last[name] = n
    out = {}
    for n, step in enumerate(schedule):
        entries = [{"id": name, "tokens": t, "want": list(range(len(t)))} for name, t in step]
        logits = player.step(entries, [name for name, _ in step if last[name] == n])
        at = 0
        for name, t in step:
            out.setdefault(name, []).append(logits[at:at + len(t)])
            at += len(t)
    return {k: np.concatenate(v) for k, v in out.items()}


def portions(toks, sizes):
    """The tokens cut into portions of the given sizes, the last size repeated."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = sizes[min(k, len(sizes) - 1)]
        out.append(toks[at:at + n])
        at, k = at + n, k + 1
    return out


def mixed_schedule(requests, sizes, live, seed=0):
    """Requests advance by portions of changing size, up to ``live`` at a time, some left out of a step now and then."""
    rng = np.random.default_rng(seed)
    waiting = list(requests.items())
    active, steps = {}, []
    while waiting or active:
        while waiting and len(active) < live:
            name, toks = waiting.pop(0)
            active[name] = list(toks)
        step = []
        for name in list(active):
            if len(active) > 1 and rng.random() < 0.25:
                continue
            n = int(rng.choice(sizes))
            step.append((name, active[name][:n]))
            del active[name][:n]
        if not step:
            continue
        steps.append(step)
        for name in [k for k, v in active.items() if not v]:
            del active[name]
    return steps
