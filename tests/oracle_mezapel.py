"""A plain, slow Mezapel decoder: one function per mechanism, whole sequences at once, no cache, no batching.

What the product's CPU and CUDA op sets are compared against.  It shares no code with them: weights are a dict of
tensors by checkpoint name, the configuration is the parsed ``config.json`` dict, arithmetic is in ``dtype`` (float64
unless asked otherwise).
"""
import math

import torch


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------------------------------------ norms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------------------------------------ embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; the first token of a sequence, which has none before it, takes the last row."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embedding(tokens, w, e):
    b = e["bigram"]
    rows = bigram_rows([int(t) for t in tokens], b["buckets"], b["mul_prev"], b["mul_cur"])
    return w["embed"][torch.as_tensor(tokens)] * e["scale"] + w["bigram"][torch.tensor(rows)]


# ------------------------------------------------------------------------------------------------ residual streams
def gather_streams(xs, weights):
    """sum_s weights[s] x_s"""
    return sum(weights[s] * xs[s] for s in range(len(xs)))


def spread_streams(xs, y, mix, out):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, all at once."""
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out[t] * y for t in range(n)]


# ------------------------------------------------------------------------------------------------ rotation
def plain_frequencies(base, dims):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(base, dims, c):
    """Fast pairs keep their frequency, slow ones are divided by the factor, a linear ramp over the pair's index between."""
    def index_of(turns):
        return dims * math.log(c["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    first, last = max(math.floor(index_of(c["fast"])), 0), min(math.ceil(index_of(c["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(base, dims)):
        ramp = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(ramp * f / c["factor"] + (1.0 - ramp) * f)
    return out


def yarn_amplitude(c):
    return 1.0 + 0.1 * math.log(c["factor"])


def banded_frequencies(base, dims, c):
    """Short wavelengths are kept, long ones stretched by the factor, those between blended by their number of turns."""
    out = []
    for f in plain_frequencies(base, dims):
        wavelength = 2.0 * math.pi / f
        if wavelength < c["original"] / c["high"]:
            out.append(f)
        elif wavelength > c["original"] / c["low"]:
            out.append(f / c["factor"])
        else:
            s = (c["original"] / wavelength - c["low"]) / (c["high"] - c["low"])
            out.append((1.0 - s) * f / c["factor"] + s * f)
    return out


def rotate(x, frequencies, amplitude=1.0, first_position=0):
    """x [tokens, heads, d]; entry i of a head turns together with entry i + len(frequencies); later entries pass."""
    half = len(frequencies)
    pos = torch.arange(first_position, first_position + x.shape[0], dtype=torch.float64)
    angle = pos[:, None] * torch.tensor(frequencies, dtype=torch.float64)
    c, s = (amplitude * angle.cos()).to(x.dtype)[:, None], (amplitude * angle.sin()).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ------------------------------------------------------------------------------------------------ attention
def causal_conv(x, taps):
    """x [tokens, channels], taps [channels, n]: y_t = sum_i taps[:, i] x_(t - (n - 1) + i), zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for i in range(n):
        y = y + padded[i:i + x.shape[0]] * taps[:, i]
    return y


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def sliding(n, size):
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < size)


def chunked(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (j // size == i // size)


def sink_attention(q, k, v, scale, visible, sink, cap=None):
    """q [tokens, H, d], k [tokens, G, d], v [tokens, G, dv]; sink [H]: a score in the denominator alone."""
    share = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, dim=1), v.repeat_interleave(share, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap is not None:
        s = softcap(s, cap)
    s = s.masked_fill(~visible, float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return torch.einsum("hij,jhe->ihe", e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top)), v)


def chunk_attention(h, w, p, m, eps):
    """Norm over a whole projection, ramped rotation, attention inside chunks, a sink of score zero, one gate per head."""
    n, H, G, d, dv, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q = unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(n, G, dv)
    f, a = yarn_frequencies(rot["base"], rot["dims"], rot["scaling"]), yarn_amplitude(rot["scaling"])
    q, k = rotate(q.view(n, H, d), f, a), rotate(k.view(n, G, d), f, a)
    o = sink_attention(q, k, v, m["scale"], chunked(n, m["mask"]["size"]), torch.zeros(H, dtype=h.dtype))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(n, H * dv) @ w[p + "o"].T


def window_attention(h, w, p, m, eps):
    """Short convolutions, norm per head, banded rotation, capped scores, a sliding window, learned sinks, a gate per element."""
    n, H, G, d, dv, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q, k, v = (causal_conv(h @ w[p + c].T, w[p + c + ".conv"]) for c in "qkv")
    q, k = unit_rms(q.view(n, H, d), eps) * w[p + "q.norm"], unit_rms(k.view(n, G, d), eps) * w[p + "k.norm"]
    f = banded_frequencies(rot["base"], rot["dims"], rot["scaling"])
    o = sink_attention(rotate(q, f), rotate(k, f), v.view(n, G, dv), m["scale"], sliding(n, m["mask"]["size"]), w[p + "sink"], m["softcap"])
    return (o.reshape(n, H * dv) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ layers
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"attention": chunk_attention, "attention_2": window_attention}


def layer(xs, w, i, spec, eps):
    p = f"l{i}."

    def sublayer(xs, k, f):
        u = layer_norm(gather_streams(xs, w[f"{p}hc{k}.in"]), w[f"{p}norm{k}"], w[f"{p}norm{k}.b"], eps)
        return spread_streams(xs, f(u), w[f"{p}hc{k}.mix"], w[f"{p}hc{k}.out"])

    xs = sublayer(xs, 1, lambda u: MIXERS[spec["type"]](u, w, p + "mix.", spec["mixer"], eps))
    return xs if spec["mlp"] is None else sublayer(xs, 2, lambda u: dense(u, w, p + "mlp."))


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [tokens, vocab]; ``trace``: a list that receives the sum of the streams after every layer run."""
    w = {k: t.to(dtype) if t.is_floating_point() else t for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    xs = [embedding(tokens, w, cfg["embedding"])] * cfg["streams"]
    for i in layer_order(cfg):
        xs = layer(xs, w, i, cfg["layers"][i], eps)
        if trace is not None:
            trace.append(sum(xs))
    return layer_norm(sum(xs), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
