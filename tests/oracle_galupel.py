"""A plain, slow Galupel decoder: one function per mechanism, whole sequences at once, no cache, no batching.

What the product's CPU and CUDA op sets are compared against.  It shares no code with them: weights are a dict of
tensors by checkpoint name, the configuration is the parsed ``config.json`` dict, arithmetic is in ``dtype`` (float64
unless asked otherwise).
"""
import math

import torch


# ------------------------------------------------------------------------------------------------ norms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def grouped_rms(x, w, groups, eps):
    """Every one of ``groups`` neighbouring parts of a row is divided by its own root mean square."""
    parts = [unit_rms(p, eps) for p in x.chunk(groups, dim=-1)]
    return torch.cat(parts, dim=-1) * w


# ------------------------------------------------------------------------------------------------ rotation
def rotate_neighbours(x, base, first_position=0):
    """x [tokens, heads, d], d even: entries 2i and 2i + 1 of a head turn together by position * base^(-2i / d)."""
    d = x.shape[-1]
    pos = torch.arange(first_position, first_position + x.shape[0], dtype=torch.float64)
    out = torch.empty_like(x)
    for i in range(d // 2):
        a = pos * base ** (-2.0 * i / d)
        c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def sliding(n, size):
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < size)


def pooled(x, pool):
    """x [tokens, heads, d] -> the mean of every whole block of ``pool`` tokens."""
    blocks = x.shape[0] // pool
    return torch.stack([x[b * pool:(b + 1) * pool].mean(dim=0) for b in range(blocks)]) if blocks else x[:0]


def blocks_behind(n, size, pool):
    """[tokens, blocks]: the block's last token lies before the token's window."""
    last = torch.arange(n // pool) * pool + pool - 1
    return last[None, :] <= torch.arange(n)[:, None] - size


def softmax_attention(q, k, v, scale, visible):
    """q [tokens, H, d], k [keys, G, d], v [keys, G, dv]; visible [tokens, keys]; scale a number or one per head."""
    share = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, dim=1), v.repeat_interleave(share, dim=1)
    s = torch.einsum("ihd,jhd->hij", q * scale, k).masked_fill(~visible, float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, dim=-1), v)


def pooled_window_attention(q, k, v, scale, size, pool):
    """A sliding window of tokens and, behind it, one key and value per whole block, in one softmax."""
    n = q.shape[0]
    keys, values = torch.cat([k, pooled(k, pool)]), torch.cat([v, pooled(v, pool)])
    return softmax_attention(q, keys, values, scale, torch.cat([sliding(n, size), blocks_behind(n, size, pool)], dim=1))


def attention(h, w, p, m, eps, lent):
    """``lent``: the keys and values of every earlier layer that has some, by layer number.  Returns output, keys, values."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).view(n, H, d), eps) * w[p + "q.norm"]
    if m.get("kv_from") is None:
        k = unit_rms((h @ w[p + "k"].T).view(n, G, d), eps) * w[p + "k.norm"]
        v = (h @ w[p + "v"].T).view(n, G, dv)
    else:
        k, v = lent[m["kv_from"]]
    o = pooled_window_attention(q, k, v, (m["scale"] * w[p + "temp"])[:, None], m["mask"]["size"], m["mask"]["pool"])
    return o.reshape(n, H * dv) @ w[p + "o"].T, k, v


def latent_attention(h, w, p, m, eps):
    n, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(n, H, d + r)
    low = h @ w[p + "dkv"].T
    c = unit_rms(low[:, :R], eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).view(n, H, d)
    v = (c @ w[p + "uv"].T).view(n, H, dv)
    base = m["rot"]["base"]
    k = torch.cat([k, rotate_neighbours(low[:, None, R:], base).expand(n, H, r)], dim=-1)
    q = torch.cat([q[..., :d], rotate_neighbours(q[..., d:], base)], dim=-1)
    return softmax_attention(q, k, v, m["scale"], sliding(n, m["mask"]["size"])).reshape(n, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def choose(scores, correction, top, count, keep):
    """Experts of one token, best first: the ``top`` largest of scores + correction within the ``keep`` best of ``count`` groups of
    neighbours, a group being as good as its two best experts together."""
    c = [float(s) for s in scores + correction]
    size = len(c) // count
    groups = [range(g * size, (g + 1) * size) for g in range(count)]
    worth = [sum(sorted((c[e] for e in g), reverse=True)[:2]) for g in groups]
    kept = sorted(range(count), key=lambda g: -worth[g])[:keep]
    return sorted((e for g in kept for e in groups[g]), key=lambda e: -c[e])[:top]


def experts(h, w, p, spec):
    r = spec["router"]
    scores = 1.0 / (1.0 + torch.exp(-(h @ w[p + "router"].T)))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(scores[t], w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"]):
            out[t] += scores[t, e] * (w[f"{p}e{e}.down"] @ gelu(w[f"{p}e{e}.up"] @ h[t]))
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [tokens, vocab]; ``trace``: a list that receives the residual stream after every layer."""
    w = {k: t.to(dtype) if t.is_floating_point() else t for k, t in weights.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = grouped_rms(w["embed"][torch.as_tensor(tokens)], w["embed.norm"], groups, eps)
    lent = {}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        if l["type"] == "attention":
            y, *lent[i] = attention(x, w, p + "mix.", m, eps, lent)
        else:
            y = latent_attention(x, w, p + "mix.", m, eps)
        x = x + grouped_rms(y, w[p + "norm1"], groups, eps)
        if l["mlp"] is not None:
            x = x + grouped_rms(experts(x, w, p + "mlp.", l["mlp"]), w[p + "norm2"], groups, eps)
        if trace is not None:
            trace.append(x)
    z = grouped_rms(x, w["final.norm"], groups, eps) @ w["embed"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])
