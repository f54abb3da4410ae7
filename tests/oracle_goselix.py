"""A plain, slow Goselix decoder: one function per mechanism, whole sequences at once, no cache, no batching.

What the product's CPU and CUDA op sets are compared against.  It shares no code with them: weights are a dict of
tensors by checkpoint name, the configuration is the parsed ``config.json`` dict, arithmetic is in ``dtype`` (float64
unless asked otherwise).
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def rotate(x, base, dims, first_position=0):
    """x: [tokens, heads, d]; the first ``dims`` entries of each head are rotated, entry i together with i + dims / 2."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            angle = (first_position + t) * base ** (-2.0 * i / dims)
            c, s = math.cos(angle), math.sin(angle)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def causal_softmax_attention(q, k, v, scale):
    """q, k: [tokens, heads, d]; v: [tokens, heads, dv]."""
    n = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    hidden = torch.ones(n, n, dtype=torch.bool).triu(1)
    scores = scores.masked_fill(hidden, float("-inf"))
    weights = torch.softmax(scores, dim=-1)
    return torch.einsum("hij,jhe->ihe", weights, v)


def latent_attention(h, w, p, m, eps):
    """Keys and values are rebuilt per head from the normed latent; one rotated key part is shared by all heads."""
    n, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).view(n, H, d + r)
    both = h @ w[p + "dkv"].T
    c = rms_norm(both[:, :rank], w[p + "dkv.norm"], eps)
    k_rot = rotate(both[:, None, rank:], m["rot"]["base"], r)
    q_rot = rotate(q[:, :, d:], m["rot"]["base"], r)
    k = torch.cat([(c @ w[p + "uk"].T).view(n, H, d), k_rot.expand(n, H, r)], dim=-1)
    v = (c @ w[p + "uv"].T).view(n, H, dv)
    o = causal_softmax_attention(torch.cat([q[:, :, :d], q_rot], dim=-1), k, v, m["scale"])
    return o.reshape(n, H * dv) @ w[p + "o"].T


def retention_scan(q, k, v, decay):
    """Token by token: S <- decay S + k v^T; o = S^T q.  q, k: [tokens, heads, d], v: [tokens, heads, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    g = torch.as_tensor(decay, dtype=q.dtype).view(H, 1, 1)
    out = []
    for t in range(n):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def retention(h, w, p, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w[p + "q"].T).view(n, H, d), m["rot"]["base"], m["rot"]["dims"])
    k = rotate((h @ w[p + "k"].T).view(n, H, d), m["rot"]["base"], m["rot"]["dims"]) * d ** -0.5
    v = (h @ w[p + "v"].T).view(n, H, dv)
    o, _ = retention_scan(q, k, v, m["decay"])
    o = unit_rms(o, eps).reshape(n, H * dv) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def route(h, router, top):
    """(experts [tokens, top], weights [tokens, top]): the largest sigmoid scores, not renormalised."""
    s = 1.0 / (1.0 + torch.exp(-(h @ router.T)))
    weights, experts = torch.sort(s, dim=-1, descending=True, stable=True)
    return experts[:, :top], weights[:, :top]


def mixture(h, w, p, m):
    experts, weights = route(h, w[p + "router"], m["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(experts[t].tolist(), weights[t]):
            q = f"{p}e{e}."
            out[t] += gated_ff((s * h[t])[None], w[q + "gate"], w[q + "up"], w[q + "down"])[0]
    return out


def layer(x, w, i, spec, eps):
    """Mixer and feed-forward both read x; their sum is added to it."""
    p = f"l{i}."
    mixers = {"latent_attention": latent_attention, "retention": retention}
    y = mixers[spec["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    if spec["mlp"] is not None:
        h = rms_norm(x, w[p + "norm2"], eps)
        if spec["mlp"]["kind"] == "moe":
            y = y + mixture(h, w, p + "mlp.", spec["mlp"])
        else:
            y = y + gated_ff(h, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
    return x + y


def layer_runs(cfg):
    """[(layer, pass)] in the order they are computed; pass is None outside the loop."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [tokens, vocab]; ``trace``: a list that receives the residual stream after every layer run."""
    w = {k: t.to(dtype) if t.is_floating_point() else t for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    embedded = w["embed"][torch.as_tensor(tokens)]
    x = embedded.clone()
    for i, t in layer_runs(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            if t > 0:
                x = x + embedded
            x = x + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps)
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
