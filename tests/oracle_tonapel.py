"""A plain, slow Tonapel decoder: one function per mechanism, whole sequences at once, no cache, no batching.

What the product's CPU and CUDA op sets are compared against.  It shares no code with them: weights are a dict of
tensors by checkpoint name, the configuration is the parsed ``config.json`` dict, arithmetic is in ``dtype`` (float64
unless asked otherwise).
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def shifted_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x, taps, bias=None):
    """x [tokens, channels], taps [channels, n]: y_t = sum_i taps[:, i] x_(t - (n - 1) + i), zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for i in range(n):
        y = y + padded[i:i + x.shape[0]] * taps[:, i]
    return y if bias is None else y + bias


# ------------------------------------------------------------------------------------------------ windowed attention
def rotate(x, base, dims, first_position=0):
    """x [tokens, heads, d]; the first ``dims`` entries of each head are rotated, entry i together with i + dims / 2."""
    half = dims // 2
    pos = torch.arange(first_position, first_position + x.shape[0], dtype=torch.float64)
    angle = pos[:, None] * torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    c, s = angle.cos().to(x.dtype)[:, None], angle.sin().to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def windowed_attention(q, k, v, scale, window):
    """q [tokens, H, d], k [tokens, G, d], v [tokens, G, dv]; token i sees the tokens j with 0 <= i - j < window."""
    n, share = q.shape[0], q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(share, dim=1), v.repeat_interleave(share, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    scores = scores.masked_fill((back < 0) | (back >= window), float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(scores, dim=-1), v)


def attention(h, w, p, m):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(n, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(n, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    rot = m["rot"]
    o = windowed_attention(rotate(q, rot["base"], rot["dims"]), rotate(k, rot["base"], rot["dims"]), v, m["scale"], m["mask"]["size"])
    return o.reshape(n, H * dv) @ w[p + "o"].T + w[p + "o.b"]


# ------------------------------------------------------------------------------------------------ state-space duality
def ssd_scan(x, B, C, dt, A_log, D, S=None):
    """x [tokens, H, dv], B and C [tokens, G, N], dt [tokens, H]: S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x."""
    n, H, dv = x.shape
    share = H // B.shape[1]
    B, C = B.repeat_interleave(share, dim=1), C.repeat_interleave(share, dim=1)
    S = torch.zeros(H, B.shape[2], dv, dtype=x.dtype) if S is None else S
    ys = []
    for t in range(n):
        S = torch.exp(-torch.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        ys.append(torch.einsum("hne,hn->he", S, C[t]) + D[:, None] * x[t])
    return torch.stack(ys), S


def grouped_gate_norm(y, z, weight, groups, eps):
    """y silu(z), every one of ``groups`` equal parts divided by its own root mean square, times the weight."""
    y = y * silu(z)
    return unit_rms(y.view(y.shape[0], groups, -1), eps).reshape(y.shape) * weight


def ssd(h, w, p, m, eps):
    n, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], dim=-1)
    y, _ = ssd_scan(x.reshape(n, H, dv), B.reshape(n, G, N), C.reshape(n, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return grouped_gate_norm(y.reshape(n, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * attention(h, w, p + "left.", m["left"]) + m["right_scale"] * ssd(h, w, p + "right.", m["right"], eps)


# ------------------------------------------------------------------------------------------------ gated delta rule
def unit_vectors(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, g, beta, S=None):
    """q, k [tokens, H, d], v [tokens, H, dv], g and beta [tokens, H]: S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if S is None else S
    out = []
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def delta(h, w, p, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + c].T, w[p + c + ".conv"])) for c in "qkv")
    q, k = unit_vectors(q.view(n, G, d)) * d ** -0.5, unit_vectors(k.view(n, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_scan(q, k, v.view(n, H, dv), g, sigmoid(h @ w[p + "b"].T))
    o = unit_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(n, H, dv)
    return o.reshape(n, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forwards
def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(h, gate, up, down, limit):
    g, u = torch.clamp(h @ gate.T, max=limit), torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, top):
    """(experts [tokens, top], weights [tokens, top]): the largest logits, weighted by the softmax over these alone."""
    z, experts = torch.sort(h @ router.T, dim=-1, descending=True, stable=True)
    return experts[:, :top], torch.softmax(z[:, :top], dim=-1)


def mixture(h, w, p, m):
    experts, weights = route(h, w[p + "router"], m["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(experts[t].tolist(), weights[t]):
            q = f"{p}e{e}."
            out[t] += s * clamped_expert(h[t][None], w[q + "gate"], w[q + "up"], w[q + "down"], m["expert"]["limit"])[0]
    return out


# ------------------------------------------------------------------------------------------------ layers
def layer(x, w, i, spec, mult, eps):
    """Each sublayer is normed on its way in and on its way out; its result is added with the factor ``mult``."""
    p = f"l{i}."
    mixers = {"parallel": parallel, "delta": delta}
    y = mixers[spec["type"]](shifted_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    x = x + mult * shifted_norm(y, w[p + "norm1b"], eps)
    if spec["mlp"] is None:
        return x
    h = shifted_norm(x, w[p + "norm2"], eps)
    y = mixture(h, w, p + "mlp.", spec["mlp"]) if spec["mlp"]["kind"] == "moe" else dense(h, w, p + "mlp.")
    return x + mult * shifted_norm(y, w[p + "norm2b"], eps)


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [tokens, vocab]; ``trace``: a list that receives the residual stream after every layer."""
    w = {k: t.to(dtype) if t.is_floating_point() else t for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, cfg["residual_mult"], eps)
        if trace is not None:
            trace.append(x.clone())
    return shifted_norm(x, w["final.norm"], eps) @ w["head"].T
