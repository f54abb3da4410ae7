"""Plain-PyTorch statement of every op: the CPU execution path and the oracle for the CUDA kernels.

Each function states the math of one reference layer; accumulation is in fp32
and the result is cast back to the input dtype.

Parity:
  rms_norm / add_rms_norm   tinyvllm/layers/layernorm.py:21-45 (without the fp32 aliasing of the in-place version)
  rope_table / apply_rope   tinyvllm/layers/rotary_embedding.py:5-57 (NeoX half-split rotation, fp32)
  silu_mul                  tinyvllm/layers/activation.py:11-14
  store_kv                  tinyvllm/layers/attention.py:9-48 (plus: negative slots are skipped)
  attention                 tinyvllm/layers/attention.py:86-111 (varlen causal GQA over the paged cache,
                            bottom-right aligned mask when a prefix is cached)
  embedding                 tinyvllm/layers/embed_head.py:34-40 (masked vocab-shard lookup)
  sample                    tinyvllm/layers/sampler.py:13-21 (Gumbel-max == softmax sampling; greedy at T == 0)

KV cache layout used everywhere in this package: ``[num_blocks, kv_heads, block_size, head_dim]`` per
layer and per K/V, so one (block, head) pair is a contiguous ``block_size x head_dim`` tile that a
single bulk copy can fetch.
"""
from __future__ import annotations


import numpy as np
import torch
import torch.nn.functional as F

from . import ref_hybrid


# ----------------------------------------------------------------------------- norms
def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    xf = x.float()
    var = xf.pow(2).mean(dim=-1, keepdim=True)
    y = xf * torch.rsqrt(var + eps)
    return (y.to(x.dtype).float() * weight.float()).to(x.dtype) if x.dtype != torch.float32 else (y * weight.float())


def add_rms_norm(x: torch.Tensor, residual: torch.Tensor | None, weight: torch.Tensor, eps: float):
    """Returns (normed, new_residual); new_residual = x + residual rounded to the model dtype."""
    if residual is None:
        return rms_norm(x, weight, eps), x
    s = (x.float() + residual.float()).to(x.dtype)
    return rms_norm(s, weight, eps), s


# ----------------------------------------------------------------------------- rotary
def rope_table(max_positions: int, head_dim: int, theta: float, device="cpu", angle_dtype=torch.float32) -> torch.Tensor:
    """fp32 table ``[max_positions, head_dim]`` = cat(cos, sin) of pos * theta^(-2i/d).  ``angle_dtype=torch.float64``: the
    angles carry no rounding of their own (in fp32 an angle of 1e4 rad is off by up to 5e-4)."""
    inv_freq = 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=angle_dtype) / max(head_dim, 1)))
    t = torch.arange(max_positions, dtype=angle_dtype)
    freqs = torch.outer(t, inv_freq)
    return torch.cat((freqs.cos(), freqs.sin()), dim=-1).float().to(device)


def rotation_table(max_positions: int, frequencies: list, amplitude: float = 1.0, device="cpu") -> torch.Tensor:
    """The same from given frequencies (one per pair of entries), angles in fp64; cos and sin times ``amplitude``."""
    angles = torch.outer(torch.arange(max_positions, dtype=torch.float64), torch.tensor(frequencies, dtype=torch.float64))
    return (amplitude * torch.cat((angles.cos(), angles.sin()), dim=-1)).float().to(device)


def apply_rope(x: torch.Tensor, positions: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """x: [T, heads, d]; rotates pairs (i, i + d/2)."""
    d = x.shape[-1]
    cs = table[positions.long()]
    cos, sin = cs[:, None, :d // 2], cs[:, None, d // 2:]
    xf = x.float()
    x1, x2 = xf[..., :d // 2], xf[..., d // 2:]
    return torch.cat((x1 * cos - x2 * sin, x2 * cos + x1 * sin), dim=-1).to(x.dtype)


# ----------------------------------------------------------------------------- activation
def silu_mul(x: torch.Tensor) -> torch.Tensor:
    d = x.shape[-1] // 2
    g, u = x[..., :d].float(), x[..., d:].float()
    return (F.silu(g) * u).to(x.dtype)


# ----------------------------------------------------------------------------- linear
def linear(x: torch.Tensor, w) -> torch.Tensor:
    if not isinstance(w, torch.Tensor):     # Fp8BlockWeight: same arithmetic as the fp8 kernel
        from .quant import linear_fp8_ref
        return linear_fp8_ref(x, w)
    return F.linear(x, w)


def linear_silu_mul(x: torch.Tensor, w_gate_up) -> torch.Tensor:
    return silu_mul(linear(x, w_gate_up))


# gate and up projections (fp32) and a limit -> the feed-forward's inner activation
ACTIVATIONS = {
    "silu": lambda g, u, limit: F.silu(g) * u,
    "gelu_tanh": lambda g, u, limit: F.gelu(g, approximate="tanh") * u,
    "clamped_swish": lambda g, u, limit: (gc := g.clamp(max=limit)) * torch.sigmoid(1.702 * gc) * (u.clamp(-limit, limit) + 1.0),
}


def linear_act_mul(x: torch.Tensor, w_gate_up, act: str, limit: float = 0.0) -> torch.Tensor:
    g, u = linear(x, w_gate_up).float().chunk(2, dim=-1)
    return ACTIVATIONS[act](g, u, limit).to(x.dtype)


# the inner activation of a feed-forward without gates
PLAIN_ACTIVATIONS = {"gelu": lambda u, limit: F.gelu(u)}


def linear_act(x: torch.Tensor, w_up, act: str, limit: float = 0.0) -> torch.Tensor:
    return PLAIN_ACTIVATIONS[act](linear(x, w_up).float(), limit).to(x.dtype)


def bound_logits(x: torch.Tensor, scale: float, softcap: float) -> torch.Tensor:
    """softcap * tanh(scale * x / softcap); without a softcap scale * x."""
    z = x.float() * scale
    return (softcap * torch.tanh(z / softcap) if softcap else z).to(x.dtype)


# ----------------------------------------------------------------------------- KV cache
def store_kv(k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
             slot_mapping: torch.Tensor) -> None:
    """k, v: [T, kv_heads, d]; caches: [blocks, kv_heads, block_size, d]; slot < 0 is skipped."""
    bs = k_cache.shape[2]
    slots = slot_mapping.long()
    keep = slots >= 0
    if not bool(keep.all()):
        slots, k, v = slots[keep], k[keep], v[keep]
    blk, off = slots // bs, slots % bs
    k_cache[blk, :, off] = k.to(k_cache.dtype)
    v_cache[blk, :, off] = v.to(v_cache.dtype)


def qk_norm_rope_store(qkv: torch.Tensor, q_weight: torch.Tensor, k_weight: torch.Tensor, eps: float,
                       table: torch.Tensor, positions: torch.Tensor, slot_mapping: torch.Tensor,
                       k_cache: torch.Tensor, v_cache: torch.Tensor,
                       num_heads: int, num_kv_heads: int, head_dim: int) -> torch.Tensor:
    """Split the fused QKV projection, RMS-normalise q and k per head, rotate, write k and v into the
    paged cache and return q as ``[T, heads, d]`` (tinyvllm/models/qwen3.py:78-94)."""
    T = qkv.shape[0]
    q, k, v = qkv.split([num_heads * head_dim, num_kv_heads * head_dim, num_kv_heads * head_dim], dim=-1)
    q = rms_norm(q.reshape(T, num_heads, head_dim), q_weight, eps)
    k = rms_norm(k.reshape(T, num_kv_heads, head_dim), k_weight, eps)
    q = apply_rope(q, positions, table)
    k = apply_rope(k, positions, table)
    store_kv(k, v.reshape(T, num_kv_heads, head_dim), k_cache, v_cache, slot_mapping)
    return q


def _gather_kv(cache: torch.Tensor, table_row: torch.Tensor, length: int) -> torch.Tensor:
    """Rows 0..length-1 of one sequence from the paged cache -> [kv_heads, length, d]."""
    bs = cache.shape[2]
    nblk = (length + bs - 1) // bs
    blocks = cache[table_row[:nblk].long()]              # [nblk, kvh, bs, d]
    kvh, d = blocks.shape[1], blocks.shape[3]
    return blocks.permute(1, 0, 2, 3).reshape(kvh, nblk * bs, d)[:, :length]


def attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, cu_seqlens_q: torch.Tensor,
              context_lens: torch.Tensor, block_tables: torch.Tensor, scale: float, num_seqs: int) -> torch.Tensor:
    """Causal GQA attention of new query tokens over the paged cache.

    q: [T, heads, d] holds, for sequence s, rows cu_seqlens_q[s]:cu_seqlens_q[s+1]; these are the LAST
    ``q_len`` positions of a sequence of ``context_lens[s]`` tokens whose K/V are all in the cache already.
    Returns [T, heads * d].
    """
    T, H, d = q.shape
    out = torch.zeros(T, H, d, dtype=q.dtype, device=q.device)
    cu = cu_seqlens_q.tolist()
    lens = context_lens.tolist()
    for s in range(num_seqs):
        a, b = cu[s], cu[s + 1]
        ql, kl = b - a, lens[s]
        if ql == 0:
            continue
        k = _gather_kv(k_cache, block_tables[s], kl).float()      # [kvh, kl, d]
        v = _gather_kv(v_cache, block_tables[s], kl).float()
        g = H // k.shape[0]
        qs = q[a:b].float().permute(1, 0, 2).reshape(k.shape[0], g * ql, d)   # [kvh, g*ql, d]
        scores = torch.bmm(qs, k.transpose(1, 2)) * scale                      # [kvh, g*ql, kl]
        qpos = torch.arange(kl - ql, kl, device=q.device).repeat(g)            # row r -> query position
        mask = torch.arange(kl, device=q.device)[None, :] > qpos[:, None]
        scores.masked_fill_(mask[None], float("-inf"))
        p = torch.softmax(scores, dim=-1)
        o = torch.bmm(p, v).reshape(H, ql, d).permute(1, 0, 2)
        out[a:b] = o.to(q.dtype)
    return out.reshape(T, H * d)


# ----------------------------------------------------------------------------- 32-bit residual stream
def stream_update(x, dtype, eps, norms, start=False, a=None, b=None, ids=None, embed=None, vec=None, rows=None,
                  a_bias=None, post=None, mult=1.0, offset=0.0, groups=1):
    """The residual stream between two layers: x += a + b (the two branches of a parallel layer), += embed[ids], += vec,
    all in fp32; then one RMS norm per weight in ``norms``, each rounded once to ``dtype`` (None: the stream itself, rounded).  ``start``: x
    begins at zero.  ``rows``: norms of these rows only, and x is left as it was.  ``a_bias`` is added to a.  ``post``: a (without
    a: the embedding) is normed with this weight and multiplied by ``mult`` on its way into x.  ``offset`` is added to every norm
    weight (weights stored around zero).  ``groups``: a norm divides every one of that many equal parts of a row by its own root mean
    square."""
    def norm(v, w):
        if w is None:
            return v
        parts = v.view(v.shape[0], groups, -1)
        return (parts * torch.rsqrt(parts.pow(2).mean(dim=-1, keepdim=True) + eps)).view(v.shape) * (w.float() + offset)

    s = torch.zeros_like(x) if start else x
    if a is None and post is not None:
        s, ids = s + mult * norm(F.embedding(ids.long(), embed).float(), post), None
    if a is not None:
        a = a.float() if a_bias is None else a.float() + a_bias
        s = s + (a if post is None else mult * norm(a, post))
    if b is not None:
        s = s + b.float()
    if ids is not None:
        s = s + F.embedding(ids.long(), embed).float()
    if vec is not None:
        s = s + vec.float()
    if rows is None:
        x.copy_(s)
    else:
        s = s[rows.long()]
    return [norm(s, w).to(dtype) for w in norms]


def stream_mix(x, dtype, eps, into, norm, bias, y=None, mix=None, out=None, ids=None, prev=None, embed=None, scale=1.0, pairs=None,
               mul_prev=0, mul_cur=0, rows=None):
    """Several residual streams x [T, streams, W] (fp32) between two sublayers.  First the streams take up a sublayer's result, all at
    once: x_t <- sum_s mix[s, t] x_s + out[t] y; or, with ``ids``, every stream begins as scale * embed[id] + the pair table's row
    (prev * mul_prev + id * mul_cur) mod (rows - 1), the last row where prev < 0.  Then sum_s into[s] x_s goes through a
    layer norm (weight, bias) and is rounded once to ``dtype``.  norm=None: no result.  ``rows``: results of these rows only, and
    x is left as it was."""
    if ids is not None:
        last = pairs.shape[0] - 1
        at = torch.where(prev < 0, last, (prev.long() * mul_prev + ids.long() * mul_cur) % last)
        s = (scale * F.embedding(ids.long(), embed).float() + pairs[at].float())[:, None].expand_as(x)
    else:
        s = torch.einsum("nsw,st->ntw", x, mix) + out[:, None] * y.float()[:, None, :]
    if rows is None:
        x.copy_(s)
    else:
        s = s[rows.long()]
    if norm is None:
        return None
    u = torch.einsum("nsw,s->nw", s, into)
    u = u - u.mean(dim=-1, keepdim=True)
    return (u * torch.rsqrt(u.pow(2).mean(dim=-1, keepdim=True) + eps) * norm.float() + bias.float()).to(dtype)


def apply_partial_rope(x: torch.Tensor, positions: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """fp32 [T, heads, d]; the first ``table.shape[1]`` entries of every head are rotated, the rest pass."""
    n = table.shape[1]
    return torch.cat((apply_rope(x[..., :n].float(), positions, table), x[..., n:].float()), dim=-1)


# ----------------------------------------------------------------------------- latent attention
def latent_prepare(proj, q_rank, kv_rank, q_norm, kv_norm, eps, table, positions, slot_mapping, cache):
    """proj [T, q_rank + kv_rank + rot] -> the normed query latent; the normed key/value latent and the rotated shared key
    part go to the paged cache [blocks, block_size, kv_rank + rot].  Without ``q_norm`` the first ``q_rank`` columns are passed over and
    nothing is returned; columns after the rotated part are padding."""
    def norm(v, w):
        v = v.float()
        return v * torch.rsqrt(v.pow(2).mean(dim=-1, keepdim=True) + eps) * w.float()
    cq = None if q_norm is None else norm(proj[:, :q_rank], q_norm).to(proj.dtype)
    c = norm(proj[:, q_rank:q_rank + kv_rank], kv_norm)
    kr = apply_partial_rope(proj[:, None, q_rank + kv_rank:q_rank + cache.shape[-1]], positions, table)[:, 0]
    slots = slot_mapping.long()
    keep = slots >= 0
    flat = cache.view(-1, cache.shape[-1])
    flat[slots[keep]] = torch.cat((c, kr), dim=-1)[keep].to(cache.dtype)
    return cq


def latent_attention(q, wkv, cache, batch, table, spec):
    """q [T, heads * (dim + rot)] before rotation; wkv [heads * (dim + vdim), kv_rank] = key rows, then value rows."""
    H, d, r, dv, R = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank
    T = q.shape[0]
    q = q.reshape(T, H, d + r).float()
    q = torch.cat((q[..., :d], apply_partial_rope(q[..., d:], batch.positions, table)), dim=-1)
    out = torch.zeros(T, H, dv, dtype=cache.dtype, device=cache.device)
    w = wkv.float()
    cu, lens = batch.cu_seqlens_q.tolist(), batch.context_lens.tolist()
    bs = cache.shape[1]
    for s in range(batch.num_seqs):
        a, b = cu[s], cu[s + 1]
        n = lens[s]
        rows = cache[batch.block_tables[s, :(n + bs - 1) // bs].long()].reshape(-1, R + r)[:n].float()
        kv = rows[:, :R] @ w.t()
        k = torch.cat((kv[:, :H * d].view(n, H, d), rows[:, None, R:].expand(n, H, r)), dim=-1)
        scores = torch.einsum("qhd,khd->hqk", q[a:b], k) * spec.scale
        pos = batch.positions[a:b].long()
        back = pos[:, None] - torch.arange(n, device=q.device)[None, :]
        scores.masked_fill_((back < 0) | (back >= (spec.window or n)), float("-inf"))
        out[a:b] = torch.einsum("hqk,khe->qhe", torch.softmax(scores, dim=-1), kv[:, H * d:].view(n, H, dv)).to(out.dtype)
    return out.view(T, H * dv)


# ----------------------------------------------------------------------------- retention
def retention(qkvg, decay, state, batch, table, spec, eps):
    """qkvg [T, heads * (2 dim + 2 vdim)] = q, k, v, gate.  state [slots, heads, dim, vdim] fp32 is read and updated in place
    (a sequence's first token starts from zero).  Returns the gated, per-head normed output [T, heads * vdim]."""
    H, d, dv = spec.heads, spec.dim, spec.vdim
    T = qkvg.shape[0]
    q, k, v, g = qkvg.float().split([H * d, H * d, H * dv, H * dv], dim=-1)
    q = apply_partial_rope(q.reshape(T, H, d), batch.positions, table)
    k = apply_partial_rope(k.reshape(T, H, d), batch.positions, table) * d ** -0.5
    v = v.reshape(T, H, dv)
    o = torch.zeros(T, H, dv, device=q.device)
    cu, slots = batch.cu_seqlens_q.tolist(), batch.state_slots.tolist()
    keep = decay.view(H, 1, 1)
    for s in range(batch.num_seqs):
        a, b = cu[s], cu[s + 1]
        if int(batch.positions[a]) == 0:
            state[slots[s]].zero_()
        S = state[slots[s]]
        for t in range(a, b):
            S.mul_(keep).add_(k[t][:, :, None] * v[t][:, None, :])
            o[t] = torch.einsum("hde,hd->he", S, q[t])
    o = o * torch.rsqrt(o.pow(2).mean(dim=-1, keepdim=True) + eps)
    return (o.reshape(T, H * dv) * F.silu(g)).to(qkvg.dtype)


# ----------------------------------------------------------------------------- mixture of experts
def choose_experts(scores, correction, groups, keep):
    """Experts of every token, best first, by scores + correction within the ``keep`` best groups of neighbours (a group's worth: its two
    best experts together); ties go to the lower number."""
    c = scores if correction is None else scores + correction
    if groups > 1:
        parts = c.view(c.shape[0], groups, -1)
        worth = parts.topk(min(2, parts.shape[-1]), dim=-1).values.sum(dim=-1)
        best = torch.sort(worth, dim=-1, descending=True, stable=True).indices[:, :keep]
        out = torch.ones_like(worth, dtype=torch.bool).scatter_(1, best, False)
        c = parts.masked_fill(out[:, :, None], float("-inf")).view(c.shape)
    return torch.sort(c, dim=-1, descending=True, stable=True).indices


def moe(h, router, up, down, top, score="sigmoid", weigh="input", act="silu", limit=0.0, gated=True, correction=None, groups=1, keep=1):
    """Top-k experts.  ``score``: sigmoid of each logit, or softmax over the chosen logits; ``weigh``: the score multiplies the
    expert's input or its output.  up [experts, 2 ff (gate, up), width], or with ``gated=False`` [experts, ff, width]; down [experts, width,
    ff].  ``correction``, ``groups``, ``keep``: see ``choose_experts``; weights are the scores without the correction."""
    z = h.float() @ router.float().t()
    if score == "sigmoid":
        z = torch.sigmoid(z)
    e = choose_experts(z, correction, groups, keep)
    w = z.gather(1, e) if score == "sigmoid" else torch.softmax(z.gather(1, e)[:, :top], dim=-1)
    inner = linear_act_mul if gated else linear_act
    out = torch.zeros(h.shape[0], down.shape[1], device=h.device)
    for j in range(top):
        for x in e[:, j].unique().tolist():
            rows = (e[:, j] == x).nonzero()[:, 0]
            hx, wx = h[rows], w[rows, j, None]
            if weigh == "input":
                hx, wx = (hx.float() * wx).to(h.dtype), 1.0
            out[rows] += wx * linear(inner(hx, up[x], act, limit), down[x]).float()
    return out


# ----------------------------------------------------------------------------- embedding
def embedding(ids: torch.Tensor, weight: torch.Tensor, vocab_start: int = 0) -> torch.Tensor:
    """Rows of this rank's vocab shard; ids outside the shard give zero rows."""
    n = weight.shape[0]
    local = ids.long() - vocab_start
    ok = (local >= 0) & (local < n)
    out = F.embedding(torch.where(ok, local, torch.zeros_like(local)), weight)
    return out * ok[:, None].to(out.dtype)


# ----------------------------------------------------------------------------- sampling
_PHILOX_M0, _PHILOX_M1 = np.uint64(0xD2511F53), np.uint64(0xCD9E8D57)
_PHILOX_W0, _PHILOX_W1 = np.uint32(0x9E3779B9), np.uint32(0xBB67AE85)


def philox4x32(c0, c1, c2, c3, k0, k1):
    """Philox-4x32-10 on numpy uint32 arrays; returns four uint32 arrays."""
    c0, c1, c2, c3 = (np.asarray(c, dtype=np.uint32) for c in (c0, c1, c2, c3))
    c0, c1, c2, c3 = np.broadcast_arrays(c0, c1, c2, c3)
    k0, k1 = np.uint32(k0), np.uint32(k1)
    with np.errstate(over="ignore"):
        for _ in range(10):
            p0 = c0.astype(np.uint64) * _PHILOX_M0
            p1 = c2.astype(np.uint64) * _PHILOX_M1
            hi0, lo0 = (p0 >> np.uint64(32)).astype(np.uint32), p0.astype(np.uint32)
            hi1, lo1 = (p1 >> np.uint64(32)).astype(np.uint32), p1.astype(np.uint32)
            c0, c1, c2, c3 = hi1 ^ c1 ^ k0, lo1, hi0 ^ c3 ^ k1, lo0
            k0 = np.uint32((int(k0) + int(_PHILOX_W0)) & 0xFFFFFFFF)
            k1 = np.uint32((int(k1) + int(_PHILOX_W1)) & 0xFFFFFFFF)
    return c0, c1, c2, c3


def gumbel_noise(rows: int, vocab: int, seed: int, step: int, vocab_start: int = 0) -> np.ndarray:
    """-log(-log(u)) per (row, global vocab id), a pure function of (seed, step, row, id).

    One Philox call covers four consecutive vocab ids: counter = (id // 4, row, step, 0),
    key = seed; lane ``id % 4`` of the output is the uniform for that id.  Keying on the GLOBAL
    vocab id makes the sampled token independent of how the vocabulary is sharded.
    """
    ids = np.arange(vocab_start, vocab_start + vocab, dtype=np.int64)
    grp = (ids // 4).astype(np.uint32)
    r = np.arange(rows, dtype=np.uint32)[:, None]
    outs = philox4x32(grp[None, :], r, np.uint32(step & 0xFFFFFFFF), np.uint32(0),
                      seed & 0xFFFFFFFF, (seed >> 32) & 0xFFFFFFFF)
    lane = (ids % 4)[None, :]
    bits = np.choose(np.broadcast_to(lane, outs[0].shape), outs)
    # u = (k + 0.5) / 2^24 with k the top 24 bits.  The winners of the arg-max have u close to 1, where fp32 cannot
    # resolve 1 - u; work from w = 1 - u = (2^24 - k - 0.5) / 2^24 in fp64: E = -log(u) = -log1p(-w), noise = -log(E).
    return _gumbel_from_bits(bits)


SAMPLE_GROUP = 16


def _gumbel_from_bits(bits: np.ndarray) -> np.ndarray:
    k = (bits >> np.uint32(8)).astype(np.float64)
    w = (16777216.0 - k - 0.5) / 16777216.0
    return (-np.log(-np.log1p(-w))).astype(np.float32)


def group_gumbel_noise(rows: int, g_first: int, ngroups: int, seed: int, step: int) -> np.ndarray:
    """Gumbel noise per (row, group of 16 global vocab ids): Philox counter (g // 4, row, step, 1), lane g % 4."""
    g = np.arange(g_first, g_first + ngroups, dtype=np.int64)
    r = np.arange(rows, dtype=np.uint32)[:, None]
    outs = philox4x32((g // 4).astype(np.uint32)[None, :], r, np.uint32(step & 0xFFFFFFFF), np.uint32(1),
                      seed & 0xFFFFFFFF, (seed >> 32) & 0xFFFFFFFF)
    bits = np.choose(np.broadcast_to((g % 4)[None, :], outs[0].shape), outs)
    return _gumbel_from_bits(bits)


def sample(logits: torch.Tensor, temperatures: torch.Tensor, seed: int, step: int, vocab_start: int = 0):
    """Returns (token ids int64 [rows], winning scores fp32 [rows]) over this vocab shard.

    T == 0 -> argmax(logits), score = the maximum.  T > 0 -> a draw from softmax(logits / T), as the reference's
    ``probs / Exp(1)`` race is (tinyvllm/layers/sampler.py:13-21), in two levels so that only one random number per GROUP
    of 16 consecutive global token ids is needed: (1) the winning group is argmax_g (logsumexp_{i in g}(logit_i / T) +
    Gumbel(row, g)), which is distributed as the group holding the arg-max of per-token Gumbel-max sampling; (2) inside it
    the token is argmax_i (logit_i / T + Gumbel(row, i)).  The score returned is the winning group's, so that vocab shards
    (which start on multiples of 16) can be merged by taking the row-wise maximum.  Same procedure as csrc/include/sampling.cuh.
    """
    lf = logits.float()
    rows, vocab = lf.shape
    t = temperatures.float().to(lf.device)
    greedy = t <= 0
    inv_t = torch.where(greedy, torch.ones_like(t), 1.0 / torch.where(greedy, torch.ones_like(t), t))
    x = lf * inv_t[:, None]
    G = SAMPLE_GROUP
    g_first, g_last = vocab_start // G, (vocab_start + vocab - 1) // G
    ngroups = g_last - g_first + 1
    lead = vocab_start - g_first * G                      # ids of the first group that lie before the shard
    padded = torch.full((rows, ngroups * G), float("-inf"), device=lf.device)
    padded[:, lead:lead + vocab] = x
    grp = padded.view(rows, ngroups, G)
    gscore = torch.logsumexp(grp, dim=-1)
    gnoise = torch.from_numpy(group_gumbel_noise(rows, g_first, ngroups, seed, step)).to(lf.device)
    gscore = torch.where(greedy[:, None], grp.max(dim=-1).values, gscore + gnoise)
    best, gwin = gscore.max(dim=-1)                        # ties -> the first (lowest) group
    noise = torch.from_numpy(gumbel_noise(rows, ngroups * G, seed, step, g_first * G)).to(lf.device).view(rows, ngroups, G)
    inner = grp + torch.where(greedy[:, None, None], torch.zeros_like(noise), noise)
    pick = inner[torch.arange(rows, device=lf.device), gwin].argmax(dim=-1)
    return (g_first + gwin) * G + pick, best


# ----------------------------------------------------------------------------- op set
class RefOps(ref_hybrid.RefHybridOps):
    """The op set the model calls, stated with the functions above (CPU path and oracle)."""

    name = "ref"

    linear = staticmethod(linear)
    linear_silu_mul = staticmethod(linear_silu_mul)
    linear_act_mul = staticmethod(linear_act_mul)
    bound_logits = staticmethod(bound_logits)
    embedding = staticmethod(embedding)
    add_rms_norm = staticmethod(add_rms_norm)
    rms_norm = staticmethod(rms_norm)
    qk_norm_rope_store = staticmethod(qk_norm_rope_store)
    stream_update = staticmethod(stream_update)
    stream_mix = staticmethod(stream_mix)
    latent_prepare = staticmethod(latent_prepare)
    retention = staticmethod(retention)
    moe = staticmethod(moe)

    @staticmethod
    def latent_attention(q, weights, cache, batch, table, spec):
        return latent_attention(q, weights.ukv, cache, batch, table, spec)

    @staticmethod
    def attention(q, k_cache, v_cache, batch, scale):
        return attention(q, k_cache, v_cache, batch.cu_seqlens_q, batch.context_lens, batch.block_tables,
                         scale, batch.num_seqs)

    @staticmethod
    def select_rows(x, index):
        return x.index_select(0, index.long())

    @staticmethod
    def tp_all_reduce(y, tp):
        return tp.all_reduce(y)

    @staticmethod
    def embed_norm(ids, embed, norm_weight, eps):
        h = embed.tp.all_reduce(embedding(ids, embed.weight, embed.vocab_start))
        return add_rms_norm(h, None, norm_weight, eps)

    @staticmethod
    def row_linear_add_rms_norm(x, layer, residual, norm_weight, eps, site):
        h = layer.tp.all_reduce(linear(x, layer.weight))
        return add_rms_norm(h, residual, norm_weight, eps)

    @staticmethod
    def sample(logits, batch, vocab_start, tp):
        """Token ids [rows] (int64), identical on every rank."""
        ids, best = sample(logits, batch.temperatures, batch.seed, batch.step_index, vocab_start)
        if tp.size == 1:
            return ids
        all_best = tp.all_gather_stack(best)          # [tp, rows]
        all_ids = tp.all_gather_stack(ids)
        win = all_best.argmax(dim=0, keepdim=True)    # ties -> lowest rank == lowest vocab id
        return all_ids.gather(0, win)[0]
