"""Plain-PyTorch ops of hybrid decoders: windowed attention, short convolutions, state-space and gated-delta recurrences.

Everything that the recurrences keep or multiply is fp32; token by token.  A sequence's first token (position 0) starts from
zeros, whatever its slot held before.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F


def _runs(batch):
    """(first row, end row, slot, starts afresh) of every sequence of the step."""
    cu, slots = batch.cu_seqlens_q.tolist(), batch.state_slots.tolist()
    return [(cu[s], cu[s + 1], slots[s], int(batch.positions[cu[s]]) == 0) for s in range(batch.num_seqs)]


def bias_rope_store(proj, bias, spec, table, positions, slot_mapping, k_cache, v_cache):
    """proj [T, q | k | v] -> q [T, heads, dim] rotated; keys (rotated) and values go to the paged caches."""
    from .ref import apply_partial_rope, store_kv
    T, H, G, d = proj.shape[0], spec.heads, spec.kv_heads, spec.dim
    q, k, v = (proj.float() + bias).split([H * d, G * d, G * spec.vdim], dim=-1)
    q = apply_partial_rope(q.reshape(T, H, d), positions, table)
    k = apply_partial_rope(k.reshape(T, G, d), positions, table)
    store_kv(k, v.reshape(T, G, spec.vdim), k_cache, v_cache, slot_mapping)
    return q.to(proj.dtype)


def norm_rope_store(proj, q_norm, k_norm, eps, spec, table, positions, slot_mapping, k_cache, v_cache, temper=None):
    """proj [T, q | k | v] -> q [T, heads, dim] normed and rotated; keys (the same) and values go to the paged caches.  A norm weight of
    ``dim`` entries belongs to every head, one of all entries to the projection as a whole.  Without ``k_norm`` proj is q alone and
    nothing is stored.  ``temper`` [heads]: a factor of the queries."""
    from .ref import apply_partial_rope, store_kv
    T, H, G, d = proj.shape[0], spec.heads, spec.kv_heads, spec.dim

    def normed(x, w, heads):
        x = x.float().reshape((T, heads, d) if spec.norm == "head" else (T, heads * d))
        return apply_partial_rope((x * torch.rsqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps) * w.float()).view(T, heads, d), positions, table)

    q = proj[:, :H * d]
    if k_norm is not None:
        k, v = proj[:, H * d:].split([G * d, G * spec.vdim], dim=-1)
        store_kv(normed(k, k_norm, G), v.reshape(T, G, spec.vdim), k_cache, v_cache, slot_mapping)
    q = normed(q, q_norm, H)
    return (q if temper is None else q * temper[:, None]).to(proj.dtype)


def pool_place(block, size: int, block_size: int):
    """Where the mean of block ``block`` (an index tensor) of ``size`` tokens lies: page of the sequence, row of the page."""
    page = (block * size + size - 1) // block_size
    return page, block - page * block_size // size


def pool_blocks(k_cache, v_cache, pool, batch) -> None:
    """Means of the keys and values of the blocks that end among the step's tokens, into their places."""
    from .ref import _gather_kv
    cu, lens, bs = batch.cu_seqlens_q.tolist(), batch.context_lens.tolist(), k_cache.shape[2]
    for s in range(batch.num_seqs):
        first, end = (lens[s] - (cu[s + 1] - cu[s])) // pool.size, lens[s] // pool.size
        if first >= end:
            continue
        page, row = pool_place(torch.arange(first, end, device=k_cache.device), pool.size, bs)
        page = batch.block_tables[s].long()[page]
        for cache, means in ((k_cache, pool.k), (v_cache, pool.v)):
            x = _gather_kv(cache, batch.block_tables[s], end * pool.size)[:, first * pool.size:].float()
            means[page, :, row] = x.reshape(x.shape[0], end - first, pool.size, -1).mean(dim=2).transpose(0, 1).to(means.dtype)


def windowed_attention(q, k_cache, v_cache, batch, spec, out, scale, chunked=False, softcap=0.0, sink=None, gate=None, pool=None):
    """out [T, heads * vdim] <- scale * attention of q over the keys at most ``window - 1`` positions back, or (``chunked``) over those of
    the query's own chunk of ``window`` positions.  ``softcap`` bounds the scores; ``sink`` [heads]: one more score per head, of
    the denominator alone; ``gate`` [T, heads] or [T, heads * vdim]: its sigmoid multiplies the result.  ``pool`` (see
    ``PooledCache``): the blocks that end in this step get their means, and every query also sees the means of the blocks that end before
    its window."""
    from .ref import _gather_kv
    H, G = spec.heads, spec.kv_heads
    cu, lens = batch.cu_seqlens_q.tolist(), batch.context_lens.tolist()
    if pool is not None and pool.own:
        pool_blocks(k_cache, v_cache, pool, batch)
    for s in range(batch.num_seqs):
        a, b, n = cu[s], cu[s + 1], lens[s]
        k = _gather_kv(k_cache, batch.block_tables[s], n).float()
        v = _gather_kv(v_cache, batch.block_tables[s], n).float()
        pos, keys = batch.positions[a:b].long()[:, None], torch.arange(n, device=q.device)[None, :]
        oldest = pos // spec.window * spec.window if chunked else pos - spec.window + 1
        hidden = (keys > pos) | (keys < oldest)
        if pool is not None:
            blocks = torch.arange(n // pool.size, device=q.device)
            page, row = pool_place(blocks, pool.size, k_cache.shape[2])
            page = batch.block_tables[s].long()[page]
            k, v = (torch.cat((x, means[page, :, row].float().transpose(0, 1)), dim=1) for x, means in ((k, pool.k), (v, pool.v)))
            hidden = torch.cat((hidden, blocks[None, :] * pool.size + pool.size > oldest), dim=1)
            n = hidden.shape[1]
        k, v = k.repeat_interleave(H // G, dim=0), v.repeat_interleave(H // G, dim=0)
        scores = torch.einsum("qhd,hkd->hqk", q[a:b].float(), k) * spec.scale
        if softcap:
            scores = softcap * torch.tanh(scores / softcap)
        scores.masked_fill_(hidden, float("-inf"))
        if sink is not None:
            scores = torch.cat((scores, sink[:, None, None].expand(H, b - a, 1)), dim=-1)
        o = torch.einsum("hqk,hke->qhe", torch.softmax(scores, dim=-1)[..., :n], v)
        if gate is not None:
            o = o * torch.sigmoid(gate[a:b].float()).view(b - a, H, -1)
        out[a:b] = (scale * o.reshape(b - a, -1)).to(out.dtype)


def short_conv(x, taps, bias, state, batch, act="silu"):
    """A causal convolution over time, per channel, then silu (``act="none"``: nothing).  x [T, channels], taps [channels, n] (last column:
    the token itself), state [slots, n - 1, channels]: the inputs before the step's first token, replaced by the last ones."""
    n = taps.shape[1]
    out = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    for a, b, slot, fresh in _runs(batch):
        past = state[slot] if not fresh and n > 1 else torch.zeros(state.shape[1:], dtype=state.dtype, device=state.device)
        seq = torch.cat([past, x[a:b]]).float()
        y = sum(seq[i:i + b - a] * taps[:, i] for i in range(n))
        y = y if bias is None else y + bias
        out[a:b] = (F.silu(y) if act == "silu" else y).to(x.dtype)
        if n > 1:
            state[slot] = seq[seq.shape[0] - (n - 1):].to(state.dtype)
    return out


def state_space(xbc, z, dt, block, state, batch, out, scale):
    """xbc [T, x | B | C] -> out [T, heads * vdim] <- scale * norm(y silu(z)); state [slots, heads, N, vdim] fp32."""
    s = block.spec
    T, H, N, G, dv = xbc.shape[0], s.heads, s.state, s.groups, s.vdim
    x, B, C = xbc.float().split([s.inner, G * N, G * N], dim=-1)
    x = x.reshape(T, H, dv)
    B, C = (m.reshape(T, G, N).repeat_interleave(H // G, dim=1) for m in (B, C))
    dt = F.softplus(dt.float() + block.dt_bias, threshold=1e9)
    keep = torch.exp(-torch.exp(block.A_log) * dt)
    y = torch.zeros(T, H, dv, device=xbc.device)
    for a, b, slot, fresh in _runs(batch):
        if fresh:
            state[slot].zero_()
        S = state[slot]
        for t in range(a, b):
            S.mul_(keep[t, :, None, None]).add_(B[t][:, :, None] * (dt[t, :, None] * x[t])[:, None, :])
            y[t] = torch.einsum("hne,hn->he", S, C[t]) + block.D[:, None] * x[t]
    y = (y.reshape(T, -1) * F.silu(z.float())).view(T, s.norm_groups, -1)
    y = (y * torch.rsqrt(y.pow(2).mean(dim=-1, keepdim=True) + block.eps)).reshape(T, -1) * block.norm
    out.copy_((scale * y).to(out.dtype))


def gated_delta(qkv, gate, ba, block, state, batch):
    """qkv [T, q | k | v] after the convolutions, gate [T, heads * vdim], ba [T, b | a] -> [T, heads * vdim] normed and gated;
    state [slots, heads, dim, vdim] fp32."""
    s = block.spec
    T, H, G, d, dv = qkv.shape[0], s.heads, s.kv_heads, s.dim, s.vdim
    q, k, v = qkv.float().split([G * d, G * d, H * dv], dim=-1)
    q, k = (m.reshape(T, G, d) for m in (q, k))
    q, k = (m * torch.rsqrt(m.pow(2).sum(dim=-1, keepdim=True) + 1e-6) for m in (q, k))
    q, k = (q * d ** -0.5).repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    v = v.reshape(T, H, dv)
    beta = torch.sigmoid(ba[:, :H].float())
    keep = torch.exp(-torch.exp(block.A_log) * F.softplus(ba[:, H:].float() + block.dt_bias, threshold=1e9))
    o = torch.zeros(T, H, dv, device=qkv.device)
    for a, b, slot, fresh in _runs(batch):
        if fresh:
            state[slot].zero_()
        S = state[slot]
        for t in range(a, b):
            S.mul_(keep[t, :, None, None])
            u = beta[t, :, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
            S.add_(k[t][:, :, None] * u[:, None, :])
            o[t] = torch.einsum("hde,hd->he", S, q[t])
    o = o * torch.rsqrt(o.pow(2).mean(dim=-1, keepdim=True) + block.eps) * block.norm
    return (o.reshape(T, H * dv) * F.silu(gate.float())).to(qkv.dtype)


class RefHybridOps:
    """Mixed into ``RefOps``."""
    bias_rope_store = staticmethod(bias_rope_store)
    norm_rope_store = staticmethod(norm_rope_store)
    windowed_attention = staticmethod(windowed_attention)
    short_conv = staticmethod(short_conv)
    state_space = staticmethod(state_space)
    gated_delta = staticmethod(gated_delta)
