"""What the GPU tests of single kernels share: device metadata of a step, random tensors, comparison."""
import numpy as np
import torch

F32 = torch.float32


class Spec:
    def __init__(self, **kw):
        self.__dict__.update(kw)


class Batch:
    """Device metadata of a step: q tokens [start, end) per sequence, blocks in shuffled order."""

    def __init__(self, ranges, block, slots=None, decode=False, pad=0, seed=0):
        g = torch.Generator().manual_seed(seed)
        n = len(ranges)
        width = max(-(-e // block) for _, e in ranges)
        self.num_blocks = n * width + 3
        perm = torch.randperm(self.num_blocks, generator=g)[:n * width].view(n, width)
        q = [e - s for s, e in ranges]
        single = [x == 1 for x in q]
        self.num_single = single.index(False) if False in single else n
        self.is_prefill, self.num_seqs, self.padded_seqs = not decode, n, n + pad
        self.table_width, self.max_seqlen_q, self.max_seqlen_k = width, max(q), max(e for _, e in ranges)
        dev = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
        self.tables = perm
        self.block_tables = torch.cat([perm, torch.full((pad, width), -1)]).int().cuda()
        cu = np.cumsum([0] + q).tolist()
        self.cu_seqlens_q = dev(cu + [cu[-1]] * pad)
        self.context_lens = dev([e for _, e in ranges] + [0] * pad)
        self.positions = dev([p for s, e in ranges for p in range(s, e)] + [0] * pad)
        self.slot_mapping = dev([int(perm[i][p // block]) * block + p % block for i, (s, e) in enumerate(ranges) for p in range(s, e)] + [-1] * pad)
        ks = [0] * (self.num_single + 1) + np.cumsum([e for _, e in ranges[self.num_single:]]).tolist()
        self.cu_seqlens_k = dev(ks)
        self.kv_rows = ks[-1]
        self.state_slots = dev((slots or list(range(n))) + [-1] * pad)


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    err = (got - want).abs().max() / want.abs().max()
    assert err <= tol, f"max error {err:.3g} of the largest value (allowed {tol})"


def rope(n, dims, base=10000.0):
    from tinyllmforge_b200.ops.ref import rope_table
    return rope_table(n, dims, base, "cuda", torch.float64)


def rnd(*shape, seed=0, scale=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)
