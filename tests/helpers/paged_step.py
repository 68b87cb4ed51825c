"""A step over given sequences on a shuffled paged cache, for tests of attention kernels: the packed inputs and filled caches."""
import numpy as np
import torch

from xllm_wxh_b200.framework.step_input import StepInput, make_layout


class PagedStep:
    """`lens`: (tokens before the step, tokens in the step) per sequence; `rows`: per sequence the tensors [tokens, heads, width]
    that go to the caches (one cache per tensor).  Single tokens with a past come first, as the scheduler orders them."""

    def __init__(self, lens, rows, block, device, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.order = sorted(range(len(lens)), key=lambda i: not (lens[i][1] == 1 and lens[i][0] > 0))
        self.lens = lens
        need = [-(-(b + n) // block) for b, n in lens]
        MB = max(need)
        perm = (torch.randperm(sum(need), generator=g) + 1).tolist()
        # places that belong to no sequence hold other values
        caches = [torch.randn(sum(need) + 1, block, *t.shape[1:], generator=g).to(t.dtype) * 3 for t in rows[0]]
        L = make_layout(sum(n for _, n in lens), len(lens), MB, len(lens), 32)
        host = torch.zeros(L.total_words, dtype=torch.int32)
        at, n_dec = 0, 0
        for s, i in enumerate(self.order):
            before, n = lens[i]
            blocks = [perm.pop() for _ in range(need[i])]
            for c, t in zip(caches, rows[i]):
                for p in range(before + n):
                    c[blocks[p // block], p % block] = t[p]
            o = L.block_tables + s * L.MB_cap
            host[o:o + len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
            host[L.positions + at:L.positions + at + n] = torch.arange(before, before + n, dtype=torch.int32)
            host[L.token_seq + at:L.token_seq + at + n] = s
            host[L.slots + at:L.slots + at + n] = torch.tensor([blocks[p // block] * block + p % block for p in range(before, before + n)])
            at += n
            host[L.q_cu + s + 1] = at
            host[L.kv_lens + s] = before + n
            n_dec += n == 1 and before > 0
        hdr = np.zeros(32, dtype=np.int32)
        hdr[0], hdr[1], hdr[3], hdr[4] = at, len(lens), n_dec, len(lens) - n_dec
        hdr[5], hdr[6], hdr[17] = max(n for _, n in lens), max(b + n for b, n in lens), block
        hdr[7] = 2 if n_dec == len(lens) else 3
        hdr[21] = sum(n for b, n in lens if not (n == 1 and b > 0))
        host[L.header:L.header + 32] = torch.from_numpy(hdr)
        self.inp = StepInput(host.to(device), L, hdr)
        self.caches = [c.to(device) for c in caches]

    def step_rows(self, per_sequence):
        """Rows of the step, in its order, of per-sequence tensors [tokens, ...]."""
        return torch.cat([per_sequence[i][self.lens[i][0]:] for i in self.order])
