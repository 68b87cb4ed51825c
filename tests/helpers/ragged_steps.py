"""Steps over ragged batches with state slots on a GPU, for tests of recurrent and attention kernels."""
import numpy as np
import torch

from xllm_wxh_b200.framework.step_input import StepInput, make_layout

DEV = "cuda:0"


def status_ok():
    from xllm_wxh_b200.ops import cuda_ops
    return cuda_ops.read_status() == 0


def rel(got, want):
    return ((got.double().cpu() - want.double().cpu()).norm() / want.double().cpu().norm()).item()


def step_input(spans, slots, block=16, tables=None, pad=0):
    """Step whose sequences have run `before` tokens and bring `n` more: spans = [(before, n), ...], single decoded tokens
    first.  `pad`: padding rows and sequences behind them, as in a captured step."""
    T, B = sum(n for _, n in spans), len(spans)
    nb = max(-(-(b + n) // block) for b, n in spans)
    L = make_layout(T + pad, B + pad, nb, B, 32)
    host = torch.zeros(L.total_words, dtype=torch.int32)
    at, n_dec = 0, 0
    host[L.token_seq:L.token_seq + T + pad] = -1
    for s, (before, n) in enumerate(spans):
        assert n_dec == s or not (n == 1 and before > 0)
        n_dec += n == 1 and before > 0
        pos = torch.arange(before, before + n, dtype=torch.int32)
        host[L.positions + at:L.positions + at + n] = pos
        host[L.token_seq + at:L.token_seq + at + n] = s
        if tables is not None:
            t = torch.tensor(tables[s], dtype=torch.int32)
            host[L.block_tables + s * nb:L.block_tables + s * nb + len(t)] = t
            host[L.slots + at:L.slots + at + n] = t[pos.long() // block] * block + pos % block
        at += n
        host[L.q_cu + s + 1] = at
        host[L.kv_lens + s] = before + n
        host[L.state_slots + s] = slots[s]
    host[L.q_cu + B + 1:L.q_cu + B + pad + 1] = at
    hdr = np.zeros(32, dtype=np.int32)
    hdr[0], hdr[1], hdr[3], hdr[4] = T, B, n_dec, B - n_dec
    hdr[5], hdr[6], hdr[7], hdr[17] = max(n for _, n in spans), max(b + n for b, n in spans), 2 if n_dec == B else 3, block
    hdr[21] = sum(n for b, n in spans if not (n == 1 and b > 0))
    host[L.header:L.header + 32] = torch.from_numpy(hdr)
    return StepInput(host.to(DEV), L, hdr, padded=pad > 0)


class Ragged:
    """Sequences run in portions by a recurrent op: `steps` lists the portion of every sequence per step (0: left out)."""

    def __init__(self, lens, steps, n_slots=9, pad=0, seed=0):
        self.lens, self.steps, self.pad, self.n_slots = lens, steps, pad, n_slots
        self.slots = (torch.randperm(n_slots - 1, generator=torch.Generator().manual_seed(seed))[:len(lens)] + 1).tolist()

    def __iter__(self):
        done = [0] * len(self.lens)
        for step in self.steps:
            ids = [i for i, n in enumerate(step) if n]
            ids.sort(key=lambda i: not (step[i] == 1 and done[i] > 0))
            inp = step_input([(done[i], step[i]) for i in ids], [self.slots[i] for i in ids], pad=self.pad)
            rows = [(i, done[i], done[i] + step[i]) for i in ids]
            for i in ids:
                done[i] += step[i]
            yield inp, rows
        assert done == self.lens

    def take(self, seqs, rows):
        x = torch.cat([seqs[i][a:b] for i, a, b in rows])
        if self.pad:
            x = torch.cat([x, torch.full((self.pad,) + x.shape[1:], 7.0, dtype=x.dtype)])
        return x.to(DEV)
