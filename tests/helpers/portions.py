"""Ragged portions of a few sequences, run one step after the other, for tests of recurrent ops on the CPU."""
import torch


class Ragged:
    """Row ranges of unequal sequences for the recurrent ops: portions of given lengths, run one after the other."""

    def __init__(self, n_slots=6):
        self.n_slots = n_slots

    def steps(self, lens, cuts, seed=0):
        """lens: tokens per sequence; cuts: list of steps, each a list of portion lengths (0: left out).  Yields per step
        (q_cu, kv_lens, slots, n, rows) with rows = [(sequence, first, last), ...]."""
        g = torch.Generator().manual_seed(seed)
        slots = (torch.randperm(self.n_slots - 1, generator=g)[:len(lens)] + 1).int()
        done = [0] * len(lens)
        for step in cuts:
            ids = [i for i, c in enumerate(step) if c]
            q, rows = [0], []
            for i in ids:
                rows.append((i, done[i], done[i] + step[i]))
                q.append(q[-1] + step[i])
                done[i] += step[i]
            yield torch.tensor(q).int(), torch.tensor([done[i] for i in ids]).int(), slots[ids], len(ids), rows
        assert done == lens


CUTS = ([[7, 1, 20]], [[3, 1, 2], [1, 0, 2], [2, 0, 15], [1, 0, 1]], [[1, 1, 1]] + [[1, 0, 1]] * 6 + [[0, 0, 1]] * 13, [[2, 0, 18], [5, 1, 2]])
RAG = [7, 1, 20]


def rag(seqs, rows):
    return torch.cat([seqs[i][a:b] for i, a, b in rows])
