"""Per-layer description of a decoder whose layers differ from one another (sizes, kind of mixer, kind of feed-forward),
for designs whose configuration lists the layers one by one instead of giving one set of sizes for all."""
from __future__ import annotations

import dataclasses
from typing import List, Optional


@dataclasses.dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                      # query / key size of a head
    vdim: int                     # value size of a head
    scale: float                  # factor of q . k
    chunk: int = 0                # positions per chunk that a query may look at (0: all earlier ones)
    window: int = 0               # sliding window in positions (0: none)
    distance_bias: bool = False   # take slope_h * (i - j) off the scores, slopes from `head_slopes`
    sink: Optional[float] = None  # score of a key without a value that joins the softmax denominator (None: no sink)
    qk_norm: bool = False         # RMS norm over every query and key head

    def head_slopes(self) -> List[float]:
        """Geometric slopes 2^(-8 (h + 1) / H), h = 0 .. H - 1."""
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclasses.dataclass
class FeedForwardSpec:
    ff: int                       # inner size (of one expert in a mixture)
    act: str                      # gate activation: "silu" | "gelu_tanh"
    experts: int = 0              # experts with weights (0: a dense feed-forward)
    identity_experts: int = 0     # router outputs behind them whose expert is the identity
    top_k: int = 0
    n_group: int = 1              # equal groups of neighbouring router outputs ...
    topk_group: int = 1           # ... of which only the best ones may be chosen from
    group_score: str = "max"      # rank of a group: "max" | "top2" (sum of its two best choice scores)
    scoring: str = "softmax"      # "softmax" | "sigmoid"
    renormalize: bool = False     # chosen weights scaled to sum 1
    shared_ff: int = 0            # inner size of an expert that every token uses (0: none)

    @property
    def is_moe(self) -> bool:
        return self.experts > 0 or self.identity_experts > 0


@dataclasses.dataclass
class LayerSpec:
    mixer: AttentionSpec
    mlp: Optional[FeedForwardSpec]      # None: the layer has no feed-forward sublayer


def run_order(n_layers: int, start: int = 0, stop: int = 0, times: int = 1) -> List[int]:
    """Layer index of every layer run: layers start .. stop - 1 run `times` times in a row, the others once."""
    if not 0 <= start <= stop <= n_layers or times < 1:
        raise ValueError(f"bad layer loop: start {start}, stop {stop}, times {times} with {n_layers} layers")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n_layers))
