"""Per-layer description of a decoder whose layers differ from one another (sizes, kind of mixer, kind of feed-forward),
for designs whose configuration lists the layers one by one instead of giving one set of sizes for all."""
from __future__ import annotations

import dataclasses
import math
from typing import List, Optional, Tuple, Union


@dataclasses.dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first `dims` dimensions of a head, optionally with YaRN scaling or slowed long wavelengths."""
    dims: int
    base: float
    interleaved: bool = False     # pairs (2i, 2i + 1); else (i, i + dims / 2)
    factor: float = 0.0           # YaRN: context extension (0: no scaling) ...
    original: float = 0.0         # ... of a model of so many positions ...
    fast: float = 32.0            # ... whose dimensions of at least so many turns over them keep their frequency
    slow: float = 1.0             # ... and of at most so many turns are slowed by the factor
    by_turns: bool = False        # the ramp between the two runs over turns per original context, not over dimensions, and cos and
                                  # sin keep their size (the scaling of Llama 3.1)

    def frequencies(self) -> Tuple[List[float], float]:
        """(angle per position of every pair, factor of cos and sin)."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.factor <= 0:
            return f, 1.0
        if self.by_turns:
            turns = [self.original * x / (2 * math.pi) for x in f]
            keep = [min(max((t - self.slow) / max(self.fast - self.slow, 1e-12), 0.0), 1.0) for t in turns]
            return [x * s + x / self.factor * (1 - s) for x, s in zip(f, keep)], 1.0

        def dim_of(turns):        # dimension that turns so often over the original positions
            return self.dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(self.base))
        lo, hi = max(math.floor(dim_of(self.fast)), 0), min(math.ceil(dim_of(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(self.dims // 2)]
        return [x / self.factor * r + x * (1 - r) for x, r in zip(f, ramp)], 0.1 * math.log(self.factor) + 1


@dataclasses.dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                      # query / key size of a head
    vdim: int                     # value size of a head
    scale: float                  # factor of q . k
    chunk: int = 0                # positions per chunk that a query may look at (0: all earlier ones)
    window: int = 0               # sliding window in positions (0: none)
    keep_first: int = 0           # first positions of the sequence that stay visible behind the window
    conv: int = 0                 # taps of a causal convolution on q, k and v ahead of norm and rotation (0: none)
    mixed_scores: bool = False    # a factor per head, then every head's scores become a weighted sum over all heads' scores
    learned_sink: bool = False    # a sink score of every head's own, part of the checkpoint
    distance_bias: bool = False   # take slope_h * (i - j) off the scores, slopes from `head_slopes`
    sink: Optional[float] = None  # score of a key without a value that joins the softmax denominator (None: no sink)
    qk_norm: bool = False         # RMS norm over every query and key head
    qk_norm_all: bool = False     # RMS norm over the whole query and the whole key projection, ahead of the split into heads
    qkv_bias: bool = False        # biases on the query, key and value projections
    output_gate: bool = False     # the heads' outputs times sigmoid of a projection of the layer's input
    rot: Optional[RotarySpec] = None
    softcap: float = 0.0          # scores become softcap * tanh(score / softcap) (0: they do not)
    maps: int = 1                 # 2: differential attention, two maps of query / key size `dim` per head over the same values
    diff: float = 0.0             # constant part of the second map's factor; the normed difference is multiplied by 1 - diff

    def head_slopes(self) -> List[float]:
        """Geometric slopes 2^(-8 (h + 1) / H), h = 0 .. H - 1."""
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclasses.dataclass
class LatentAttentionSpec:
    """Attention whose keys and values are projections of one latent per token, beside one rotated key part that all heads
    share; only those two are cached."""
    heads: int
    dim: int                      # unrotated query / key size of a head
    rot_dim: int                  # rotated one
    vdim: int                     # value size of a head
    kv_rank: int                  # size of the latent
    q_rank: int                   # size of the queries' own latent
    scale: float                  # factor of the whole score
    rot: RotarySpec

    @property
    def row(self) -> int:
        """Cached elements per token."""
        return self.kv_rank + self.rot_dim


@dataclasses.dataclass
class TimeMixSpec:
    """Linear attention with a matrix state per head, a data-dependent decay per key channel and a bonus for the current
    token; its inputs are blends of every token with the one before it."""
    heads: int
    dim: int                      # key and value size of a head
    decay_rank: int = 0           # inner size of the decay's low-rank projection (0: the checkpoint's tensors tell)


@dataclasses.dataclass
class GatedLinearSpec:
    """Linear attention with a matrix state per head that decays per key channel, by a power of a gate, ahead of every token."""
    heads: int
    dim: int                      # key size of a head
    vdim: int                     # value size of a head
    tau: float                    # decay = sigmoid(z)^(1 / tau)
    decay_rank: int = 0           # inner size of the gate's low-rank projection (0: the checkpoint's tensors tell)


@dataclasses.dataclass
class MatrixMemorySpec:
    """Matrix memory with exponential input gates and one forget gate per head, kept relative to a running maximum, and a
    normaliser (xLSTM's mLSTM)."""
    heads: int
    dim: int                      # query / key size of a head
    vdim: int                     # value size of a head
    gate_cap: float               # bound of both gates ahead of their exponential


@dataclasses.dataclass
class SelectiveScanSpec:
    """Diagonal state space layer with data-dependent step sizes, input and output vectors, behind a short causal
    convolution."""
    inner: int                    # channels
    state: int                    # states per channel
    conv: int                     # taps of the convolution
    dt_rank: int                  # inner size of the step sizes' low-rank projection


@dataclasses.dataclass
class ParallelSpec:
    """Two mixers side by side on the same input; their outputs are added with a factor each."""
    left: AttentionSpec
    right: Union[TimeMixSpec, GatedLinearSpec]
    left_scale: float = 1.0
    right_scale: float = 1.0
    branch_norm: bool = False     # every branch's output is normed over the model width ahead of its factor


Mixer = Union[AttentionSpec, LatentAttentionSpec, SelectiveScanSpec, MatrixMemorySpec, ParallelSpec]


def attention_of(mixer: Mixer) -> Optional[AttentionSpec]:
    """The attention part of a mixer: what its layer keeps in the paged cache as keys and values of heads (None: nothing)."""
    if isinstance(mixer, ParallelSpec):
        return mixer.left
    return mixer if isinstance(mixer, AttentionSpec) else None


@dataclasses.dataclass
class FeedForwardSpec:
    ff: int                       # inner size (of one expert in a mixture)
    act: str                      # gate activation "silu" | "gelu_tanh" | "clamped", or "relu2": squared relu without a gate
    limit: float = 0.0            # "clamped": bound of the gate (from above) and of the other factor (both sides)
    experts: int = 0              # experts with weights (0: a dense feed-forward)
    identity_experts: int = 0     # router outputs behind them whose expert is the identity
    top_k: int = 0
    n_group: int = 1              # equal groups of neighbouring router outputs ...
    topk_group: int = 1           # ... of which only the best ones may be chosen from
    group_score: str = "max"      # rank of a group: "max" | "top2" (sum of its two best choice scores)
    scoring: str = "softmax"      # "softmax" | "sigmoid" | "softmax_chosen": over the chosen logits only
    renormalize: bool = False     # chosen weights scaled to sum 1
    shared_ff: int = 0            # inner size of an expert that every token uses (0: none)

    @property
    def is_moe(self) -> bool:
        return self.experts > 0 or self.identity_experts > 0


@dataclasses.dataclass
class LayerSpec:
    mixer: Mixer
    mlp: Optional[FeedForwardSpec]      # None: the layer has no feed-forward sublayer


def run_order(n_layers: int, start: int = 0, stop: int = 0, times: int = 1) -> List[int]:
    """Layer index of every layer run: layers start .. stop - 1 run `times` times in a row, the others once."""
    if not 0 <= start <= stop <= n_layers or times < 1:
        raise ValueError(f"bad layer loop: start {start}, stop {stop}, times {times} with {n_layers} layers")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n_layers))


def pass_starts(n_layers: int, start: int = 0, stop: int = 0, times: int = 1) -> List[int]:
    """Index in `run_order` of the first run of every pass through the loop (empty: no loop)."""
    run_order(n_layers, start, stop, times)
    return [start + t * (stop - start) for t in range(times)] if stop > start else []
