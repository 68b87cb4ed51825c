"""A model design beside the framework's closest other one at equal layer sizes (`bench.py --compare-design movolorn|falalix|babadra|govuvik`):
tokens per second of the decoder layers in prefill and decode, and the design's own kernels beside the like kernels with their
distance from the roofline.  Random weights; kernel and layer times come from CUDA-graph replay between CUDA events, with
weights, caches and activations rotated through (or larger than) more memory than L2 holds."""
from __future__ import annotations

import dataclasses
import json
import os
from typing import Callable, Dict, List

import numpy as np
import torch

from ..framework.step_input import StepInput, make_layout
from ..models.args import ModelArgs, QuantArgs, preset
from ..models.layer_spec import AttentionSpec, LatentAttentionSpec, MatrixMemorySpec, ParallelSpec, RotarySpec, SelectiveScanSpec
from ..models.registry import get_model_class
from . import cuda_ops as c
from . import moe_cuda
from .bench_kernels import time_graph

DEV = "cuda:0"
# (model, closest one, which of the model's kinds of layer)
PAIRS = {"movolorn": [("movolorn-8b", "qwen3-8b", ""), ("movolorn-30b-a3b", "qwen3-30b-a3b", "")],
         "falalix": [("falalix-8b", "qwen3-8b", "parallel"), ("falalix-8b", "qwen3-8b", "scan"), ("falalix-8b", "qwen3-8b", "")],
         "babadra": [("babadra-8b", "deepseek-8b", "latent"), ("babadra-8b", "qwen3-8b", "two-map"),
                     ("babadra-30b-a3b", "qwen3-30b-a3b", "two-map")],
         "govuvik": [("govuvik-30b-a3b", "qwen3-30b-a3b", "parallel"), ("govuvik-30b-a3b", "qwen3-30b-a3b", "memory"),
                     ("govuvik-30b-a3b", "qwen3-30b-a3b", "")]}
KINDS = {"parallel": lambda m: isinstance(m, ParallelSpec), "scan": lambda m: isinstance(m, SelectiveScanSpec),
         "latent": lambda m: isinstance(m, LatentAttentionSpec), "two-map": lambda m: getattr(m, "maps", 1) == 2,
         "memory": lambda m: isinstance(m, MatrixMemorySpec)}


def args_of(name: str) -> ModelArgs:
    if name == "deepseek-8b":            # the attention of deepseek-v3 with the width, heads and feed-forward of qwen3-8b, in bf16
        return dataclasses.replace(preset("deepseek-v3"), hidden_size=4096, n_heads=32, n_kv_heads=32, intermediate_size=12288, vocab_size=151936,
                                   n_routed_experts=0, quant=QuantArgs(), rope_scaling_factor=4.0, rope_original_max_position=8192,
                                   max_position_embeddings=32768)
    return preset(name)


# Issue rates that bound recurrent kernels in fp32, per second over 148 SMs at 1.9 GHz: 128 multiply-adds and 16 exponentials
# per SM and clock (nominal; there is no measured figure for them).
FMA_RATE, EXP_RATE = 148 * 128 * 1.9e9, 148 * 16 * 1.9e9
STEPS = [("prefill", 1, 8192, 8192), ("prefill", 8, 1024, 1024), ("decode", 256, 1, 1152), ("decode", 32, 1, 8192)]


def peaks() -> Dict[str, float]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return {"hbm_gbs": p["hbm_gbs"], "bf16_tflops": p["bf16_tflops"], "what": "measured"}
    except (OSError, KeyError, ValueError):
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "what": "fallback"}


def step_input(seqs: int, q_len: int, kv_len: int, block: int, vocab: int) -> StepInput:
    """`seqs` equal sequences of kv_len tokens whose last q_len are in the step, on shuffled blocks."""
    T, nb = seqs * q_len, -(-kv_len // block)
    L = make_layout(T, seqs, nb, seqs, 32)
    host = torch.zeros(L.total_words, dtype=torch.int32)
    bt = (torch.randperm(seqs * nb) + 1).int().view(seqs, nb)
    pos = torch.arange(kv_len - q_len, kv_len).repeat(seqs)
    seq = torch.arange(seqs).repeat_interleave(q_len)
    host[L.tokens:L.tokens + T] = torch.randint(0, vocab, (T,)).int()
    host[L.positions:L.positions + T] = pos.int()
    host[L.token_seq:L.token_seq + T] = seq.int()
    host[L.slots:L.slots + T] = (bt[seq, pos // block] * block + (pos % block)).int()
    host[L.q_cu:L.q_cu + seqs + 1] = (torch.arange(seqs + 1) * q_len).int()
    host[L.kv_lens:L.kv_lens + seqs] = kv_len
    host[L.state_slots:L.state_slots + seqs] = torch.randperm(seqs).int() + 1
    host[L.block_tables:L.block_tables + seqs * nb] = bt.reshape(-1)
    hdr = np.zeros(32, dtype=np.int32)
    dec = q_len == 1
    hdr[0], hdr[1], hdr[3], hdr[4], hdr[5], hdr[6] = T, seqs, seqs if dec else 0, 0 if dec else seqs, q_len, kv_len
    hdr[7], hdr[17], hdr[21] = 2 if dec else 0, block, 0 if dec else T
    host[L.header:L.header + 32] = torch.from_numpy(hdr)
    return StepInput(host.to(DEV), L, hdr)


def cut_to_layers(a: ModelArgs, n: int, kind: str = "") -> ModelArgs:
    """n layers, all of one kind (a key of KINDS) where a model has several and one is named."""
    kw = dict(n_layers=n)
    if a.layer_specs:
        specs = [s for s in a.layer_specs if not kind or KINDS[kind](s.mixer)]
        kw.update(layer_specs=specs[:n], layer_runs=list(range(n)), pass_starts=[])
    return dataclasses.replace(a, **kw)


@torch.inference_mode()
def layer_throughput(name: str, layers: int, block: int, kind: str = "") -> List[Dict]:
    args = cut_to_layers(args_of(name), layers, kind)
    model = get_model_class(args.model_type)(args, device=DEV, dtype=torch.bfloat16).init_random(0)
    if hasattr(model, "finalize_weights"):
        model.finalize_weights()
    rows = []
    for kind, seqs, q_len, kv_len in STEPS:
        inp = step_input(seqs, q_len, kv_len, block, args.vocab_size)
        blocks = seqs * (-(-kv_len // block)) + 1
        kv = [tuple(torch.randn(s, device=DEV, dtype=torch.bfloat16) for s in pair) for pair in model.kv_cache_shapes(blocks, block)]
        if hasattr(model, "state_cache_shapes"):
            inp.states = [tuple(torch.zeros(s, device=DEV, dtype=dt) for s, dt in run) for run in model.state_cache_shapes(seqs + 1)]
        us = time_graph([lambda: model.forward(inp, kv)] * 3)
        rows.append({"step": kind, "sequences": seqs, "tokens": seqs * q_len, "context": kv_len, "us_per_layer": round(us / layers, 1),
                     "tokens_per_s_per_layer": round(seqs * q_len / us * layers * 1e6)})
        del kv
    del model
    torch.cuda.empty_cache()
    return rows


def _rotated(make: Callable[[], tuple], nbytes: float) -> List[tuple]:
    """Enough copies of a kernel's inputs that a pass over all of them leaves nothing of the first in L2."""
    return [make() for _ in range(min(64, max(2, int(400e6 / max(nbytes, 1)) + 1)))]


def _bf(*shape, std=1.0):
    return (torch.randn(*shape, device=DEV) * std).to(torch.bfloat16)


class Rows:
    """Kernels of a design beside the like ones: microseconds and fraction of the roofline of each."""

    def __init__(self):
        self.pk = peaks()
        self.rows = []

    def add(self, what, ours, like, bytes_ours=0.0, bytes_like=0.0, flops=0.0, flops_like=None, fma=0.0, fma_like=0.0):
        def frac(us, nbytes, ops, fp32):
            bound = max(nbytes / (self.pk["hbm_gbs"] * 1e3), ops / (self.pk["bf16_tflops"] * 1e6), fp32 / FMA_RATE * 1e6)
            return bound / us
        fo, fl = frac(ours, bytes_ours, flops, fma), frac(like, bytes_like, flops if flops_like is None else flops_like, fma_like)
        self.rows.append({"what": what, "us": round(ours, 1), "like_us": round(like, 1), "roofline": round(fo, 3), "like_roofline": round(fl, 3),
                          "farther_by": round(fl / fo, 2)})

    def add_alone(self, what, us, nbytes, fma=0.0, exps=0.0):
        """A kernel without a like one: its bound is the slowest of memory, fp32 multiply-adds and exponentials."""
        bounds = {"memory": nbytes / (self.pk["hbm_gbs"] * 1e3), "fp32": fma / FMA_RATE * 1e6, "exp": exps / EXP_RATE * 1e6}
        by = max(bounds, key=bounds.get)
        self.rows.append({"what": what, "us": round(us, 1), "roofline": round(bounds[by] / us, 3), "bound_by": by})


@torch.inference_mode()
def movolorn_kernels() -> List[Dict]:
    table_rows = Rows()
    add, rows = table_rows.add, table_rows.rows
    # ---- attention
    for H, G, chunk in ((32, 8, 8192), (32, 4, 8192)):
        spec = AttentionSpec(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5)
        slopes, sinks = torch.tensor(spec.head_slopes(), device=DEV), torch.zeros(H, device=DEV)
        for kind, seqs, q_len, kv in STEPS:
            inp = step_input(seqs, q_len, kv, 16, 1000)
            nb = seqs * (-(-kv // 16)) + 1
            row = (H + 2 * G) * 128
            cache_bytes = 2.0 * seqs * kv * G * 128 * 2
            sets = _rotated(lambda: (_bf(seqs * q_len, row), _bf(nb, 16, G, 128), _bf(nb, 16, G, 128)), cache_bytes + seqs * q_len * row * 2)
            sets = sets[:8]
            view = lambda q: q[:, :H * 128].unflatten(1, (H, 128))
            o = time_graph([lambda s=s: c.paged_attention_ext(view(s[0]), s[1], s[2], inp, spec.scale, -1, chunk, slopes, sinks) for s in sets])
            k = time_graph([lambda s=s: c.paged_attention(view(s[0]), s[1], s[2], inp, spec.scale) for s in sets])
            byts = cache_bytes + 2.0 * seqs * q_len * H * 128 * 2
            fl = 4.0 * H * 128 * seqs * (q_len * (kv - q_len) + q_len * (q_len + 1) / 2)
            add(f"attention {kind} {seqs} x {q_len} of {kv}, {H}/{G} heads", o, k, byts, byts, fl if kind == "prefill" else 0.0)
    # ---- norms around the residual, per-head norm + cache write
    for T, H in ((8192, 4096), (256, 4096), (8192, 2048), (256, 2048)):
        w = _bf(H)
        sets = _rotated(lambda: (_bf(T, H), torch.randn(T, H, device=DEV), _bf(T, H)), T * H * 10.0)
        o = time_graph([lambda s=s: c.post_norm_add_norm(s[0], s[1], w, w, 1e-6) for s in sets])
        k = time_graph([lambda s=s: c.add_rms_norm(s[0], s[2], w, 1e-6) for s in sets])
        add(f"norm + residual + norm, {T} x {H}", o, k, T * H * 12.0, T * H * 8.0)
    cs = torch.randn(8192, 128, device=DEV)
    for T, H, G in ((8192, 32, 8), (256, 32, 8)):
        w = _bf(128)
        inp = step_input(1, T, T, 16, 1000)
        row = (H + 2 * G) * 128
        sets = _rotated(lambda: (_bf(T, row), _bf(T // 16 + 1, 16, G, 128), _bf(T // 16 + 1, 16, G, 128)), T * row * 2.0)
        o = time_graph([lambda s=s: c.qknorm_kvwrite(s[0], inp.slots, w, w, 1e-6, s[1], s[2], H, G) for s in sets])
        k = time_graph([lambda s=s: c.rope_qknorm_kvwrite(s[0], inp.positions, inp.slots, cs, w, w, 1e-6, s[1], s[2], H, G, 128) for s in sets])
        add(f"q / k norm + cache write, {T} tokens", o, k, T * (2.0 * H + 4 * G) * 256, T * (2.0 * H + 5 * G) * 256 + T * 512.0)
    ids = torch.randint(0, 151936, (8192,), device=DEV).int()
    table, w = _bf(151936, 2048), _bf(2048)
    o = time_graph([lambda: c.embed_rms_norm(ids, table, 2.0, w, 1e-6)] * 8)
    k = time_graph([lambda: c.rms_norm(c.embedding(ids, table), w, 1e-6)] * 8)
    add("embedding + first norm, 8192 x 2048", o, k, 8192 * 2048 * 8.0, 8192 * 2048 * 8.0)
    del table
    # ---- gated feed-forward product
    for T in (8192, 256):
        sets = _rotated(lambda: (_bf(T, 4096), _bf(24576, 4096, std=0.02)), 24576 * 8192.0)[:3]
        o = time_graph([lambda s=s: c.linear_gated(s[0], s[1], "gelu_tanh") for s in sets])
        k = time_graph([lambda s=s: c.linear_swiglu(s[0], s[1]) for s in sets])
        b = 24576 * 8192.0 + T * (8192.0 + 24576.0)
        add(f"gate / up product + gate, {T} x 24576 x 4096", o, k, b, b, 2.0 * T * 24576 * 4096)
    # ---- router and mixture (128 router outputs: 124 experts + 4 identity, against 128 experts)
    E, ident, H, I, top = 128, 4, 2048, 768, 8
    wr, corr = _bf(E, H, std=0.02), torch.randn(E, device=DEV) * 0.01
    w13, w2 = _bf(E, 2 * I, H, std=0.02), _bf(E, H, I, std=0.02)
    moe_cuda.interleave_w13(w13)
    for T in (8192, 256):
        sets = _rotated(lambda: (_bf(T, H), torch.randn(T, H, device=DEV), _bf(T, H)), T * H * 10.0)[:16]

        def ours_router(s):
            return c.moe_router(c.linear_f32(s[0], wr), top, "softmax", False, corr, 8, 4, 1.0, "max")

        def like_router(s):
            return c.moe_router(c.linear(s[0], wr), top, "softmax", True)
        o = time_graph([lambda s=s: ours_router(s) for s in sets])
        k = time_graph([lambda s=s: like_router(s) for s in sets])
        add(f"router product + choice, {T} x {E}", o, k, T * H * 2.0 + E * H * 2.0 + T * 64.0, T * H * 2.0 + E * H * 2.0 + T * 64.0,
            2.0 * T * E * H)
        wts, idx = like_router(sets[0])
        n = E - ident

        def ours_mix(s):
            y, dst = moe_cuda.expert_rows(s[0], w13[:n], w2[:n], idx, "silu", True)
            return moe_cuda.combine_post_norm_add_norm(y, dst, idx, wts, s[0], None, n, s[1], w, w, 1e-6)

        def like_mix(s):
            return c.add_rms_norm(moe_cuda.moe_experts(s[0], w13, w2, wts, idx, 0, True), s[2], w, 1e-6)
        o = time_graph([lambda s=s: ours_mix(s) for s in sets])
        k = time_graph([lambda s=s: like_mix(s) for s in sets])
        b = 3.0 * E * I * H * 2
        local = float((idx < n).sum())
        rows_like = float(idx.numel())
        add(f"mixture to the next sublayer's input, {T} tokens", o, k, b * n / E + T * H * 12.0, b + T * H * 8.0, 6.0 * rows_like * I * H)
        rows[-1]["expert_rows"] = [int(local), int(rows_like)]
        # the combine with its norms alone
        y, dst = moe_cuda.expert_rows(sets[0][0], w13[:n], w2[:n], idx, "silu", True)
        r = moe_cuda.moe_sort(idx, 0, E)
        o = time_graph([lambda s=s: moe_cuda.combine_post_norm_add_norm(y, dst, idx, wts, s[0], None, n, s[1], w, w, 1e-6) for s in sets])
        k = time_graph([lambda s=s: c.add_rms_norm(moe_cuda.combine(y, r, wts, T), s[2], w, 1e-6) for s in sets])
        add(f"combine + norms, {T} tokens", o, k, T * H * (2.0 * top + 12), T * H * (2.0 * top + 10))
    return rows


@torch.inference_mode()
def falalix_kernels() -> List[Dict]:
    R = Rows()
    add, alone = R.add, R.add_alone
    H = 4096
    # ---- attention with a window and kept first keys, beside the same window without
    for kind, seqs, q_len, kv in STEPS:
        heads, G, window, keep = 32, 8, 4096, 128
        inp = step_input(seqs, q_len, kv, 16, 1000)
        nb, row = seqs * (-(-kv // 16)) + 1, (heads + 2 * G) * 128
        seen = min(kv, window + keep)
        cache_bytes = 2.0 * seqs * (kv if kind == "prefill" else seen) * G * 128 * 2
        sets = _rotated(lambda: (_bf(seqs * q_len, row), _bf(nb, 16, G, 128), _bf(nb, 16, G, 128)), cache_bytes + seqs * q_len * row * 2)[:8]
        view = lambda q: q[:, :heads * 128].unflatten(1, (heads, 128))
        o = time_graph([lambda s=s: c.paged_attention_ext(view(s[0]), s[1], s[2], inp, 128 ** -0.5, window, 0, None, None, keep) for s in sets])
        k = time_graph([lambda s=s: c.paged_attention(view(s[0]), s[1], s[2], inp, 128 ** -0.5, window) for s in sets])
        byts = cache_bytes + 2.0 * seqs * q_len * heads * 128 * 2
        first = kv - q_len
        pairs = sum(min(p + 1, window + keep) for p in range(first, kv)) * seqs
        add(f"attention {kind} {seqs} x {q_len} of {kv}, window {window} + {keep}", o, k, byts, byts,
            4.0 * heads * 128 * pairs if kind == "prefill" else 0.0)
    # ---- norms, cache write, gates
    cs = torch.randn(8192, 128, device=DEV)
    for T in (8192, 256):
        w, wa = _bf(H), (_bf(4096), _bf(1024))
        sets = _rotated(lambda: (_bf(T, H), torch.randn(T, H, device=DEV), _bf(T, H)), T * H * 10.0)
        o = time_graph([lambda s=s: c.add_norm(s[0], s[1], 0.3, w, 1e-6) for s in sets])
        k = time_graph([lambda s=s: c.add_rms_norm(s[0], s[2], w, 1e-6) for s in sets])
        add(f"residual + norm, {T} x {H}", o, k, T * H * 12.0, T * H * 8.0)
        inp = step_input(1, T, T, 16, 1000)
        sets = _rotated(lambda: (_bf(T, 10240), _bf(T // 16 + 1, 16, 8, 128), _bf(T // 16 + 1, 16, 8, 128), _bf(T, 6144)), T * 10240 * 2.0)[:24]
        o = time_graph([lambda s=s: c.qknorm_all_kvwrite(s[0], inp.slots, wa[0], wa[1], 1e-6, s[1], s[2], 32, 8) for s in sets])
        k = time_graph([lambda s=s: c.rope_qknorm_kvwrite(s[3], inp.positions, inp.slots, cs, w, w, 1e-6, s[1], s[2], 32, 8, 128) for s in sets])
        add(f"q / k norm + cache write, {T} tokens", o, k, T * 96.0 * 256, T * 104.0 * 256 + T * 512.0)
        sets = _rotated(lambda: (_bf(T, 4096), _bf(T, 10240), torch.empty(T, 8192, device=DEV, dtype=torch.bfloat16), _bf(T, 8192)), T * 4096 * 6.0)[:24]
        o = time_graph([lambda s=s: c.gate_into(s[0], s[1][:, 6144:], 0.5, s[2][:, :4096]) for s in sets])
        k = time_graph([lambda s=s: c.silu_and_mul(s[3]) for s in sets])
        add(f"output gate, {T} x 4096", o, k, T * 4096 * 6.0, T * 4096 * 6.0)
        # ---- products with an epilogue
        sets = _rotated(lambda: (_bf(T, H), _bf(12288, H, std=0.02)), 12288 * 8192.0)[:4]
        o = time_graph([lambda s=s: c.act_linear(s[0], s[1], "relu2") for s in sets])
        k = time_graph([lambda s=s: c.linear(s[0], s[1]) for s in sets])
        b = 12288 * 8192.0 + T * (8192.0 + 24576.0)
        add(f"up product + squared relu, {T} x 12288 x 4096", o, k, b, b, 2.0 * T * 12288 * H)
    # ---- recurrent kernels, which have no like one
    C, N, taps, heads, d = 8192, 16, 4, 64, 64
    for kind, seqs, q_len, kv in STEPS[:3]:
        T = seqs * q_len
        inp = step_input(seqs, q_len, kv, 16, 1000)
        new = kv == q_len
        sets = [(_bf(T, H), _bf(5, H), _bf(seqs + 1, H)) for _ in range(8)]
        alone(f"token shift, {kind} {seqs} x {q_len}", time_graph([lambda s=s: c.token_shift(s[0], s[1], s[2], inp) for s in sets]), T * H * 12.0)
        del sets
        sets = [(_bf(T, 2 * C), _bf(taps, C), _bf(C), _bf(seqs + 1, taps - 1, C)) for _ in range(4 if kind == "prefill" else 16)]
        alone(f"convolution, {kind} {seqs} x {q_len}", time_graph([lambda s=s: c.causal_conv(s[0][:, :C], s[1], s[2], s[3], inp, "silu") for s in sets]),
              T * C * 4.0 + (0 if new else 2) * seqs * 3 * C * 2.0)
        del sets
        A = -torch.rand(C, N, device=DEV)
        D, bias = torch.randn(C, device=DEV), torch.randn(C, device=DEV) - 3
        sets = [(_bf(T, C), torch.randn(T, C, device=DEV), _bf(T, 288), _bf(T, 2 * C), torch.zeros(seqs + 1, C, N, device=DEV)) for _ in range(3)]
        us = time_graph([lambda s=s: c.selective_scan(s[0], s[1], bias, A, s[2][:, 256:272], s[2][:, 272:], D, s[3][:, C:], s[4], inp) for s in sets])
        alone(f"selective scan, {kind} {seqs} x {q_len}, {C} channels x {N}", us, T * C * 10.0 + (1 if new else 2) * seqs * C * N * 4.0,
              3.0 * T * C * N, 1.0 * T * C * N)
        del sets
        n = heads * d
        u, w0, nw = torch.randn(heads, d, device=DEV), torch.randn(n, device=DEV) - 3, _bf(n)
        sets = [(_bf(T, n), _bf(T, n), _bf(T, n), torch.randn(T, n, device=DEV), _bf(T, n), torch.empty(T, 2 * n, device=DEV, dtype=torch.bfloat16),
                 torch.zeros(seqs + 1, heads, d, d, device=DEV)) for _ in range(3)]
        us = time_graph([lambda s=s: c.time_mix(s[0], s[1], s[2], s[3], w0, u, s[4], nw, 0.5, 1e-6, s[6], inp, s[5][:, n:]) for s in sets])
        alone(f"time mixing, {kind} {seqs} x {q_len}, {heads} heads of {d}", us, T * n * 14.0 + (1 if new else 2) * seqs * n * d * 4.0, 3.0 * T * n * d,
              2.0 * T * n)
        del sets
    return R.rows


@torch.inference_mode()
def babadra_kernels() -> List[Dict]:
    R = Rows()
    add = R.add
    H, heads = 4096, 32
    # ---- differential attention beside attention with as many query, key and value columns
    factor, bound = torch.tensor([0.7], device=DEV), 1.02 * 64         # norm weights of one
    for G in (8, 4):
        for kind, seqs, q_len, kv in STEPS:
            inp = step_input(seqs, q_len, kv, 16, 1000)
            nb, row, T = seqs * (-(-kv // 16)) + 1, (heads + 2 * G) * 128, seqs * q_len
            cache_bytes = 2.0 * seqs * kv * G * 128 * 2
            sets = _rotated(lambda: (_bf(T, row), _bf(nb, 16, G, 128), _bf(nb, 16, G, 128)), cache_bytes + T * row * 2)[:8]
            o = time_graph([lambda s=s: c.paged_attention_ext(s[0][:, :heads * 128].unflatten(1, (2 * heads, 64)), s[1].view(nb, 16, 2 * G, 64), s[2], inp,
                                                              64 ** -0.5, softcap=50.0, mix=(factor, 0.4, 1e-6), bound=bound) for s in sets])
            k = time_graph([lambda s=s: c.paged_attention(s[0][:, :heads * 128].unflatten(1, (heads, 128)), s[1], s[2], inp, 128 ** -0.5) for s in sets])
            byts = cache_bytes + 2.0 * T * heads * 128 * 2
            pairs = seqs * (q_len * (kv - q_len) + q_len * (q_len + 1) / 2)
            # products: both maps' scores, and both maps' sums of the values
            fo, fk = (2.0 * 2 * 64 + 2.0 * 2 * 128) * heads * pairs, 4.0 * 128 * heads * pairs
            if kind == "prefill":
                add(f"two-map attention {kind} {seqs} x {q_len} of {kv}, {heads}/{G} heads", o, k, byts, byts, fo, fk)
            else:
                add(f"two-map attention {kind} {seqs} x {q_len} of {kv}, {heads}/{G} heads", o, k, byts, byts)
            del sets
    # ---- latent attention: from the projected queries to the heads' outputs
    dim, rd, C, nq, dv = 128, 64, 512, 1536, 128
    uk, uv = _bf(heads, C, dim, std=0.05), _bf(heads, dv, C, std=0.05)
    table = torch.randn(8192, rd, device=DEV)
    kc = uk.transpose(1, 2).contiguous()
    w_q, w_c, w_down = _bf(nq), _bf(C), _bf(nq + C + rd, H, std=0.02)
    w_qa, w_kva = w_down[:nq].contiguous(), w_down[nq:].contiguous()
    for kind, seqs, q_len, kv in STEPS:
        inp = step_input(seqs, q_len, kv, 16, 1000)
        nb, T = seqs * (-(-kv // 16)) + 1, seqs * q_len
        rot = (table, inp.positions, True)
        sets = _rotated(lambda: (_bf(T, heads * (dim + rd)), _bf(nb, 16, C + rd), _bf(T, C + rd), _bf(T, H)), seqs * kv * 1152.0)[:8]
        o = time_graph([lambda s=s: c.latent_attention_mla(s[0].view(T, heads, dim + rd), uk, uv, s[1], inp, rot, 0.07, dim) for s in sets])

        def like(s):
            a, b = c.mla_prepare(s[0].view(T, heads, dim + rd), s[2], inp.positions, inp.slots, table, w_c, 1e-6, s[1], kc, dim, rd, C)
            return c.mla_v_up(c.mla_attention(a, b, s[1], inp, 0.07, C), uv)
        k = time_graph([lambda s=s: like(s) for s in sets])
        pairs = seqs * (q_len * (kv - q_len) + q_len * (q_len + 1) / 2)
        fl = 2.0 * heads * ((2 * C + rd) * pairs + T * C * (dim + dv))
        byts = seqs * kv * (C + rd) * 2.0 + T * heads * (dim + rd + dv) * 2.0
        add(f"latent attention {kind} {seqs} x {q_len} of {kv}, {heads} heads", o, k, byts, byts, fl)
        if (seqs, q_len) not in ((1, 8192), (256, 1)):
            continue
        # ---- what lies ahead of it: down products, norms, rotation, cache write
        o = time_graph([lambda s=s: c.latent_down(c.linear(s[3], w_down), nq, C, w_q, w_c, 1e-6, rot, inp.slots, s[1]) for s in sets])
        k = time_graph([lambda s=s: (c.rms_norm(c.linear(s[3], w_qa), w_q, 1e-6), c.linear(s[3], w_kva)) for s in sets])
        n = nq + C + rd
        add(f"down products + norms, {T} tokens", o, k, T * (H * 2.0 + n * 2) + n * H * 2.0, T * (H * 4.0 + n * 2) + n * H * 2.0, 2.0 * T * n * H)
        low = [_bf(T, n) for _ in range(8 if T > 1000 else 32)]
        o = time_graph([lambda x=x: c.latent_down(x, nq, C, w_q, w_c, 1e-6, rot, inp.slots, sets[0][1]) for x in low])
        k = time_graph([lambda x=x: (c.rms_norm(x[:, :nq], w_q, 1e-6), c.rms_norm(x[:, nq:nq + C], w_c, 1e-6)) for x in low])
        add(f"norms + rotation + cache write of {T} latents", o, k, T * n * 4.0, T * (nq + C) * 4.0)
    # ---- norms, embedding, q / k norm with rotation
    cs = torch.randn(8192, 128, device=DEV)
    t64 = torch.randn(8192, 64, device=DEV)
    pos = _bf(8192, H)
    for T in (8192, 256):
        w, w64, w128 = _bf(H), _bf(64), _bf(128)
        sets = _rotated(lambda: (_bf(T, H), torch.randn(T, H, device=DEV), _bf(T, H)), T * H * 10.0)
        k = time_graph([lambda s=s: c.add_rms_norm(s[0], s[2], w, 1e-6) for s in sets])
        o = time_graph([lambda s=s: c.add_norm(s[0], s[1], 1.0, w, 1e-6, w, 1.0) for s in sets])
        add(f"layer scale + residual + norm, {T} x {H}", o, k, T * H * 12.0, T * H * 8.0)
        ids, at = torch.randint(0, 30000, (T,), device=DEV).int(), torch.arange(T, device=DEV).int()
        emb = _bf(30000, H)
        o = time_graph([lambda s=s: c.add_norm(s[0], s[1], 1.0, w, 1e-6, w, 1.0, (ids, emb, 2.0, at, pos)) for s in sets])
        add(f"the same at the head of a pass, {T} x {H}", o, k, T * H * 16.0, T * H * 8.0)
        o = time_graph([lambda: c.embed_rms_norm(ids, emb, 2.0, w, 1e-6, at, pos, 1.0)] * 8)
        k = time_graph([lambda: c.rms_norm(c.embedding(ids, emb), w, 1e-6)] * 8)
        add(f"embedding + positions + first norm, {T} x {H}", o, k, T * H * 10.0, T * H * 8.0)
        inp, row = step_input(1, T, T, 16, 1000), 48 * 128
        sets = _rotated(lambda: (_bf(T, row), _bf(T // 16 + 1, 16, 8, 128), _bf(T // 16 + 1, 16, 8, 128)), T * row * 2.0)[:24]
        o = time_graph([lambda s=s: c.qknorm_kvwrite(s[0], inp.slots, w64, w64, 1e-6, s[1].view(-1, 16, 16, 64), s[2], 64, 16, (t64, inp.positions, False))
                        for s in sets])
        k = time_graph([lambda s=s: c.rope_qknorm_kvwrite(s[0], inp.positions, inp.slots, cs, w128, w128, 1e-6, s[1], s[2], 32, 8, 128) for s in sets])
        add(f"q / k norm + rotation + cache write, {T} tokens", o, k, T * 104.0 * 256 + T * 256.0, T * 104.0 * 256 + T * 512.0)
        # ---- products with an epilogue
        sets = _rotated(lambda: (_bf(T, H), _bf(24576, H, std=0.02)), 24576 * 8192.0)[:3]
        o = time_graph([lambda s=s: c.linear_gated(s[0], s[1], "clamped", 7.0) for s in sets])
        k = time_graph([lambda s=s: c.linear_swiglu(s[0], s[1]) for s in sets])
        b = 24576 * 8192.0 + T * (8192.0 + 24576.0)
        add(f"gate / up product + clamped gate, {T} x 24576 x {H}", o, k, b, b, 2.0 * T * 24576 * H)
        del sets
    x, head = _bf(256, H), _bf(151936, H, std=0.02)
    o, k = time_graph([lambda: c.linear_softcap(x, head, 30.0)] * 3), time_graph([lambda: c.linear(x, head)] * 3)
    add("bounded logits, 256 x 151936", o, k, 151936 * (H * 2.0 + 512.0), 151936 * (H * 2.0 + 512.0), 2.0 * 256 * 151936 * H)
    del x, head
    # ---- router and mixture
    E, W, I, top = 128, 2048, 768, 8
    wr, br = _bf(E, W, std=0.02), torch.randn(E, device=DEV) * 0.01
    w13, w2, ls, w = _bf(E, 2 * I, W, std=0.02), _bf(E, W, I, std=0.02), _bf(W), _bf(W)
    moe_cuda.interleave_w13(w13)
    for T in (8192, 256):
        sets = _rotated(lambda: (_bf(T, W), torch.randn(T, W, device=DEV), _bf(T, W)), T * W * 10.0)[:16]
        o = time_graph([lambda s=s: c.moe_router(c.linear_f32(s[0], wr), top, "softmax_chosen", bias=br) for s in sets])
        k = time_graph([lambda s=s: c.moe_router(c.linear(s[0], wr), top, "softmax", True) for s in sets])
        b = T * W * 2.0 + E * W * 2.0 + T * 64.0
        add(f"router product + choice, {T} x {E}", o, k, b, b, 2.0 * T * E * W)
        wts, idx = c.moe_router(c.linear(sets[0][0], wr), top, "softmax", True)

        def ours_mix(s):
            y, dst = moe_cuda.expert_rows(s[0], w13, w2, idx, "clamped", True, 7.0)
            return moe_cuda.combine_add_norm(y, dst, wts, ls, s[1], w, 1e-6, 1.0)
        o = time_graph([lambda s=s: ours_mix(s) for s in sets])
        k = time_graph([lambda s=s: c.add_rms_norm(moe_cuda.moe_experts(s[0], w13, w2, wts, idx, 0, True), s[2], w, 1e-6) for s in sets])
        b = 3.0 * E * I * W * 2
        add(f"mixture to the next sublayer's input, {T} tokens", o, k, b + T * W * 12.0, b + T * W * 8.0, 6.0 * T * top * I * W)
    return R.rows


@torch.inference_mode()
def govuvik_kernels() -> List[Dict]:
    R = Rows()
    add, alone = R.add, R.add_alone
    W, heads, G, d, window = 2048, 32, 4, 128, 4096
    # ---- attention with mixed scores and sinks, beside attention with the same window
    sinks = torch.zeros(heads, device=DEV)
    for kind, seqs, q_len, kv in STEPS:
        inp = step_input(seqs, q_len, kv, 16, 1000)
        nb, T, row = seqs * (-(-kv // 16)) + 1, seqs * q_len, (heads + 2 * G) * d
        cache_bytes = 2.0 * seqs * (kv if kind == "prefill" else min(kv, window)) * G * d * 2
        sets = _rotated(lambda: (_bf(T, heads * G * d, std=0.1), _bf(nb, 16, G, d), _bf(nb, 16, G, d), _bf(T, row)), cache_bytes + T * row * 2)[:8]
        o = time_graph([lambda s=s: c.paged_attention_ext(s[0].view(T, heads, G * d), s[1].view(nb, 16, 1, G * d), s[2], inp, d ** -0.5, window,
                                                          sinks=sinks) for s in sets])
        k = time_graph([lambda s=s: c.paged_attention(s[3][:, :heads * d].unflatten(1, (heads, d)), s[1], s[2], inp, d ** -0.5, window) for s in sets])
        pairs = sum(min(p + 1, window) for p in range(kv - q_len, kv)) * seqs
        fk = 4.0 * heads * d * pairs
        io = T * heads * d * 2.0
        # ours: scores, their mix, sums of the values; q enters with the columns of every key head
        add(f"attention {kind} {seqs} x {q_len} of {kv}, window {window}, {heads}/{G} heads", o, k, cache_bytes + io * (1 + G), cache_bytes + 2 * io,
            fk + 2.0 * heads * heads * pairs if kind == "prefill" else 0.0, fk if kind == "prefill" else 0.0)
        del sets
    # ---- norms, cache write, convolutions
    cs, t64 = torch.randn(8192, 128, device=DEV), torch.randn(8192, 64, device=DEV)
    mix, w, w128 = torch.eye(heads, device=DEV) + 0.1, _bf(W), _bf(128)
    qw, kw, emb = _bf(heads * d), _bf(G * d), _bf(30000, W)
    for T in (8192, 256):
        inp, row = step_input(1, T, T, 16, 1000), (heads + 2 * G) * d
        new = step_input(T, 1, 1152, 16, 1000) if T == 256 else step_input(1, T, T, 16, 1000)
        sets = _rotated(lambda: (_bf(T, row), _bf(T // 16 + 1, 16, G, d), _bf(T // 16 + 1, 16, G, d)), T * row * 2.0)[:24]
        rot = (t64, inp.positions, False)
        o = time_graph([lambda s=s: c.qknorm_all_kvwrite(s[0], inp.slots, qw, kw, 1e-6, s[1], s[2], heads, G, rot, mix) for s in sets])
        k = time_graph([lambda s=s: c.rope_qknorm_kvwrite(s[0], inp.positions, inp.slots, cs, w128, w128, 1e-6, s[1], s[2], heads, G, d) for s in sets])
        add(f"q / k norm + rotation + score mix + cache write, {T} tokens", o, k, T * (heads * (1.0 + G) + 4 * G) * d * 2 + T * 256.0,
            T * (2.0 * heads + 4 * G) * d * 2 + T * 512.0, fma=1.0 * T * heads * heads * d)
        slots = T if T == 256 else 1
        for what, C in (("input", W), ("q, k, v", row)):
            sets = _rotated(lambda: (_bf(T, C), _bf(4, C), _bf(C), _bf(slots + 1, 3, C)), T * C * 4.0)[:16]
            o = time_graph([lambda s=s: c.causal_conv(s[0], s[1], None, s[3], new, "none", C == W) for s in sets])
            k = time_graph([lambda s=s: c.causal_conv(s[0], s[1], s[2], s[3], new, "silu") for s in sets])
            b = T * C * 4.0 + (2 * T * 3 * C * 2.0 if T == 256 else 0)
            add(f"convolution on {what}, {T} x {C}", o, k, b, b)
        sets = _rotated(lambda: (_bf(T, W), torch.randn(T, W, device=DEV), _bf(T, W)), T * W * 10.0)
        o = time_graph([lambda s=s: c.branches_post_norm_add_norm(s[0], s[2], w, w, 0.5, s[1], w, w, 1e-6) for s in sets])
        k = time_graph([lambda s=s: c.post_norm_add_norm(s[0], s[1], w, w, 1e-6) for s in sets])
        add(f"two branch norms + norm + residual + norm, {T} x {W}", o, k, T * W * 14.0, T * W * 12.0)
        ids = torch.randint(0, 30000, (T,), device=DEV).int()
        o = time_graph([lambda: c.embed_rms_norm(ids, emb, 1.0, w, 1e-6, w_rows=w)] * 8)
        k = time_graph([lambda: c.rms_norm(c.embedding(ids, emb), w, 1e-6)] * 8)
        add(f"embedding + its norm + first norm, {T} x {W}", o, k, T * W * 8.0, T * W * 8.0)
    # ---- matrix states beside time mixing, per element of the state the same work
    for kind, seqs, q_len, kv in STEPS[:3]:
        T = seqs * q_len
        inp = step_input(seqs, q_len, kv, 16, 1000)
        passes = 1 if kv == q_len else 2
        n, hd = 4096, 64
        u, w0, nw = torch.randn(n // hd, hd, device=DEV), torch.randn(n, device=DEV) - 3, _bf(n)
        sets = [(_bf(T, n), _bf(T, n), _bf(T, n), torch.randn(T, n, device=DEV), _bf(T, n), torch.empty(T, n, device=DEV, dtype=torch.bfloat16),
                 torch.zeros(seqs + 1, n // hd, hd, hd, device=DEV)) for _ in range(3)]
        k = time_graph([lambda s=s: c.time_mix(s[0], s[1], s[2], s[3], w0, u, s[4], nw, 0.5, 1e-6, s[6], inp, s[5]) for s in sets])
        kb, kf = T * n * 14.0 + passes * seqs * n * hd * 4.0, 3.0 * T * n * hd
        del sets
        H, dk, dv = 16, 64, 128
        row = H * (2 * dk + 2 * dv)
        cut = lambda x: (x[:, :H * dk], x[:, H * dk:2 * H * dk], x[:, 2 * H * dk:2 * H * dk + H * dv])
        bias, nw = torch.randn(H * dk, device=DEV) + 2, _bf(dv)
        sets = [(_bf(T, row), torch.randn(T, H * dk, device=DEV), torch.zeros(seqs + 1, H, dk, dv, device=DEV)) for _ in range(4)]
        o = time_graph([lambda s=s: c.gated_memory(*cut(s[0]), s[1], bias, 1 / 16, s[0][:, -H * dv:], nw, 1e-6, s[2], inp) for s in sets])
        add(f"gated linear attention, {kind} {seqs} x {q_len}, {H} heads of {dk} x {dv}", o, k,
            T * (row * 2.0 + H * dk * 4 + H * dv * 2) + passes * seqs * H * dk * dv * 4.0, kb, fma=3.0 * T * H * dk * dv, fma_like=kf)
        del sets
        H = 32
        row = H * (2 * dk + 2 * dv)
        bias, nw = torch.randn(2 * H, device=DEV) + 2, _bf(H * dv)
        sets = [(_bf(T, row), torch.randn(T, 2 * H, device=DEV), torch.zeros(seqs + 1, H, dk * dv + dk, device=DEV), torch.zeros(seqs + 1, H, device=DEV))
                for _ in range(4)]
        o = time_graph([lambda s=s: c.matrix_memory(*cut(s[0]), s[1], bias, 15.0, s[0][:, -H * dv:], nw, 1e-6, s[2], s[3], inp) for s in sets])
        add(f"matrix memory, {kind} {seqs} x {q_len}, {H} heads of {dk} x {dv}", o, k,
            T * (row * 2.0 + H * 8 + H * dv * 2) + passes * seqs * H * dk * dv * 4.0, kb, fma=3.0 * T * H * dk * dv, fma_like=kf)
        del sets
    # ---- router and mixture: experts without gates, of as many weights
    E, top, ff, I = 128, 8, 1152, 768
    wr = _bf(E, W, std=0.02)
    up, down = _bf(E, ff, W, std=0.02), _bf(E, W, ff, std=0.02)
    w13, w2 = _bf(E, 2 * I, W, std=0.02), _bf(E, W, I, std=0.02)
    moe_cuda.interleave_w13(w13)
    for T in (8192, 256):
        sets = _rotated(lambda: (_bf(T, W), torch.randn(T, W, device=DEV), _bf(T, W)), T * W * 10.0)[:16]
        o = time_graph([lambda s=s: c.moe_router(c.linear_f32(s[0], wr), top, "softmax_chosen") for s in sets])
        k = time_graph([lambda s=s: c.moe_router(c.linear(s[0], wr), top, "softmax", True) for s in sets])
        b = T * W * 2.0 + E * W * 2.0 + T * 64.0
        add(f"router product + choice, {T} x {E}", o, k, b, b, 2.0 * T * E * W)
        wts, idx = c.moe_router(c.linear(sets[0][0], wr), top, "softmax", True)

        def ours_mix(s):
            y, dst = moe_cuda.expert_rows(s[0], up, down, idx, "relu2")
            return moe_cuda.combine_post_norm_add_norm(y, dst, idx, wts, s[0], None, E, s[1], w, w, 1e-6)
        o = time_graph([lambda s=s: ours_mix(s) for s in sets])
        k = time_graph([lambda s=s: c.add_rms_norm(moe_cuda.moe_experts(s[0], w13, w2, wts, idx, 0, True), s[2], w, 1e-6) for s in sets])
        b = 3.0 * E * I * W * 2
        add(f"mixture to the next sublayer's input, {T} tokens", o, k, b + T * W * 12.0, b + T * W * 8.0, 6.0 * T * top * I * W)
    # ---- small products
    h, a1 = _bf(8192, W), _bf(8192, 16)
    gw, a2 = _bf(64, W, std=0.02), _bf(1024, 16)
    alone("gates of the matrix memory, 8192 x 64 x 2048", time_graph([lambda: c.linear_f32(h, gw)] * 4), 8192 * (W * 2.0 + 256))
    alone("decay's second factor, 8192 x 1024 x 16", time_graph([lambda: c.linear_f32(a1, a2)] * 4), 8192 * (32.0 + 4096))
    return R.rows


KERNELS = {"movolorn": movolorn_kernels, "falalix": falalix_kernels, "babadra": babadra_kernels, "govuvik": govuvik_kernels}


def run(design: str, layers: int = 4, block: int = 16) -> Dict:
    out = {"design": design, "layers": layers, "block_size": block, "peaks": peaks(), "models": []}
    seen: Dict[str, List[Dict]] = {}
    for ours, like, kind in PAIRS[design]:
        if like not in seen:
            seen[like] = layer_throughput(like, layers, block)
        a, b = layer_throughput(ours, layers, block, kind), seen[like]
        out["models"].append({"model": ours + (f" ({kind} layers)" if kind else ""), "closest": like,
                              "steps": [dict(x, closest_us_per_layer=y["us_per_layer"], ratio=round(y["us_per_layer"] / x["us_per_layer"], 3))
                                        for x, y in zip(a, b)]})
    out["kernels"] = KERNELS[design]()
    out["device_status"] = c.read_status()
    return out
