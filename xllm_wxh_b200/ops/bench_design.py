"""A model design beside the framework's closest other one at equal layer sizes (`bench.py --compare-design movolorn`):
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
from ..models.args import ModelArgs, preset
from ..models.layer_spec import AttentionSpec
from ..models.registry import get_model_class
from . import cuda_ops as c
from . import moe_cuda
from .bench_kernels import time_graph

DEV = "cuda:0"
PAIRS = {"movolorn": [("movolorn-8b", "qwen3-8b"), ("movolorn-30b-a3b", "qwen3-30b-a3b")]}
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
    host[L.block_tables:L.block_tables + seqs * nb] = bt.reshape(-1)
    hdr = np.zeros(32, dtype=np.int32)
    dec = q_len == 1
    hdr[0], hdr[1], hdr[3], hdr[4], hdr[5], hdr[6] = T, seqs, seqs if dec else 0, 0 if dec else seqs, q_len, kv_len
    hdr[7], hdr[17], hdr[21] = 2 if dec else 0, block, 0 if dec else T
    host[L.header:L.header + 32] = torch.from_numpy(hdr)
    return StepInput(host.to(DEV), L, hdr)


def cut_to_layers(a: ModelArgs, n: int) -> ModelArgs:
    kw = dict(n_layers=n)
    if a.layer_specs:
        kw.update(layer_specs=a.layer_specs[:n], layer_runs=a.layer_runs[:n])
    return dataclasses.replace(a, **kw)


@torch.inference_mode()
def layer_throughput(name: str, layers: int, block: int) -> List[Dict]:
    args = cut_to_layers(preset(name), layers)
    model = get_model_class(args.model_type)(args, device=DEV, dtype=torch.bfloat16).init_random(0).finalize_weights()
    rows = []
    for kind, seqs, q_len, kv_len in STEPS:
        inp = step_input(seqs, q_len, kv_len, block, args.vocab_size)
        blocks = seqs * (-(-kv_len // block)) + 1
        kv = [tuple(torch.randn(s, device=DEV, dtype=torch.bfloat16) for s in pair) for pair in model.kv_cache_shapes(blocks, block)]
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


@torch.inference_mode()
def kernel_pairs() -> List[Dict]:
    """Each kernel of the design beside the like one: microseconds, bytes or FLOPs of each, and the fraction of the roofline."""
    pk = peaks()
    rows = []

    def add(what, ours, like, bytes_ours=0.0, bytes_like=0.0, flops=0.0):
        def frac(us, nbytes):
            bound = max(nbytes / (pk["hbm_gbs"] * 1e3), flops / (pk["bf16_tflops"] * 1e6))
            return bound / us
        fo, fl = frac(ours, bytes_ours), frac(like, bytes_like)
        rows.append({"what": what, "us": round(ours, 1), "like_us": round(like, 1), "roofline": round(fo, 3), "like_roofline": round(fl, 3),
                     "farther_by": round(fl / fo, 2)})
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


def run(design: str, layers: int = 4, block: int = 16) -> Dict:
    out = {"design": design, "layers": layers, "block_size": block, "peaks": peaks(), "models": []}
    for ours, like in PAIRS[design]:
        a, b = layer_throughput(ours, layers, block), layer_throughput(like, layers, block)
        out["models"].append({"model": ours, "closest": like,
                              "steps": [dict(x, closest_us_per_layer=y["us_per_layer"], ratio=round(y["us_per_layer"] / x["us_per_layer"], 3))
                                        for x, y in zip(a, b)]})
    out["kernels"] = kernel_pairs()
    out["device_status"] = c.read_status()
    return out
