"""Movolorn: a decoder-only model whose configuration lists its layers one by one.

Every sublayer is normed before and after (x += norm_b(f(norm_a(x))), fp32 residual).  Attention has per-head q / k norms,
no rotation, a per-head linear distance bias, chunks of positions and a sink in the softmax denominator; the feed-forward
is a tanh-gelu-gated MLP or a mixture with identity experts, groups of experts and a shared expert.  A range of layers may
run several times with the same weights; every run has a KV cache of its own, so the caches (and everything that follows
them: paging, prefix cache, host tier, hand-off) are counted in layer runs.

The mechanisms live in `ops` and take their constants as parameters; this file only loads weights and strings the ops
together.  Between two sublayers there is one kernel (post norm + residual + next norm); a mixture's combine is part of it.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..parallel.comm import Comm
from .args import ModelArgs
from .layer_spec import FeedForwardSpec, LayerSpec
from .qwen import _DT, WeightInit
from .registry import register_model


class MixerWeights:
    def __init__(self):
        self.qkv_w = self.o_w = self.q_norm = self.k_norm = None
        self.slopes = self.sinks = None         # fp32 [heads], or None


class FeedForwardWeights:
    def __init__(self):
        self.gate_up_w = self.down_w = None     # dense, or the shared expert of a mixture: [2 ff, H], [H, ff]
        self.router_w = self.correction = None  # mixture: [outputs, H], fp32 [outputs]
        self.w13 = self.w2 = None               # mixture: [experts, 2 ff, H], [experts, H, ff]
        self.interleaved = self.w13_interleaved = False


class BlockWeights:
    def __init__(self, spec: LayerSpec):
        self.norm1 = self.norm1b = self.norm2 = self.norm2b = None
        self.mix = MixerWeights()
        self.mlp = FeedForwardWeights() if spec.mlp is not None else None


@register_model("movolorn")
class MovolornForCausalLM:
    def __init__(self, args: ModelArgs, comm: Optional[Comm] = None, device="cpu", dtype: Optional[torch.dtype] = None):
        self.args = args
        self.comm = comm or Comm()
        if self.comm.tp_size > 1 or self.comm.ep_size > 1 or self.comm.dp_size > 1:
            raise ValueError("movolorn runs on one device: tensor, expert and data parallelism are not implemented for it")
        self.device = torch.device(device)
        self.dtype = dtype or _DT[args.dtype]
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"movolorn runs in bfloat16 or float32, not {self.dtype}")
        self.layers: List[BlockWeights] = [BlockWeights(s) for s in args.layer_specs]
        self.embed = self.final_norm = self.lm_head = None
        self.layer_hook = None       # callable(run index), right after a run's attention (its KV is written by then)
        self.residual_hook = None    # callable(run index, fp32 residual), after a run's last sublayer (tests, tools)

    # ------------------------------------------------------------------ weights
    def kv_cache_shapes(self, num_blocks: int, block_size: int):
        out = []
        for li in self.args.layer_runs:
            m = self.args.layer_specs[li].mixer
            out.append(((num_blocks, block_size, m.kv_heads, m.dim), (num_blocks, block_size, m.kv_heads, m.vdim)))
        return out

    @staticmethod
    def tensor_shapes(a: ModelArgs) -> Dict[str, tuple]:
        """Checkpoint tensor names and shapes of a configuration."""
        H = a.hidden_size
        out = {"embed": (a.vocab_size, H), "final.norm": (H,), "head": (a.vocab_size, H)}
        for i, s in enumerate(a.layer_specs):
            p, m, f = f"l{i}.", s.mixer, s.mlp
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f is not None else ()):
                out[p + n] = (H,)
            out[p + "mix.q"], out[p + "mix.k"] = (m.heads * m.dim, H), (m.kv_heads * m.dim, H)
            out[p + "mix.v"], out[p + "mix.o"] = (m.kv_heads * m.vdim, H), (H, m.heads * m.vdim)
            if m.qk_norm:
                out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (m.dim,)
            if f is None:
                continue
            parts = {}
            if not f.is_moe:
                parts[""] = f.ff
            else:
                n = f.experts + f.identity_experts
                out[p + "mlp.router"], out[p + "mlp.correction"] = (n, H), (n,)
                parts.update({f"e{e}.": f.ff for e in range(f.experts)})
                if f.shared_ff:
                    parts["shared."] = f.shared_ff
            for q, ff in parts.items():
                out[p + f"mlp.{q}gate"], out[p + f"mlp.{q}up"], out[p + f"mlp.{q}down"] = (ff, H), (ff, H), (H, ff)
        return out

    def _fill(self, get) -> "MovolornForCausalLM":
        """Build the weights from `get(name)` (checkpoint names, any dtype, any device)."""
        dev = lambda n: get(n).to(self.device, self.dtype).contiguous()

        def cat(*names):
            return torch.cat([dev(n) for n in names], 0)
        self.embed, self.final_norm, self.lm_head = dev("embed"), dev("final.norm"), dev("head")
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, f = f"l{i}.", s.mlp
            L.norm1, L.norm1b = dev(p + "norm1"), dev(p + "norm1b")
            L.mix.qkv_w, L.mix.o_w = cat(p + "mix.q", p + "mix.k", p + "mix.v"), dev(p + "mix.o")
            m = s.mixer
            if m.qk_norm:
                L.mix.q_norm, L.mix.k_norm = dev(p + "mix.q.norm"), dev(p + "mix.k.norm")
            if m.distance_bias:
                L.mix.slopes = torch.tensor(m.head_slopes(), dtype=torch.float32, device=self.device)
            if m.sink is not None:
                L.mix.sinks = torch.full((m.heads,), m.sink, dtype=torch.float32, device=self.device)
            if f is None:
                continue
            L.norm2, L.norm2b = dev(p + "norm2"), dev(p + "norm2b")
            p += "mlp."
            W = L.mlp
            W.interleaved = W.w13_interleaved = False
            if not f.is_moe:
                W.gate_up_w, W.down_w = cat(p + "gate", p + "up"), dev(p + "down")
                continue
            W.router_w = dev(p + "router")
            W.correction = get(p + "correction").to(self.device, torch.float32).contiguous()
            H = self.args.hidden_size
            W.w13 = torch.empty((f.experts, 2 * f.ff, H), dtype=self.dtype, device=self.device)
            W.w2 = torch.empty((f.experts, H, f.ff), dtype=self.dtype, device=self.device)
            for e in range(f.experts):
                W.w13[e, :f.ff].copy_(get(p + f"e{e}.gate"))
                W.w13[e, f.ff:].copy_(get(p + f"e{e}.up"))
                W.w2[e].copy_(get(p + f"e{e}.down"))
            if f.shared_ff:
                W.gate_up_w, W.down_w = cat(p + "shared.gate", p + "shared.up"), dev(p + "shared.down")
        return self

    def load_weights(self, ckpt) -> "MovolornForCausalLM":
        want = self.tensor_shapes(self.args)
        for n, shape in want.items():
            if not ckpt.has(n):
                raise ValueError(f"the checkpoint has no tensor '{n}'")
            if tuple(ckpt.get(n).shape) != shape:
                raise ValueError(f"tensor '{n}' has shape {tuple(ckpt.get(n).shape)}, the configuration asks for {shape}")
        return self._fill(ckpt.get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "MovolornForCausalLM":
        wi = WeightInit(seed, std, self.dtype, self.device)
        shapes = self.tensor_shapes(self.args)

        def get(name):
            if name.endswith((".norm", ".norm1", ".norm1b", ".norm2", ".norm2b")):
                return wi.ones(shapes[name])
            if name.endswith(".correction"):
                return torch.zeros(shapes[name], dtype=torch.float32, device=self.device)
            return wi.normal(name, shapes[name])
        return self._fill(get)

    def finalize_weights(self) -> "MovolornForCausalLM":
        """On CUDA in bf16 the gate / up rows are interleaved in groups of 16, so that the GEMM epilogue applies the gate."""
        if self.device.type != "cuda" or self.dtype != torch.bfloat16 or self.args.hidden_size % 8:
            return self
        from ..ops import cuda_ops, moe_cuda
        for L in self.layers:
            W = L.mlp
            if W is None:
                continue
            if W.gate_up_w is not None and not W.interleaved and W.down_w.shape[1] % 16 == 0:
                W.gate_up_w = cuda_ops.interleave_gate_up(W.gate_up_w)
                W.interleaved = True
            if W.w13 is not None and not W.w13_interleaved and W.w13.shape[0] > 0 and W.w2.shape[2] % 16 == 0:
                moe_cuda.interleave_w13(W.w13)
                W.w13_interleaved = True
        return self

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """Tensors under their checkpoint names (before `finalize_weights`)."""
        sd = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head}
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, f = f"l{i}.", s.mixer, s.mlp
            sd[p + "norm1"], sd[p + "norm1b"] = L.norm1, L.norm1b
            sd[p + "mix.q"], sd[p + "mix.k"], sd[p + "mix.v"] = L.mix.qkv_w.split([m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim])
            sd[p + "mix.o"] = L.mix.o_w
            if m.qk_norm:
                sd[p + "mix.q.norm"], sd[p + "mix.k.norm"] = L.mix.q_norm, L.mix.k_norm
            if f is None:
                continue
            W = L.mlp
            assert not (W.interleaved or W.w13_interleaved), "state_dict() must be taken before finalize_weights()"
            sd[p + "norm2"], sd[p + "norm2b"] = L.norm2, L.norm2b
            p += "mlp."
            if f.is_moe:
                sd[p + "router"], sd[p + "correction"] = W.router_w, W.correction
                for e in range(f.experts):
                    sd[p + f"e{e}.gate"], sd[p + f"e{e}.up"], sd[p + f"e{e}.down"] = W.w13[e, :f.ff], W.w13[e, f.ff:], W.w2[e]
            q = p + ("shared." if f.is_moe else "")
            if W.gate_up_w is not None:
                (sd[q + "gate"], sd[q + "up"]), sd[q + "down"] = W.gate_up_w.chunk(2), W.down_w
        return {k: v.contiguous() for k, v in sd.items()}

    # ------------------------------------------------------------------ forward
    def _feed_forward(self, L: BlockWeights, f: FeedForwardSpec, h: torch.Tensor, x: torch.Tensor, w_next: torch.Tensor) -> torch.Tensor:
        """The second sublayer from its normed input h; adds to x and returns the next sublayer's input."""
        W, eps = L.mlp, self.args.rms_norm_eps
        if not f.is_moe:
            y = ops.linear(ops.gated_linear(h, W.gate_up_w, f.act, W.interleaved), W.down_w)
            return ops.post_norm_add_norm(y, x, L.norm2b, w_next, eps)
        weights, ids = ops.moe_router(ops.linear_f32(h, W.router_w), f.top_k, f.scoring, f.renormalize, W.correction, f.n_group,
                                      f.topk_group, 1.0, f.group_score)
        shared = None
        if W.gate_up_w is not None:
            shared = ops.linear(ops.gated_linear(h, W.gate_up_w, f.act, W.interleaved), W.down_w)
        return ops.moe_post_norm_add_norm(h, W.w13, W.w2, weights, ids, shared, f.experts, x, L.norm2b, w_next, eps, f.act,
                                          W.w13_interleaved)

    def forward(self, inp, kv_caches) -> torch.Tensor:
        """Returns the final-normed hidden states [T, H]."""
        a, eps, runs = self.args, self.args.rms_norm_eps, self.args.layer_runs
        x, h = ops.embed_rms_norm(inp.tokens, self.embed, a.embedding_scale, self.layers[runs[0]].norm1, eps)
        for r, li in enumerate(runs):
            L, s = self.layers[li], a.layer_specs[li]
            m = s.mixer
            w_next = self.layers[runs[r + 1]].norm1 if r + 1 < len(runs) else self.final_norm
            k_cache, v_cache = kv_caches[r]
            qkv = ops.linear(h, L.mix.qkv_w)
            q = ops.qknorm_kvwrite(qkv, inp.slots, L.mix.q_norm, L.mix.k_norm, eps, k_cache, v_cache, m.heads, m.kv_heads)
            o = ops.paged_attention_ext(q.view(-1, m.heads, m.dim), k_cache, v_cache, inp, m.scale, m.window, m.chunk, L.mix.slopes,
                                        L.mix.sinks)
            if self.layer_hook is not None:
                self.layer_hook(r)
            y = ops.linear(o, L.mix.o_w)
            if s.mlp is None:
                h = ops.post_norm_add_norm(y, x, L.norm1b, w_next, eps)
            else:
                h = ops.post_norm_add_norm(y, x, L.norm1b, L.norm2, eps)
                h = self._feed_forward(L, s.mlp, h, x, w_next)
            if self.residual_hook is not None:
                self.residual_hook(r, x)
        return h

    def logits(self, hidden: torch.Tensor, sample_idx: torch.Tensor, gather: bool = True) -> torch.Tensor:
        sel = hidden.index_select(0, sample_idx.long()) if sample_idx is not None else hidden
        return ops.linear(sel, self.lm_head)

    def pooled_embedding(self, hidden: torch.Tensor, sample_idx: torch.Tensor) -> torch.Tensor:
        """Last-token pooling + L2 normalisation (embedding task)."""
        return torch.nn.functional.normalize(hidden.index_select(0, sample_idx.long()).float(), dim=-1)

    def weight_bytes(self) -> int:
        from ..runtime.sleep import iter_weight_slots
        seen = {}
        for get, _ in iter_weight_slots(self):
            t = get()
            seen[t.data_ptr()] = t.numel() * t.element_size()
        return sum(seen.values())
