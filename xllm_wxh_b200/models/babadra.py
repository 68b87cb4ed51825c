"""Babadra: a decoder-only model whose configuration lists its layers one by one, with two kinds of attention.

Latent attention caches one normed latent per token and one rotated key part that all heads share (YaRN-scaled interleaved
rotation), and runs in absorbed form.  Differential attention takes the difference of two attention maps over the same values
(normed and rotated queries and keys, scores bounded by a tanh).  The feed-forward is a clamped gated one, dense or a mixture whose
weights are the softmax over the chosen experts' logits.  Sublayers are normed before only (weights stored around zero) and enter
an fp32 residual through a vector each; a learned position vector joins the embedding; logits are bounded by a tanh.  A range of
layers may run several times with the same weights: the embedding is added again ahead of every pass but the first, and every run
has a cache of its own.

The mechanisms live in `ops` and take their constants as parameters; this file only loads weights and strings the ops together.
Between two sublayers there is one kernel: layer scale, residual, the embedding at the head of a pass and the next norm; a
mixture's combine is part of it.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..parallel.comm import Comm
from .args import ModelArgs
from .layer_spec import AttentionSpec, FeedForwardSpec, LatentAttentionSpec, RotarySpec
from .qwen import _DT, WeightInit
from .registry import register_model

AROUND_ZERO = 1.0           # what norm1, norm2 and the final norm add to their stored weights


class LatentWeights:
    def __init__(self):
        self.down_w = None                      # rows: query latent, key/value latent, rotated key part
        self.q_norm = self.kv_norm = None
        self.uq_w = None
        self.uk_w = self.uv_w = None            # [heads, kv_rank, dim], [heads, vdim, kv_rank]
        self.o_w = None


class TwoMapWeights:
    def __init__(self):
        self.qkv_w = self.q_norm = self.k_norm = None
        self.lam = None                         # fp32 [4, dim]: lq1, lk1, lq2, lk2
        self.factor = None                      # fp32 [1], of the second map
        self.bound = 0.0                        # of |q . k|, from the norms' weights
        self.o_w = None


class FeedForwardWeights:
    def __init__(self):
        self.gate_up_w = self.down_w = None     # dense: [2 ff, H], [H, ff]
        self.router_w = self.router_b = None    # mixture: [experts, H], fp32 [experts]
        self.w13 = self.w2 = None               # mixture: [experts, 2 ff, H], [experts, H, ff]
        self.interleaved = False


class BlockWeights:
    def __init__(self, spec):
        self.norm1 = self.norm2 = self.ls1 = self.ls2 = None
        self.mix = LatentWeights() if isinstance(spec.mixer, LatentAttentionSpec) else TwoMapWeights()
        self.mlp = FeedForwardWeights() if spec.mlp is not None else None


@register_model("babadra")
class BabadraForCausalLM:
    def __init__(self, args: ModelArgs, comm: Optional[Comm] = None, device="cpu", dtype: Optional[torch.dtype] = None):
        self.args = args
        self.comm = comm or Comm()
        if self.comm.tp_size > 1 or self.comm.ep_size > 1 or self.comm.dp_size > 1:
            raise ValueError("babadra runs on one device: tensor, expert and data parallelism are not implemented for it")
        self.device = torch.device(device)
        self.dtype = dtype or _DT[args.dtype]
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"babadra runs in bfloat16 or float32, not {self.dtype}")
        self.layers: List[BlockWeights] = [BlockWeights(s) for s in args.layer_specs]
        self.embed = self.positions = self.final_norm = self.lm_head = None
        # rotation tables, one per distinct rotation; they are no weights and stay through sleep
        self.cos_sin: Dict[RotarySpec, torch.Tensor] = {}
        for s in args.layer_specs:
            if s.mixer.rot is not None and s.mixer.rot not in self.cos_sin:
                self.cos_sin[s.mixer.rot] = ops.ref.rotary_table(s.mixer.rot, args.max_position_embeddings, self.device)
        self.layer_hook = None       # callable(run index), right after a run's mixer (its cache is written by then)
        self.residual_hook = None    # callable(run index, fp32 residual), after a run's last sublayer (tests, tools)

    # ------------------------------------------------------------------ cache
    def kv_cache_shapes(self, num_blocks: int, block_size: int):
        """Per layer run: latents with the shared key part, or the keys of both maps and the values."""
        out, at = [], (num_blocks, block_size)
        for li in self.args.layer_runs:
            m = self.args.layer_specs[li].mixer
            out.append((at + (m.row,),) if isinstance(m, LatentAttentionSpec) else
                       (at + (m.kv_heads * m.maps, m.dim), at + (m.kv_heads, m.vdim)))
        return out

    # ------------------------------------------------------------------ weights
    @staticmethod
    def tensor_shapes(a: ModelArgs) -> Dict[str, tuple]:
        """Checkpoint tensor names and shapes of a configuration."""
        H = a.hidden_size
        out = {"embed": (a.vocab_size, H), "pos": (a.position_rows, H), "final.norm": (H,), "head": (a.vocab_size, H)}
        for i, s in enumerate(a.layer_specs):
            p, m, f = f"l{i}.", s.mixer, s.mlp
            out[p + "norm1"] = out[p + "ls1"] = (H,)
            if isinstance(m, LatentAttentionSpec):
                out.update({p + "mix.dq": (m.q_rank, H), p + "mix.dq.norm": (m.q_rank,), p + "mix.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                            p + "mix.dkv": (m.row, H), p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                            p + "mix.uv": (m.heads * m.vdim, m.kv_rank)})
            else:
                out.update({p + "mix.q": (m.heads * m.maps * m.dim, H), p + "mix.k": (m.kv_heads * m.maps * m.dim, H),
                            p + "mix.v": (m.kv_heads * m.vdim, H)})
                out.update({p + "mix." + n: (m.dim,) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
            out[p + "mix.o"] = (H, m.heads * m.vdim)
            if f is None:
                continue
            out[p + "norm2"] = out[p + "ls2"] = (H,)
            if f.is_moe:
                out[p + "mlp.router"], out[p + "mlp.router.b"] = (f.experts, H), (f.experts,)
            for q in [f"e{e}." for e in range(f.experts)] or [""]:
                out[p + f"mlp.{q}gate"], out[p + f"mlp.{q}up"], out[p + f"mlp.{q}down"] = (f.ff, H), (f.ff, H), (H, f.ff)
        return out

    def _fill(self, get) -> "BabadraForCausalLM":
        """Build the weights from `get(name)` (checkpoint names, any dtype, any device)."""
        dev = lambda n: get(n).to(self.device, self.dtype).contiguous()
        f32 = lambda n: get(n).to(self.device, torch.float32).contiguous()
        H = self.args.hidden_size
        self.embed, self.positions, self.final_norm, self.lm_head = dev("embed"), dev("pos"), dev("final.norm"), dev("head")
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, f, W = f"l{i}.", s.mixer, s.mlp, L.mix
            L.norm1, L.ls1 = dev(p + "norm1"), dev(p + "ls1")
            q = p + "mix."
            if isinstance(m, LatentAttentionSpec):
                W.down_w = torch.cat([dev(q + "dq"), dev(q + "dkv")], 0)
                W.q_norm, W.kv_norm, W.uq_w = dev(q + "dq.norm"), dev(q + "dkv.norm"), dev(q + "uq")
                W.uk_w = dev(q + "uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2).contiguous()
                W.uv_w = dev(q + "uv").view(m.heads, m.vdim, m.kv_rank)
            else:
                W.qkv_w = torch.cat([dev(q + n) for n in "qkv"], 0)
                W.q_norm, W.k_norm = dev(q + "q.norm"), dev(q + "k.norm")
                turn = m.rot.frequencies()[1] if m.rot is not None else 1.0
                # a normed row is no longer than sqrt(dim); 2 % for the rounding of q and k
                W.bound = 1.02 * m.dim * float(W.q_norm.abs().max()) * float(W.k_norm.abs().max()) * max(1.0, turn * turn)
                W.lam = torch.stack([f32(q + n) for n in ("lq1", "lk1", "lq2", "lk2")])
                W.factor = (torch.exp((W.lam[0] * W.lam[1]).sum()) - torch.exp((W.lam[2] * W.lam[3]).sum()) + m.diff).reshape(1)
            W.o_w = dev(q + "o")
            if f is None:
                continue
            L.norm2, L.ls2 = dev(p + "norm2"), dev(p + "ls2")
            p, W = p + "mlp.", L.mlp
            W.interleaved = False
            if not f.is_moe:
                W.gate_up_w, W.down_w = torch.cat([dev(p + "gate"), dev(p + "up")], 0), dev(p + "down")
                continue
            W.router_w, W.router_b = dev(p + "router"), f32(p + "router.b")
            W.w13 = torch.empty((f.experts, 2 * f.ff, H), dtype=self.dtype, device=self.device)
            W.w2 = torch.empty((f.experts, H, f.ff), dtype=self.dtype, device=self.device)
            for e in range(f.experts):
                W.w13[e, :f.ff].copy_(get(p + f"e{e}.gate"))
                W.w13[e, f.ff:].copy_(get(p + f"e{e}.up"))
                W.w2[e].copy_(get(p + f"e{e}.down"))
        return self

    def load_weights(self, ckpt) -> "BabadraForCausalLM":
        for n, shape in self.tensor_shapes(self.args).items():
            if not ckpt.has(n):
                raise ValueError(f"the checkpoint has no tensor '{n}'")
            if tuple(ckpt.get(n).shape) != shape:
                raise ValueError(f"tensor '{n}' has shape {tuple(ckpt.get(n).shape)}, the configuration asks for {shape}")
        return self._fill(ckpt.get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "BabadraForCausalLM":
        wi = WeightInit(seed, std, self.dtype, self.device)
        shapes = self.tensor_shapes(self.args)

        def get(name):
            last = name.rsplit(".", 1)[-1]
            if name.endswith(("q.norm", "k.norm", "dq.norm", "dkv.norm")):
                return wi.ones(shapes[name])
            if last in ("norm", "norm1", "norm2") or name.endswith("router.b"):
                return torch.zeros(shapes[name], dtype=torch.float32, device=self.device)
            if last in ("ls1", "ls2"):
                return wi.ones(shapes[name]) * 0.5
            return wi.normal(name, shapes[name])
        return self._fill(get)

    def finalize_weights(self) -> "BabadraForCausalLM":
        """On CUDA in bf16 the gate / up rows are interleaved in groups of 16, so that the GEMM epilogue applies the gate."""
        if self.device.type != "cuda" or self.dtype != torch.bfloat16 or self.args.hidden_size % 8:
            return self
        from ..ops import cuda_ops, moe_cuda
        for L in self.layers:
            W = L.mlp
            if W is None or W.interleaved:
                continue
            if W.w13 is not None and W.w2.shape[2] % 16 == 0:
                moe_cuda.interleave_w13(W.w13)
                W.interleaved = True
            elif W.gate_up_w is not None and W.down_w.shape[1] % 16 == 0:
                W.gate_up_w = cuda_ops.interleave_gate_up(W.gate_up_w)
                W.interleaved = True
        return self

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """Tensors under their checkpoint names (before `finalize_weights`)."""
        sd = {"embed": self.embed, "pos": self.positions, "final.norm": self.final_norm, "head": self.lm_head}
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, f, W = f"l{i}.", s.mixer, s.mlp, L.mix
            sd[p + "norm1"], sd[p + "ls1"] = L.norm1, L.ls1
            q = p + "mix."
            if isinstance(m, LatentAttentionSpec):
                sd[q + "dq"], sd[q + "dkv"] = W.down_w.split([m.q_rank, m.row])
                sd[q + "dq.norm"], sd[q + "dkv.norm"], sd[q + "uq"] = W.q_norm, W.kv_norm, W.uq_w
                sd[q + "uk"], sd[q + "uv"] = W.uk_w.transpose(1, 2).reshape(-1, m.kv_rank), W.uv_w.reshape(-1, m.kv_rank)
            else:
                sd[q + "q"], sd[q + "k"], sd[q + "v"] = W.qkv_w.split([m.heads * m.maps * m.dim, m.kv_heads * m.maps * m.dim, m.kv_heads * m.vdim])
                sd[q + "q.norm"], sd[q + "k.norm"] = W.q_norm, W.k_norm
                sd.update({q + n: W.lam[j] for j, n in enumerate(("lq1", "lk1", "lq2", "lk2"))})
            sd[q + "o"] = W.o_w
            if f is None:
                continue
            W = L.mlp
            assert not W.interleaved, "state_dict() must be taken before finalize_weights()"
            sd[p + "norm2"], sd[p + "ls2"] = L.norm2, L.ls2
            p += "mlp."
            if not f.is_moe:
                (sd[p + "gate"], sd[p + "up"]), sd[p + "down"] = W.gate_up_w.chunk(2), W.down_w
                continue
            sd[p + "router"], sd[p + "router.b"] = W.router_w, W.router_b
            for e in range(f.experts):
                sd[p + f"e{e}.gate"], sd[p + f"e{e}.up"], sd[p + f"e{e}.down"] = W.w13[e, :f.ff], W.w13[e, f.ff:], W.w2[e]
        return {k: v.contiguous() for k, v in sd.items()}

    # ------------------------------------------------------------------ forward
    def _rotation(self, rot: Optional[RotarySpec], inp):
        return None if rot is None else (self.cos_sin[rot], inp.positions, rot.interleaved)

    def _latent(self, W: LatentWeights, m: LatentAttentionSpec, h: torch.Tensor, inp, kv) -> torch.Tensor:
        rot = self._rotation(m.rot, inp)
        c_q = ops.latent_down(ops.linear(h, W.down_w), m.q_rank, m.kv_rank, W.q_norm, W.kv_norm, self.args.rms_norm_eps, rot, inp.slots, kv[0])
        q = ops.linear(c_q, W.uq_w).view(-1, m.heads, m.dim + m.rot_dim)
        return ops.latent_attention(q, W.uk_w, W.uv_w, kv[0], inp, rot, m.scale, m.dim)

    def _two_map(self, W: TwoMapWeights, m: AttentionSpec, h: torch.Tensor, inp, kv) -> torch.Tensor:
        eps, n_q = self.args.rms_norm_eps, m.heads * m.maps
        q = ops.qknorm_kvwrite(ops.linear(h, W.qkv_w), inp.slots, W.q_norm, W.k_norm, eps, kv[0], kv[1], n_q, m.kv_heads * m.maps,
                               self._rotation(m.rot, inp))
        return ops.paged_attention_ext(q.unflatten(1, (n_q, m.dim)), kv[0], kv[1], inp, m.scale, softcap=m.softcap,
                                       mix=(W.factor, 1.0 - m.diff, eps), bound=W.bound)

    def _feed_forward(self, L: BlockWeights, f: FeedForwardSpec, h: torch.Tensor, x: torch.Tensor, w_next: torch.Tensor, lead) -> torch.Tensor:
        """The second sublayer from its normed input h; adds to x and returns the next sublayer's input."""
        W, eps = L.mlp, self.args.rms_norm_eps
        if not f.is_moe:
            y = ops.linear(ops.gated_linear(h, W.gate_up_w, f.act, W.interleaved, f.limit), W.down_w)
            return ops.add_norm(y, x, 1.0, w_next, eps, L.ls2, AROUND_ZERO, lead)
        weights, ids = ops.moe_router(ops.linear_f32(h, W.router_w), f.top_k, f.scoring, bias=W.router_b)
        return ops.moe_add_norm(h, W.w13, W.w2, weights, ids, L.ls2, x, w_next, eps, f.act, W.interleaved, f.limit, AROUND_ZERO, lead)

    def forward(self, inp, kv_caches) -> torch.Tensor:
        """Returns the final-normed hidden states [T, H]."""
        a, eps, runs = self.args, self.args.rms_norm_eps, self.args.layer_runs
        again = (inp.tokens, self.embed, a.embedding_scale, inp.positions, self.positions)
        x, h = ops.embed_rms_norm(inp.tokens, self.embed, a.embedding_scale, self.layers[runs[0]].norm1, eps, inp.positions, self.positions,
                                  AROUND_ZERO)
        for r, li in enumerate(runs):
            L, s = self.layers[li], a.layer_specs[li]
            w_next = self.layers[runs[r + 1]].norm1 if r + 1 < len(runs) else self.final_norm
            lead = again if r + 1 in a.pass_starts[1:] else None          # the next run opens a further pass
            fused = lead if self.residual_hook is None else None
            mixer = self._latent if isinstance(s.mixer, LatentAttentionSpec) else self._two_map
            o = mixer(L.mix, s.mixer, h, inp, kv_caches[r])
            if self.layer_hook is not None:
                self.layer_hook(r)
            y = ops.linear(o, L.mix.o_w)
            if s.mlp is None:
                h = ops.add_norm(y, x, 1.0, w_next, eps, L.ls1, AROUND_ZERO, fused)
            else:
                h = ops.add_norm(y, x, 1.0, L.norm2, eps, L.ls1, AROUND_ZERO)
                h = self._feed_forward(L, s.mlp, h, x, w_next, fused)
            if self.residual_hook is not None:
                self.residual_hook(r, x)
                if lead is not None:
                    h = ops.lead_norm(lead, x, w_next, eps, AROUND_ZERO)
        return h

    def logits(self, hidden: torch.Tensor, sample_idx: torch.Tensor, gather: bool = True) -> torch.Tensor:
        sel = hidden.index_select(0, sample_idx.long()) if sample_idx is not None else hidden
        cap = self.args.logit_softcap
        return ops.linear_softcap(sel, self.lm_head, cap) if cap > 0 else ops.linear(sel, self.lm_head)

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
