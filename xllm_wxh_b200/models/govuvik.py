"""Govuvik: a decoder-only model whose configuration lists its layers one by one, every one of them with recurrent state.

A layer's mixer is a matrix memory with exponential gates (xLSTM's mLSTM), or two branches side by side: sliding-window attention
(short convolutions on queries, keys and values, norms over the whole query and key projection, partial rotation, a learned sink
per head, and scores that are mixed over the heads ahead of the softmax) and gated linear attention (a matrix state per head with a
decay of its own for every key channel); both branches' outputs are normed and averaged.  What a mixer reads goes through a short
causal convolution first.  The feed-forward is a mixture of experts without gates (squared relu) whose weights are the softmax over
the chosen experts' logits.  Sublayers are normed before and after, the residual is fp32, the embedding is normed, logits are
bounded by a tanh.

Mixed scores: a head's score is a sum over all heads of products of their queries and keys, so one product of all key heads' keys
side by side with a query row that holds the weighted queries of every key head (`ops.qknorm_all_kvwrite` with `mix`) gives it at
once; attention then runs as with a single, wide key head beside several value heads.

Every layer has state records (convolution inputs, matrix states) that belong to a slot the scheduler gives a sequence from its
first step to its last one (see `csrc/core/state_slots.h`), and attention layers a paged KV cache beside them.  The mechanisms live
in `ops` and take their constants as parameters; this file only loads weights and strings the ops together.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..parallel.comm import Comm
from .args import ModelArgs
from .layer_spec import FeedForwardSpec, MatrixMemorySpec, ParallelSpec, RotarySpec, attention_of
from .qwen import _DT, WeightInit
from .registry import register_model


class Rows:
    """Several projections of one input as one product: where each one's columns lie in its output."""

    def __init__(self, weights, align: int):
        self.at, parts, n = [], [], 0
        for w in weights:
            rows = -(-w.shape[0] // align) * align
            self.at.append((n, n + w.shape[0]))
            parts.append(torch.nn.functional.pad(w, (0, 0, 0, rows - w.shape[0])))
            n += rows
        self.w = torch.cat(parts, 0).contiguous()

    def split(self, y: torch.Tensor) -> List[torch.Tensor]:
        return [y[:, a:b] for a, b in self.at]

    def parts(self) -> List[torch.Tensor]:
        return [self.w[a:b] for a, b in self.at]


class ParallelWeights:
    def __init__(self):
        self.ins = None                         # attention q, k, v together; linear attention q, k, v, gate, decay's first factor
        self.conv_w = None                      # [taps, attention q + k + v columns]
        self.q_norm = self.k_norm = None
        self.talk = self.temp = None            # fp32, as stored
        self.mix = self.sink = None             # fp32: [heads, heads] talk times temp, [heads]
        self.a2_w = self.a2_b = None            # [heads * dim, rank (padded)], fp32 bias
        self.norm = None
        self.left_o = self.right_o = self.left_out = self.right_out = None


class MemoryWeights:
    def __init__(self):
        self.ins = None                         # q, k, v, gate
        self.gates_w = self.gates_b = None      # [2 heads, H]: input gates, forget gates; fp32 biases
        self.norm = self.o_w = None


class ExpertWeights:
    def __init__(self):
        self.router_w = self.up_w = self.down_w = None      # [E, H], [E, ff, H], [E, H, ff]


class BlockWeights:
    def __init__(self, spec):
        self.norm1 = self.norm1b = self.norm2 = self.norm2b = None
        self.conv_w = None                      # [taps, H]
        self.mix = ParallelWeights() if isinstance(spec.mixer, ParallelSpec) else MemoryWeights()
        self.mlp = ExpertWeights() if spec.mlp is not None else None


@register_model("govuvik")
class GovuvikForCausalLM:
    def __init__(self, args: ModelArgs, comm: Optional[Comm] = None, device="cpu", dtype: Optional[torch.dtype] = None):
        self.args = args
        self.comm = comm or Comm()
        if self.comm.tp_size > 1 or self.comm.ep_size > 1 or self.comm.dp_size > 1:
            raise ValueError("govuvik runs on one device: tensor, expert and data parallelism are not implemented for it")
        self.device = torch.device(device)
        self.dtype = dtype or _DT[args.dtype]
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"govuvik runs in bfloat16 or float32, not {self.dtype}")
        self.layers: List[BlockWeights] = [BlockWeights(s) for s in args.layer_specs]
        self.embed = self.embed_norm = self.final_norm = self.lm_head = None
        # rotation tables, one per distinct rotation; they are no weights and stay through sleep
        self.cos_sin: Dict[RotarySpec, torch.Tensor] = {}
        for s in args.layer_specs:
            a = attention_of(s.mixer)
            if a is not None and a.rot is not None and a.rot not in self.cos_sin:
                self.cos_sin[a.rot] = ops.ref.rotary_table(a.rot, args.max_position_embeddings, self.device)
        self.layer_hook = None       # callable(run index), right after a run's mixer (its cache is written by then)
        self.residual_hook = None    # callable(run index, fp32 residual), after a run's last sublayer (tests, tools)

    # ------------------------------------------------------------------ caches
    def kv_cache_shapes(self, num_blocks: int, block_size: int):
        out = []
        for li in self.args.layer_runs:
            m = attention_of(self.args.layer_specs[li].mixer)
            out.append(() if m is None else ((num_blocks, block_size, m.kv_heads, m.dim), (num_blocks, block_size, m.kv_heads, m.vdim)))
        return out

    def state_cache_shapes(self, slots: int):
        """(shape, dtype) of every layer run's state tensors: the last inputs of the input convolution; then the last projected
        queries, keys and values and the heads' matrices, or the heads' matrices with their normalisers and the running maxima."""
        out, H = [], self.args.hidden_size
        for li in self.args.layer_runs:
            m = self.args.layer_specs[li].mixer
            mine = [((slots, self.args.input_conv - 1, H), self.dtype)]
            if isinstance(m, ParallelSpec):
                a, t = m.left, m.right
                mine += [((slots, a.conv - 1, a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)), self.dtype),
                         ((slots, t.heads, t.dim, t.vdim), torch.float32)]
            else:
                mine += [((slots, m.heads, m.dim * m.vdim + m.dim), torch.float32), ((slots, m.heads), torch.float32)]
            out.append(tuple(mine))
        return out

    # ------------------------------------------------------------------ weights
    @staticmethod
    def tensor_shapes(a: ModelArgs) -> Dict[str, tuple]:
        """Checkpoint tensor names and shapes of a configuration; 0 stands for a size that only the checkpoint tells."""
        H = a.hidden_size
        out = {"embed": (a.vocab_size, H), "embed.norm": (H,), "final.norm": (H,), "head": (a.vocab_size, H)}
        for i, s in enumerate(a.layer_specs):
            p, m, f = f"l{i}.", s.mixer, s.mlp
            out.update({p + "norm1": (H,), p + "norm1b": (H,), p + "canon1": (H, a.input_conv)})
            if f is not None:
                out.update({p + "norm2": (H,), p + "norm2b": (H,), p + "mlp.router": (f.experts, H)})
                for e in range(f.experts):
                    out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = (f.ff, H), (H, f.ff)
            p += "mix."
            if isinstance(m, MatrixMemorySpec):
                k, v = m.heads * m.dim, m.heads * m.vdim
                out.update({p + "q": (k, H), p + "k": (k, H), p + "v": (v, H), p + "g": (v, H), p + "o": (H, v), p + "norm": (v,),
                            p + "i": (m.heads, H), p + "i.b": (m.heads,), p + "f": (m.heads, H), p + "f.b": (m.heads,)})
                continue
            l, t, q = m.left, m.right, p + "left."
            for n, rows in (("q", l.heads * l.dim), ("k", l.kv_heads * l.dim), ("v", l.kv_heads * l.vdim)):
                out[q + n], out[q + n + ".conv"] = (rows, H), (rows, l.conv)
                if n != "v":
                    out[q + n + ".norm"] = (rows,)
            out.update({q + "talk": (l.heads, l.heads), q + "temp": (l.heads,), q + "sink": (l.heads,), q + "o": (H, l.heads * l.vdim),
                        q + "out": (H,)})
            q, k, v = p + "right.", t.heads * t.dim, t.heads * t.vdim
            out.update({q + "q": (k, H), q + "k": (k, H), q + "v": (v, H), q + "g": (v, H), q + "o": (H, v), q + "norm": (t.vdim,),
                        q + "a1": (t.decay_rank, H), q + "a2": (k, t.decay_rank), q + "a2.b": (k,), q + "out": (H,)})
        return out

    def _fill(self, get) -> "GovuvikForCausalLM":
        """Build the weights from `get(name)` (checkpoint names, any dtype, any device)."""
        dev = lambda n: get(n).to(self.device, self.dtype).contiguous()
        f32 = lambda n: get(n).to(self.device, torch.float32).contiguous()
        align = 8 if self.dtype == torch.bfloat16 else 1        # rows of the tensor-core products start on 16-byte boundaries
        H = self.args.hidden_size
        self.embed, self.embed_norm, self.final_norm, self.lm_head = dev("embed"), dev("embed.norm"), dev("final.norm"), dev("head")
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, f, W = f"l{i}.", s.mixer, s.mlp, L.mix
            L.norm1, L.norm1b, L.conv_w = dev(p + "norm1"), dev(p + "norm1b"), dev(p + "canon1").t().contiguous()
            if f is not None:
                L.norm2, L.norm2b, M, q = dev(p + "norm2"), dev(p + "norm2b"), L.mlp, p + "mlp."
                M.router_w = dev(q + "router")
                M.up_w = torch.empty((f.experts, f.ff, H), dtype=self.dtype, device=self.device)
                M.down_w = torch.empty((f.experts, H, f.ff), dtype=self.dtype, device=self.device)
                for e in range(f.experts):
                    M.up_w[e].copy_(get(q + f"e{e}.up"))
                    M.down_w[e].copy_(get(q + f"e{e}.down"))
            p += "mix."
            if isinstance(m, MatrixMemorySpec):
                W.ins = Rows([dev(p + c) for c in "qkvg"], align)
                W.gates_w, W.gates_b = torch.cat([dev(p + "i"), dev(p + "f")]), torch.cat([f32(p + "i.b"), f32(p + "f.b")])
                W.norm, W.o_w = dev(p + "norm"), dev(p + "o")
                continue
            l, r = p + "left.", p + "right."
            W.ins = Rows([torch.cat([dev(l + c) for c in "qkv"])] + [dev(r + c) for c in ("q", "k", "v", "g", "a1")], align)
            W.conv_w = torch.cat([dev(l + c + ".conv") for c in "qkv"]).t().contiguous()
            W.q_norm, W.k_norm, W.sink = dev(l + "q.norm"), dev(l + "k.norm"), f32(l + "sink")
            W.talk, W.temp = f32(l + "talk"), f32(l + "temp")
            W.mix = (W.talk * W.temp).contiguous()
            a2 = dev(r + "a2")
            W.a2_w, W.a2_b = torch.nn.functional.pad(a2, (0, -a2.shape[1] % align)).contiguous(), f32(r + "a2.b")
            W.norm, W.left_o, W.right_o = dev(r + "norm"), dev(l + "o"), dev(r + "o")
            W.left_out, W.right_out = dev(l + "out"), dev(r + "out")
        return self

    def load_weights(self, ckpt) -> "GovuvikForCausalLM":
        want = self.tensor_shapes(self.args)
        for n, shape in want.items():
            if not ckpt.has(n):
                raise ValueError(f"the checkpoint has no tensor '{n}'")
            got = tuple(ckpt.get(n).shape)
            if len(got) != len(shape) or any(b and a != b for a, b in zip(got, shape)):
                raise ValueError(f"tensor '{n}' has shape {got}, the configuration asks for {shape}")
        for i, s in enumerate(self.args.layer_specs):
            if isinstance(s.mixer, ParallelSpec):
                p = f"l{i}.mix.right."
                rank = ckpt.get(p + "a1").shape[0]
                if ckpt.get(p + "a2").shape[1] != rank:
                    raise ValueError(f"tensors '{p}a1' and '{p}a2' differ in their inner size")
                s.mixer.right.decay_rank = int(rank)
        return self._fill(ckpt.get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "GovuvikForCausalLM":
        wi = WeightInit(seed, std, self.dtype, self.device)
        for s in self.args.layer_specs:
            if isinstance(s.mixer, ParallelSpec) and s.mixer.right.decay_rank == 0:
                s.mixer.right.decay_rank = 16
        shapes = self.tensor_shapes(self.args)

        def get(name):
            shape, last = shapes[name], name.rsplit(".", 1)[-1]
            if "norm" in last or last in ("out", "temp"):
                return wi.ones(shape)
            if last == "talk":
                return torch.eye(shape[0], device=self.device) + wi.normal(name, shape)
            if last == "sink" or name.endswith(".i.b"):
                return torch.zeros(shape, device=self.device)
            if name.endswith(".f.b"):
                return torch.linspace(3.0, 6.0, shape[0], device=self.device)
            return wi.normal(name, shape)
        return self._fill(get)

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """Tensors under their checkpoint names."""
        sd = {"embed": self.embed, "embed.norm": self.embed_norm, "final.norm": self.final_norm, "head": self.lm_head}
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, f, W = f"l{i}.", s.mixer, s.mlp, L.mix
            sd.update({p + "norm1": L.norm1, p + "norm1b": L.norm1b, p + "canon1": L.conv_w.t()})
            if f is not None:
                sd.update({p + "norm2": L.norm2, p + "norm2b": L.norm2b, p + "mlp.router": L.mlp.router_w})
                for e in range(f.experts):
                    sd[p + f"mlp.e{e}.up"], sd[p + f"mlp.e{e}.down"] = L.mlp.up_w[e], L.mlp.down_w[e]
            p += "mix."
            if isinstance(m, MatrixMemorySpec):
                sd.update(dict(zip((p + "q", p + "k", p + "v", p + "g"), W.ins.parts())))
                sd[p + "i"], sd[p + "f"] = W.gates_w.chunk(2)
                sd[p + "i.b"], sd[p + "f.b"] = W.gates_b.chunk(2)
                sd[p + "norm"], sd[p + "o"] = W.norm, W.o_w
                continue
            a, t, l, r = m.left, m.right, p + "left.", p + "right."
            rows = [a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim]
            qkv, *right = W.ins.parts()
            for c, w, conv in zip("qkv", qkv.split(rows), W.conv_w.t().split(rows)):
                sd[l + c], sd[l + c + ".conv"] = w, conv
            sd.update({l + "q.norm": W.q_norm, l + "k.norm": W.k_norm, l + "talk": W.talk, l + "temp": W.temp, l + "sink": W.sink,
                       l + "o": W.left_o, l + "out": W.left_out})
            sd.update(dict(zip((r + "q", r + "k", r + "v", r + "g", r + "a1"), right)))
            sd.update({r + "a2": W.a2_w[:, :t.decay_rank], r + "a2.b": W.a2_b, r + "norm": W.norm, r + "o": W.right_o, r + "out": W.right_out})
        return {k: v.contiguous() for k, v in sd.items()}

    # ------------------------------------------------------------------ forward
    def _parallel(self, W: ParallelWeights, m: ParallelSpec, h: torch.Tensor, inp, kv, state):
        """Both branches' outputs."""
        a, t, eps = m.left, m.right, self.args.rms_norm_eps
        qkv, q, k, v, g, low = W.ins.split(y := ops.linear(h, W.ins.w))
        qkv = ops.causal_conv(qkv, W.conv_w, None, state[1], inp)
        rot = None if a.rot is None else (self.cos_sin[a.rot], inp.positions, False)
        wide = ops.qknorm_all_kvwrite(qkv, inp.slots, W.q_norm, W.k_norm, eps, kv[0], kv[1], a.heads, a.kv_heads, rot, W.mix)
        o = ops.paged_attention_ext(wide.unflatten(1, (a.heads, a.kv_heads * a.dim)), kv[0].flatten(2).unsqueeze(2), kv[1], inp, a.scale,
                                    a.window, sinks=W.sink)
        low = y[:, W.ins.at[-1][0]:][:, :W.a2_w.shape[1]]        # with the padding of its rows, which is zero
        d = ops.gated_memory(q, k, v, ops.linear_f32(low, W.a2_w), W.a2_b, 1.0 / t.tau, g, W.norm, eps, state[2], inp)
        return ops.linear(o, W.left_o), ops.linear(d, W.right_o)

    def _memory(self, W: MemoryWeights, m: MatrixMemorySpec, h: torch.Tensor, inp, state) -> torch.Tensor:
        q, k, v, g = W.ins.split(ops.linear(h, W.ins.w))
        o = ops.matrix_memory(q, k, v, ops.linear_f32(h, W.gates_w), W.gates_b, m.gate_cap, g, W.norm, self.args.rms_norm_eps, state[1],
                              state[2], inp)
        return ops.linear(o, W.o_w)

    def _feed_forward(self, L: BlockWeights, f: FeedForwardSpec, h: torch.Tensor, x: torch.Tensor, w_next: torch.Tensor) -> torch.Tensor:
        """The second sublayer from its normed input h; adds to x and returns the next sublayer's input."""
        M = L.mlp
        weights, ids = ops.moe_router(ops.linear_f32(h, M.router_w), f.top_k, f.scoring)
        return ops.moe_post_norm_add_norm(h, M.up_w, M.down_w, weights, ids, None, f.experts, x, L.norm2b, w_next, self.args.rms_norm_eps,
                                          f.act)

    def forward(self, inp, kv_caches) -> torch.Tensor:
        """Returns the final-normed hidden states [T, H]."""
        a, eps, runs = self.args, self.args.rms_norm_eps, self.args.layer_runs
        x, h = ops.embed_rms_norm(inp.tokens, self.embed, a.embedding_scale, self.layers[runs[0]].norm1, eps, w_rows=self.embed_norm)
        for r, li in enumerate(runs):
            L, s, state = self.layers[li], a.layer_specs[li], inp.states[r]
            w_next = self.layers[runs[r + 1]].norm1 if r + 1 < len(runs) else self.final_norm
            w_mid = w_next if s.mlp is None else L.norm2
            h = ops.causal_conv(h, L.conv_w, None, state[0], inp, residual=True)
            if isinstance(s.mixer, ParallelSpec):
                left, right = self._parallel(L.mix, s.mixer, h, inp, kv_caches[r], state)
                if self.layer_hook is not None:
                    self.layer_hook(r)
                h = ops.branches_post_norm_add_norm(left, right, L.mix.left_out, L.mix.right_out, s.mixer.left_scale, x, L.norm1b, w_mid, eps)
            else:
                y = self._memory(L.mix, s.mixer, h, inp, state)
                if self.layer_hook is not None:
                    self.layer_hook(r)
                h = ops.post_norm_add_norm(y, x, L.norm1b, w_mid, eps)
            if s.mlp is not None:
                h = self._feed_forward(L, s.mlp, h, x, w_next)
            if self.residual_hook is not None:
                self.residual_hook(r, x)
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
