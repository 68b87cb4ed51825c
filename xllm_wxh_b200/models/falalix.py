"""Falalix: a decoder-only model whose configuration lists its layers one by one, most of them with recurrent state.

A layer's mixer is a selective scan behind a short convolution, or two branches side by side: attention (biased projections,
norms over the whole query and key projection, no rotation, a sliding window with kept first positions, a sigmoid output
gate) and time mixing (a matrix state per head with a decay of its own for every key channel).  Sublayers are normed before
only and enter an fp32 residual with a constant factor; the dense feed-forward squares its relu.  A range of layers may run
several times with the same weights; ahead of every pass a product of the residual and the embedding replaces the residual.

Every layer run has a paged KV cache (attention) and state records (recurrent parts) of its own.  The state belongs to a
slot that the scheduler gives a sequence from its first step to its last one; see `csrc/core/state_slots.h`.

The mechanisms live in `ops` and take their constants as parameters; this file only loads weights and strings the ops
together.  The two branches' outputs land side by side in one buffer, scaled, so that one product with both output weights
adds them in fp32.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..parallel.comm import Comm
from .args import ModelArgs
from .layer_spec import ParallelSpec, SelectiveScanSpec, attention_of
from .qwen import _DT, WeightInit
from .registry import register_model

MIXES = "rkvgw"             # inputs of time mixing, in the order of its blend weights


class ParallelWeights:
    def __init__(self):
        self.qkvg_w = self.qkvg_b = self.q_norm = self.k_norm = None       # rows q, k, v, gate; the gate's bias is zero
        self.mu = None                          # [5, H] blend weights in the order of MIXES
        self.rkvg_w = None                      # [4, heads * dim, H]
        self.w1 = self.w2 = None                # decay's low-rank projection
        self.w0 = self.u = None                 # fp32
        self.norm = None
        self.o_w = None                         # [H, attention heads * vdim + time mixing heads * dim]


class ScanWeights:
    def __init__(self):
        self.in_w = self.conv_w = self.conv_b = None     # conv_w: [taps, channels]
        self.x_w = self.dt_w = None             # bf16: rows / columns padded with zeros to multiples of 8
        self.dt_b = self.A = self.D = None      # fp32
        self.A_log = None                       # as stored
        self.o_w = None


class FeedForwardWeights:
    def __init__(self):
        self.up_w = self.down_w = None


class BlockWeights:
    def __init__(self, spec):
        self.norm1 = self.norm2 = None
        self.mix = ParallelWeights() if isinstance(spec.mixer, ParallelSpec) else ScanWeights()
        self.mlp = FeedForwardWeights() if spec.mlp is not None else None


def _pad(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    return torch.nn.functional.pad(w, (0, cols - w.shape[1], 0, rows - w.shape[0])).contiguous()


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


@register_model("falalix")
class FalalixForCausalLM:
    def __init__(self, args: ModelArgs, comm: Optional[Comm] = None, device="cpu", dtype: Optional[torch.dtype] = None):
        self.args = args
        self.comm = comm or Comm()
        if self.comm.tp_size > 1 or self.comm.ep_size > 1 or self.comm.dp_size > 1:
            raise ValueError("falalix runs on one device: tensor, expert and data parallelism are not implemented for it")
        self.device = torch.device(device)
        self.dtype = dtype or _DT[args.dtype]
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"falalix runs in bfloat16 or float32, not {self.dtype}")
        self.layers: List[BlockWeights] = [BlockWeights(s) for s in args.layer_specs]
        self.embed = self.final_norm = self.lm_head = None
        self.loop_in = self.loop_step = None
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
        """(shape, dtype) of every layer run's state tensors: selective scan: its states and the convolution's last inputs;
        time mixing: the heads' matrices and the last input row."""
        out = []
        for li in self.args.layer_runs:
            m = self.args.layer_specs[li].mixer
            if isinstance(m, SelectiveScanSpec):
                out.append((((slots, m.inner, m.state), torch.float32), ((slots, m.conv - 1, m.inner), self.dtype)))
            else:
                t = m.right
                out.append((((slots, t.heads, t.dim, t.dim), torch.float32), ((slots, self.args.hidden_size), self.dtype)))
        return out

    # ------------------------------------------------------------------ weights
    @staticmethod
    def tensor_shapes(a: ModelArgs) -> Dict[str, tuple]:
        """Checkpoint tensor names and shapes of a configuration; 0 stands for a size that only the checkpoint tells."""
        H = a.hidden_size
        out = {"embed": (a.vocab_size, H), "final.norm": (H,), "head": (a.vocab_size, H)}
        if a.pass_starts:
            out["loop.in"], out["loop.step"] = (H, 2 * H), (len(a.pass_starts), H)
        for i, s in enumerate(a.layer_specs):
            p, m = f"l{i}.", s.mixer
            out[p + "norm1"] = (H,)
            if s.mlp is not None:
                out[p + "norm2"], out[p + "mlp.up"], out[p + "mlp.down"] = (H,), (s.mlp.ff, H), (H, s.mlp.ff)
            p += "mix."
            if isinstance(m, SelectiveScanSpec):
                out.update({p + "in": (2 * m.inner, H), p + "conv": (m.inner, m.conv), p + "conv.b": (m.inner,),
                            p + "x": (m.dt_rank + 2 * m.state, m.inner), p + "dt": (m.inner, m.dt_rank), p + "dt.b": (m.inner,),
                            p + "A_log": (m.inner, m.state), p + "D": (m.inner,), p + "o": (H, m.inner)})
                continue
            a_, t = m.left, m.right
            for n, rows in (("q", a_.heads * a_.dim), ("k", a_.kv_heads * a_.dim), ("v", a_.kv_heads * a_.vdim)):
                out[f"{p}left.{n}"], out[f"{p}left.{n}.b"] = (rows, H), (rows,)
            out.update({p + "left.q.norm": (a_.heads * a_.dim,), p + "left.k.norm": (a_.kv_heads * a_.dim,),
                        p + "left.g": (a_.heads * a_.vdim, H), p + "left.o": (H, a_.heads * a_.vdim)})
            p, n = p + "right.", t.heads * t.dim
            out.update({p + "mu." + c: (H,) for c in MIXES})
            out.update({p + c: (n, H) for c in "rkvg"})
            out.update({p + "w1": (t.decay_rank, H), p + "w2": (n, t.decay_rank), p + "w0": (n,), p + "u": (t.heads, t.dim),
                        p + "norm": (n,), p + "o": (H, n)})
        return out

    def _fill(self, get) -> "FalalixForCausalLM":
        """Build the weights from `get(name)` (checkpoint names, any dtype, any device)."""
        dev = lambda n: get(n).to(self.device, self.dtype).contiguous()
        f32 = lambda n: get(n).to(self.device, torch.float32).contiguous()
        pad8 = _up8 if self.dtype == torch.bfloat16 else (lambda n: n)
        H = self.args.hidden_size
        self.embed, self.final_norm, self.lm_head = dev("embed"), dev("final.norm"), dev("head")
        if self.args.pass_starts:
            self.loop_in, self.loop_step = ops.split_columns(dev("loop.in"), H), f32("loop.step")
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, W = f"l{i}.", s.mixer, L.mix
            L.norm1 = dev(p + "norm1")
            if s.mlp is not None:
                L.norm2, L.mlp.up_w, L.mlp.down_w = dev(p + "norm2"), dev(p + "mlp.up"), dev(p + "mlp.down")
            p += "mix."
            if isinstance(m, SelectiveScanSpec):
                W.in_w, W.conv_w, W.conv_b, W.o_w = dev(p + "in"), dev(p + "conv").t().contiguous(), dev(p + "conv.b"), dev(p + "o")
                W.x_w = _pad(dev(p + "x"), pad8(m.dt_rank + 2 * m.state), m.inner)
                W.dt_w = _pad(dev(p + "dt"), m.inner, pad8(m.dt_rank))
                W.dt_b, W.D, W.A_log = f32(p + "dt.b"), f32(p + "D"), dev(p + "A_log")
                W.A = -torch.exp(f32(p + "A_log"))
                continue
            q = p + "left."
            W.qkvg_w = torch.cat([dev(q + n) for n in "qkvg"], 0)
            W.qkvg_b = torch.cat([dev(q + n + ".b") for n in "qkv"] + [torch.zeros(m.left.heads * m.left.vdim, dtype=self.dtype,
                                                                                   device=self.device)])
            W.q_norm, W.k_norm = dev(q + "q.norm"), dev(q + "k.norm")
            t = p + "right."
            W.mu = torch.stack([dev(t + "mu." + c) for c in MIXES])
            W.rkvg_w = torch.stack([dev(t + c) for c in "rkvg"])
            W.w1, W.w2, W.w0, W.u, W.norm = dev(t + "w1"), dev(t + "w2"), f32(t + "w0"), f32(t + "u"), dev(t + "norm")
            W.o_w = torch.cat([dev(q + "o"), dev(t + "o")], 1).contiguous()
        return self

    def load_weights(self, ckpt) -> "FalalixForCausalLM":
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
                rank = ckpt.get(p + "w1").shape[0]
                if ckpt.get(p + "w2").shape[1] != rank:
                    raise ValueError(f"tensors '{p}w1' and '{p}w2' differ in their inner size")
                s.mixer.right.decay_rank = int(rank)
        return self._fill(ckpt.get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "FalalixForCausalLM":
        wi = WeightInit(seed, std, self.dtype, self.device)
        for s in self.args.layer_specs:
            if isinstance(s.mixer, ParallelSpec) and s.mixer.right.decay_rank == 0:
                s.mixer.right.decay_rank = 32
        shapes = self.tensor_shapes(self.args)

        def get(name):
            shape = shapes[name]
            if "norm" in name.rsplit(".", 1)[-1] or name.endswith(".D"):
                return wi.ones(shape)
            if ".mu." in name:
                return wi.ones(shape) * 0.5
            if name.endswith(".A_log"):
                return torch.log(torch.arange(1, shape[1] + 1, dtype=torch.float32, device=self.device)).expand(shape)
            if name.endswith(".right.w0"):
                return torch.full(shape, -2.0, device=self.device)
            if name.endswith(".dt.b"):
                return torch.full(shape, -4.0, device=self.device)
            return wi.normal(name, shape)
        return self._fill(get)

    def state_dict(self) -> Dict[str, torch.Tensor]:
        """Tensors under their checkpoint names."""
        H = self.args.hidden_size
        sd = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head}
        if self.loop_in is not None:
            sd["loop.in"], sd["loop.step"] = self.loop_in[:, -2 * H:], self.loop_step
        for i, (L, s) in enumerate(zip(self.layers, self.args.layer_specs)):
            p, m, W = f"l{i}.", s.mixer, L.mix
            sd[p + "norm1"] = L.norm1
            if L.mlp is not None:
                sd[p + "norm2"], sd[p + "mlp.up"], sd[p + "mlp.down"] = L.norm2, L.mlp.up_w, L.mlp.down_w
            p += "mix."
            if isinstance(m, SelectiveScanSpec):
                sd.update({p + "in": W.in_w, p + "conv": W.conv_w.t(), p + "conv.b": W.conv_b, p + "x": W.x_w[:m.dt_rank + 2 * m.state],
                           p + "dt": W.dt_w[:, :m.dt_rank], p + "dt.b": W.dt_b, p + "A_log": W.A_log, p + "D": W.D, p + "o": W.o_w})
                continue
            a = m.left
            n_o = a.heads * a.vdim
            rows = [a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, n_o]
            for c, w, b in zip("qkvg", W.qkvg_w.split(rows), W.qkvg_b.split(rows)):
                sd[f"{p}left.{c}"] = w
                if c != "g":
                    sd[f"{p}left.{c}.b"] = b
            sd[p + "left.q.norm"], sd[p + "left.k.norm"] = W.q_norm, W.k_norm
            sd[p + "left.o"], sd[p + "right.o"] = W.o_w[:, :n_o], W.o_w[:, n_o:]
            p += "right."
            sd.update({p + "mu." + c: W.mu[j] for j, c in enumerate(MIXES)})
            sd.update({p + c: W.rkvg_w[j] for j, c in enumerate("rkvg")})
            sd.update({p + "w1": W.w1, p + "w2": W.w2, p + "w0": W.w0, p + "u": W.u, p + "norm": W.norm})
        return {k: v.contiguous() for k, v in sd.items()}

    # ------------------------------------------------------------------ forward
    def _parallel(self, W: ParallelWeights, m: ParallelSpec, h: torch.Tensor, inp, kv, state) -> torch.Tensor:
        a, t, eps = m.left, m.right, self.args.rms_norm_eps
        n_o, n_t = a.heads * a.vdim, t.heads * t.dim
        both = torch.empty((h.shape[0], n_o + n_t), dtype=h.dtype, device=h.device)
        qkvg = ops.linear(h, W.qkvg_w, W.qkvg_b)
        q = ops.qknorm_all_kvwrite(qkvg, inp.slots, W.q_norm, W.k_norm, eps, kv[0], kv[1], a.heads, a.kv_heads)
        o = ops.paged_attention_ext(q.unflatten(1, (a.heads, a.dim)), kv[0], kv[1], inp, a.scale, a.window, 0, None, None, a.keep_first)
        ops.gate_into(o, qkvg[:, -n_o:], m.left_scale, both[:, :n_o])
        mixed = ops.token_shift(h, W.mu, state[1], inp)
        r, k, v, g = (ops.linear(mixed[j], W.rkvg_w[j]) for j in range(4))
        z = ops.linear_f32(ops.act_linear(mixed[4], W.w1, "tanh"), W.w2)
        ops.time_mix(r, k, v, z, W.w0, W.u, g, W.norm, m.right_scale, eps, state[0], inp, both[:, n_o:])
        return ops.linear(both, W.o_w)

    def _scan(self, W: ScanWeights, m: SelectiveScanSpec, h: torch.Tensor, inp, state) -> torch.Tensor:
        xz = ops.linear(h, W.in_w)
        x = ops.conv_silu(xz[:, :m.inner], W.conv_w, W.conv_b, state[1], inp)
        low = ops.linear(x, W.x_w)
        dt = ops.linear_f32(low[:, :W.dt_w.shape[1]], W.dt_w)
        B, C = low[:, m.dt_rank:m.dt_rank + m.state], low[:, m.dt_rank + m.state:m.dt_rank + 2 * m.state]
        return ops.linear(ops.selective_scan(x, dt, W.dt_b, W.A, B, C, W.D, xz[:, m.inner:], state[0], inp), W.o_w)

    def forward(self, inp, kv_caches) -> torch.Tensor:
        """Returns the final-normed hidden states [T, H]."""
        a, eps, runs = self.args, self.args.rms_norm_eps, self.args.layer_runs
        passes = {r: t for t, r in enumerate(a.pass_starts)}
        x, h = ops.embed_rms_norm(inp.tokens, self.embed, a.embedding_scale, self.layers[runs[0]].norm1, eps)
        for r, li in enumerate(runs):
            L, s = self.layers[li], a.layer_specs[li]
            if r in passes:
                both = ops.split_rows(x, inp.tokens, self.embed, a.embedding_scale)
                h = ops.replace_norm(ops.linear_f32(both, self.loop_in), self.loop_step[passes[r]], x, L.norm1, eps)
            w_next = self.layers[runs[r + 1]].norm1 if r + 1 < len(runs) else self.final_norm
            if isinstance(s.mixer, SelectiveScanSpec):
                y = self._scan(L.mix, s.mixer, h, inp, inp.states[r])
            else:
                y = self._parallel(L.mix, s.mixer, h, inp, kv_caches[r], inp.states[r])
            if self.layer_hook is not None:
                self.layer_hook(r)
            h = ops.add_norm(y, x, a.residual_mult, w_next if s.mlp is None else L.norm2, eps)
            if s.mlp is not None:
                h = ops.add_norm(ops.linear(ops.act_linear(h, L.mlp.up_w, s.mlp.act), L.mlp.down_w), x, a.residual_mult, w_next, eps)
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
