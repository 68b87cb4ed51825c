"""Govuvik on the CPU path in fp32: configuration, each mechanism against the plain statement of tests/oracle_govuvik.py, whole
models through the engine (portions, decoding, batches, blocks and state slots used again), greedy generation, the replay
program."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import oracle_govuvik as O
from tests.helpers import govuvik_models as M
from tests.helpers.portions import CUTS, RAG, Ragged, rag
from xllm_wxh_b200 import LLM, SamplingParams, ops
from xllm_wxh_b200.models.args import args_from_hf_config, preset
from xllm_wxh_b200.models.layer_spec import MatrixMemorySpec, ParallelSpec, RotarySpec
from xllm_wxh_b200.models.registry import get_model_class

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 1e-4        # a row whose products with its own key nearly vanish is normed up; all others are below 1e-5


def f64(sd):
    return {k: v.double() for k, v in sd.items()}


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    cfg = M.mixed_config()
    sd = M.weights(cfg, 1)
    return cfg, f64(sd), M.save(cfg, sd, tmp_path_factory.mktemp("govuvik"))


# ----------------------------------------------------------------------------- configuration
def test_config_reader_takes_everything_from_the_file():
    a = args_from_hf_config(M.mixed_config(width=88, vocab=301))
    assert (a.model_type, a.hidden_size, a.vocab_size, a.rms_norm_eps, a.logit_softcap, a.input_conv) == ("govuvik", 88, 301, 3e-6, 12.0, 3)
    assert a.layer_runs == [0, 1, 2, 3, 4]
    m, p, q = a.layer_specs[3].mixer, a.layer_specs[2].mixer, a.layer_specs[1].mixer
    assert isinstance(m, MatrixMemorySpec) and (m.heads, m.dim, m.vdim, m.gate_cap) == (2, 40, 24, 12.0)
    assert isinstance(p, ParallelSpec) and p.branch_norm and (p.left_scale, p.right_scale) == (0.5, 0.5)
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.window, p.left.conv) == (4, 1, 40, 56, 33, 5)
    assert (p.right.heads, p.right.dim, p.right.vdim, p.right.tau) == (2, 48, 24, 1.0)
    assert p.left.rot == RotarySpec(40, 3e3) and q.left.rot == RotarySpec(10, 3e3, False, 5.0, 60.0, 3.0, 1.5, True)
    f = a.layer_specs[3].mlp
    assert a.layer_specs[0].mlp is None and (f.ff, f.experts, f.top_k, f.act, f.scoring) == (24, 9, 4, "relu2", "softmax_chosen")
    model = get_model_class("govuvik")(a)
    kv, st = model.kv_cache_shapes(5, 16), model.state_cache_shapes(4)
    assert kv[0] == () and kv[2] == ((5, 16, 1, 40), (5, 16, 1, 56))
    assert st[2] == (((4, 2, 88), torch.bfloat16), ((4, 4, 256), torch.bfloat16), ((4, 2, 48, 24), torch.float32))
    assert st[3] == (((4, 2, 88), torch.bfloat16), ((4, 2, 40 * 24 + 40), torch.float32), ((4, 2), torch.float32))


def test_config_reader_rejects_what_it_does_not_know():
    for edit in (lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][1]["mlp"].update(kind="dense"),
                 lambda c: c["layers"][1]["mixer"]["left"].update(heads=5), lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26),
                 lambda c: c["layers"][1]["mlp"]["router"].update(top=6), lambda c: c["layers"][0]["mixer"].update(gate_cap=0),
                 lambda c: c["layers"][1]["mixer"]["right"].update(tau=0), lambda c: c["canon"].update(taps=0)):
        cfg = copy.deepcopy(M.mixed_config())
        edit(cfg)
        with pytest.raises(ValueError):
            args_from_hf_config(cfg)


def test_loading_checks_names_and_shapes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 0)
    for i, (name, edit) in enumerate([("l0.mix.left.talk", lambda d: d.pop("l0.mix.left.talk")), ("l1.mlp.e6.up", lambda d: d.pop("l1.mlp.e6.up")),
                                      ("l1.mix.f.b", lambda d: d.update({"l1.mix.f.b": sd["l1.mix.f.b"].repeat(2)})),
                                      ("l0.mix.right.a1", lambda d: d.update({"l0.mix.right.a1": sd["l0.mix.right.a1"][:-1]}))]):
        bad = dict(sd)
        edit(bad)
        with pytest.raises(ValueError, match=name):
            M.engine(M.save(cfg, bad, tmp_path / str(i)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_dict_round_trip(mixed, dtype):
    cfg, sd, path = mixed
    m = M.engine(path, dtype=dtype).worker.model
    got = m.state_dict()
    assert set(got) == set(sd)
    for k in sd:
        assert torch.equal(got[k].double(), sd[k]), k
    assert m.weight_bytes() > 0


# ----------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 8192), (5.0, 1.5, 3.0, 60), (2.0, 2.0, 2.0, 100)])
def test_rotation_frequencies(scaling):
    for dims, base in ((24, 5e5), (64, 1e4), (6, 20.0)):
        rot = {"dims": dims, "base": base}
        kw = {}
        if scaling:
            rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
            kw = dict(factor=scaling[0], original=scaling[3], fast=scaling[2], slow=scaling[1], by_turns=True)
        if scaling and scaling[1] == scaling[2]:          # no ramp: every wavelength is kept or slowed
            rot["scaling"]["high"] = scaling[2] + 1e-9
        got, mult = RotarySpec(dims, base, **kw).frequencies()
        assert mult == 1.0 and np.allclose(got, O.frequencies(rot), rtol=1e-12, atol=0)


def test_scaled_rotation_has_all_three_ranges():
    f = [1e4 ** (-2 * i / 64) for i in range(32)]
    got = O.frequencies({"dims": 64, "base": 1e4, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}})
    kept, slowed = [a == b for a, b in zip(f, got)], [abs(a / 8 - b) < 1e-12 for a, b in zip(f, got)]
    assert any(kept) and any(slowed) and sum(kept) + sum(slowed) < 32 and not any(a and b for a, b in zip(kept, slowed))


@pytest.mark.parametrize("rot", [None, (10, 3e3), (24, 100.0), (2, 7.0)])
def test_mixed_scores_are_products_with_all_keys_side_by_side(rot):
    """Queries of `qknorm_all_kvwrite` with a mixing matrix against the sum over heads of normed, turned and weighted scores."""
    g = torch.Generator().manual_seed(5)
    T, H, G, d, dv = 12, 6, 3, 24, 7
    qkv = torch.randn(T, (H + G) * d + G * dv + 5, generator=g) * 1e-2           # small rows: eps matters
    qw, kw, talk, temp = (torch.randn(*s, generator=g) for s in ((H * d,), (G * d,), (H, H), (H,)))
    kc, vc = torch.zeros(4, 4, G, d), torch.zeros(4, 4, G, dv)
    slots, pos = torch.randperm(16, generator=g)[:T].int(), torch.arange(T)
    table = None if rot is None else (ops.ref.rotary_table(RotarySpec(*rot), 64), pos, False)
    cfg = None if rot is None else {"dims": rot[0], "base": rot[1]}
    a, b, c, _ = qkv.split([H * d, G * d, G * dv, 5], -1)
    q = O.rotate(O.rms_norm(a, qw, 1e-4).view(T, H, d), cfg)
    k = O.rotate(O.rms_norm(b, kw, 1e-4).view(T, G, d), cfg)
    plain = ops.qknorm_all_kvwrite(qkv.clone(), slots, qw, kw, 1e-4, kc, vc, H, G, table)
    assert torch.allclose(plain.view(T, H, d), q, atol=1e-5)
    kc.zero_(), vc.zero_()
    wide = ops.qknorm_all_kvwrite(qkv.clone(), slots, qw, kw, 1e-4, kc, vc, H, G, table, talk * temp)
    keys = kc.view(-1, G * d)[slots.long()]
    assert torch.allclose(keys, k.flatten(1), atol=1e-5) and torch.equal(vc.view(-1, G * dv)[slots.long()], c)
    want = O.mix_scores(O.raw_scores(q, k, 0.7), temp, talk)
    assert torch.allclose(torch.einsum("thx,jx->htj", wide.view(T, H, G * d), keys) * 0.7, want, atol=1e-4)


def test_attention_over_one_wide_key_head():
    g = torch.Generator().manual_seed(4)
    n, H, G, d, dv = 40, 4, 2, 8, 6
    for size in (1, 3, 16, 17, 64):
        q, k, v = torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, G, dv, generator=g)
        temp, talk, sink = torch.randn(H, generator=g), torch.randn(H, H, generator=g), torch.randn(H, generator=g) * 2
        bt = torch.tensor([[2, 1, 3]]).int()
        kc, vc = torch.zeros(4, 16, 1, G * d), torch.zeros(4, 16, G, dv)
        for t in range(n):
            kc[bt[0, t // 16], t % 16, 0], vc[bt[0, t // 16], t % 16] = k[t].flatten(), v[t]
        wide = torch.einsum("hjg,tjgd->thjd", (talk * temp).view(H, G, -1), q.view(n, G, -1, d)).reshape(n, H, G * d)
        want = O.attention_core(q, k, v, 0.5, temp, talk, sink, size).flatten(1)
        for m in (n, 1, 2, 17):
            got = ops.paged_attention_ext(wide[n - m:], kc, vc, Inputs(m, n, bt), 0.5, size, sinks=sink)
            assert torch.allclose(got, want[n - m:], atol=1e-5)


class Inputs:
    def __init__(self, m, n, bt):
        self.q_cu, self.kv_lens, self.block_tables, self.n_seqs = torch.tensor([0, m]), torch.tensor([n]), bt, 1


def test_window_and_sink():
    see = O.visible_matrix(9, 3)
    assert see[6].nonzero().flatten().tolist() == [4, 5, 6] and see[1].nonzero().flatten().tolist() == [0, 1]
    s, sink = torch.tensor([[0.3, -2.0, 1.0]]), torch.tensor(4.0)
    e = torch.exp(s)
    assert torch.allclose(O.softmax_with_sink(s, sink), e / (e.sum() + math.exp(4.0)))


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("residual", [False, True])
@pytest.mark.parametrize("cuts", CUTS)
def test_conv(cuts, residual, taps):
    g = torch.Generator().manual_seed(2)
    C = 9
    x, w = [torch.randn(n, C, generator=g) for n in RAG], torch.randn(C, taps, generator=g)
    state = torch.full((6, taps - 1, C), 1e3)                     # what earlier owners of the slots left behind
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.causal_conv(rag(x, rows), w.t(), None, state, q, kv, sl, n, "none", residual)
        assert torch.allclose(got, rag([O.causal_conv(s, w) + residual * s for s in x], rows), atol=1e-5)


@pytest.mark.parametrize("tau", [1.0, 11.0])
@pytest.mark.parametrize("cuts", CUTS)
def test_gated_linear_attention(cuts, tau):
    g = torch.Generator().manual_seed(1)
    H, d, dv, eps = 2, 6, 5, 1e-4
    q_, k, z = ([torch.randn(n, H * d, generator=g) for n in RAG] for _ in range(3))
    v, gate = ([torch.randn(n, H * dv, generator=g) for n in RAG] for _ in range(2))
    bias, nw = torch.randn(H * d, generator=g), torch.randn(dv, generator=g)
    want = []
    for i in range(3):
        o = O.gated_linear_core(q_[i].view(-1, H, d) * d ** -0.5, k[i].view(-1, H, d), v[i].view(-1, H, dv),
                                O.channel_decay(z[i] + bias, tau).view(-1, H, d))
        want.append(O.rms_norm(o, nw, eps).flatten(1) * O.silu(gate[i]))
    state = torch.full((6, H, d, dv), 1e3)
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.gated_memory(*(rag(x, rows) for x in (q_, k, v, z)), bias, 1 / tau, rag(gate, rows), nw, eps, state, q, kv, sl, n)
        assert torch.allclose(got, rag(want, rows), atol=1e-4)


@pytest.mark.parametrize("level", [-6.0, 0.0, 5.0])
@pytest.mark.parametrize("cuts", CUTS)
def test_matrix_memory(cuts, level):
    """Input gates far below, around and above the running maximum's start at 0; the normaliser small and large."""
    g = torch.Generator().manual_seed(3)
    H, d, dv, eps, cap = 2, 6, 5, 1e-4, 7.0
    q_, k = ([torch.randn(n, H * d, generator=g) for n in RAG] for _ in range(2))
    v, gate = ([torch.randn(n, H * dv, generator=g) for n in RAG] for _ in range(2))
    z = [torch.randn(n, 2 * H, generator=g) * 3 for n in RAG]
    bias, nw = torch.cat([torch.full((H,), level), torch.full((H,), 2.0)]), torch.randn(H * dv, generator=g)
    want = []
    for i in range(3):
        log_i, f = O.soft_bound(z[i] + bias, cap).split(H, -1)
        o = O.matrix_memory_core(q_[i].view(-1, H, d) * d ** -0.5, k[i].view(-1, H, d), v[i].view(-1, H, dv), log_i, O.log_sigmoid(f))
        want.append(O.rms_norm(o, 1.0, eps).flatten(1) * nw * O.sigmoid(gate[i]))
    state, top = torch.full((6, H, d * dv + d), 1e3), torch.full((6, H), 1e3)
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.matrix_memory(*(rag(x, rows) for x in (q_, k, v, z)), bias, cap, rag(gate, rows), nw, eps, state, top, q, kv, sl, n)
        assert torch.allclose(got, rag(want, rows), atol=1e-4)


def test_matrix_memory_is_a_weighted_mean_of_its_past():
    """Without the running maximum: sums of plain exponentials, the normaliser at least 1."""
    g = torch.Generator().manual_seed(9)
    n, d, dv = 12, 4, 3
    q, k, v = (torch.randn(n, 1, w, generator=g).double() for w in (d, d, dv))
    li, lf = torch.randn(n, 1, generator=g).double(), -torch.rand(n, 1, generator=g).double()
    got = O.matrix_memory_core(q, k, v, li, lf)[:, 0]
    for t in range(n):
        w = torch.stack([torch.exp(li[s, 0] + lf[s + 1:t + 1, 0].sum()) for s in range(t + 1)]) * (k[:t + 1, 0] @ q[t, 0])
        assert torch.allclose(got[t], (w[:, None] * v[:t + 1, 0]).sum(0) / max(abs(w.sum()), 1.0), rtol=1e-4)


def test_norm_kernels():
    g = torch.Generator().manual_seed(5)
    T, W = 6, 24
    x, a, b = (torch.randn(T, W, generator=g) for _ in range(3))
    wa, wb, wp, wn = (torch.randn(W, generator=g) for _ in range(4))
    got = x.clone()
    h = ops.branches_post_norm_add_norm(a, b, wa, wb, 0.5, got, wp, wn, 1e-3)
    y = (O.rms_norm(a, wa, 1e-3) + O.rms_norm(b, wb, 1e-3)) / 2
    want = x + O.rms_norm(y, wp, 1e-3)
    assert torch.allclose(got, want, atol=1e-5) and torch.allclose(h, O.rms_norm(want, wn, 1e-3), atol=1e-5)
    table, ids = torch.randn(9, W, generator=g) * 1e-2, torch.tensor([3, 0, 8, 3, 1]).int()
    x, h = ops.embed_rms_norm(ids, table, 1.0, wn, 1e-3, w_rows=wa)
    want = O.rms_norm(table[ids.long()], wa, 1e-3)
    assert torch.allclose(x, want, atol=1e-5) and torch.allclose(h, O.rms_norm(want, wn, 1e-3), atol=1e-5)


def test_experts_without_a_gate():
    g = torch.Generator().manual_seed(6)
    T, W, ff, E, top = 11, 16, 12, 5, 3
    h, x = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g)
    up, down, router = torch.randn(E, ff, W, generator=g) / 4, torch.randn(E, W, ff, generator=g) / 4, torch.randn(E, W, generator=g)
    sd = {"router": router, **{f"e{e}.up": up[e] for e in range(E)}, **{f"e{e}.down": down[e] for e in range(E)}}
    y = O.feed_forward(sd, "", {"router": {"top": top}}, h)
    w, ids = ops.moe_router(ops.linear_f32(h, router), top, "softmax_chosen")
    one = torch.ones(W)
    want = x + O.rms_norm(y, one, 1e-5)
    got = ops.moe_post_norm_add_norm(h, up, down, w, ids, None, E, x, one, one, 1e-5, "relu2")
    assert torch.allclose(x, want, atol=1e-5) and torch.allclose(got, O.rms_norm(want, one, 1e-5), atol=1e-5)


# ----------------------------------------------------------------------------- whole models through the engine
def test_layers_one_by_one(mixed):
    cfg, sd, path = mixed
    toks = M.tokens(45, cfg["vocab"], 7)
    want = []
    logits = O.forward(sd, cfg, toks, want)
    eng, got = M.engine(path), []
    eng.worker.model.residual_hook = lambda r, x: got.append(x.clone())
    out = M.replay(eng, {"a": toks}, [[("a", 45)]])["a"]
    assert len(got) == len(want) == 5
    for r, (a, b) in enumerate(zip(got, want)):
        assert M.row_error(a, b).max() < TOL, r
    assert M.row_error(out, logits).max() < TOL


@pytest.mark.parametrize("cuts", [(2,), (1, 2, 3, 5, 8, 13, 21, 34), (16, 16, 16, 16), (19, 19, 19, 19), (18, 2, 17, 2, 40), (2,) * 40])
def test_portions_and_decoding_equal_the_whole(mixed, cuts):
    cfg, sd, path = mixed
    toks = M.tokens(101, cfg["vocab"], 8)
    want = O.forward(sd, cfg, toks)
    got = M.replay(M.engine(path), {"a": toks}, M.alone("a", toks, *cuts))["a"]
    assert M.row_error(got, want).max() < TOL


SEQS = [("a", 70), ("b", 9), ("c", 40), ("d", 23), ("e", 66), ("f", 31)]
STEPS = [[("a", 30), ("b", 8)], [("c", 5), ("a", 2), ("b", 1)], [("d", 20)], [("a", 1), ("d", 1), ("c", 33)], [("a", 37), ("d", 2), ("c", 2)],
         [("e", 50), ("f", 2)], [("f", 28), ("e", 1)], [("e", 15), ("f", 1)]]


@pytest.mark.parametrize("block_size", [4, 16, 64])
def test_unequal_batches_blocks_and_slots_used_again(mixed, block_size):
    """Four live requests of unequal length, portions beside single tokens, requests left out of steps; blocks and state slots
    are just enough for the live ones, so later requests get what earlier ones gave back."""
    cfg, sd, path = mixed
    seqs = {n: M.tokens(c, cfg["vocab"], 20 + i) for i, (n, c) in enumerate(SEQS)}
    room = sum(-(-n // block_size) for n in (70, 40, 23, 9))
    eng = M.engine(path, block_size=block_size, blocks=room + 1, num_state_slots=3)
    for t in (t for run in eng.worker.state_caches for t in run):
        t.fill_(1e4)                                             # a state that is taken over shows
    got = M.replay(eng, seqs, STEPS)
    for n, toks in seqs.items():
        assert M.row_error(got[n], O.forward(sd, cfg, toks)).max() < TOL, n


def test_odd_sizes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 2)
    toks = M.tokens(40, cfg["vocab"], 9)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 13, 9))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


@pytest.mark.parametrize("layers", ["memory", "parallel"])
def test_models_of_one_kind_of_layer(tmp_path, layers):
    """No attention at all (the paged cache holds nothing), and attention in every layer."""
    one = M.memory() if layers == "memory" else M.parallel()
    cfg = M.config([(one, M.moe()), (one, None)])
    sd = M.weights(cfg, 3)
    toks = M.tokens(50, cfg["vocab"], 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 20, 7))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


def test_long_decoding(tmp_path):
    cfg = M.config([(M.parallel(window=48), M.moe()), (M.memory(), None)], width=40, vocab=97)
    sd = M.weights(cfg, 3)
    toks = M.tokens(300, 97, 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 3))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


# Every mechanism shows in the logits of these models: an oracle with one planted mistake is far from the right one.
def _shift(x):
    return torch.cat([torch.zeros_like(x[:1]), x[:-1]])


MISTAKES = {
    "window one longer": ("visible_matrix", lambda f: lambda n, s: f(n, s + 1)),
    "window one shorter": ("visible_matrix", lambda f: lambda n, s: f(n, max(1, s - 1))),
    "no window": ("visible_matrix", lambda f: lambda n, s: f(n, 1 << 20)),
    "sink left out": ("softmax_with_sink", lambda f: lambda s, sink: torch.softmax(s, -1)),
    "heads not mixed": ("mix_scores", lambda f: lambda s, temp, talk: s * temp[:, None, None]),
    "mixed the other way": ("mix_scores", lambda f: lambda s, temp, talk: f(s, temp, talk.T)),
    "factor behind the mix": ("mix_scores", lambda f: lambda s, temp, talk: f(s, temp * 0 + 1, talk) * temp[:, None, None]),
    "no factor": ("mix_scores", lambda f: lambda s, temp, talk: f(s, temp * 0 + 1, talk)),
    "no rotation": ("rotate", lambda f: lambda x, rot: x),
    "positions one late": ("rotate", lambda f: lambda x, rot: x if not rot else f(torch.cat([x[:1], x]), rot)[1:] if x.shape[1] != 3 else f(x, rot)),
    "rotation not scaled": ("frequencies", lambda f: lambda rot: f({**rot, "scaling": None})),
    "convolutions one late": ("causal_conv", lambda f: lambda x, w: f(_shift(x), w)),
    "convolutions without the past": ("causal_conv", lambda f: lambda x, w: x * w[:, -1]),
    "embedding not normed": ("embed", lambda f: lambda sd, t, eps: sd["embed"][torch.as_tensor(t)]),
    "root of the decay": ("channel_decay", lambda f: lambda z, tau: f(z, 1.0)),
    "decay of the next token": ("channel_decay", lambda f: lambda z, tau: torch.roll(f(z, tau), 1, 0)),
    "output ahead of the update": ("gated_linear_core", lambda f: lambda q, k, v, a: f(q, k, v, a) - (q * k).sum(-1, keepdim=True) * v),
    "memory without input gates": ("matrix_memory_core", lambda f: lambda q, k, v, i, g: f(q, k, v, i * 0, g)),
    "memory without forgetting": ("matrix_memory_core", lambda f: lambda q, k, v, i, g: f(q, k, v, i, g * 0)),
    "gates not bounded": ("soft_bound", lambda f: lambda z, cap: z),
    "memory gate is silu": ("sigmoid", lambda f: lambda z: z * f(z)),
    "plain relu": ("squared_relu", lambda f: lambda z: z.clamp(min=0)),
    "experts weighted alike": ("route", lambda f: lambda l, top: (f(l, top)[0], torch.ones(top, dtype=l.dtype) / top)),
    "one expert less": ("route", lambda f: lambda l, top: f(l, max(1, top - 1))),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_a_planted_mistake_would_show(mixed, name, monkeypatch):
    cfg, sd, _ = mixed
    toks = M.tokens(60, cfg["vocab"], 11)
    right = O.forward(sd, cfg, toks)
    attr, wrap = MISTAKES[name]
    monkeypatch.setattr(O, attr, wrap(getattr(O, attr)))
    assert M.row_error(O.forward(sd, cfg, toks), right).max() > 20 * TOL


def test_far_tokens_show_through_the_states(tmp_path):
    """One token far back, behind every window: other values of it move the last logits, in a prompt and in decoding."""
    cfg = M.config([(M.parallel(window=5, tau=30.0), M.moe()), (M.memory(), None)], vocab=60)
    sd = M.weights(cfg, 12)
    for place in (0, 1, 30):
        toks = M.tokens(64, 60, 13)
        other = list(toks)
        other[place] = (toks[place] + 17) % 60
        path = M.save(cfg, sd, tmp_path / str(place))
        a, b = (M.replay(M.engine(path), {"a": t}, M.alone("a", t, 40))["a"] for t in (toks, other))
        assert M.row_error(a[63:], b[63:]).max() > 5 * TOL
        assert M.row_error(b, O.forward(f64(sd), cfg, other)).max() < TOL


# ----------------------------------------------------------------------------- generation
@pytest.mark.parametrize("kw", [{}, dict(max_tokens_per_batch=24, max_tokens_per_chunk_for_prefill=7), dict(enable_prefix_cache=True),
                                dict(enable_schedule_overlap=True), dict(use_mix_scheduler=True), dict(blocks=16), dict(num_state_slots=2),
                                dict(num_state_slots=1, enable_schedule_overlap=True)])
def test_greedy_generation(mixed, kw):
    """LLM.generate through the scheduler: chunked prefill, overlap, preemption (few blocks), fewer state slots than requests; a
    prefix cache that is asked for stays off, since a cached prefix has no state to go on from."""
    cfg, sd, path = mixed
    prompts = [M.tokens(n, cfg["vocab"], 30 + n) for n in (5, 33, 18, 41)]
    prompts.append(prompts[3][:32] + [7, 9])
    eng = M.engine(path, **kw)
    llm = LLM(model=path, devices="cpu", engine=eng)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == O.greedy(sd, cfg, p, 8)
    assert not eng.opt.enable_prefix_cache
    eng.step()
    assert eng.scheduler.num_free_state_slots == eng.worker.num_state_slots


def test_sleep_and_wakeup(mixed):
    cfg, sd, path = mixed
    eng = M.engine(path)
    llm = LLM(model=path, devices="cpu", engine=eng)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    for level in (1, 2):
        assert eng.sleep(level) and eng.worker.state_caches == [] and eng.wakeup()
        assert llm.generate([[1, 2, 3]], sp)[0].outputs[0].token_ids == O.greedy(sd, cfg, [1, 2, 3], 6)


def test_presets_are_described():
    for name in ("govuvik-30b-a3b",):
        a = preset(name)
        assert a.model_type == "govuvik" and len(a.layer_runs) == a.n_layers == len(a.layer_specs)
        assert len(get_model_class("govuvik").tensor_shapes(a)) > 48


# ----------------------------------------------------------------------------- the replay program
def test_trace_run_program(mixed, tmp_path):
    cfg, sd, path = mixed
    seqs = {"x": M.tokens(30, cfg["vocab"], 40), "y": M.tokens(12, cfg["vocab"], 41)}
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": seqs["x"][:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": seqs["x"][20:21], "want": []}, {"id": "y", "tokens": seqs["y"], "want": [11, 3]}],
              "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": seqs["x"][21:22], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "x", "tokens": seqs["x"][22:], "want": [7]}], "end": ["x"]}]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out",
                        str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    X, Y = O.forward(sd, cfg, seqs["x"]), O.forward(sd, cfg, seqs["y"])
    for step, want in ((0, X[[0, 19]]), (1, Y[[11, 3]]), (3, X[[29]])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{step}.f32", "<f4").reshape(len(want), -1))
        assert M.row_error(got, want).max() < TOL
