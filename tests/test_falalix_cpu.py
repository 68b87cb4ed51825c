"""Falalix on the CPU path in fp32: configuration, each mechanism against the plain statement of tests/oracle_falalix.py, whole
models through the engine (portions, decoding, batches, blocks and state slots used again), greedy generation, the replay
program; and the scheduler's state slots."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import oracle_falalix as O
from tests.helpers import falalix_models as M
from tests.helpers.portions import CUTS, RAG, Ragged, rag
from xllm_wxh_b200 import LLM, SamplingParams, _core, ops
from xllm_wxh_b200.config import Options
from xllm_wxh_b200.models.args import args_from_hf_config, preset
from xllm_wxh_b200.models.layer_spec import ParallelSpec, SelectiveScanSpec, pass_starts
from xllm_wxh_b200.models.registry import get_model_class

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 2e-5


def f64(sd):
    return {k: v.double() for k, v in sd.items()}


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    cfg = M.mixed_config()
    sd = M.weights(cfg, 1)
    return cfg, f64(sd), M.save(cfg, sd, tmp_path_factory.mktemp("falalix"))


# ----------------------------------------------------------------------------- configuration
def test_config_reader_takes_everything_from_the_file():
    a = args_from_hf_config(M.mixed_config(width=88, vocab=301))
    assert (a.model_type, a.hidden_size, a.vocab_size, a.rms_norm_eps, a.residual_mult) == ("falalix", 88, 301, 3e-6, 0.6)
    assert a.layer_runs == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and a.pass_starts == [1, 4, 7]
    s, p = a.layer_specs[2].mixer, a.layer_specs[3].mixer
    assert isinstance(s, SelectiveScanSpec) and (s.inner, s.state, s.conv, s.dt_rank) == (88, 20, 3, 8)
    assert isinstance(p, ParallelSpec) and (p.left_scale, p.right_scale) == (1.3, 0.4)
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.window, p.left.keep_first) == (6, 3, 40, 56, 33, 2)
    assert (p.right.heads, p.right.dim) == (2, 48)
    assert a.layer_specs[0].mlp is None and a.layer_specs[1].mlp.ff == 80 and a.layer_specs[1].mlp.act == "relu2"
    model = get_model_class("falalix")(a)
    kv, st = model.kv_cache_shapes(5, 16), model.state_cache_shapes(4)
    assert len(kv) == len(st) == 11
    assert kv[0] == () and kv[3] == kv[6] == ((5, 16, 3, 40), (5, 16, 3, 56))
    assert st[2] == (((4, 88, 20), torch.float32), ((4, 2, 88), torch.bfloat16))
    assert st[3] == (((4, 2, 48, 48), torch.float32), ((4, 88), torch.bfloat16))


def test_config_reader_rejects_what_it_does_not_know():
    for edit in (lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][1]["mlp"].update(kind="moe"),
                 lambda c: c["layers"][1]["mixer"]["left"].update(heads=5), lambda c: c["loop"].update(stop=9),
                 lambda c: c["layers"][0]["mixer"].update(state=0)):
        cfg = copy.deepcopy(M.mixed_config())
        edit(cfg)
        with pytest.raises(ValueError):
            args_from_hf_config(cfg)


def test_pass_starts():
    assert pass_starts(4) == [] and pass_starts(4, 2, 2, 5) == []
    assert pass_starts(4, 0, 4, 2) == [0, 4] and pass_starts(6, 2, 3, 3) == [2, 3, 4]


def test_loading_checks_names_and_shapes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 0)
    for i, (name, edit) in enumerate([("l0.mix.right.mu.w", lambda d: d.pop("l0.mix.right.mu.w")), ("loop.step", lambda d: d.pop("loop.step")),
                                      ("l1.mix.x", lambda d: d.update({"l1.mix.x": sd["l1.mix.x"][:-1]})),
                                      ("l0.mix.right.w1", lambda d: d.update({"l0.mix.right.w1": sd["l0.mix.right.w1"][:-1]}))]):
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
@pytest.mark.parametrize("cuts", CUTS)
def test_token_shift(cuts):
    g = torch.Generator().manual_seed(0)
    W = 10
    h, mu = [torch.randn(n, W, generator=g) for n in RAG], torch.rand(5, W, generator=g)
    last = torch.full((6, W), 1e3)                                # what earlier owners of the slots left behind
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.token_shift(rag(h, rows), mu, last, q, kv, sl, n)
        for j in range(5):
            assert torch.allclose(got[j], rag([O.token_mix(x, mu[j]) for x in h], rows), atol=1e-6)


@pytest.mark.parametrize("cuts", CUTS)
def test_time_mix(cuts):
    g = torch.Generator().manual_seed(1)
    H, d, eps = 2, 6, 1e-4
    r, k, v, z, gate = ([torch.randn(n, H * d, generator=g) for n in RAG] for _ in range(5))
    w0, u, nw = torch.randn(H * d, generator=g) - 2, torch.randn(H, d, generator=g), torch.randn(H * d, generator=g)
    want = []
    for i in range(3):
        w = torch.exp(-torch.exp(z[i] + w0)).view(-1, H, d)
        o = O.time_mix_core(*(x[i].view(-1, H, d) for x in (r, k, v)), w, u)
        want.append(0.3 * (o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)).flatten(1) * nw * O.silu(gate[i]))
    state = torch.full((6, H, d, d), 1e3)
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        out = torch.empty(int(q[-1]), H * d)
        ops.ref.time_mix(*(rag(x, rows) for x in (r, k, v, z)), w0, u, rag(gate, rows), nw, 0.3, eps, state, q, kv, sl, n, out)
        assert torch.allclose(out, rag(want, rows), atol=1e-4)


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("cuts", CUTS)
def test_conv(cuts, taps):
    g = torch.Generator().manual_seed(2)
    C = 9
    x, w, b = [torch.randn(n, C, generator=g) for n in RAG], torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    state = torch.full((6, taps - 1, C), 1e3)
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.conv_silu(rag(x, rows), w.t(), b, state, q, kv, sl, n)
        assert torch.allclose(got, rag([O.silu(O.causal_conv(s, w, b)) for s in x], rows), atol=1e-5)


@pytest.mark.parametrize("cuts", CUTS)
def test_selective_scan(cuts):
    g = torch.Generator().manual_seed(3)
    C, N = 7, 5
    x, dt, z = ([torch.randn(n, C, generator=g) for n in RAG] for _ in range(3))
    B, Cm = ([torch.randn(n, N, generator=g) for n in RAG] for _ in range(2))
    A, D, bias = -torch.rand(C, N, generator=g) * 2, torch.randn(C, generator=g), torch.randn(C, generator=g) - 2
    want = [O.scan_core(x[i], O.softplus(dt[i] + bias), A, B[i], Cm[i], D) * O.silu(z[i]) for i in range(3)]
    state = torch.full((6, C, N), 1e3)
    for q, kv, sl, n, rows in Ragged().steps(RAG, cuts):
        got = ops.ref.selective_scan(*(rag(t, rows) for t in (x, dt)), bias, A, rag(B, rows), rag(Cm, rows), D, rag(z, rows), state, q, kv, sl, n)
        assert torch.allclose(got, rag(want, rows), atol=1e-4)


def test_window_with_kept_first_keys():
    """Rows of the visibility: the kept keys, then a gap, then the window that ends at the query."""
    see = O.visible_matrix(12, 3, 2)
    assert see[9].nonzero().flatten().tolist() == [0, 1, 7, 8, 9] and see[2].nonzero().flatten().tolist() == [0, 1, 2]
    assert all(bool(see[i, j]) == O.visible(i, j, 3, 2) for i in range(12) for j in range(12))
    g = torch.Generator().manual_seed(4)
    n, H, G, d, dv = 40, 4, 2, 8, 6
    for size, keep in ((3, 2), (1, 0), (7, 30), (64, 5), (16, 16)):
        q, k, v = torch.randn(n, H, d, generator=g), torch.randn(n, G, d, generator=g), torch.randn(n, G, dv, generator=g)
        bt = torch.tensor([[2, 1, 3]]).int()
        kc, vc = torch.zeros(4, 16, G, d), torch.zeros(4, 16, G, dv)
        for t in range(n):
            kc[bt[0, t // 16], t % 16], vc[bt[0, t // 16], t % 16] = k[t], v[t]
        want = O.attention_core(q, k, v, 0.5, size, keep).flatten(1)
        for m in (n, 1, 2, 17):
            got = ops.ref.paged_attention(q[n - m:], kc, vc, torch.tensor([0, m]), torch.tensor([n]), bt, 1, 0.5, size, 0, None, None, keep)
            assert torch.allclose(got, want[n - m:], atol=1e-5)


def test_norms_and_gate():
    g = torch.Generator().manual_seed(5)
    T, H, G, d, dv = 6, 4, 2, 10, 7
    qkv = torch.randn(T, (H + G) * d + G * dv + 5, generator=g) * 1e-2           # small rows: eps matters
    qw, kw = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    kc, vc = torch.zeros(4, 4, G, d), torch.zeros(4, 4, G, dv)
    slots = torch.tensor([5, 6, 7, 12, 13, 14]).int()
    q = ops.qknorm_all_kvwrite(qkv.clone(), slots, qw, kw, 1e-4, kc, vc, H, G)
    a, b, c, _ = qkv.split([H * d, G * d, G * dv, 5], -1)
    assert torch.allclose(q, O.rms_norm(a, qw, 1e-4), atol=1e-6)
    assert torch.allclose(kc.view(-1, G * d)[slots.long()], O.rms_norm(b, kw, 1e-4), atol=1e-6)
    assert torch.equal(vc.view(-1, G * dv)[slots.long()], c)
    x, y, wn = torch.randn(T, 24, generator=g), torch.randn(T, 24, generator=g), torch.randn(24, generator=g)
    got = x.clone()
    h = ops.add_norm(y, got, 0.3, wn, 1e-5)
    assert torch.allclose(got, x + 0.3 * y, atol=1e-6) and torch.allclose(h, O.rms_norm(x + 0.3 * y, wn, 1e-5), atol=1e-5)
    step = torch.randn(24, generator=g)
    h = ops.replace_norm(y, step, got, wn, 1e-5)
    assert torch.allclose(got, y + step) and torch.allclose(h, O.rms_norm(y + step, wn, 1e-5), atol=1e-5)
    out = torch.zeros(T, 30)
    ops.gate_into(y, x, 1.7, out[:, 3:27])
    assert torch.allclose(out[:, 3:27], 1.7 * y * O.sigmoid(x), atol=1e-6) and out[:, :3].abs().sum() == 0


def test_product_of_the_residual_keeps_more_than_16_bits():
    g = torch.Generator().manual_seed(6)
    W = 64
    table, w = torch.randn(9, W, generator=g).bfloat16(), (torch.randn(40, 2 * W, generator=g) / 8).bfloat16()
    x, ids = torch.randn(5, W, generator=g), torch.tensor([3, 0, 8, 3, 1]).int()
    want = torch.cat([x.double(), table[ids.long()].double()], -1) @ w.double().T
    got = ops.linear_f32(ops.split_rows(x, ids, table, 1.0), ops.split_columns(w, W))
    assert (got.double() - want).abs().max() < 2e-4
    got = ops.linear_f32(ops.split_rows(x, ids, table.float(), 1.0), ops.split_columns(w.float(), W))
    assert (got.double() - want).abs().max() < 1e-5


def test_activations():
    x, w = torch.linspace(-9, 9, 60).reshape(6, 10), torch.eye(10)
    assert torch.allclose(ops.act_linear(x, w, "relu2"), O.squared_relu(x)) and torch.allclose(ops.act_linear(x, w, "tanh"), torch.tanh(x))


# ----------------------------------------------------------------------------- whole models through the engine
def test_layers_one_by_one(mixed):
    cfg, sd, path = mixed
    toks = M.tokens(45, cfg["vocab"], 7)
    want = []
    logits = O.forward(sd, cfg, toks, want)
    eng, got = M.engine(path), []
    eng.worker.model.residual_hook = lambda r, x: got.append(x.clone())
    out = M.replay(eng, {"a": toks}, [[("a", 45)]])["a"]
    assert len(got) == len(want) == 11
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


def test_replay_refuses_what_has_no_slot(mixed):
    cfg, _, path = mixed
    eng = M.engine(path, num_state_slots=2)
    a, b, c = (eng.add_request([]) for _ in range(3))
    eng.step_portions([(a, [1, 2], []), (b, [3], [])])
    with pytest.raises(RuntimeError, match="state slot"):
        eng.step_portions([(a, [1], []), (c, [3], [])])
    eng.cancel(b)
    assert len(eng.step_portions([(a, [1], [0]), (c, [3], [0])])) == 2
    assert eng.scheduler.num_free_state_slots == 0


def test_odd_sizes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 2)
    toks = M.tokens(40, cfg["vocab"], 9)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 13, 9))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


@pytest.mark.parametrize("layers", ["scan", "parallel"])
def test_models_of_one_kind_of_layer(tmp_path, layers):
    """No attention at all (the paged cache holds nothing), and attention in every layer; no loop."""
    one = M.scan() if layers == "scan" else M.parallel()
    cfg = M.config([(one, M.dense()), (one, None)])
    sd = M.weights(cfg, 3)
    toks = M.tokens(50, cfg["vocab"], 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 20, 7))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


def test_long_decoding(tmp_path):
    cfg = M.config([(M.parallel(window=48, keep_first=17), M.dense()), (M.scan(inner=24), None)], width=40, vocab=97)
    sd = M.weights(cfg, 3)
    toks = M.tokens(300, 97, 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 3))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


# Every mechanism shows in the logits of these models: an oracle with one planted mistake is far from the right one.
MISTAKES = {
    "window one longer": ("visible_matrix", lambda f: lambda n, s, k: f(n, s + 1, k)),
    "window one shorter": ("visible_matrix", lambda f: lambda n, s, k: f(n, max(1, s - 1), k)),
    "one more kept key": ("visible_matrix", lambda f: lambda n, s, k: f(n, s, k + 1)),
    "one kept key less": ("visible_matrix", lambda f: lambda n, s, k: f(n, s, k - 1)),
    "no window": ("visible_matrix", lambda f: lambda n, s, k: f(n, 1 << 20, k)),
    "no rows before": ("shifted", lambda f: lambda h: torch.zeros_like(h)),
    "own row as the one before": ("shifted", lambda f: lambda h: h),
    "no bonus": ("time_mix_core", lambda f: lambda r, k, v, w, u: f(r, k, v, w, u * 0)),
    "decay of the next token": ("decay", lambda f: lambda *a: torch.roll(f(*a), 1, 0)),
    "decay without its projection": ("decay", lambda f: lambda sd, p, m: torch.exp(-torch.exp(sd[p + "w0"])).expand(len(m), -1)),
    "convolution one late": ("causal_conv", lambda f: lambda x, w, b: f(O.shifted(x), w, b)),
    "step without bias": ("softplus", lambda f: lambda z: f(z + 1)),
    "no D": ("scan_core", lambda f: lambda x, dt, A, B, C, D: f(x, dt, A, B, C, D * 0)),
    "plain relu": ("squared_relu", lambda f: lambda z: z.clamp(min=0)),
    "gate is silu": ("sigmoid", lambda f: lambda z: z * f(z)),
    "loop run once": ("schedule", lambda f: lambda cfg: f({**cfg, "loop": {**cfg["loop"], "times": 1}})),
    "passes not entered": ("enter_pass", lambda f: lambda sd, x, x0, t: x),
    "step vector of the first pass": ("enter_pass", lambda f: lambda sd, x, x0, t: f(sd, x, x0, 0)),
    "pass without the embedding": ("enter_pass", lambda f: lambda sd, x, x0, t: f(sd, x, x0 * 0, t)),
    "keys not normed": ("project_qkv", lambda f: lambda sd, p, h, eps: (f(sd, p, h, eps)[0], h @ sd[p + "k"].T + sd[p + "k.b"],
                                                                        f(sd, p, h, eps)[2])),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_a_planted_mistake_would_show(mixed, name, monkeypatch):
    cfg, sd, _ = mixed
    toks = M.tokens(60, cfg["vocab"], 11)
    right = O.forward(sd, cfg, toks)
    attr, wrap = MISTAKES[name]
    monkeypatch.setattr(O, attr, wrap(getattr(O, attr)))
    assert M.row_error(O.forward(sd, cfg, toks), right).max() > 100 * TOL


def test_far_tokens_show_through_state_and_kept_keys(tmp_path):
    """One token far back, behind every window: other values of it move the last logits, in a prompt and in decoding."""
    cfg = M.config([(M.parallel(window=5, keep_first=2), M.dense()), (M.scan(), None)], vocab=60)
    sd = M.weights(cfg, 12)
    for place in (0, 1, 2, 30):
        toks = M.tokens(64, 60, 13)
        other = list(toks)
        other[place] = (toks[place] + 17) % 60
        path = M.save(cfg, sd, tmp_path / str(place))
        a, b = (M.replay(M.engine(path), {"a": t}, M.alone("a", t, 40))["a"] for t in (toks, other))
        assert M.row_error(a[63:], b[63:]).max() > 20 * TOL
        assert M.row_error(b, O.forward(f64(sd), cfg, other)).max() < TOL


# ----------------------------------------------------------------------------- generation
@pytest.mark.parametrize("kw", [{}, dict(max_tokens_per_batch=24, max_tokens_per_chunk_for_prefill=7), dict(enable_prefix_cache=True),
                                dict(enable_schedule_overlap=True), dict(use_mix_scheduler=True), dict(blocks=16), dict(num_state_slots=2),
                                dict(num_state_slots=1, enable_schedule_overlap=True), dict(num_state_slots=3, use_mix_scheduler=True),
                                dict(enable_chunked_prefill=False, num_state_slots=2)])
def test_greedy_generation(mixed, kw):
    """LLM.generate through the scheduler: chunked prefill, overlap, preemption (few blocks), fewer state slots than requests; a
    prefix cache that is asked for stays off, since a cached prefix has no state to go on from."""
    cfg, sd, path = mixed
    prompts = [M.tokens(n, cfg["vocab"], 30 + n) for n in (5, 33, 18, 41)]
    prompts.append(prompts[3][:32] + [7, 9])
    eng = M.engine(path, **kw)
    llm = LLM(model=path, devices="cpu", engine=eng)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == O.greedy(sd, cfg, p, 12)
    assert not eng.opt.enable_prefix_cache
    eng.step()
    assert eng.scheduler.num_free_state_slots == eng.worker.num_state_slots


def test_several_samples_of_a_prompt_and_beams(mixed):
    cfg, sd, path = mixed
    llm = LLM(model=path, devices="cpu", engine=M.engine(path, num_state_slots=3))
    sp = SamplingParams(temperature=0.9, n=4, seed=3, max_tokens=5, ignore_eos=True)
    a, b = ([s.token_ids for s in llm.generate([[1, 2, 3]], sp)[0].outputs] for _ in range(2))
    assert a == b and len(a) == 4 and len({tuple(x) for x in a}) > 1
    out = llm.generate([[4, 5, 6, 7]], SamplingParams(temperature=0.0, beam_width=3, max_tokens=3, ignore_eos=True))[0]
    assert len(out.outputs[0].token_ids) == 3


def test_refused_combinations(mixed, monkeypatch):
    _, _, path = mixed
    for kw in (dict(num_speculative_tokens=2), dict(enable_disagg_pd=True, instance_role="PREFILL")):
        with pytest.raises(ValueError):
            M.engine(path, **kw)
    so = _core.SchedulerOptions()
    so.num_state_slots = 2
    with pytest.raises(ValueError):
        _core.Scheduler(so, 8, 4, True, 0)


def test_sleep_and_wakeup(mixed):
    cfg, sd, path = mixed
    eng = M.engine(path)
    llm = LLM(model=path, devices="cpu", engine=eng)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    for level in (1, 2):
        assert eng.sleep(level) and eng.worker.state_caches == [] and eng.wakeup()
        assert llm.generate([[1, 2, 3]], sp)[0].outputs[0].token_ids == O.greedy(sd, cfg, [1, 2, 3], 6)


def test_preset_is_described():
    a = preset("falalix-8b")
    assert a.model_type == "falalix" and len(a.layer_runs) == a.n_layers == len(a.layer_specs)
    opts = Options(model="preset:falalix-8b")
    assert opts.num_state_slots == 0


# ----------------------------------------------------------------------------- the scheduler's state slots
def scheduler(slots, **kw):
    so = _core.SchedulerOptions()
    so.num_state_slots = slots
    for k, v in kw.items():
        setattr(so, k, v)
    return _core.Scheduler(so, 64, 4, False, 0)


def run_step(s):
    b = s.schedule()[0]
    L = _core.BatchLayout(256, 16, 64, 16, 32)
    buf = np.full(L.total_words, -7, dtype=np.int32)
    assert b.build(L, buf.ctypes.data, L.total_words, 4) == 0
    ids = [e[1] for e in b.entries()]
    got = dict(zip(ids, buf[L.state_slots:L.state_slots + len(ids)].tolist()))
    assert (buf[L.state_slots + len(ids):L.state_slots + 16] == 0).all()          # padding rows: slot 0
    if not b.empty:
        s.process_output(b.id, np.full(b.num_sample_rows, 5, dtype=np.int32), None)
    return got


def test_a_sequence_keeps_its_slot_and_gives_it_back():
    s = scheduler(2)
    stop = _core.StopCriteria()
    stop.max_tokens = 3
    a, b, c = (s.add_request(list(range(n)), _core.SamplingParams(), stop) for n in (5, 3, 4))
    first = run_step(s)
    assert sorted(first) == sorted([a, b]) and sorted(first.values()) == [1, 2] and s.num_free_state_slots == 0
    assert run_step(s) == first                                  # the third waits for a slot
    assert run_step(s) == first
    late = run_step(s)                                           # both are done
    assert list(late) == [c] and late[c] in (1, 2)
    s.cancel(c)
    run_step(s)
    assert s.num_free_state_slots == 2


def test_preemption_gives_the_slot_back():
    s = scheduler(4, max_tokens_per_batch=64)
    stop = _core.StopCriteria()
    stop.max_tokens = 100
    ids = [s.add_request(list(range(60)), _core.SamplingParams(), stop) for _ in range(4)]
    held = {}
    for _ in range(60):
        got = run_step(s)
        assert len(set(got.values())) == len(got) and 0 not in got.values()
        for i, slot in got.items():
            held.setdefault(i, set()).add(slot)
    assert len(held) == 4 and s.stats()["num_preemptions"] > 0
    for i in ids:
        s.cancel(i)
    s.schedule()
    assert s.num_free_state_slots == 4


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
    assert not os.path.exists(tmp_path / "o" / "2.f32")
