"""Movolorn on the CPU path in fp32: configuration, each mechanism against the plain statement of tests/oracle_movolorn.py,
whole models through the engine (portions, decoding, batches, blocks used again), greedy generation, the replay program."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import oracle_movolorn as O
from tests.helpers import movolorn_models as M
from xllm_wxh_b200 import LLM, SamplingParams, ops
from xllm_wxh_b200.models.args import args_from_hf_config, preset
from xllm_wxh_b200.models.layer_spec import run_order
from xllm_wxh_b200.models.registry import get_model_class

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 2e-5


def f64(sd):
    return {k: v.double() for k, v in sd.items()}


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    cfg = M.mixed_config()
    sd = M.weights(cfg, 1)
    return cfg, f64(sd), M.save(cfg, sd, tmp_path_factory.mktemp("movolorn"))


# ----------------------------------------------------------------------------- configuration
def test_config_reader_takes_everything_from_the_file():
    a = args_from_hf_config(M.mixed_config(width=88, vocab=301))
    assert (a.model_type, a.hidden_size, a.vocab_size, a.rms_norm_eps, a.embedding_scale) == ("movolorn", 88, 301, 3e-6, 1.7)
    assert a.layer_runs == [0, 1, 2, 1, 2, 1, 2, 3] and a.n_layers == 8
    m, f = a.layer_specs[1].mixer, a.layer_specs[1].mlp
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.chunk) == (6, 2, 40, 56, 19)
    assert (f.experts, f.identity_experts, f.top_k, f.n_group, f.topk_group, f.shared_ff) == (6, 2, 3, 4, 2, 64)
    assert a.layer_specs[2].mlp is None
    g = a.layer_specs[3].mlp
    assert (g.identity_experts, g.n_group, g.topk_group, g.shared_ff) == (0, 1, 1, 0)
    assert a.layer_specs[0].mlp.act == "gelu_tanh" and g.act == "silu"
    shapes = get_model_class("movolorn")(a).kv_cache_shapes(5, 16)
    assert len(shapes) == 8 and shapes[1] == ((5, 16, 2, 40), (5, 16, 2, 56)) == shapes[3]


def test_config_reader_rejects_what_it_does_not_know():
    for edit in (lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                 lambda c: c["layers"][0]["mixer"].update(heads=5), lambda c: c["loop"].update(stop=9),
                 lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3)):
        cfg = copy.deepcopy(M.mixed_config())
        edit(cfg)
        with pytest.raises(ValueError):
            args_from_hf_config(cfg)


def test_run_order():
    assert run_order(3) == [0, 1, 2]
    assert run_order(4, 0, 4, 2) == [0, 1, 2, 3, 0, 1, 2, 3]
    assert run_order(4, 2, 3, 3) == [0, 1, 2, 2, 2, 3]
    assert run_order(4, 2, 2, 5) == [0, 1, 2, 3]


def test_loading_checks_names_and_shapes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 0)
    bad = dict(sd)
    del bad["l1.mlp.e3.up"]
    with pytest.raises(ValueError, match="l1.mlp.e3.up"):
        M.engine(M.save(cfg, bad, tmp_path / "a"))
    bad = dict(sd, **{"l0.mix.k": sd["l0.mix.k"][:-1]})
    with pytest.raises(ValueError, match="l0.mix.k"):
        M.engine(M.save(cfg, bad, tmp_path / "b"))


def test_state_dict_round_trip(mixed):
    cfg, sd, path = mixed
    m = M.engine(path).worker.model
    got = m.state_dict()
    assert set(got) == set(sd)
    for k in sd:
        assert torch.equal(got[k].double(), sd[k]), k
    assert m.weight_bytes() > 0


# ----------------------------------------------------------------------------- mechanisms
def test_embedding_scale_and_norm():
    g = torch.Generator().manual_seed(0)
    table, w = torch.randn(11, 20, generator=g), torch.randn(20, generator=g)
    ids = torch.tensor([3, 0, 10, 3], dtype=torch.int32)
    x, h = ops.embed_rms_norm(ids, table, 2.5, w, 1e-3)
    want = O.embed({"embed": table}, {"embedding": {"scale": 2.5}}, ids.tolist())
    assert torch.allclose(x, want) and x.dtype == torch.float32
    assert torch.allclose(h, O.rms_norm(want, w, 1e-3), atol=1e-6)


def test_norm_before_and_after_with_eps_inside_the_root():
    g = torch.Generator().manual_seed(1)
    x, y = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g) * 1e-3      # small rows: eps matters
    wp, wn = torch.randn(24, generator=g), torch.randn(24, generator=g)
    want_x = x + O.rms_norm(y, wp, 1e-5)
    got = x.clone()
    h = ops.post_norm_add_norm(y, got, wp, wn, 1e-5)
    assert torch.allclose(got, want_x, atol=1e-6) and torch.allclose(h, O.rms_norm(want_x, wn, 1e-5), atol=1e-6)


def test_qk_norm_and_cache_write():
    g = torch.Generator().manual_seed(2)
    T, H, G, d, dv = 6, 4, 2, 10, 7
    qkv = torch.randn(T, (H + G) * d + G * dv, generator=g)
    qw, kw = torch.randn(d, generator=g), torch.randn(d, generator=g)
    kc, vc = torch.zeros(4, 4, G, d), torch.zeros(4, 4, G, dv)
    slots = torch.tensor([5, 6, 7, 12, 13, 14], dtype=torch.int32)
    q = ops.qknorm_kvwrite(qkv.clone(), slots, qw, kw, 1e-6, kc, vc, H, G)
    a, b, c = qkv.split([H * d, G * d, G * dv], -1)
    assert torch.allclose(q.view(T, H, d), O.rms_norm(a.view(T, H, d), qw, 1e-6), atol=1e-6)
    assert torch.allclose(kc.view(-1, G, d)[slots.long()], O.rms_norm(b.view(T, G, d), kw, 1e-6), atol=1e-6)
    assert torch.equal(vc.view(-1, G, dv)[slots.long()], c.view(T, G, dv))
    assert kc.view(-1, G, d)[0].abs().sum() == 0


def test_gate_activations():
    x = torch.linspace(-9, 9, 60).reshape(3, 20)
    for act, f in (("silu", O.silu), ("gelu_tanh", O.gelu_tanh)):
        assert torch.allclose(ops.ref.gated_act(x, act), f(x[:, :10]) * x[:, 10:], atol=1e-5)


@pytest.mark.parametrize("groups", [None, (4, 2), (2, 1), (6, 6)])
def test_router(groups):
    g = torch.Generator().manual_seed(3)
    z = torch.randn(64, 12, generator=g) * 1.5
    corr = torch.randn(12, generator=g) * 0.5 - 1.0                # choice scores of both signs
    r = {"top": 3}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    n, k = groups or (1, 1)
    w, ids = ops.moe_router(z, 3, "softmax", False, corr, n, k, 1.0, "max")
    for t in range(64):
        want = O.route(z[t].double(), corr.double(), r)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double(), torch.stack([x for _, x in want]), atol=1e-6)


def test_mixture_with_identity_and_shared_experts():
    cfg = M.config([(M.attn(), M.moe())])
    sd = {k: v.float() for k, v in M.weights(cfg, 4).items()}
    mlp, p = cfg["layers"][0]["mlp"], "l0.mlp."
    h = torch.randn(20, cfg["width"], generator=torch.Generator().manual_seed(5))
    w, ids = ops.moe_router(ops.linear_f32(h, sd[p + "router"]), 3, "softmax", False, sd[p + "correction"], 4, 2, 1.0, "max")
    assert (ids >= 6).any() and (ids < 6).any()
    w13 = torch.stack([torch.cat([sd[f"{p}e{e}.gate"], sd[f"{p}e{e}.up"]]) for e in range(6)])
    w2 = torch.stack([sd[f"{p}e{e}.down"] for e in range(6)])
    shared = O.gated_ff(sd, p + "shared.", h, O.silu)
    x = torch.randn(20, cfg["width"], generator=torch.Generator().manual_seed(6))
    want = x + O.rms_norm(O.moe(sd, p, mlp, h), sd["l0.norm2b"], 1e-6)
    out = ops.moe_post_norm_add_norm(h, w13, w2, w, ids, shared, 6, x, sd["l0.norm2b"], sd["final.norm"], 1e-6)
    assert torch.allclose(x, want, atol=1e-4) and torch.allclose(out, O.rms_norm(want, sd["final.norm"], 1e-6), atol=1e-4)


# ----------------------------------------------------------------------------- whole models through the engine
def test_layers_one_by_one(mixed):
    cfg, sd, path = mixed
    toks = M.tokens(45, cfg["vocab"], 7)
    want = []
    logits = O.forward(sd, cfg, toks, want)
    eng, got = M.engine(path), []
    eng.worker.model.residual_hook = lambda r, x: got.append(x.clone())
    out = M.replay(eng, {"a": toks}, [[("a", 45)]])["a"]
    assert len(got) == len(want) == 8
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


@pytest.mark.parametrize("block_size", [4, 16, 64])
def test_unequal_batches_and_blocks_used_again(mixed, block_size):
    """Four live requests of unequal length, portions beside single tokens, requests left out of steps; the cache holds
    little more than the live ones, so later requests get blocks that earlier ones gave back."""
    cfg, sd, path = mixed
    seqs = {n: M.tokens(c, cfg["vocab"], 20 + i) for i, (n, c) in enumerate([("a", 70), ("b", 9), ("c", 40), ("d", 23), ("e", 66), ("f", 31)])}
    steps = [[("a", 30), ("b", 8)], [("c", 5), ("a", 2), ("b", 1)], [("d", 20)], [("a", 1), ("d", 1), ("c", 33)], [("a", 37), ("d", 2), ("c", 2)],
             [("e", 50), ("f", 2)], [("f", 28), ("e", 1)], [("e", 15), ("f", 1)]]
    room = sum(-(-n // block_size) for n in (70, 40, 23, 9))
    eng = M.engine(path, block_size=block_size, blocks=room + 1)
    got = M.replay(eng, seqs, steps)
    for n, toks in seqs.items():
        assert M.row_error(got[n], O.forward(sd, cfg, toks)).max() < TOL, n


def test_replay_refuses_what_does_not_fit(mixed):
    cfg, sd, path = mixed
    eng = M.engine(path, block_size=16, blocks=4)
    r = eng.add_request([])
    eng.step_portions([(r, M.tokens(40, cfg["vocab"], 1), [])])
    with pytest.raises(RuntimeError, match="no room"):
        eng.step_portions([(r, M.tokens(10, cfg["vocab"], 2), [])])
    with pytest.raises(RuntimeError, match="wanted place"):
        eng.step_portions([(r, [1, 2], [2])])
    with pytest.raises(RuntimeError, match="unknown"):
        eng.step_portions([(r + 5, [1], [])])
    out = eng.step_portions([(r, [1, 2], [1])])
    assert out[0].shape == (1, cfg["vocab"])


def test_odd_sizes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 2)
    toks = M.tokens(40, cfg["vocab"], 9)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 13, 9))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


def test_long_decoding(tmp_path):
    cfg = M.config([(M.attn(chunk=48), M.dense()), (M.attn(heads=2, kv_heads=1, chunk=90), M.moe())], width=40, vocab=97)
    sd = M.weights(cfg, 3)
    toks = M.tokens(300, 97, 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 3))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


# Every mechanism shows in the logits of these models: an oracle with one planted mistake is far from the right one.
MISTAKES = {
    "chunk one longer": ("visible_matrix", lambda f: lambda n, c: f(n, c + 1)),
    "no chunks": ("visible_matrix", lambda f: lambda n, c: f(n, 1 << 20)),
    "no sink": ("softmax_plus_one", lambda f: lambda s: torch.softmax(s, -1)),
    "no distance bias": ("distance_bias", lambda f: lambda n, s, d: f(n, s, d) * 0),
    "slopes of the next head": ("head_slope", lambda f: lambda h, H: f(h + 1, H)),
    "weight of the choice score": ("route", lambda f: lambda z, c, r: [(e, w + c[e]) for e, w in f(z, c, r)]),
    "silu for gelu": ("gelu_tanh", lambda f: O.silu),
    "loop run once": ("layer_order", lambda f: lambda cfg: list(range(len(cfg["layers"])))),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_a_planted_mistake_would_show(mixed, name, monkeypatch):
    cfg, sd, _ = mixed
    toks = M.tokens(60, cfg["vocab"], 11)
    right = O.forward(sd, cfg, toks)
    attr, wrap = MISTAKES[name]
    monkeypatch.setattr(O, attr, wrap(getattr(O, attr)))
    assert M.row_error(O.forward(sd, cfg, toks), right).max() > 100 * TOL


# ----------------------------------------------------------------------------- generation
@pytest.mark.parametrize("kw", [{}, dict(max_tokens_per_batch=24, max_tokens_per_chunk_for_prefill=7), dict(enable_prefix_cache=True),
                                dict(enable_schedule_overlap=True), dict(use_mix_scheduler=True), dict(blocks=16)])
def test_greedy_generation(mixed, kw):
    """LLM.generate through the scheduler: chunked prefill, prefix cache, overlap, preemption (few blocks)."""
    cfg, sd, path = mixed
    prompts = [M.tokens(n, cfg["vocab"], 30 + n) for n in (5, 33, 18, 41)]
    prompts.append(prompts[3][:32] + [7, 9])                    # shares two blocks with another prompt
    llm = LLM(model=path, devices="cpu", engine=M.engine(path, **kw))
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == O.greedy(sd, cfg, p, 12)


def test_sampling_and_embedding(mixed):
    cfg, _, path = mixed
    llm = LLM(model=path, devices="cpu", engine=M.engine(path))
    sp = SamplingParams(temperature=0.8, top_k=20, seed=5, max_tokens=6, ignore_eos=True, logprobs=True, top_logprobs=2)
    a, b = (llm.generate([[1, 2, 3]], sp)[0].outputs[0].token_ids for _ in range(2))
    assert a == b and len(a) == 6


def test_presets_are_described():
    for name in ("movolorn-8b", "movolorn-30b-a3b"):
        a = preset(name)
        assert a.model_type == "movolorn" and len(a.layer_runs) == a.n_layers == len(a.layer_specs)


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
