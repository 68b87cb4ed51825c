"""Babadra on the CPU path in fp32: configuration, each mechanism against the plain statement of tests/oracle_babadra.py, whole
models through the engine (portions, decoding, batches, blocks used again), greedy generation, the replay program."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import oracle_babadra as O
from tests.helpers import babadra_models as M
from tests.helpers.paged_step import PagedStep
from xllm_wxh_b200 import LLM, SamplingParams, ops
from xllm_wxh_b200.models.args import args_from_hf_config, preset
from xllm_wxh_b200.models.layer_spec import LatentAttentionSpec, RotarySpec
from xllm_wxh_b200.models.registry import get_model_class

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 2e-5


def f64(sd):
    return {k: v.double() for k, v in sd.items()}


def gen(seed):
    return torch.Generator().manual_seed(seed)


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    cfg = M.mixed_config()
    sd = M.weights(cfg, 1)
    return cfg, f64(sd), M.save(cfg, sd, tmp_path_factory.mktemp("babadra"))


# ----------------------------------------------------------------------------- configuration
def test_config_reader_takes_everything_from_the_file():
    a = args_from_hf_config(M.mixed_config(width=88, vocab=301))
    assert (a.model_type, a.hidden_size, a.vocab_size, a.rms_norm_eps, a.embedding_scale) == ("babadra", 88, 301, 3e-5, 1.7)
    assert (a.position_rows, a.max_position_embeddings, a.logit_softcap) == (512, 512, 6.0)
    assert a.layer_runs == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and a.n_layers == 11 and a.pass_starts == [1, 4, 7]
    two, lat, plain = a.layer_specs[0].mixer, a.layer_specs[1].mixer, a.layer_specs[3].mixer
    assert (two.heads, two.kv_heads, two.dim, two.vdim, two.maps, two.diff, two.softcap) == (4, 2, 32, 40, 2, 0.35, 9.0)
    assert two.rot == RotarySpec(16, 5000.0) and plain.rot == RotarySpec(8, 9000.0, True)
    assert (lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank, lat.q_rank, lat.row) == (4, 24, 16, 40, 48, 56, 64)
    assert lat.rot == RotarySpec(16, 9000.0, True, 3.0, 96.0, 8.0, 1.5)
    e, d = a.layer_specs[3].mlp, a.layer_specs[1].mlp
    assert (e.ff, e.experts, e.top_k, e.limit, e.scoring) == (32, 5, 2, 1.9, "softmax_chosen") and (d.ff, d.limit, d.is_moe) == (80, 1.1, False)
    assert a.layer_specs[2].mlp is None
    shapes = get_model_class("babadra")(a).kv_cache_shapes(5, 16)
    assert len(shapes) == 11 and shapes[0] == ((5, 16, 4, 32), (5, 16, 2, 40)) and shapes[1] == ((5, 16, 64),) == shapes[4]
    odd = args_from_hf_config(M.odd_config())
    assert odd.logit_softcap == 0 and odd.layer_specs[1].mixer.softcap == 0 and odd.pass_starts == [0, 3]


def test_config_reader_rejects_what_it_does_not_know():
    for edit in (lambda c: c["layers"][0].update(type="recurrent"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                 lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["loop"].update(stop=9),
                 lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14),
                 lambda c: c["layers"][0]["mlp"]["router"].update(top=7), lambda c: c["layers"][1]["mixer"].update(kv_rank=0)):
        cfg = copy.deepcopy(M.mixed_config())
        edit(cfg)
        with pytest.raises(ValueError):
            args_from_hf_config(cfg)


def test_loading_checks_names_and_shapes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 0)
    bad = dict(sd)
    del bad["l0.mlp.e3.up"]
    with pytest.raises(ValueError, match="l0.mlp.e3.up"):
        M.engine(M.save(cfg, bad, tmp_path / "a"))
    for name in ("pos", "l0.mix.dkv", "l1.mix.k", "l1.ls2"):
        bad = dict(sd, **{name: sd[name][:-1]})
        with pytest.raises(ValueError, match=name):
            M.engine(M.save(cfg, bad, tmp_path / name))


def test_state_dict_round_trip(mixed):
    cfg, sd, path = mixed
    m = M.engine(path).worker.model
    got = m.state_dict()
    assert set(got) == set(sd)
    for k in sd:
        assert torch.equal(got[k].double(), sd[k]), k
    assert m.weight_bytes() > 0


# ----------------------------------------------------------------------------- mechanisms
ROTATIONS = [(16, 100.0, None), (24, 1e6, None), (32, 9000.0, (3.0, 96, 8.0, 1.5)), (12, 500.0, (0.5, 40, 4.0, 1.0)),
             (8, 50.0, (4.0, 1e9, 2.0, 1.9)), (10, 1e4, (2.0, 30, 6.0, 1.0)), (2, 77.0, None), (64, 1e5, (40.0, 4096, 32.0, 1.0))]


@pytest.mark.parametrize("dims,base,scaling", ROTATIONS)
@pytest.mark.parametrize("interleaved", [False, True])
def test_rotation(dims, base, scaling, interleaved):
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    spec = RotarySpec(dims, base, interleaved, *(scaling or ()))
    x = torch.randn(70, 3, dims + 5, generator=gen(dims))
    table = ops.ref.rotary_table(spec, 300)
    for first in (0, 229):
        got = ops.ref.apply_rotary(x, (table, torch.arange(first, first + 70, dtype=torch.int32), interleaved))
        assert torch.allclose(got.double(), O.rotate(x.double(), rot, interleaved, first), atol=1e-5)
    assert torch.equal(got[..., dims:], x[..., dims:])


def test_embedding_with_positions_and_norm_around_zero():
    table, pos, w = (torch.randn(n, 20, generator=gen(n)) for n in (11, 9, 1))
    ids, at = torch.tensor([3, 0, 10, 3], dtype=torch.int32), torch.tensor([0, 1, 2, 3], dtype=torch.int32)
    x, h = ops.embed_rms_norm(ids, table, 2.5, w[0], 1e-3, at, pos, 1.0)
    want = O.embed({"embed": table, "pos": pos}, {"embedding": {"scale": 2.5}}, ids.tolist())
    assert torch.allclose(x, want) and x.dtype == torch.float32
    assert torch.allclose(h, O.centred_norm(want, w[0], 1e-3), atol=1e-6)


@pytest.mark.parametrize("again", [False, True])
def test_layer_scale_residual_and_embedding_at_the_head_of_a_pass(again):
    x, y, table, pos = (torch.randn(n, 24, generator=gen(n)) for n in (5, 6, 7, 8))
    y, vec, w = y[:5] * 1e-3, torch.randn(24, generator=gen(1)), torch.randn(24, generator=gen(2))
    ids, at = torch.tensor([6, 0, 2, 2, 5], dtype=torch.int32), torch.tensor([7, 0, 3, 4, 1], dtype=torch.int32)
    lead = (ids, table, 1.9, at, pos) if again else None
    want = x + vec * y + (table[ids.long()] * 1.9 + pos[at.long()] if again else 0)
    got = x.clone()
    h = ops.add_norm(y, got, 1.0, w, 1e-5, vec, 1.0, lead)
    assert torch.allclose(got, want, atol=1e-6) and torch.allclose(h, O.centred_norm(want, w, 1e-5), atol=1e-6)
    if again:
        got = x + vec * y
        assert torch.allclose(ops.lead_norm(lead, got, w, 1e-5, 1.0), h, atol=1e-6) and torch.allclose(got, want, atol=1e-6)


def test_qk_norm_rotation_and_cache_write():
    T, H, G, d, dv = 6, 4, 2, 10, 7
    rot = {"dims": 6, "base": 30.0}
    qkv = torch.randn(T, 2 * (H + G) * d + G * dv, generator=gen(2))
    qw, kw = torch.randn(2, d, generator=gen(3))
    kc, vc = torch.zeros(4, 4, 2 * G, d), torch.zeros(4, 4, G, dv)
    slots, at = torch.tensor([5, 6, 7, 12, 13, 14], dtype=torch.int32), torch.arange(3, 9, dtype=torch.int32)
    table = ops.ref.rotary_table(RotarySpec(6, 30.0), 20)
    q = ops.qknorm_kvwrite(qkv.clone(), slots, qw, kw, 1e-6, kc, vc, 2 * H, 2 * G, (table, at, False))
    a, b, c = qkv.split([2 * H * d, 2 * G * d, G * dv], -1)
    assert torch.allclose(q.view(T, H, 2, d), O.rotate(O.plain_norm(a.view(T, H, 2, d), qw, 1e-6), rot, False, 3), atol=1e-5)
    assert torch.allclose(kc.view(-1, G, 2, d)[slots.long()], O.rotate(O.plain_norm(b.view(T, G, 2, d), kw, 1e-6), rot, False, 3), atol=1e-5)
    assert torch.equal(vc.view(-1, G, dv)[slots.long()], c.view(T, G, dv))
    assert kc.view(-1, 2 * G, d)[0].abs().sum() == 0


def two_map_step(lens, H, G, d, dv, block, seed=0, edit=None, device="cpu", dtype=torch.float32):
    """(step, queries of the step [T, 2 H, d], per-sequence q / k / v in double) with random or edited rows."""
    g, seqs = gen(seed), []
    for before, n in lens:
        q, k, v = (torch.randn(before + n, *s, generator=g) for s in ((H, 2, d), (G, 2, d), (G, dv)))
        if edit:
            edit(q, k, v)
        seqs.append([t.to(dtype) for t in (q, k, v)])
    step = PagedStep(lens, [(k.flatten(1, 2), v) for _, k, v in seqs], block, device, seed)
    return step, step.step_rows([q.flatten(1, 2) for q, _, _ in seqs]).to(device), [[t.double() for t in s] for s in seqs]


@pytest.mark.parametrize("cap", [0.0, 1.5, 40.0])
@pytest.mark.parametrize("block", [4, 16])
def test_two_map_attention(cap, block):
    lens = [(0, 1), (0, 20), (29, 1), (7, 2), (50, 1), (5, 34)]
    step, q, seqs = two_map_step(lens, 6, 2, 12, 10, block)
    lam, diff, eps = torch.tensor([0.8]), 0.4, 1e-4
    got = ops.paged_attention_ext(q, *step.caches, step.inp, 0.5, softcap=cap, mix=(lam, 1 - diff, eps))
    want = step.step_rows([O.two_map_core(*s, 0.5, cap, lam.double(), diff, eps).flatten(1) for s in seqs])
    assert torch.allclose(got.double(), want, atol=1e-5)


def planted(at, strength):
    """One key of both maps that every query finds, with a value of its own."""
    def edit(q, k, v):
        q[:] = q * 0.05 + 1.0
        k[:] = k * 0.05
        k[at] = strength
        v[at] = 30.0 * torch.sign(v[at])
    return edit


@pytest.mark.parametrize("at", [0, 1, 3, 4, 15, 16, 31, 47])
def test_one_key_that_stands_out(at):
    """Keys at page borders, far behind and right at the query: rows from the key's own on see it, earlier ones do not."""
    lens = [(0, 60), (at, 1), (at, 2), (at + 1, 1), (59, 1)]
    step, q, seqs = two_map_step(lens, 4, 1, 16, 8, 4, seed=at, edit=planted(at, 2.0))
    mix = (torch.tensor([0.3]), 1.0, 1e-6)
    got = ops.paged_attention_ext(q, *step.caches, step.inp, 0.4, softcap=50.0, mix=mix)
    want = step.step_rows([O.two_map_core(*s, 0.4, 50.0, 0.3, 0.0, 1e-6).flatten(1) for s in seqs])
    assert torch.allclose(got.double(), want, atol=1e-4)
    first = O.two_map_core(*seqs[0], 0.4, 50.0, 0.3, 0.0, 1e-6)
    sign = torch.sign(seqs[0][2][at, 0])
    sees = ((first * sign).flatten(1) > 0.5).all(-1)
    assert sees[at:].all() and not sees[:at].any()


@pytest.mark.parametrize("sizes", [(4, 24, 16, 40, 48, 56), (1, 8, 2, 5, 30, 7), (3, 40, 8, 24, 16, 12)])
def test_latent_attention(sizes):
    H, d, r, dv, C, R = sizes
    layer = M.latent(heads=H, dim=d, rot_dim=r, vdim=dv, kv_rank=C, q_rank=R)
    cfg = M.config([(layer, None)])
    sd = {k: v.float() for k, v in M.weights(cfg, 4).items()}
    m, p, W = layer["mixer"], "l0.mix.", cfg["width"]
    sd[p + "o"] = torch.eye(H * dv)                    # compare the heads' outputs
    lens = [(0, 9), (20, 1), (11, 5), (0, 1)]
    hs = [torch.randn(b + n, W, generator=gen(b + n)) for b, n in lens]
    down = torch.cat([sd[p + "dq"], sd[p + "dkv"]])
    spec = RotarySpec(r, m["rot"]["base"], True, *(m["rot"]["scaling"][k] for k in ("factor", "original", "fast", "slow")))
    table = ops.ref.rotary_table(spec, 64)
    rows = []
    for h in hs:                                       # the past of every sequence, through a step of its own
        n = h.shape[0]
        cache = torch.zeros(1, n, C + r)
        ops.latent_down(h @ down.T, R, C, sd[p + "dq.norm"], sd[p + "dkv.norm"], 3e-5, (table, torch.arange(n), True), torch.arange(n), cache)
        rows.append((cache[0, :, None, :],))
    step = PagedStep(lens, rows, 4, "cpu")
    cache = step.caches[0][:, :, 0]
    rot = (table, step.inp.positions, True)
    cq = ops.latent_down(step.step_rows(hs) @ down.T, R, C, sd[p + "dq.norm"], sd[p + "dkv.norm"], 3e-5, rot, step.inp.slots, cache)
    q = (cq @ sd[p + "uq"].T).view(-1, H, d + r)
    got = ops.latent_attention(q, sd[p + "uk"].view(H, d, C).transpose(1, 2), sd[p + "uv"].view(H, dv, C), cache, step.inp, rot, m["scale"], d)
    d64 = {k: v.double() for k, v in sd.items()}
    want = step.step_rows([O.latent_attention(d64, p, m, h.double(), 3e-5) for h in hs])
    assert torch.allclose(got.double(), want, atol=2e-5)


def test_clamped_gate():
    x = torch.linspace(-9, 9, 60).reshape(3, 20)
    for limit in (0.3, 1.0, 4.0):
        assert torch.allclose(ops.ref.gated_act(x, "clamped", limit), O.clamped_gate(x[:, :10], x[:, 10:], limit), atol=1e-6)
    big = torch.tensor([[50.0, 50.0]])
    assert torch.allclose(ops.ref.gated_act(big, "clamped", 2.0), torch.tensor([[2.0 / (1 + math.exp(-3.404)) * 3.0]]), atol=1e-5)


@pytest.mark.parametrize("top", [1, 3, 12])
def test_router(top):
    z, b = torch.randn(64, 12, generator=gen(3)) * 40, torch.randn(12, generator=gen(4)) * 30      # gaps that exp cannot hold
    w, ids = ops.moe_router(z, top, "softmax_chosen", bias=b)
    for t in range(64):
        want = O.route(z[t].double(), b.double(), top)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double(), torch.stack([x for _, x in want]), atol=1e-6)


def test_mixture():
    cfg = M.config([(M.latent(), M.moe())])
    sd = {k: v.float() for k, v in M.weights(cfg, 4).items()}
    mlp, p = cfg["layers"][0]["mlp"], "l0.mlp."
    h, x = torch.randn(20, cfg["width"], generator=gen(5)), torch.randn(20, cfg["width"], generator=gen(6))
    w, ids = ops.moe_router(ops.linear_f32(h, sd[p + "router"]), 3, "softmax_chosen", bias=sd[p + "router.b"])
    w13 = torch.stack([torch.cat([sd[f"{p}e{e}.gate"], sd[f"{p}e{e}.up"]]) for e in range(6)])
    w2 = torch.stack([sd[f"{p}e{e}.down"] for e in range(6)])
    want = x + sd["l0.ls2"] * O.moe(sd, p, mlp, h)
    out = ops.moe_add_norm(h, w13, w2, w, ids, sd["l0.ls2"], x, sd["final.norm"], 1e-6, "clamped", limit=0.8, w_offset=1.0)
    assert torch.allclose(x, want, atol=1e-4) and torch.allclose(out, O.centred_norm(want, sd["final.norm"], 1e-6), atol=1e-4)


def test_bounded_logits():
    x, w = torch.randn(5, 16, generator=gen(1)) * 4, torch.randn(9, 16, generator=gen(2))
    assert torch.allclose(ops.linear_softcap(x, w, 7.0), O.softcap(x @ w.T, 7.0), atol=1e-5)


# ----------------------------------------------------------------------------- whole models through the engine
@pytest.mark.parametrize("hooked", [True, False])
def test_layers_one_by_one(mixed, hooked):
    cfg, sd, path = mixed
    toks = M.tokens(45, cfg["vocab"], 7)
    want = []
    logits = O.forward(sd, cfg, toks, want)
    eng, got = M.engine(path), []
    if hooked:
        eng.worker.model.residual_hook = lambda r, x: got.append(x.clone())
    out = M.replay(eng, {"a": toks}, [[("a", 45)]])["a"]
    assert len(got) == (len(want) if hooked else 0) and len(want) == 11
    for r, (a, b) in enumerate(zip(got, want)):
        assert M.row_error(a, b).max() < TOL, r
    assert M.row_error(out, logits).max() < TOL


@pytest.mark.parametrize("cuts", [(2,), (1, 2, 3, 5, 8, 13, 21, 34), (16, 16, 16, 16), (15, 2, 17, 2, 40), (2,) * 40])
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
    got = M.replay(M.engine(path, block_size=block_size, blocks=room + 1), seqs, steps)
    for n, toks in seqs.items():
        assert M.row_error(got[n], O.forward(sd, cfg, toks)).max() < TOL, n


def test_odd_sizes(tmp_path):
    cfg = M.odd_config()
    sd = M.weights(cfg, 2)
    toks = M.tokens(40, cfg["vocab"], 9)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 13, 9))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


def test_long_decoding(tmp_path):
    cfg = M.config([(M.latent(heads=2), M.dense()), (M.two_map(heads=2, kv_heads=1), M.moe())], width=40, vocab=97)
    sd = M.weights(cfg, 3)
    toks = M.tokens(300, 97, 10)
    got = M.replay(M.engine(M.save(cfg, sd, tmp_path)), {"a": toks}, M.alone("a", toks, 3))["a"]
    assert M.row_error(got, O.forward(f64(sd), cfg, toks)).max() < TOL


def test_no_more_tokens_than_positions(tmp_path):
    """The learned position table ends a sequence."""
    cfg = M.config([(M.latent(heads=2), M.dense())], width=40, vocab=97, positions=24)
    eng = M.engine(M.save(cfg, M.weights(cfg, 3), tmp_path))
    out = LLM(model="", devices="cpu", engine=eng).generate([M.tokens(10, 97, 1)], SamplingParams(temperature=0.0, max_tokens=60, ignore_eos=True))
    assert 10 < 10 + len(out[0].outputs[0].token_ids) <= 24


# Every mechanism shows in the logits of these models: an oracle with one planted mistake is far from the right one.
MISTAKES = {
    "no position vectors": ("embed", lambda f: lambda sd, c, t: f(dict(sd, pos=sd["pos"] * 0), c, t)),
    "position vectors scaled": ("embed", lambda f: lambda sd, c, t: f(dict(sd, pos=sd["pos"] * 1.7), c, t)),
    "norm weights not around zero": ("centred_norm", lambda f: O.plain_norm),
    "no key before the own one": ("causal", lambda f: lambda n: f(n) & f(n).T),
    "the next key": ("causal", lambda f: lambda n: f(n) | torch.diag(torch.ones(n - 1, dtype=torch.bool), 1)),
    "no frequency scaling": ("frequencies", lambda f: lambda r: (f(dict(r, scaling=None))[0], f(r)[1])),
    "no amplitude of the scaling": ("frequencies", lambda f: lambda r: (f(r)[0], 1.0)),
    "other pairs": ("rotate", lambda f: lambda x, r, i, first=0: f(x, r, not i, first)),
    "unbounded scores and logits": ("softcap", lambda f: lambda s, c: s),
    "second map left out": ("difference", lambda f: lambda a, b, l, d, e: f(a, b, 0.0, d, e)),
    "difference not normed": ("difference", lambda f: lambda a, b, l, d, e: (a - l * b) * (1 - d)),
    "difference not scaled": ("difference", lambda f: lambda a, b, l, d, e: f(a, b, l, 0.0, e)),
    "constant factor only": ("mix_factor", lambda f: lambda sd, p, d: d),
    "unclamped gate": ("clamped_gate", lambda f: lambda g, u, l: f(g, u, 1e9)),
    "gate clamped on both sides": ("clamped_gate", lambda f: lambda g, u, l: f(g.clamp(min=-l), u, l)),
    "weights of all experts' softmax": ("route", lambda f: lambda z, b, t: [(e, torch.softmax(z + b, -1)[e]) for e, _ in f(z, b, t)]),
    "bias not in the weights": ("route", lambda f: lambda z, b, t: [(e, w) for (e, _), w in zip(f(z, b, t), torch.softmax(
        torch.stack([z[e] for e, _ in f(z, b, t)]), -1))]),
    "loop run once": ("layer_order", lambda f: lambda cfg: [(i, False) for i in range(len(cfg["layers"]))]),
    "embedding not added again": ("layer_order", lambda f: lambda cfg: [(i, False) for i, _ in f(cfg)]),
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


def test_sampling(mixed):
    cfg, _, path = mixed
    llm = LLM(model=path, devices="cpu", engine=M.engine(path))
    sp = SamplingParams(temperature=0.8, top_k=20, seed=5, max_tokens=6, ignore_eos=True, logprobs=True, top_logprobs=2)
    a, b = (llm.generate([[1, 2, 3]], sp)[0].outputs[0].token_ids for _ in range(2))
    assert a == b and len(a) == 6


def test_presets_are_described():
    for name in ("babadra-8b", "babadra-30b-a3b"):
        a = preset(name)
        assert a.model_type == "babadra" and len(a.layer_runs) == a.n_layers == len(a.layer_specs)
        assert {type(s.mixer) for s in a.layer_specs} > {LatentAttentionSpec}


# ----------------------------------------------------------------------------- the replay program
def test_trace_run_program(mixed, tmp_path):
    cfg, sd, path = mixed
    seqs = {"x": M.tokens(30, cfg["vocab"], 40), "y": M.tokens(12, cfg["vocab"], 41)}
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": seqs["x"][:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": seqs["x"][20:21], "want": []}, {"id": "y", "tokens": seqs["y"], "want": [11, 3]}],
              "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": seqs["x"][21:], "want": [8]}], "end": ["x"]}]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out",
                        str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(3)]
    X, Y = O.forward(sd, cfg, seqs["x"]), O.forward(sd, cfg, seqs["y"])
    for step, want in ((0, X[[0, 19]]), (1, Y[[11, 3]]), (2, X[[29]])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{step}.f32", "<f4").reshape(len(want), -1))
        assert M.row_error(got, want).max() < TOL
