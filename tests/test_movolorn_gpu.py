"""Movolorn on a GPU: every kernel against the plain fp32 statement of its mechanism, whole models in bf16 and in true 32-bit
against tests/oracle_movolorn.py, decoding through CUDA graphs, greedy generation through the scheduler."""
import math

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

from tests import oracle_movolorn as O
from tests.helpers import movolorn_models as M
from xllm_wxh_b200 import LLM, SamplingParams, ops
from xllm_wxh_b200.framework.step_input import StepInput, make_layout
from xllm_wxh_b200.models.layer_spec import AttentionSpec

DEV = "cuda:0"


def status_ok():
    from xllm_wxh_b200.ops import cuda_ops
    return cuda_ops.read_status() == 0


def rel(got, want):
    return ((got.double().cpu() - want.double().cpu()).norm() / want.double().cpu().norm()).item()


# ----------------------------------------------------------------------------- attention
class Paged:
    """Sequences of given (tokens before the step, tokens in the step) with random q / k / v in a shuffled paged cache."""

    def __init__(self, lens, H, G, d, dv, block, dtype, seed=0, edit=None):
        g = torch.Generator().manual_seed(seed)
        self.seqs = []
        for before, n in lens:
            T = before + n
            q, k, v = (torch.randn(T, h, w, generator=g) for h, w in ((H, d), (G, d), (G, dv)))
            if edit:
                edit(q, k, v)
            self.seqs.append([t.to(dtype) for t in (q, k, v)])
        self.lens = lens = sorted(range(len(lens)), key=lambda i: not (lens[i][1] == 1 and lens[i][0] > 0)), lens
        order, lens = self.lens
        need = [-(-(b + n) // block) for b, n in lens]
        MB = max(need)
        perm = (torch.randperm(sum(need), generator=g) + 1).tolist()
        kc = torch.randn(sum(need) + 1, block, G, d, generator=g).to(dtype)        # other places hold other values
        vc = torch.randn(sum(need) + 1, block, G, dv, generator=g).to(dtype)
        L = make_layout(sum(n for _, n in lens), len(lens), MB, len(lens), 32)
        host = torch.zeros(L.total_words, dtype=torch.int32)
        rows, at, n_dec = [], 0, 0
        for s, i in enumerate(order):
            before, n = lens[i]
            blocks = [perm.pop() for _ in range(need[i])]
            q, k, v = self.seqs[i]
            for t in range(before + n):
                kc[blocks[t // block], t % block], vc[blocks[t // block], t % block] = k[t], v[t]
            o = L.block_tables + s * L.MB_cap
            host[o:o + len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
            host[L.positions + at:L.positions + at + n] = torch.arange(before, before + n, dtype=torch.int32)
            host[L.token_seq + at:L.token_seq + at + n] = s
            at += n
            host[L.q_cu + s + 1] = at
            host[L.kv_lens + s] = before + n
            n_dec += n == 1 and before > 0
            rows.append(q[before:])
        hdr = np.zeros(32, dtype=np.int32)
        hdr[0], hdr[1], hdr[3], hdr[4] = at, len(lens), n_dec, len(lens) - n_dec
        hdr[5], hdr[6], hdr[17] = max(n for _, n in lens), max(b + n for b, n in lens), block
        hdr[7] = 2 if n_dec == len(lens) else 3
        hdr[21] = sum(n for b, n in lens if not (n == 1 and b > 0))
        host[L.header:L.header + 32] = torch.from_numpy(hdr)
        self.inp = StepInput(host.to(DEV), L, hdr)
        self.q, self.kc, self.vc = torch.cat(rows).to(DEV), kc.to(DEV), vc.to(DEV)

    def want(self, scale, chunk):
        order, lens = self.lens
        out = []
        for i in order:
            q, k, v = (t.double() for t in self.seqs[i])
            out.append(O.attention_core(q, k, v, scale, chunk)[lens[i][0]:].flatten(1))
        return torch.cat(out)

    def got(self, scale, chunk):
        H = self.q.shape[1]
        spec = AttentionSpec(heads=H, kv_heads=self.kc.shape[2], dim=0, vdim=0, scale=0)
        return ops.paged_attention_ext(self.q, self.kc, self.vc, self.inp, scale, -1, chunk,
                                       torch.tensor(spec.head_slopes(), device=DEV), torch.zeros(H, device=DEV))


HEADS = [(4, 1, 56, 40), (8, 2, 128, 128), (6, 2, 64, 64), (3, 3, 16, 96), (5, 1, 128, 24), (2, 2, 8, 8), (12, 1, 72, 64),
         (4, 2, 20, 36), (2, 1, 160, 144), (20, 1, 32, 32)]
LENS = [(0, 1), (0, 200), (129, 1), (37, 2), (250, 1), (5, 64), (128, 130), (63, 1), (64, 1)]


@pytest.mark.parametrize("heads", HEADS)
@pytest.mark.parametrize("chunk,block", [(37, 16), (96, 64), (128, 32), (1 << 20, 128)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_attention(heads, chunk, block, dtype):
    p = Paged(LENS, *heads, block, dtype, seed=sum(heads))
    scale = 2.0 / math.sqrt(heads[2])
    got, want = p.got(scale, chunk), p.want(scale, chunk)
    assert rel(got, want) < (8e-3 if dtype == torch.bfloat16 else 1e-5)
    assert (got.double().cpu() - want).abs().max() < (0.06 if dtype == torch.bfloat16 else 1e-4)
    assert status_ok()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("chunk", [32, 50, 64, 100])
def test_one_key_just_inside_or_outside_a_chunk(chunk, dtype):
    """One key per sequence stands out by far (its value too): rows of its chunk behind it see it, all others do not.  The
    keys lie at the first and last place of a chunk, at block borders, and at the start of the sequence."""
    H, G, d, dv = 4, 2, 64, 64
    for planted in (0, 1, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 2 * chunk, 15, 16, 63, 64):
        def edit(q, k, v):
            q[:] = q * 0.05 + 1.0
            k[:] = k * 0.05
            k[planted] = 2.0
            v[planted] = 30.0
        n = 2 * chunk + 9
        lens = [(0, n), (planted, 1), (planted, 2)] + [(t, 1) for t in (chunk - 1, chunk, 2 * chunk - 1, 2 * chunk) if t > planted]
        lens = [x for x in lens if sum(x) > planted and x != (0, 1)]
        p = Paged(lens, H, G, d, dv, 16, dtype, seed=planted, edit=edit)
        got, want = p.got(0.1, chunk), p.want(0.1, chunk)
        assert rel(got, want) < (8e-3 if dtype == torch.bfloat16 else 1e-5), planted
        # rows that must not see the planted key stay small
        dark = want.abs().max(-1).values < 5
        assert dark.any() and got.cpu()[dark].abs().max() < 6, planted
    assert status_ok()


def test_sink_dominates_when_scores_are_low():
    """Scores far below 0: the one in the denominator outweighs every key; and the first token has only itself and the sink."""
    def edit(q, k, v):
        q[:], k[:] = 1.0, -1.0
    for dtype in (torch.bfloat16, torch.float32):
        for lens in ([(0, 40), (30, 1), (0, 1)], [(600, 1), (900, 1)], [(0, 300)]):
            p = Paged(lens, 4, 2, 64, 64, 16, dtype, edit=edit)
            assert rel(p.got(0.05, 1 << 20), p.want(0.05, 1 << 20)) < 1e-2


def test_long_context_splits_and_merges():
    """Few sequences over many keys: the key ranges are split in decode and prefill, the sink joins once."""
    p = Paged([(5000, 1), (4100, 1), (3000, 1)], 8, 2, 128, 128, 64, torch.bfloat16)
    assert rel(p.got(0.25, 1 << 20), p.want(0.25, 1 << 20)) < 1e-2
    p = Paged([(3900, 100)], 4, 2, 64, 96, 64, torch.bfloat16)
    assert rel(p.got(0.25, 1 << 20), p.want(0.25, 1 << 20)) < 1e-2
    p = Paged([(3900, 100), (4095, 1)], 4, 2, 128, 128, 64, torch.bfloat16)
    assert rel(p.got(0.25, 3000), p.want(0.25, 3000)) < 1e-2
    assert status_ok()


# ----------------------------------------------------------------------------- the other kernels
@pytest.mark.parametrize("H", [67, 72, 336, 2048, 4096, 5120, 9000])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_norm_kernels(H, dtype):
    g = torch.Generator().manual_seed(H)
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    T = 37
    y, wp, wn = (torch.randn(s, generator=g).to(dtype) for s in ((T, H), (H,), (H,)))
    y[3] *= 1e-4                                               # eps matters
    x = torch.randn(T, H, generator=g)
    xd = x.to(DEV)
    h = ops.post_norm_add_norm(y.to(DEV), xd, wp.to(DEV), wn.to(DEV), 1e-6)
    want = x.double() + O.rms_norm(y.double(), wp.double(), 1e-6)
    assert rel(xd, want) < 2e-6 and rel(h, O.rms_norm(want, wn.double(), 1e-6)) < tol
    table = torch.randn(50, H, generator=g).to(dtype)
    ids = torch.randint(0, 50, (T,), generator=g).int()
    xe, he = ops.embed_rms_norm(ids.to(DEV), table.to(DEV), 3.5, wn.to(DEV), 1e-6)
    assert rel(xe, table[ids.long()].double() * 3.5) < 1e-6
    assert rel(he, O.rms_norm(table[ids.long()].double() * 3.5, wn.double(), 1e-6)) < tol


@pytest.mark.parametrize("dims", [(4, 2, 56, 40), (3, 1, 128, 64), (2, 2, 21, 13), (5, 1, 8, 256), (2, 1, 300, 264)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_qknorm_kvwrite_kernel(dims, dtype):
    H, G, d, dv = dims
    g = torch.Generator().manual_seed(sum(dims))
    T = 29
    qkv = torch.randn(T, (H + G) * d + G * dv, generator=g).to(dtype)
    qw, kw = (1 + 0.3 * torch.randn(2, d, generator=g)).to(dtype)
    kc, vc = torch.zeros(8, 16, G, d, dtype=dtype), torch.zeros(8, 16, G, dv, dtype=dtype)
    slots = torch.randperm(100, generator=g)[:T].int()
    kd, vd = kc.to(DEV), vc.to(DEV)
    q = ops.qknorm_kvwrite(qkv.to(DEV), slots.to(DEV), qw.to(DEV), kw.to(DEV), 1e-6, kd, vd, H, G)
    a, b, c = qkv.double().split([H * d, G * d, G * dv], -1)
    tol = 4e-3 if dtype == torch.bfloat16 else 1e-6
    assert rel(q, O.rms_norm(a.reshape(T, H, d), qw.double(), 1e-6).flatten(1)) < tol
    assert rel(kd.view(-1, G, d)[slots.long().to(DEV)], O.rms_norm(b.reshape(T, G, d), kw.double(), 1e-6)) < tol
    assert torch.equal(vd.view(-1, G, dv)[slots.long().to(DEV)].cpu().double(), c.reshape(T, G, dv))
    rest = torch.ones(128, dtype=torch.bool)
    rest[slots.long()] = False
    assert kd.view(128, -1).cpu()[rest].abs().sum() == 0 and vd.view(128, -1).cpu()[rest].abs().sum() == 0


@pytest.mark.parametrize("M_,N,K", [(1, 10, 272), (300, 132, 256), (77, 67, 51), (130, 520, 80), (5, 3, 8)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_products(M_, N, K, dtype):
    g = torch.Generator().manual_seed(M_ + N + K)
    x, w = torch.randn(M_, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) / math.sqrt(K)).to(dtype)
    want = x.double() @ w.double().T
    assert rel(ops.linear_f32(x.to(DEV), w.to(DEV)), want) < 1e-6
    assert rel(ops.linear(x.to(DEV), w.to(DEV)), want) < (4e-3 if dtype == torch.bfloat16 else 1e-6)
    assert status_ok()


@pytest.mark.parametrize("act,f", [("silu", O.silu), ("gelu_tanh", O.gelu_tanh)])
@pytest.mark.parametrize("M_,ff,K", [(3, 80, 272), (400, 1024, 512), (150, 45, 64)])
def test_gated_linear(act, f, M_, ff, K):
    from xllm_wxh_b200.ops import cuda_ops
    g = torch.Generator().manual_seed(ff)
    x, w = torch.randn(M_, K, generator=g) * 2, torch.randn(2 * ff, K, generator=g) / math.sqrt(K)
    for dtype in (torch.bfloat16, torch.float32):
        xt, wt = x.to(dtype), w.to(dtype)
        want = f(xt.double() @ wt[:ff].double().T) * (xt.double() @ wt[ff:].double().T)
        tol = 8e-3 if dtype == torch.bfloat16 else 3e-6
        assert rel(ops.gated_linear(xt.to(DEV), wt.to(DEV), act), want) < tol
        if dtype == torch.bfloat16 and ff % 16 == 0:
            assert rel(ops.gated_linear(xt.to(DEV), cuda_ops.interleave_gate_up(wt.to(DEV)), act, True), want) < tol
    assert status_ok()


@pytest.mark.parametrize("E,top,groups", [(14, 3, (7, 3)), (128, 8, (8, 4)), (9, 3, (1, 1)), (40, 5, (20, 3))])
def test_router_kernel(E, top, groups):
    g = torch.Generator().manual_seed(E)
    z = torch.randn(50, E, generator=g) * 2
    corr = torch.randn(E, generator=g) * 0.3 - 0.5
    w, ids = ops.moe_router(z.to(DEV), top, "softmax", False, corr.to(DEV), groups[0], groups[1], 1.0, "max")
    r = {"top": top, "groups": {"count": groups[0], "keep": groups[1]}}
    for t in range(50):
        want = O.route(z[t].double(), corr.double(), r)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double().cpu(), torch.stack([x for _, x in want]), rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("width,ff,experts,identity,shared", [(272, 80, 7, 3, 112), (512, 64, 12, 0, 0), (67, 27, 5, 1, 9)])
@pytest.mark.parametrize("T", [1, 7, 300])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_mixture_kernels(width, ff, experts, identity, shared, T, dtype):
    mlp = M.moe(ff=ff, experts=experts, identity=identity, top=3, groups=None, shared=shared)
    cfg = M.config([(M.attn(), mlp)], width=width)
    sd = {k: v.to(dtype) for k, v in M.weights(cfg, T).items()}
    p = "l0.mlp."
    g = torch.Generator().manual_seed(T)
    h, x = torch.randn(T, width, generator=g).to(dtype), torch.randn(T, width, generator=g)
    dev = {k: v.to(DEV) for k, v in sd.items()}
    w, ids = ops.moe_router(ops.linear_f32(h.to(DEV), dev[p + "router"]), 3, "softmax", False, dev[p + "correction"].float(), 1, 1, 1.0, "max")
    w13 = torch.stack([torch.cat([dev[f"{p}e{e}.gate"], dev[f"{p}e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([dev[f"{p}e{e}.down"] for e in range(experts)])
    sh = None
    if shared:
        sh = ops.linear(ops.gated_linear(h.to(DEV), torch.cat([dev[p + "shared.gate"], dev[p + "shared.up"]])), dev[p + "shared.down"])
    from xllm_wxh_b200.ops import moe_cuda
    d = {k: v.double() for k, v in sd.items()}
    want_y = torch.zeros(T, width, dtype=torch.float64)
    for t in range(T):                                        # the experts that the kernel chose (checked above on its own)
        for e, wt in zip(ids[t].tolist(), w[t].double().cpu()):
            want_y[t] += wt * (O.gated_ff(d, f"{p}e{e}.", h[t:t + 1].double(), O.silu)[0] if e < experts else h[t].double())
    if shared:
        want_y += O.gated_ff(d, p + "shared.", h.double(), O.silu)
    want = x.double() + O.rms_norm(want_y, d["l0.norm2b"], 1e-6)
    tol = 8e-3 if dtype == torch.bfloat16 else 5e-6
    for inter in (False, True):
        if inter and (dtype != torch.bfloat16 or ff % 16):
            continue
        xd = x.to(DEV)
        out = ops.moe_post_norm_add_norm(h.to(DEV), moe_cuda.interleave_w13(w13.clone()) if inter else w13, w2, w, ids, sh, experts, xd,
                                         dev["l0.norm2b"], dev["final.norm"], 1e-6, "silu", inter)
        assert rel(xd, want) < tol and rel(out, O.rms_norm(want, d["final.norm"], 1e-6)) < tol
    assert status_ok()


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in (("mixed", M.mixed_config()), ("odd", M.odd_config()),
                      ("wide", M.config([(M.attn(heads=8, kv_heads=2, dim=128, vdim=128, chunk=200), M.dense(ff=512)),
                                         (M.attn(heads=8, kv_heads=4, dim=64, vdim=64, chunk=90), M.moe(ff=128, shared=128))],
                                        width=256, vocab=1024, loop=(1, 2, 2)))):
        sd = M.weights(cfg, 5)
        out[name] = cfg, {k: v.double() for k, v in sd.items()}, M.save(cfg, sd, tmp_path_factory.mktemp(name))
    return out


def check(got, want, dtype):
    e = M.row_error(got, want)
    if dtype == "float32":
        assert e.max() < 1e-4, e.max()
    else:                       # a close call of a router may go the other way in bf16
        assert e.median() < 0.02 and e.quantile(0.9) < 0.06, (e.median(), e.quantile(0.9))


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_whole_portions_and_decoding(models, name, dtype):
    cfg, sd, path = models[name]
    toks = M.tokens(230, cfg["vocab"], 50)
    res = []
    want = O.forward(sd, cfg, toks, res)
    eng, got = M.engine(path, DEV, dtype), []
    eng.worker.model.residual_hook = lambda r, x: got.append(x[:230].cpu())
    out = M.replay(eng, {"a": toks}, [[("a", 230)]])["a"]
    for a, b in zip(got, res):
        check(a, b, dtype)
    eng.worker.model.residual_hook = None
    check(out, want, dtype)
    for cuts in ((190,), (2, 3, 64, 7, 99), (37, 37, 37, 37)):
        part = M.replay(eng, {"a": toks}, M.alone("a", toks, *cuts))["a"]
        check(part, want, dtype)
        # the way the tokens are cut changes nothing beyond rounding
        e = M.row_error(part, out)
        assert e.median() < (1e-5 if dtype == "float32" else 0.02)
    g = eng.worker._graphs
    assert g is not None and g.num_replays > 40 and status_ok()


@pytest.mark.parametrize("block_size", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batches_and_blocks_used_again(models, dtype, block_size):
    cfg, sd, path = models["mixed"]
    seqs = {n: M.tokens(c, cfg["vocab"], 60 + i) for i, (n, c) in enumerate([("a", 70), ("b", 9), ("c", 40), ("d", 23), ("e", 66), ("f", 31)])}
    steps = [[("a", 30), ("b", 8)], [("c", 5), ("a", 2), ("b", 1)], [("d", 20)], [("a", 1), ("d", 1), ("c", 33)], [("a", 37), ("d", 2), ("c", 2)],
             [("e", 50), ("f", 2)], [("f", 28), ("e", 1)], [("e", 15), ("f", 1)]]
    room = sum(-(-n // block_size) for n in (70, 40, 23, 9))
    got = M.replay(M.engine(path, DEV, dtype, block_size=block_size, blocks=room + 1), seqs, steps)
    for n, toks in seqs.items():
        check(got[n], O.forward(sd, cfg, toks), dtype)
    assert status_ok()


@pytest.mark.parametrize("kw", [{}, dict(enable_graph=False), dict(enable_schedule_overlap=True, enable_prefill_piecewise_graph=True),
                                dict(max_tokens_per_batch=24, max_tokens_per_chunk_for_prefill=7), dict(enable_prefix_cache=True),
                                dict(blocks=16)])
def test_greedy_generation_in_32_bit(models, kw):
    cfg, sd, path = models["mixed"]
    prompts = [M.tokens(n, cfg["vocab"], 70 + n) for n in (5, 33, 18, 41)]
    prompts.append(prompts[3][:32] + [7, 9])
    llm = LLM(model=path, devices=DEV, engine=M.engine(path, DEV, "float32", **kw))
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == O.greedy(sd, cfg, p, 16)
    assert status_ok()


def test_bf16_generation_follows_its_own_logits(models):
    """Greedy tokens of the bf16 engine, fed back through the replayed steps, are the maxima of those logits."""
    cfg, _, path = models["wide"]
    eng = M.engine(path, DEV, "bfloat16", enable_schedule_overlap=True)
    prompts = [M.tokens(n, cfg["vocab"], 80 + n) for n in (150, 3, 64)]
    outs = LLM(model=path, devices=DEV, engine=eng).generate(prompts, SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True))
    same = total = 0
    for p, o in zip(prompts, outs):
        seq = p + o.outputs[0].token_ids
        rows = M.replay(M.engine(path, DEV, "bfloat16"), {"a": seq[:-1]}, [[("a", len(seq) - 1)]])["a"]
        same += (rows[len(p) - 1:].argmax(-1) == torch.tensor(seq[len(p):])).sum().item()
        total += len(seq) - len(p)
    assert same >= 0.9 * total


def test_sleep_and_wakeup_keep_the_outputs(models):
    cfg, _, path = models["mixed"]
    eng = M.engine(path, DEV, "bfloat16")
    llm = LLM(model=path, devices=DEV, engine=eng)
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    first = [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)]
    for level in (1, 2):
        assert eng.sleep(level) and eng.wakeup()
        assert [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)] == first
