"""Falalix on a GPU: every kernel against the plain statement of its mechanism, whole models in bf16 and in true 32-bit against
tests/oracle_falalix.py, decoding through CUDA graphs, state slots used again, greedy generation through the scheduler."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

from tests import oracle_falalix as O
from tests.helpers import falalix_models as M
from tests.helpers.ragged_steps import DEV, Ragged, rel, status_ok, step_input
from xllm_wxh_b200 import LLM, SamplingParams, ops

DTYPES = [torch.bfloat16, torch.float32]


LENS = [300, 1, 70, 2, 33]
STEPS = [
    [[300, 1, 70, 2, 33]],
    [[1, 1, 2, 1, 17], [1, 0, 1, 1, 0], [2, 0, 31, 0, 1], [150, 0, 1, 0, 1], [1, 0, 35, 0, 14]] + [[1, 0, 0, 0, 0]] * 20 + [[125, 0, 0, 0, 0]],
    [[64, 0, 64, 0, 32], [65, 1, 6, 2, 1], [171, 0, 0, 0, 0]],
]


def ragged(steps, pad):
    return Ragged(LENS, STEPS[steps], pad=pad)


# ----------------------------------------------------------------------------- recurrent kernels
@pytest.mark.parametrize("pad", [0, 5])
@pytest.mark.parametrize("steps", [0, 1, 2])
@pytest.mark.parametrize("W", [64, 67, 2560])
@pytest.mark.parametrize("dtype", DTYPES)
def test_token_shift(W, dtype, steps, pad):
    g = torch.Generator().manual_seed(W)
    h = [torch.randn(n, W, generator=g).to(dtype) for n in LENS]
    mu = torch.rand(5, W, generator=g).to(dtype)
    want = [torch.stack([O.token_mix(x.double(), mu[j].double()) for j in range(5)], 1) for x in h]
    rg = ragged(steps, pad)
    last = torch.full((rg.n_slots, W), 1e4, dtype=dtype, device=DEV)
    for inp, rows in rg:
        got = ops.token_shift(rg.take(h, rows), mu.to(DEV), last, inp)
        n = sum(b - a for _, a, b in rows)
        assert rel(got[:, :n].transpose(0, 1), torch.cat([want[i][a:b] for i, a, b in rows])) < (4e-3 if dtype == torch.bfloat16 else 1e-6)
        assert got[:, n:].abs().sum() == 0
    assert (last[0] == 1e4).all() and status_ok()


@pytest.mark.parametrize("pad", [0, 5])
@pytest.mark.parametrize("steps", [0, 1, 2])
@pytest.mark.parametrize("C,taps", [(64, 4), (1032, 4), (72, 3), (40, 2), (27, 4), (24, 1), (48, 6), (19, 1), (21, 9)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_conv(C, taps, dtype, steps, pad):
    g = torch.Generator().manual_seed(C + taps)
    x = [torch.randn(n, 2 * C, generator=g).to(dtype) for n in LENS]              # a strided half of wider rows
    w, b = torch.randn(C, taps, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype)
    want = [O.silu(O.causal_conv(s[:, :C].double(), w.double(), b.double())) for s in x]
    rg = ragged(steps, pad)
    state = torch.full((rg.n_slots, taps - 1, C), 1e4, dtype=dtype, device=DEV)
    for inp, rows in rg:
        got = ops.conv_silu(rg.take(x, rows)[:, :C], w.t().contiguous().to(DEV), b.to(DEV), state, inp)
        n = sum(q - p for _, p, q in rows)
        assert rel(got[:n], torch.cat([want[i][p:q] for i, p, q in rows])) < (4e-3 if dtype == torch.bfloat16 else 2e-6)
        assert got[n:].abs().sum() == 0
    assert status_ok()


@pytest.mark.parametrize("rows", [0, 48])
@pytest.mark.parametrize("pad", [0, 5])
@pytest.mark.parametrize("steps", [0, 1, 2])
@pytest.mark.parametrize("H,d", [(3, 64), (2, 32), (2, 128), (3, 48), (1, 8), (2, 96), (3, 21), (2, 9), (1, 160), (2, 132), (1, 139)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_time_mix(H, d, dtype, steps, pad, rows, monkeypatch):
    from xllm_wxh_b200.ops import cuda_ops
    monkeypatch.setattr(cuda_ops, "mix_force_rows", rows)        # rows per segment of longer portions (0: chosen)
    g = torch.Generator().manual_seed(H * d)
    n_ = H * d
    r, k, v, gate = ([torch.randn(n, n_, generator=g).to(dtype) for n in LENS] for _ in range(4))
    z = [torch.randn(n, n_, generator=g) for n in LENS]
    w0, u, nw = torch.rand(n_, generator=g) * 5 - 5, torch.randn(H, d, generator=g), (1 + 0.2 * torch.randn(n_, generator=g)).to(dtype)
    want = []
    for i in range(len(LENS)):
        w = torch.exp(-torch.exp(z[i].double() + w0.double())).view(-1, H, d)
        o = O.time_mix_core(*(x[i].double().view(-1, H, d) for x in (r, k, v)), w, u.double())
        o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-5)
        want.append(0.4 * o.flatten(1) * nw.double() * O.silu(gate[i].double()))
    rg = ragged(steps, pad)
    state = torch.full((rg.n_slots, H, d, d), 1e4, device=DEV)
    for inp, rows in rg:
        T = sum(b - a for _, a, b in rows)
        out = torch.full((T + pad, n_ + 24), 5.0, dtype=dtype, device=DEV)
        q = [rg.take(x, rows) for x in (r, k, v, z)]
        ops.time_mix(*q, w0.to(DEV), u.to(DEV), rg.take(gate, rows), nw.to(DEV), 0.4, 1e-5, state, inp, out[:, 24:])
        assert rel(out[:T, 24:], torch.cat([want[i][a:b] for i, a, b in rows])) < (4e-3 if dtype == torch.bfloat16 else 2e-5)
        assert (out[:, :24] == 5).all() and out[T:, 24:].abs().sum() == 0
    assert (state[0] == 1e4).all() and status_ok()


@pytest.mark.parametrize("rows", [0, 64, 16, 2, 130])
def test_time_mix_of_long_and_many_portions(rows, monkeypatch):
    """Segments: several per sequence, sequences of all lengths around a segment's, more sequences than a warp has lanes."""
    H, d = 2, 64
    g = torch.Generator().manual_seed(0)
    from xllm_wxh_b200.ops import cuda_ops
    monkeypatch.setattr(cuda_ops, "mix_force_rows", rows)
    lens = [900, 64, 65, 63, 128, 129, 2, 1, 3] + [2 + i % 5 for i in range(60)]
    r, k, v, gate, z = ([torch.randn(n, H * d, generator=g) for n in lens] for _ in range(5))
    w0, u, nw = torch.rand(H * d, generator=g) * 5 - 6, torch.randn(H, d, generator=g), torch.ones(H * d)
    rg = Ragged(lens, [lens], n_slots=100)
    state = torch.full((100, H, d, d), 1e4, device=DEV)
    (inp, rows), = list(rg)
    out = torch.empty(sum(lens), H * d, device=DEV)
    ops.time_mix(*(rg.take(x, rows) for x in (r, k, v, z)), w0.to(DEV), u.to(DEV), rg.take(gate, rows), nw.to(DEV), 1.0, 1e-5, state, inp, out)
    at = 0
    for i, a, b in rows:
        if lens[i] > 8 or i % 7 == 0:
            w = torch.exp(-torch.exp(z[i].double() + w0.double())).view(-1, H, d)
            o = O.time_mix_core(*(x[i].double().view(-1, H, d) for x in (r, k, v)), w, u.double())
            o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-5)).flatten(1) * O.silu(gate[i].double())
            assert rel(out[at:at + b - a], o) < 2e-5, lens[i]
        at += b - a
    assert status_ok()


@pytest.mark.parametrize("pad", [0, 5])
@pytest.mark.parametrize("steps", [0, 1, 2])
@pytest.mark.parametrize("C,N", [(64, 16), (200, 16), (40, 32), (27, 5), (19, 1), (36, 4), (33, 64), (24, 8), (20, 100), (12, 140), (300, 12)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_selective_scan(C, N, dtype, steps, pad):
    g = torch.Generator().manual_seed(C + N)
    x, z = ([torch.randn(n, C, generator=g).to(dtype) for n in LENS] for _ in range(2))
    BC = [torch.randn(n, 2 * N + 3, generator=g).to(dtype) for n in LENS]
    dt = [torch.randn(n, C, generator=g) for n in LENS]
    A = -torch.exp(torch.log(torch.arange(1, N + 1).float()).expand(C, N) + 0.3 * torch.randn(C, N, generator=g))
    D, bias = torch.randn(C, generator=g), torch.rand(C, generator=g) * 4 - 5
    want = [O.scan_core(x[i].double(), O.softplus(dt[i].double() + bias.double()), A.double(), BC[i][:, 3:3 + N].double(),
                        BC[i][:, 3 + N:].double(), D.double()) * O.silu(z[i].double()) for i in range(len(LENS))]
    rg = ragged(steps, pad)
    state = torch.full((rg.n_slots, C, N), 1e4, device=DEV)
    for inp, rows in rg:
        T = sum(b - a for _, a, b in rows)
        low = rg.take(BC, rows)
        got = ops.selective_scan(rg.take(x, rows), rg.take(dt, rows), bias.to(DEV), A.to(DEV), low[:, 3:3 + N], low[:, 3 + N:], D.to(DEV),
                                 rg.take(z, rows), state, inp)
        assert rel(got[:T], torch.cat([want[i][a:b] for i, a, b in rows])) < (4e-3 if dtype == torch.bfloat16 else 5e-6)
        assert got[T:].abs().sum() == 0
    assert (state[0] == 1e4).all() and status_ok()


def test_a_record_outside_the_state_is_reported():
    """A slot that the state tensors do not have: nothing is read or written there, the status word tells."""
    from xllm_wxh_b200.ops import cuda_ops
    inp = step_input([(4, 1), (0, 3)], [7, 8])
    last = torch.zeros(4, 64, device=DEV)
    ops.token_shift(torch.randn(4, 64, device=DEV), torch.rand(5, 64, device=DEV), last, inp)
    assert cuda_ops.read_status() != 0 and last.abs().sum() == 0          # reading clears the word
    assert status_ok()


# ----------------------------------------------------------------------------- attention with kept first keys
def attention_case(spans, H, G, d, dv, size, keep, block, dtype, seed=0, edit=None, pad=0, scale=None):
    g = torch.Generator().manual_seed(seed)
    scale = scale or 2.0 / math.sqrt(d)
    need = [-(-(b + n) // block) for b, n in spans]
    perm = (torch.randperm(sum(need), generator=g) + 1).tolist()
    tables = [[perm.pop() for _ in range(k)] for k in need]
    kc = torch.randn(sum(need) + 1, block, G, d, generator=g).to(dtype)
    vc = torch.randn(sum(need) + 1, block, G, dv, generator=g).to(dtype)
    qs, want = [], []
    for (before, n), t in zip(spans, tables):
        T = before + n
        q, k, v = (torch.randn(T, h, w, generator=g) for h, w in ((H, d), (G, d), (G, dv)))
        if edit:
            edit(q, k, v)
        q, k, v = (x.to(dtype) for x in (q, k, v))
        blocks = torch.tensor(t)[torch.arange(T) // block]
        kc[blocks, torch.arange(T) % block], vc[blocks, torch.arange(T) % block] = k, v
        qs.append(q[before:])
        want.append(O.attention_core(q.double(), k.double(), v.double(), scale, size, keep)[before:].flatten(1))
    q = torch.cat(qs + [torch.zeros(pad, H, d, dtype=dtype)])
    inp = step_input(spans, [1] * len(spans), block, tables, pad)
    got = ops.paged_attention_ext(q.to(DEV), kc.to(DEV), vc.to(DEV), inp, scale, size, 0, None, None, keep)
    return got[:got.shape[0] - pad], torch.cat(want)


HEADS = [(4, 1, 56, 40), (8, 2, 128, 128), (6, 2, 64, 48), (3, 3, 16, 96), (5, 1, 128, 24), (4, 2, 20, 36), (2, 1, 160, 144)]
SPANS = [(129, 1), (250, 1), (63, 1), (64, 1), (500, 1), (0, 1), (0, 200), (37, 2), (5, 64), (128, 130), (300, 150)]


@pytest.mark.parametrize("heads", HEADS)
@pytest.mark.parametrize("size,keep,block,pad", [(37, 20, 16, 0), (96, 1, 64, 3), (128, 64, 32, 0), (1 << 20, 5, 128, 0), (1, 3, 16, 0), (64, 130, 64, 0),
                                                 (10, 65, 16, 3), (200, 0, 64, 0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention(heads, size, keep, block, pad, dtype):
    got, want = attention_case(SPANS, *heads, size, keep, block, dtype, seed=sum(heads), pad=pad)
    assert rel(got, want) < (8e-3 if dtype == torch.bfloat16 else 1e-5)
    assert (got.double().cpu() - want).abs().max() < (0.06 if dtype == torch.bfloat16 else 1e-4)
    assert status_ok()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", [(40, 20), (64, 64), (33, 1), (100, 15), (16, 48)])
def test_one_key_just_inside_or_outside(size, keep, dtype):
    """One key stands out by far (its value too): rows that see it come out large, all others small.  It lies among the kept
    first keys, right behind them, at block and tile borders; the rows lie around the place where it leaves the window."""
    for planted in sorted({0, keep - 1, keep, keep + 1, 15, 16, 63, 64, 70}):
        def edit(q, k, v):
            q[:] = q * 0.05 + 1.0
            k[:] = k * 0.05
            k[planted] = 2.0
            v[planted] = 30.0
        end = planted + size
        spans = [(p, 1) for p in (end - 2, end - 1, end, end + 1, end + 200) if p > planted]
        spans += [(0, end + 9), (max(planted, end - 3), 7), (end + 130, 70)]
        got, want = attention_case(spans, 4, 2, 64, 64, size, keep, 16, dtype, seed=planted, edit=edit, scale=0.1)
        assert rel(got, want) < (8e-3 if dtype == torch.bfloat16 else 1e-5), planted
        seen = want.abs().max(-1).values > 5
        assert (got.cpu()[~seen].abs() < 6).all() and (got.cpu()[seen].abs().max(-1).values > 4).all(), planted
    assert status_ok()


def test_long_context_splits_and_merges():
    """Few sequences over many keys: key ranges, the kept keys among them, are split in decode and prefill."""
    for spans, heads, size, keep in (([(5000, 1), (4100, 1), (3000, 1)], (8, 2, 128, 128), 2600, 300), ([(3900, 100)], (4, 2, 64, 96), 3000, 200),
                                     ([(4095, 1), (3900, 100)], (4, 2, 128, 128), 1 << 20, 5), ([(3900, 100)], (4, 2, 64, 64), 1500, 2000),
                                     ([(4000, 1)], (4, 4, 64, 64), 100, 3000)):
        got, want = attention_case(spans, *heads, size, keep, 64, torch.bfloat16, scale=0.25)
        assert rel(got, want) < 1e-2
    assert status_ok()


# ----------------------------------------------------------------------------- the other kernels
@pytest.mark.parametrize("H", [67, 72, 336, 2048, 4096, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_kernels(H, dtype):
    g = torch.Generator().manual_seed(H)
    tol = 5e-3 if dtype == torch.bfloat16 else 2e-6
    T = 37
    y, w = torch.randn(T, H, generator=g).to(dtype), torch.randn(H, generator=g).to(dtype)
    x, y32, vec = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g), torch.randn(H, generator=g)
    x[3], y[3], y32[4] = x[3] * 1e-4, y[3] * 1e-4, -vec                  # eps matters
    xd = x.to(DEV)
    h = ops.add_norm(y.to(DEV), xd, 0.37, w.to(DEV), 1e-6)
    want = x.double() + 0.37 * y.double()
    assert rel(xd, want) < 1e-6 and rel(h, O.rms_norm(want, w.double(), 1e-6)) < tol
    h = ops.replace_norm(y32.to(DEV), vec.to(DEV), xd, w.to(DEV), 1e-6)
    want = y32.double() + vec.double()
    assert rel(xd, want) < 1e-6 and rel(h, O.rms_norm(want, w.double(), 1e-6)) < tol
    table, ids = torch.randn(50, H, generator=g).to(dtype), torch.randint(0, 50, (T,), generator=g).int()
    rows = ops.split_rows(x.to(DEV), ids.to(DEV), table.to(DEV), 1.0).cpu()
    assert torch.equal(rows, ops.ref.split_rows(x, ids, table, 1.0))


@pytest.mark.parametrize("dims", [(4, 2, 56, 40), (3, 1, 128, 64), (2, 2, 21, 13), (5, 1, 8, 256), (32, 8, 128, 128)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_qknorm_all_and_gate(dims, dtype):
    H, G, d, dv = dims
    g = torch.Generator().manual_seed(sum(dims))
    T, n = 29, H * dv
    row = torch.randn(T, (H + G) * d + G * dv + n, generator=g).to(dtype)
    qw, kw = (1 + 0.3 * torch.randn(H * d, generator=g)).to(dtype), (1 + 0.3 * torch.randn(G * d, generator=g)).to(dtype)
    kd, vd = torch.zeros(8, 16, G, d, dtype=dtype, device=DEV), torch.zeros(8, 16, G, dv, dtype=dtype, device=DEV)
    slots = torch.randperm(100, generator=g)[:T].int()
    rd = row.to(DEV)
    q = ops.qknorm_all_kvwrite(rd, slots.to(DEV), qw.to(DEV), kw.to(DEV), 1e-6, kd, vd, H, G)
    a, b, c, gate = row.double().split([H * d, G * d, G * dv, n], -1)
    tol = 4e-3 if dtype == torch.bfloat16 else 1e-6
    assert rel(q, O.rms_norm(a, qw.double(), 1e-6)) < tol
    assert rel(kd.view(-1, G * d)[slots.long().to(DEV)], O.rms_norm(b, kw.double(), 1e-6)) < tol
    assert torch.equal(vd.view(-1, G * dv)[slots.long().to(DEV)].cpu().double(), c)
    rest = torch.ones(128, dtype=torch.bool)
    rest[slots.long()] = False
    assert kd.view(128, -1).cpu()[rest].abs().sum() == 0 and vd.view(128, -1).cpu()[rest].abs().sum() == 0
    assert torch.equal(rd[:, -n:].cpu(), row[:, -n:])
    o, both = torch.randn(T, n, generator=g).to(dtype), torch.zeros(T, n + 16, dtype=dtype, device=DEV)
    ops.gate_into(o.to(DEV), rd[:, -n:], 0.8, both[:, :n])
    assert rel(both[:, :n], 0.8 * o.double() * O.sigmoid(gate)) < tol and both[:, n:].abs().sum() == 0


@pytest.mark.parametrize("M_,N,K", [(1, 16, 272), (300, 128, 256), (77, 67, 51), (130, 520, 80), (5, 3, 8), (400, 1024, 2048), (64, 4096, 2304)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_products(M_, N, K, dtype):
    g = torch.Generator().manual_seed(M_ + N + K)
    x, w = torch.randn(M_, K, generator=g).to(dtype), (2 * torch.randn(N, K, generator=g) / math.sqrt(K)).to(dtype)
    b = torch.randn(N, generator=g).to(dtype)
    y = x.double() @ w.double().T
    tol = 4e-3 if dtype == torch.bfloat16 else 2e-6
    xd, wd = x.to(DEV), w.to(DEV)
    assert rel(ops.linear(xd, wd, b.to(DEV)), y + b.double()) < tol
    assert rel(ops.act_linear(xd, wd, "tanh"), torch.tanh(y)) < tol
    assert rel(ops.act_linear(xd, wd, "relu2"), O.squared_relu(y)) < tol
    assert status_ok()


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in (("mixed", M.mixed_config()), ("odd", M.odd_config()),
                      ("wide", M.config([(M.parallel(heads=8, kv_heads=2, dim=128, vdim=128, window=150, keep_first=70, t_heads=4, t_dim=64), M.dense(ff=512)),
                                         (M.scan(inner=512, state=16, conv=4, dt_rank=16), None),
                                         (M.parallel(heads=8, kv_heads=4, dim=64, vdim=64, window=64, keep_first=8, t_heads=2, t_dim=128), M.dense(ff=256))],
                                        width=256, vocab=1024, loop=(1, 3, 2)))):
        sd = M.weights(cfg, 5)
        out[name] = cfg, {k: v.double() for k, v in sd.items()}, M.save(cfg, sd, tmp_path_factory.mktemp(name))
    return out


def check(got, want, dtype):
    e = M.row_error(got, want)
    if dtype == "float32":
        assert e.max() < 1e-4, e.max()
    else:
        assert e.median() < 0.03 and e.quantile(0.9) < 0.06 and e.max() < 0.2, (e.median(), e.quantile(0.9), e.max())


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
        assert e.median() < (1e-5 if dtype == "float32" else 0.03)
    g = eng.worker._graphs
    assert g is not None and g.num_replays > 40 and status_ok()


SEQS = [("a", 70), ("b", 9), ("c", 40), ("d", 23), ("e", 66), ("f", 31)]
PLAN = [[("a", 30), ("b", 8)], [("c", 5), ("a", 2), ("b", 1)], [("d", 20)], [("a", 1), ("d", 1), ("c", 33)], [("a", 37), ("d", 2), ("c", 2)],
        [("e", 50), ("f", 2)], [("f", 28), ("e", 1)], [("e", 15), ("f", 1)]]


@pytest.mark.parametrize("kw", [dict(block_size=16), dict(block_size=64), dict(block_size=16, enable_prefill_piecewise_graph=True)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batches_blocks_and_slots_used_again(models, dtype, kw):
    cfg, sd, path = models["mixed"]
    seqs = {n: M.tokens(c, cfg["vocab"], 60 + i) for i, (n, c) in enumerate(SEQS)}
    room = sum(-(-n // kw["block_size"]) for n in (70, 40, 23, 9))
    eng = M.engine(path, DEV, dtype, blocks=room + 1, num_state_slots=3, **kw)
    for t in (t for run in eng.worker.state_caches for t in run):
        t.fill_(1e4)
    for _ in range(3):                                           # graphs of steps with portions are captured when they come back
        got = M.replay(eng, seqs, PLAN)
        for n, toks in seqs.items():
            check(got[n], O.forward(sd, cfg, toks), dtype)
    assert status_ok()


@pytest.mark.parametrize("kw", [{}, dict(enable_graph=False), dict(enable_schedule_overlap=True, enable_prefill_piecewise_graph=True),
                                dict(max_tokens_per_batch=24, max_tokens_per_chunk_for_prefill=7), dict(num_state_slots=2),
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


def test_long_decoding(models):
    cfg, sd, path = models["wide"]
    toks = M.tokens(700, cfg["vocab"], 90)
    want = O.forward(sd, cfg, toks)
    got = M.replay(M.engine(path, DEV, "float32"), {"a": toks}, M.alone("a", toks, 40))["a"]
    check(got, want, "float32")


def test_sleep_and_wakeup_keep_the_outputs(models):
    cfg, _, path = models["mixed"]
    eng = M.engine(path, DEV, "bfloat16")
    llm = LLM(model=path, devices=DEV, engine=eng)
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    first = [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)]
    for level in (1, 2):
        assert eng.sleep(level) and eng.wakeup()
        assert [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)] == first
