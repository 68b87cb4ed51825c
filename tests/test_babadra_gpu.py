"""Babadra on a GPU: every kernel against the plain statement of its mechanism, whole models in bf16 and in true 32-bit against
tests/oracle_babadra.py, decoding through CUDA graphs, greedy generation through the scheduler."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

from tests import oracle_babadra as O
from tests.helpers import babadra_models as M
from tests.helpers.paged_step import PagedStep
from tests.test_babadra_cpu import ROTATIONS, planted, two_map_step
from xllm_wxh_b200 import LLM, SamplingParams, ops
from xllm_wxh_b200.models.layer_spec import RotarySpec

DEV = "cuda:0"
BOTH = pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])


def status_ok():
    from xllm_wxh_b200.ops import cuda_ops
    return cuda_ops.read_status() == 0


def rel(got, want):
    return ((got.double().cpu() - want.double().cpu()).norm() / want.double().cpu().norm()).item()


def tol(dtype, bf=8e-3, f=1e-5):
    return bf if dtype == torch.bfloat16 else f


# ----------------------------------------------------------------------------- differential attention
# tensor cores: both maps' keys in 64 / 128 / 256 columns, more than 16 query rows per value head; fp32 pipe: odd and larger sizes
TWO_MAP = [(4, 1, 32, 40), (8, 2, 64, 128), (6, 3, 24, 64), (2, 2, 128, 96), (10, 1, 64, 64), (4, 2, 72, 16), (12, 1, 40, 128), (3, 1, 20, 12),
           (2, 1, 136, 40), (4, 2, 64, 160)]
LENS = [(0, 1), (0, 200), (129, 1), (37, 2), (250, 1), (5, 64), (128, 130), (63, 1), (64, 1)]


def two_map_want(step, seqs, scale, cap, lam, diff, eps):
    return step.step_rows([O.two_map_core(*s, scale, cap, lam, diff, eps).flatten(1) for s in seqs])


@pytest.mark.parametrize("heads", TWO_MAP)
@pytest.mark.parametrize("cap,block", [(0.0, 16), (2.0, 64), (50.0, 32), (50.0, 128)])
@BOTH
def test_two_map_attention(heads, cap, block, dtype):
    step, q, seqs = two_map_step(LENS, *heads, block, sum(heads), device=DEV, dtype=dtype)
    scale, lam, diff, eps = 2.0 / math.sqrt(heads[2]), 0.7, 0.45, 1e-3
    got = ops.paged_attention_ext(q, *step.caches, step.inp, scale, softcap=cap, mix=(torch.tensor([lam], device=DEV), 1 - diff, eps))
    want = two_map_want(step, seqs, scale, cap, lam, diff, eps)
    assert rel(got, want) < tol(dtype, 1.2e-2) and status_ok()


@BOTH
@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 127, 128, 129, 191])
def test_one_key_that_stands_out(at, dtype):
    """Keys at page and tile borders, at the start, far behind and right at the query."""
    lens = [(0, 200), (at, 1), (at, 2), (at + 1, 1), (199, 1), (300, 1), (190, 40)]
    lens = [(b, n) for b, n in lens if b + n > at]
    step, q, seqs = two_map_step(lens, 4, 2, 64, 64, 16, at, planted(at, 2.0), DEV, dtype)
    got = ops.paged_attention_ext(q, *step.caches, step.inp, 0.1, softcap=50.0, mix=(torch.tensor([0.3], device=DEV), 1.0, 1e-6))
    want = two_map_want(step, seqs, 0.1, 50.0, 0.3, 0.0, 1e-6)
    assert (got.double().cpu() - want).abs().max() < tol(dtype, 0.15, 1e-3) and rel(got, want) < tol(dtype, 2e-2)
    assert status_ok()


def test_long_context_splits_and_merges():
    """Few sequences over many keys: key ranges are split, and the maps are combined by the merge."""
    from xllm_wxh_b200.ops import cuda_ops
    mix = (torch.tensor([0.6], device=DEV), 0.5, 1e-5)
    for lens, heads in (([(5000, 1), (4100, 1), (3000, 1)], (8, 2, 64, 128)), ([(3900, 100)], (4, 2, 64, 96)), ([(2500, 1)], (10, 1, 128, 64)),
                        ([(3900, 100), (4095, 1)], (4, 1, 40, 128))):
        step, q, seqs = two_map_step(lens, *heads, 64, 1, device=DEV, dtype=torch.bfloat16)
        want = two_map_want(step, seqs, 0.25, 30.0, 0.6, 0.5, 1e-5)
        for splits in (1, 3):
            cuda_ops.prefill_kv_split(splits)
            try:
                assert rel(ops.paged_attention_ext(q, *step.caches, step.inp, 0.25, softcap=30.0, mix=mix), want) < 1.2e-2
            finally:
                cuda_ops.prefill_kv_split(1)
    assert status_ok()


def test_bounded_scores_keep_their_accuracy():
    """Small products, products around the change of formula, and products far past the bound."""
    for size in (0.02, 0.5, 2.0, 30.0):
        def edit(q, k, v):
            q *= size
        step, q, seqs = two_map_step([(0, 150), (150, 1)], 4, 2, 64, 64, 64, 3, edit, DEV, torch.bfloat16)
        want = two_map_want(step, seqs, 0.3, 4.0, 0.2, 0.0, 1e-6)
        largest = max(float(torch.einsum("nhid,mhid->hinm", x, y.repeat_interleave(2, 1)).abs().max()) for x, y, _ in seqs)
        for bound in (0.0, largest):
            got = ops.paged_attention_ext(q, *step.caches, step.inp, 0.3, softcap=4.0, mix=(torch.tensor([0.2], device=DEV), 1.0, 1e-6), bound=bound)
            assert rel(got, want) < 1.2e-2


# ----------------------------------------------------------------------------- latent attention
# (heads, unrotated, rotated, value, latent): tensor cores with 64 .. 256 columns and more than 16 heads, the 512 + 64 column kernels,
# the fp32 pipe
LATENT = [(4, 48, 16, 40, 64), (20, 32, 16, 24, 48), (3, 64, 64, 64, 128), (8, 32, 32, 64, 224), (5, 16, 8, 16, 120), (16, 128, 64, 128, 512),
          (48, 64, 64, 32, 512), (4, 128, 64, 32, 512), (1, 64, 64, 48, 512), (6, 128, 64, 64, 512), (3, 13, 6, 11, 21), (1, 24, 40, 136, 200)]


def latent_step(lens, sizes, block, dtype, seed=0, edit=None):
    H, d, r, dv, C = sizes
    g = torch.Generator().manual_seed(seed)
    q = [torch.randn(b + n, H, d + r, generator=g) for b, n in lens]
    c = [torch.randn(b + n, 1, C + r, generator=g) for b, n in lens]
    uk, uv = torch.randn(H, d, C, generator=g) / math.sqrt(C), torch.randn(H, dv, C, generator=g) / math.sqrt(C)
    if edit:
        edit(q, c)
    q, c, uk, uv = [t.to(dtype) for t in q], [t.to(dtype) for t in c], uk.to(dtype), uv.to(dtype)
    return PagedStep(lens, [(t,) for t in c], block, DEV, seed), q, c, uk, uv


def latent_want(step, q, c, uk, uv, d, rot, scale):
    out = []
    for i, (b, n) in enumerate(step.lens):
        lat, key = c[i][:, 0, :uk.shape[2]].double(), c[i][:, 0, uk.shape[2]:].double()
        qr = O.rotate(q[i][..., d:].double(), rot, True)
        o = [O.attend((q[i][:, h, :d].double() @ (lat @ uk[h].double().T).T + qr[:, h] @ key.T) * scale, lat @ uv[h].double().T)
             for h in range(uk.shape[0])]
        out.append(torch.cat(o, -1))
    return step.step_rows(out)


@pytest.mark.parametrize("sizes", LATENT)
@pytest.mark.parametrize("block", [16, 64])
@BOTH
def test_latent_attention(sizes, block, dtype):
    d, r = sizes[1], sizes[2]
    step, q, c, uk, uv = latent_step(LENS, sizes, block, dtype, sum(sizes))
    table = ops.ref.rotary_table(RotarySpec(r, 100.0, True), 400, DEV)
    rot = (table, step.inp.positions, True)
    got = ops.latent_attention(step.step_rows(q).to(DEV), uk.transpose(1, 2).contiguous().to(DEV), uv.to(DEV), step.caches[0][:, :, 0], step.inp,
                               rot, 1.5 / math.sqrt(d + r), d)
    want = latent_want(step, q, c, uk, uv, d, {"dims": r, "base": 100.0}, 1.5 / math.sqrt(d + r))
    assert rel(got, want) < tol(dtype, 1.2e-2) and status_ok()


@pytest.mark.parametrize("sizes", [(4, 48, 16, 40, 64), (20, 32, 16, 24, 48), (3, 64, 64, 64, 128), (16, 128, 64, 128, 512)])
@pytest.mark.parametrize("at", [0, 15, 16, 63, 64, 130])
def test_one_latent_that_stands_out(sizes, at):
    """One latent that every query finds: rows from its own on see it, earlier ones do not."""
    H, d, r, dv, C = sizes

    def edit(q, c):
        for i in range(len(q)):
            q[i] *= 0.05
            q[i][..., :d] += 1.0
            c[i] *= 0.05
            c[i][at, 0, :C] = 2.0
    step, q, c, uk, uv = latent_step([(0, 180), (at, 1), (at + 3, 2), (170, 1)], sizes, 16, torch.bfloat16, at, edit)
    uk = uk.abs()                                      # the planted latent's products with every head's query are large
    rot = (ops.ref.rotary_table(RotarySpec(r, 100.0, True), 400, DEV), step.inp.positions, True)
    scale = 30.0 / (d * C ** 0.5)
    got = ops.latent_attention(step.step_rows(q).to(DEV), uk.transpose(1, 2).contiguous().to(DEV), uv.to(DEV), step.caches[0][:, :, 0], step.inp,
                               rot, scale, d)
    want = latent_want(step, q, c, uk, uv, d, {"dims": r, "base": 100.0}, scale)
    assert rel(got, want) < 2e-2 and status_ok()
    n = want.abs().amax(-1)
    assert n.min() < 0.2 * n.max() or at == 0          # it stands out where it is seen


# ----------------------------------------------------------------------------- the other kernels
@pytest.mark.parametrize("dims,base,scaling", ROTATIONS)
@pytest.mark.parametrize("interleaved", [False, True])
@BOTH
def test_rotations(dims, base, scaling, interleaved, dtype):
    """Behind the norm of q and k (partly rotated heads of aligned and odd sizes), and alone into a strided view."""
    spec = RotarySpec(dims, base, interleaved, *(scaling or ()))
    rot = {"dims": dims, "base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None}
    table = ops.ref.rotary_table(spec, 500, DEV)
    g = torch.Generator().manual_seed(dims)
    for d, dv in ((dims, 16), (dims + 8 - dims % 8 + 16, 24), (dims + 3, 5)):
        T, H, G, first = 29, 3, 1, 400
        qkv = torch.randn(T, 2 * (H + G) * d + G * dv, generator=g).to(dtype)
        qw, kw = (1 + 0.3 * torch.randn(2, d, generator=g)).to(dtype)
        kc, vc = torch.zeros(8, 16, 2 * G, d, dtype=dtype, device=DEV), torch.zeros(8, 16, G, dv, dtype=dtype, device=DEV)
        slots = torch.randperm(100, generator=g)[:T].int()
        at = torch.arange(first, first + T, dtype=torch.int32, device=DEV)
        q = ops.qknorm_kvwrite(qkv.to(DEV), slots.to(DEV), qw.to(DEV), kw.to(DEV), 1e-4, kc, vc, 2 * H, 2 * G, (table, at, interleaved))
        a, b, c = qkv.double().split([2 * H * d, 2 * G * d, G * dv], -1)
        turned = lambda t, n, w: O.rotate(O.plain_norm(t.reshape(T, n, d), w.double(), 1e-4), rot, interleaved, first)
        assert rel(q, turned(a, 2 * H, qw).flatten(1)) < tol(dtype, 4e-3, 2e-6)
        assert rel(kc.view(-1, 2 * G, d)[slots.long().to(DEV)], turned(b, 2 * G, kw)) < tol(dtype, 4e-3, 2e-6)
        assert torch.equal(vc.view(-1, G, dv)[slots.long().to(DEV)].cpu().double(), c.reshape(T, G, dv))
        x = torch.randn(T, H, dims + 7, generator=g).to(dtype).to(DEV)
        out = torch.zeros(T, H, dims + 9, dtype=dtype, device=DEV)
        ops.rotate_into(x[..., 7:], (table, at, interleaved), out[..., :dims])
        assert rel(out[..., :dims], O.rotate(x[..., 7:].double().cpu(), rot, interleaved, first)) < tol(dtype, 4e-3, 2e-6)
        assert out[..., dims:].abs().sum() == 0


@pytest.mark.parametrize("nq,nc,r", [(56, 48, 16), (1536, 512, 64), (19, 21, 6), (8, 200, 8)])
@BOTH
def test_latent_down_kernel(nq, nc, r, dtype):
    g = torch.Generator().manual_seed(nq)
    T = 33
    low = torch.randn(T, nq + nc + r, generator=g).to(dtype)
    low[2] *= 1e-3                                             # eps matters
    qw, kw = (1 + 0.3 * torch.randn(nq, generator=g)).to(dtype), (1 + 0.3 * torch.randn(nc, generator=g)).to(dtype)
    cache = torch.zeros(5, 16, nc + r, dtype=dtype, device=DEV)
    slots = torch.randperm(80, generator=g)[:T].int()
    table = ops.ref.rotary_table(RotarySpec(r, 60.0, True), 200, DEV)
    at = torch.arange(100, 100 + T, dtype=torch.int32, device=DEV)
    cq = ops.latent_down(low.to(DEV), nq, nc, qw.to(DEV), kw.to(DEV), 1e-5, (table, at, True), slots.to(DEV), cache)
    x = low.double()
    assert rel(cq, O.plain_norm(x[:, :nq], qw.double(), 1e-5)) < tol(dtype, 4e-3, 2e-6)
    rows = cache.view(-1, nc + r)[slots.long().to(DEV)]
    assert rel(rows[:, :nc], O.plain_norm(x[:, nq:nq + nc], kw.double(), 1e-5)) < tol(dtype, 4e-3, 2e-6)
    assert rel(rows[:, nc:], O.rotate(x[:, nq + nc:], {"dims": r, "base": 60.0}, True, 100)) < tol(dtype, 4e-3, 2e-6)
    rest = torch.ones(80, dtype=torch.bool)
    rest[slots.long()] = False
    assert cache.view(80, -1).cpu()[rest].abs().sum() == 0


@pytest.mark.parametrize("H,T,K,N", [(4, 300, 48, 64), (3, 1, 128, 512), (20, 129, 40, 72), (5, 130, 200, 24), (2, 40, 13, 21), (1, 7, 64, 8)])
@BOTH
def test_products_of_heads(H, T, K, N, dtype):
    g = torch.Generator().manual_seed(T)
    wide = torch.randn(T, H, K + 24, generator=g).to(dtype)
    w = (torch.randn(H, N, K, generator=g) / math.sqrt(K)).to(dtype)
    want = torch.einsum("thk,hnk->htn", wide[..., :K].double(), w.double())
    views = [(wide.to(DEV)[..., :K].transpose(0, 1), "token-major"), (wide[..., :K].transpose(0, 1).contiguous().to(DEV), "head-major")]
    for x, _ in views:
        for out in (torch.zeros(H, T, N, dtype=dtype, device=DEV), torch.zeros(T, H, N + 16, dtype=dtype, device=DEV)[..., :N].transpose(0, 1)):
            assert rel(ops.heads_linear(x, w.to(DEV), out), want) < tol(dtype, 4e-3, 2e-6)
            assert out._base is None or out._base[..., N:].abs().sum() == 0
    assert status_ok()


@pytest.mark.parametrize("H", [67, 72, 336, 2048, 4096, 9000])
@BOTH
def test_norm_kernels(H, dtype):
    g = torch.Generator().manual_seed(H)
    T, V, P = 37, 50, 60
    table, pos, y, ls, w = (torch.randn(s, generator=g).to(dtype) for s in ((V, H), (P, H), (T, H), (H,), (H,)))
    y[3] *= 1e-4
    ids, at = torch.randint(0, V, (T,), generator=g).int(), torch.randint(0, P, (T,), generator=g).int()
    d = [t.to(DEV) for t in (ids, table, at, pos, y, ls, w)]
    rows = table[ids.long()].double() * 3.5 + pos[at.long()].double()
    x, h = ops.embed_rms_norm(d[0], d[1], 3.5, d[6], 1e-3, d[2], d[3], 1.0)
    assert rel(x, rows) < 1e-6 and rel(h, O.centred_norm(rows, w.double(), 1e-3)) < tol(dtype, 5e-3, 2e-6)
    lead = (d[0], d[1], 3.5, d[2], d[3])
    x0 = torch.randn(T, H, generator=g)
    for again in (None, lead):
        x = x0.to(DEV)
        h = ops.add_norm(d[4], x, 1.0, d[6], 1e-3, d[5], 1.0, again)
        want = x0.double() + ls.double() * y.double() + (rows if again else 0)
        assert rel(x, want) < 1e-6 and rel(h, O.centred_norm(want, w.double(), 1e-3)) < tol(dtype, 5e-3, 2e-6)
    x = x0.to(DEV)
    h = ops.lead_norm(lead, x, d[6], 1e-3, 1.0)
    assert rel(x, x0.double() + rows) < 1e-6 and rel(h, O.centred_norm(x0.double() + rows, w.double(), 1e-3)) < tol(dtype, 5e-3, 2e-6)


@pytest.mark.parametrize("M_,ff,K", [(3, 80, 272), (400, 1024, 512), (150, 45, 64), (64, 512, 4096)])
@BOTH
def test_clamped_gate_and_bounded_products(M_, ff, K, dtype):
    from xllm_wxh_b200.ops import cuda_ops
    g = torch.Generator().manual_seed(ff)
    x, w = (torch.randn(M_, K, generator=g) * 2).to(dtype), (torch.randn(2 * ff, K, generator=g) / math.sqrt(K)).to(dtype)
    a, b = x.double() @ w[:ff].double().T, x.double() @ w[ff:].double().T
    for limit in (0.7, 5.0):
        want = O.clamped_gate(a, b, limit)
        assert rel(ops.gated_linear(x.to(DEV), w.to(DEV), "clamped", False, limit), want) < tol(dtype, 1e-2, 3e-6)
        if dtype == torch.bfloat16 and ff % 16 == 0:
            assert rel(ops.gated_linear(x.to(DEV), cuda_ops.interleave_gate_up(w.to(DEV)), "clamped", True, limit), want) < 8e-3
    for cap in (0.5, 20.0):
        assert rel(ops.linear_softcap(x.to(DEV), w.to(DEV), cap), O.softcap(x.double() @ w.double().T, cap)) < tol(dtype, 4e-3, 2e-6)
    assert status_ok()


@pytest.mark.parametrize("E,top", [(14, 3), (128, 8), (1, 1), (40, 32), (500, 5)])
def test_router_kernel(E, top):
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(50, E, generator=g) * 40, torch.randn(E, generator=g) * 20
    w, ids = ops.moe_router(z.to(DEV), top, "softmax_chosen", bias=b.to(DEV))
    for t in range(50):
        want = O.route(z[t], b, top)                       # in fp32, as the kernel adds the bias
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].cpu(), torch.stack([x for _, x in want]), rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("width,ff,experts,top", [(272, 80, 7, 3), (512, 64, 12, 5), (67, 27, 5, 2)])
@pytest.mark.parametrize("T", [1, 7, 300])
@BOTH
def test_mixture_kernels(width, ff, experts, top, T, dtype):
    from xllm_wxh_b200.ops import moe_cuda
    cfg = M.config([(M.latent(), M.moe(ff=ff, experts=experts, top=top))], width=width)
    sd = {k: v.to(dtype) for k, v in M.weights(cfg, T).items()}
    p, g = "l0.mlp.", torch.Generator().manual_seed(T)
    h, x = torch.randn(T, width, generator=g).to(dtype), torch.randn(T, width, generator=g)
    dev = {k: v.to(DEV) for k, v in sd.items()}
    w, ids = ops.moe_router(ops.linear_f32(h.to(DEV), dev[p + "router"]), top, "softmax_chosen", bias=dev[p + "router.b"].float())
    w13 = torch.stack([torch.cat([dev[f"{p}e{e}.gate"], dev[f"{p}e{e}.up"]]) for e in range(experts)])
    w2 = torch.stack([dev[f"{p}e{e}.down"] for e in range(experts)])
    d = {k: v.double() for k, v in sd.items()}
    y = torch.zeros(T, width, dtype=torch.float64)
    for t in range(T):                                        # the experts that the kernel chose (checked above on its own)
        for e, wt in zip(ids[t].tolist(), w[t].double().cpu()):
            y[t] += wt * O.gated_ff(d, f"{p}e{e}.", h[t:t + 1].double(), 0.8)[0]
    lead = (torch.arange(T, dtype=torch.int32, device=DEV) % 9, dev["embed"], 1.3, torch.arange(T, dtype=torch.int32, device=DEV), dev["pos"])
    rows = d["embed"][torch.arange(T) % 9] * 1.3 + d["pos"][:T]
    for inter in (False, True):
        if inter and (dtype != torch.bfloat16 or ff % 16):
            continue
        wi = moe_cuda.interleave_w13(w13.clone()) if inter else w13
        for again in (None, lead):
            xd, want = x.to(DEV), x.double() + d["l0.ls2"] * y + (rows if again else 0)
            out = ops.moe_add_norm(h.to(DEV), wi, w2, w, ids, dev["l0.ls2"], xd, dev["final.norm"], 1e-6, "clamped", inter, 0.8, 1.0, again)
            assert rel(xd, want) < tol(dtype, 8e-3, 5e-6)
            assert rel(out, O.centred_norm(want, d["final.norm"], 1e-6)) < tol(dtype, 8e-3, 5e-6)
    assert status_ok()


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    wide = M.config([(M.latent(heads=16, dim=128, rot_dim=64, vdim=64, kv_rank=512, q_rank=96), M.dense(ff=512)),
                     (M.two_map(heads=8, kv_heads=2, dim=64, vdim=128, dims=64), M.moe(ff=128)),
                     (M.latent(heads=24, dim=32, rot_dim=32, vdim=32, kv_rank=160, q_rank=64), None),
                     (M.two_map(heads=12, kv_heads=1, dim=96, vdim=64, dims=48), M.dense(ff=256))],
                    width=256, vocab=1024, loop=(0, 2, 2))
    out = {}
    for name, cfg in (("mixed", M.mixed_config()), ("odd", M.odd_config()), ("wide", wide)):
        sd = M.weights(cfg, 5)
        out[name] = cfg, {k: v.double() for k, v in sd.items()}, M.save(cfg, sd, tmp_path_factory.mktemp(name))
    return out


def check(got, want, dtype):
    e = M.row_error(got, want)
    if dtype == "float32":
        assert e.max() < 1e-4, e.max()
    else:                       # a close call of a router may go the other way in bf16
        assert e.median() < 0.03 and e.quantile(0.9) < 0.08, (e.median(), e.quantile(0.9))


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_whole_portions_and_decoding(models, name, dtype):
    cfg, sd, path = models[name]
    toks = M.tokens(230, cfg["vocab"], 50)
    res = []
    want = O.forward(sd, cfg, toks, res)
    eng, got = M.engine(path, DEV, dtype), []
    eng.worker.model.residual_hook = lambda r, x: got.append(x[:230].cpu())
    hooked = M.replay(eng, {"a": toks}, [[("a", 230)]])["a"]
    assert len(got) == len(res)
    for a, b in zip(got, res):
        check(a, b, dtype)
    eng.worker.model.residual_hook = None
    out = M.replay(eng, {"a": toks}, [[("a", 230)]])["a"]
    check(out, want, dtype)
    check(hooked, want, dtype)
    for cuts in ((190,), (2, 3, 64, 7, 99), (37, 37, 37, 37), (2,) * 95):
        part = M.replay(eng, {"a": toks}, M.alone("a", toks, *cuts))["a"]
        check(part, want, dtype)
        # the way the tokens are cut changes nothing beyond rounding
        e = M.row_error(part, out)
        assert e.median() < (1e-5 if dtype == "float32" else 0.03)
    g = eng.worker._graphs
    assert g is not None and g.num_replays > 40 and status_ok()


@pytest.mark.parametrize("block_size", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batches_and_blocks_used_again(models, name, dtype, block_size):
    cfg, sd, path = models[name]
    seqs = {n: M.tokens(c, cfg["vocab"], 60 + i) for i, (n, c) in enumerate([("a", 70), ("b", 9), ("c", 40), ("d", 23), ("e", 66), ("f", 31)])}
    steps = [[("a", 30), ("b", 8)], [("c", 5), ("a", 2), ("b", 1)], [("d", 20)], [("a", 1), ("d", 1), ("c", 33)], [("a", 37), ("d", 2), ("c", 2)],
             [("e", 50), ("f", 2)], [("f", 28), ("e", 1)], [("e", 15), ("f", 1)]]
    room = sum(-(-n // block_size) for n in (70, 40, 23, 9))
    got = M.replay(M.engine(path, DEV, dtype, block_size=block_size, blocks=room + 1), seqs, steps)
    for n, toks in seqs.items():
        check(got[n], O.forward(sd, cfg, toks), dtype)
    assert status_ok()


def test_long_decoding(models):
    cfg, sd, path = models["mixed"]
    toks = M.tokens(400, cfg["vocab"], 10)
    want = O.forward(sd, cfg, toks)
    for dtype in ("float32", "bfloat16"):
        check(M.replay(M.engine(path, DEV, dtype), {"a": toks}, M.alone("a", toks, 3))["a"], want, dtype)
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
    llm = LLM(model=path, devices=DEV, engine=(eng := M.engine(path, DEV, "bfloat16")))
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    first = [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)]
    for level in (1, 2):
        assert eng.sleep(level) and eng.wakeup()
        assert [o.outputs[0].token_ids for o in llm.generate([[1, 2, 3], [9] * 20], sp)] == first
