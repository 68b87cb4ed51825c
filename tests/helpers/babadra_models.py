"""Small random Babadra models for tests: configuration dictionaries, weights, checkpoint directories."""
import math

import torch

from tests.helpers.movolorn_models import alone, engine, replay, row_error, save, tokens  # noqa: F401


def latent(heads=4, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=56, base=9000.0, scaling=(3.0, 96, 8.0, 1.5), scale=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "q_rank": q_rank, "rot": rot, "scale": scale or 1.4 / math.sqrt(dim + rot_dim)}}


def two_map(heads=4, kv_heads=2, dim=32, vdim=40, dims=16, base=5000.0, softcap=9.0, diff=0.35, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": dims, "base": base}, "diff": diff,
         "scale": scale or 1.2 / math.sqrt(dim)}
    if softcap:
        m["softcap"] = softcap
    return {"type": "attention", "mixer": m}


def dense(ff=80, limit=1.1):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff=48, experts=6, top=3, limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=72, vocab=210, loop=None, eps=3e-5, emb_scale=1.7, positions=512, logit_softcap=6.0):
    cfg = {"architecture": "Babadra", "embedding": {"scale": emb_scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "max_positions": positions, "layers": [{**m, "mlp": f} for m, f in layers]}
    if logit_softcap:
        cfg["logit_softcap"] = logit_softcap
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def mixed_config(width=72, vocab=210):
    """Every branch in one model: both mixers with and without a feed-forward, layers of different sizes, scaled and plain
    rotations, partly and wholly rotated heads, a looped range in the middle."""
    return config([
        (two_map(), moe()),
        (latent(), dense()),
        (two_map(heads=6, kv_heads=3, dim=24, vdim=56, dims=24, softcap=4.0, diff=0.7), None),
        (latent(heads=3, dim=40, rot_dim=8, vdim=24, kv_rank=72, q_rank=32, scaling=None), moe(ff=32, experts=5, top=2, limit=1.9)),
        (two_map(heads=5, kv_heads=1, dim=48, vdim=64, dims=32, softcap=30.0, diff=0.2), dense(ff=96, limit=2.5)),
    ], width=width, vocab=vocab, loop=(1, 4, 3))


def odd_config():
    """Sizes that no vector load or tensor-core tile divides; a loop over everything; one expert of one, no bounds on scores
    and logits."""
    return config([
        (latent(heads=3, dim=13, rot_dim=6, vdim=11, kv_rank=21, q_rank=19, scaling=(2.0, 30, 6.0, 1.0)), moe(ff=27, experts=7, top=7)),
        (two_map(heads=2, kv_heads=1, dim=21, vdim=13, dims=10, softcap=0, diff=0.9), dense(ff=45)),
        (two_map(heads=3, kv_heads=3, dim=9, vdim=17, dims=2), moe(ff=19, experts=1, top=1, limit=0.4)),
    ], width=67, vocab=131, loop=(0, 3, 2), logit_softcap=0)


def shapes(cfg):
    H = cfg["width"]
    out = {"embed": (cfg["vocab"], H), "head": (cfg["vocab"], H), "pos": (cfg["max_positions"], H), "final.norm": (H,)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out[p + "norm1"] = out[p + "ls1"] = (H,)
        q = p + "mix."
        if layer["type"] == "latent_attention":
            out.update({q + "dq": (m["q_rank"], H), q + "dq.norm": (m["q_rank"],), q + "uq": (m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        q + "dkv": (m["kv_rank"] + m["rot_dim"], H), q + "dkv.norm": (m["kv_rank"],),
                        q + "uk": (m["heads"] * m["dim"], m["kv_rank"]), q + "uv": (m["heads"] * m["vdim"], m["kv_rank"])})
        else:
            out.update({q + "q": (m["heads"] * 2 * m["dim"], H), q + "k": (m["kv_heads"] * 2 * m["dim"], H), q + "v": (m["kv_heads"] * m["vdim"], H)})
            out.update({q + n: (m["dim"],) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
        out[q + "o"] = (H, m["heads"] * m["vdim"])
        if not f:
            continue
        out[p + "norm2"] = out[p + "ls2"] = (H,)
        p += "mlp."
        nets = [("", f.get("ff"))]
        if f["kind"] == "moe":
            n = f["router"]["experts"]
            out[p + "router"], out[p + "router.b"] = (n, H), (n,)
            nets = [(f"e{e}.", f["expert"]["ff"]) for e in range(n)]
        for q, ff in nets:
            out[p + q + "gate"] = out[p + q + "up"] = (ff, H)
            out[p + q + "down"] = (H, ff)
    return out


def weights(cfg, seed=0):
    """bf16 values: norm weights away from their neutral value, sharp attention in both maps (q / k norm weights near 1.5), scores
    and logits that the bounds bend, gates on both sides of their limits, layer scales of both signs, position vectors that weigh
    as much as tokens, router biases that decide some choices."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name.endswith(("mix.q.norm", "mix.k.norm")):
            t = 1.5 + 0.3 * r
        elif name.endswith(("dq.norm", "dkv.norm")):
            t = 1.3 + 0.3 * r
        elif last.startswith("norm"):
            t = 0.3 * r
        elif last in ("ls1", "ls2"):
            t = 0.8 * torch.sign(r) + 0.3 * r
        elif last[:2] in ("lq", "lk"):
            t = 0.3 * r
        elif last == "b":
            t = 0.8 * r
        elif last in ("embed", "pos"):
            t = r
        elif last in ("gate", "up", "head"):
            t = r * (1.5 / math.sqrt(shape[1]))
        else:
            t = r / math.sqrt(shape[1])
        sd[name] = t.to(torch.bfloat16)
    return sd
