"""Small random Govuvik models for tests: configuration dictionaries, weights, checkpoint directories."""
import math

import torch

from tests.helpers.movolorn_models import alone, engine, replay, row_error, save, tokens  # noqa: F401


def parallel(heads=6, kv_heads=3, dim=24, vdim=16, window=19, conv=3, rot=10, base=3e3, scaling=(5.0, 1.5, 3.0, 60), scale=None, g_heads=3,
             g_dim=20, g_vdim=12, tau=5.0):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or 1.2 / math.sqrt(dim),
                 "mask": {"size": window}, "rot": r},
        "right": {"heads": g_heads, "dim": g_dim, "vdim": g_vdim, "tau": tau}}}


def memory(heads=3, dim=20, vdim=28, cap=6.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def moe(ff=40, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=72, vocab=210, taps=3, softcap=12.0, eps=3e-6):
    cfg = {"architecture": "Govuvik", "norm": {"eps": eps}, "vocab": vocab, "width": width, "canon": {"taps": taps},
           "layers": [{**m, "mlp": f} for m, f in layers]}
    if softcap:
        cfg["logit_softcap"] = softcap
    return cfg


def mixed_config(width=72, vocab=210):
    """Every branch in one model: both mixers with and without a feed-forward, layers of different sizes."""
    return config([
        (memory(), None),
        (parallel(), moe()),
        (parallel(heads=4, kv_heads=1, dim=40, vdim=56, window=33, conv=5, rot=40, scaling=None, g_heads=2, g_dim=48, g_vdim=24, tau=1.0), None),
        (memory(heads=2, dim=40, vdim=24, cap=12.0), moe(ff=24, experts=9, top=4)),
        (parallel(heads=4, kv_heads=4, dim=32, vdim=32, window=7, conv=2, rot=2, base=50.0, g_heads=4, g_dim=8, g_vdim=40, tau=30.0), moe(experts=3, top=3)),
    ], width=width, vocab=vocab)


def odd_config():
    """Sizes that no vector load or tensor-core tile divides; one tap, a window of one, one expert, no bound of the logits."""
    return config([
        (parallel(heads=3, kv_heads=3, dim=21, vdim=13, window=11, conv=1, rot=6, g_heads=3, g_dim=9, g_vdim=14), moe(ff=45, experts=1, top=1)),
        (memory(heads=1, dim=7, vdim=30), moe(ff=33, experts=7, top=1)),
        (parallel(heads=5, kv_heads=1, dim=18, vdim=10, window=1, conv=7, rot=18, scaling=None, g_heads=1, g_dim=30, g_vdim=5), None),
        (memory(heads=5, dim=9, vdim=6, cap=2.0), None),
    ], width=67, vocab=131, taps=1, softcap=None)


def shapes(cfg, decay_rank=7):
    H = cfg["width"]
    out = {"embed": (cfg["vocab"], H), "head": (cfg["vocab"], H), "final.norm": (H,), "embed.norm": (H,)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out.update({p + "norm1": (H,), p + "norm1b": (H,), p + "canon1": (H, cfg["canon"]["taps"])})
        if f:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            out.update({p + "norm2": (H,), p + "norm2b": (H,), p + "mlp.router": (n, H)})
            for e in range(n):
                out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = (ff, H), (H, ff)
        p += "mix."
        if layer["type"] == "mlstm":
            h, d, v = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({p + "q": (d, H), p + "k": (d, H), p + "v": (v, H), p + "g": (v, H), p + "o": (H, v), p + "norm": (v,), p + "i": (h, H),
                        p + "i.b": (h,), p + "f": (h, H), p + "f.b": (h,)})
            continue
        a, t = m["left"], m["right"]
        for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            out[f"{p}left.{n}"], out[f"{p}left.{n}.conv"] = (rows, H), (rows, a["conv"])
            if n != "v":
                out[f"{p}left.{n}.norm"] = (rows,)
        out.update({p + "left.talk": (a["heads"], a["heads"]), p + "left.temp": (a["heads"],), p + "left.sink": (a["heads"],),
                    p + "left.o": (H, a["heads"] * a["vdim"]), p + "left.out": (H,)})
        p, d, v = p + "right.", t["heads"] * t["dim"], t["heads"] * t["vdim"]
        out.update({p + "q": (d, H), p + "k": (d, H), p + "v": (v, H), p + "g": (v, H), p + "o": (H, v), p + "norm": (t["vdim"],),
                    p + "a1": (decay_rank, H), p + "a2": (d, decay_rank), p + "a2.b": (d,), p + "out": (H,)})
    return out


def weights(cfg, seed=0, decay_rank=7):
    """bf16 values: norm weights away from 1, sharp attention with mixed heads and sinks of either sign, decays and forget gates from
    a few tokens to hundreds, input gates of every size, convolutions that weigh every tap."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in shapes(cfg, decay_rank).items():
        r, u = torch.randn(shape, generator=g), torch.rand(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = 1.4 + 0.3 * r
        elif last.startswith("norm") or last in ("out", "temp"):
            t = 1.0 + 0.25 * r
        elif last == "talk":
            t = torch.eye(shape[0]) + 0.35 * r
        elif last == "sink":
            t = 1.5 * r
        elif last.startswith(("canon", "conv")):
            t = 0.5 * r
        elif name.endswith("a2.b"):
            t = 1 + 5 * u
        elif name.endswith("f.b"):
            t = -1 + 7 * u
        elif name.endswith("i.b"):
            t = -4 + 6 * u
        elif last == "router":
            t = r * (2.0 / math.sqrt(shape[1]))
        elif last == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[1])
        sd[name] = t.to(torch.bfloat16)
    return sd
