"""Small random Falalix models for tests: configuration dictionaries, weights, checkpoint directories."""
import math

import torch

from tests.helpers.movolorn_models import alone, engine, replay, row_error, save, tokens  # noqa: F401


def parallel(heads=4, kv_heads=2, dim=24, vdim=16, window=19, keep_first=5, scale=None, t_heads=3, t_dim=20, left=0.7, right=1.1):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 / math.sqrt(dim),
                 "mask": {"size": window, "keep_first": keep_first}},
        "left_scale": left, "right": {"heads": t_heads, "dim": t_dim}, "right_scale": right}}


def scan(inner=56, state=12, conv=4, dt_rank=6):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "conv": conv, "dt_rank": dt_rank}}


def dense(ff=80):
    return {"kind": "dense", "ff": ff}


def config(layers, width=72, vocab=210, loop=None, eps=3e-6, residual_mult=0.6):
    cfg = {"architecture": "Falalix", "norm": {"eps": eps}, "vocab": vocab, "width": width, "residual_mult": residual_mult,
           "layers": [{**m, "mlp": f} for m, f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def mixed_config(width=72, vocab=210):
    """Every branch in one model: both mixers with and without a feed-forward, layers of different sizes, a looped range in
    the middle."""
    return config([
        (scan(), None),
        (parallel(), dense()),
        (scan(inner=88, state=20, conv=3, dt_rank=8), dense(ff=56)),
        (parallel(heads=6, kv_heads=3, dim=40, vdim=56, window=33, keep_first=2, t_heads=2, t_dim=48, left=1.3, right=0.4), None),
        (parallel(heads=3, kv_heads=1, dim=32, vdim=32, window=7, keep_first=11, t_heads=4, t_dim=32), dense(ff=96)),
    ], width=width, vocab=vocab, loop=(1, 4, 3))


def odd_config():
    """Sizes that no vector load or tensor-core tile divides; a loop over everything; one tap, one state, no kept keys."""
    return config([
        (parallel(heads=2, kv_heads=1, dim=21, vdim=13, window=11, keep_first=3, t_heads=3, t_dim=9), dense(ff=45)),
        (scan(inner=27, state=5, conv=5, dt_rank=3), None),
        (scan(inner=19, state=1, conv=1, dt_rank=1), dense(ff=33)),
        (parallel(heads=3, kv_heads=3, dim=18, vdim=10, window=1, keep_first=0, t_heads=1, t_dim=30), None),
    ], width=67, vocab=131, loop=(0, 4, 2))


def shapes(cfg, decay_rank=7):
    H = cfg["width"]
    out = {"embed": (cfg["vocab"], H), "head": (cfg["vocab"], H), "final.norm": (H,)}
    if cfg.get("loop"):
        out["loop.in"], out["loop.step"] = (H, 2 * H), (cfg["loop"]["times"], H)
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out[p + "norm1"] = (H,)
        if f:
            out[p + "norm2"], out[p + "mlp.up"], out[p + "mlp.down"] = (H,), (f["ff"], H), (H, f["ff"])
        p += "mix."
        if layer["type"] == "mamba1":
            c, n, r = m["inner"], m["state"], m["dt_rank"]
            out.update({p + "in": (2 * c, H), p + "conv": (c, m["conv"]), p + "conv.b": (c,), p + "x": (r + 2 * n, c), p + "dt": (c, r),
                        p + "dt.b": (c,), p + "A_log": (c, n), p + "D": (c,), p + "o": (H, c)})
            continue
        a, t = m["left"], m["right"]
        for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            out[f"{p}left.{n}"], out[f"{p}left.{n}.b"] = (rows, H), (rows,)
            if n != "v":
                out[f"{p}left.{n}.norm"] = (rows,)
        out[p + "left.g"], out[p + "left.o"] = (a["heads"] * a["vdim"], H), (H, a["heads"] * a["vdim"])
        p, n = p + "right.", t["heads"] * t["dim"]
        out.update({p + "mu." + c: (H,) for c in "rkvgw"})
        out.update({p + c: (n, H) for c in "rkvg"})
        out.update({p + "w1": (decay_rank, H), p + "w2": (n, decay_rank), p + "w0": (n,), p + "u": (t["heads"], t["dim"]), p + "norm": (n,),
                    p + "o": (H, n)})
    return out


def weights(cfg, seed=0, decay_rank=7):
    """bf16 values: norm weights away from 1, sharp attention, decays from nearly 1 to a few steps, blends of every size."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in shapes(cfg, decay_rank).items():
        r, u = torch.randn(shape, generator=g), torch.rand(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = 1.5 + 0.3 * r
        elif last.startswith("norm"):
            t = 1.0 + 0.2 * r
        elif ".mu." in name:
            t = 0.1 + 0.8 * u
        elif last == "w0":
            t = -5 + 5.5 * u
        elif last == "A_log":
            t = torch.log(torch.arange(1, shape[1] + 1).float()).expand(shape) + 0.2 * r
        elif name.endswith("dt.b"):
            t = -4 + 3 * u
        elif last in ("D", "u", "b") or name == "loop.step":
            t = 0.5 * r
        elif last == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[1])
        sd[name] = t.to(torch.bfloat16)
    return sd
