"""Small random Movolorn models for tests: configuration dictionaries, weights, checkpoint directories."""
import json
import math
import os

import torch


def attn(heads=4, kv_heads=2, dim=24, vdim=16, chunk=37, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 / math.sqrt(dim), "mask": {"size": chunk}}


def dense(ff=80):
    return {"kind": "dense", "ff": ff}


def moe(ff=48, experts=6, identity=2, top=3, groups=(4, 2), shared=64):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=72, vocab=210, loop=None, eps=3e-6, emb_scale=1.7):
    cfg = {"architecture": "Movolorn", "embedding": {"scale": emb_scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def mixed_config(width=72, vocab=210):
    """Every branch in one model: dense and mixture layers, one layer without a feed-forward, layers of different sizes, a
    looped range in the middle, router options on and off."""
    return config([
        (attn(), dense()),
        (attn(heads=6, kv_heads=2, dim=40, vdim=56, chunk=19), moe()),
        (attn(heads=3, kv_heads=3, dim=16, vdim=24, chunk=50), None),
        (attn(heads=5, kv_heads=1, dim=32, vdim=32, chunk=64), moe(ff=32, experts=5, identity=0, top=2, groups=None, shared=0)),
    ], width=width, vocab=vocab, loop=(1, 3, 3))


def odd_config():
    """Sizes that no vector load or tensor-core tile divides."""
    return config([(attn(heads=2, kv_heads=1, dim=21, vdim=13, chunk=11), dense(ff=45)),
                   (attn(heads=3, kv_heads=1, dim=18, vdim=10, chunk=7), moe(ff=27, experts=5, identity=1, top=2, groups=(3, 2), shared=9))],
                  width=67, vocab=131)


def shapes(cfg):
    H = cfg["width"]
    out = {"embed": (cfg["vocab"], H), "head": (cfg["vocab"], H), "final.norm": (H,)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out[p + "norm1"] = out[p + "norm1b"] = (H,)
        out[p + "mix.q"] = (m["heads"] * m["dim"], H)
        out[p + "mix.k"] = (m["kv_heads"] * m["dim"], H)
        out[p + "mix.v"] = (m["kv_heads"] * m["vdim"], H)
        out[p + "mix.o"] = (H, m["heads"] * m["vdim"])
        out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (m["dim"],)
        if not f:
            continue
        out[p + "norm2"] = out[p + "norm2b"] = (H,)
        nets = {"": f.get("ff")}
        if f["kind"] == "moe":
            n = f["router"]["experts"] + f["router"].get("identity", 0)
            out[p + "mlp.router"], out[p + "mlp.correction"] = (n, H), (n,)
            nets = {f"e{e}.": f["expert"]["ff"] for e in range(f["router"]["experts"])}
            if f.get("shared"):
                nets["shared."] = f["shared"]["ff"]
        for q, ff in nets.items():
            out[p + "mlp." + q + "gate"] = out[p + "mlp." + q + "up"] = (ff, H)
            out[p + "mlp." + q + "down"] = (H, ff)
    return out


def weights(cfg, seed=0):
    """bf16 values: norm weights away from 1, sharp attention (q / k norm weights near 1.5), router corrections of both signs
    whose differences exceed what the scores can make up for in some experts only."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape in shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name.endswith(("q.norm", "k.norm")):
            t = 1.5 + 0.3 * r
        elif last.startswith("norm"):
            t = 1.0 + 0.2 * r
        elif last == "correction":
            t = -0.6 + 0.4 * r
        elif last == "router":
            t = r * (2.0 / math.sqrt(shape[1]))
        elif last == "embed":
            t = r
        else:
            t = r / math.sqrt(shape[1])
        sd[name] = t.to(torch.bfloat16)
    return sd


def save(cfg, sd, path):
    from xllm_wxh_b200.utils.safetensors_io import save_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(os.path.join(path, "model.safetensors"), sd)
    return str(path)


def engine(path, device="cpu", dtype="float32", block_size=16, blocks=64, **kw):
    from xllm_wxh_b200.config import Options
    from xllm_wxh_b200.runtime.engine import LLMEngine
    o = dict(enable_prefix_cache=False, max_tokens_per_batch=512, max_seqs_per_batch=16, max_model_len=2048, enable_numa_binding=False)
    o.update(kw)
    return LLMEngine(Options(model=path, devices=device, dtype=dtype, block_size=block_size, num_kv_blocks=blocks, **o))


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def replay(eng, sequences, steps):
    """Run `steps` ([(name, count)] per step) over `sequences` (name -> tokens) with all logits wanted; a request ends with
    its last token.  Returns name -> [n, vocab]."""
    ids, at, out = {}, {}, {}
    for step in steps:
        portions = []
        for name, count in step:
            if name not in ids:
                ids[name], at[name] = eng.add_request([]), 0
            lo = at[name]
            portions.append((ids[name], sequences[name][lo:lo + count], list(range(count))))
            at[name] = lo + count
        for (name, _), rows in zip(step, eng.step_portions(portions)):
            out.setdefault(name, []).append(torch.tensor(rows))
        for name, _ in step:
            if at[name] == len(sequences[name]):
                eng.cancel(ids[name])
    return {k: torch.cat(v) for k, v in out.items()}


def alone(name, seq, *cuts):
    """Steps of one request: the given portions, then single tokens."""
    rest = len(seq) - sum(cuts)
    return [[(name, c)] for c in cuts] + [[(name, 1)]] * rest


def row_error(got, want):
    """Root mean square difference of each row (mean taken off) over the spread of all wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()
