"""Plain, slow statement of the Babadra design, one function per mechanism, used as the oracle of its tests.

Whole sequences, dense score matrices, explicit loops over heads, maps and experts; keys and values are expanded from the latent
for every head; no paging, no batching, no fused steps.  It imports nothing of the package: a configuration is the parsed
`config.json` dictionary and the weights are a dictionary of tensors under the checkpoint's names.  All arithmetic is in the
dtype of the weights it is given (tests use float32 or float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def plain_norm(x, w, eps):
    return rms(x, eps) * w


def centred_norm(x, w, eps):
    """The weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def embed(sd, cfg, tokens):
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return sd["embed"][ids] * cfg["embedding"]["scale"] + sd["pos"][:len(ids)]


# ----------------------------------------------------------------------------- rotation
def frequencies(rot):
    n = rot["dims"] // 2
    f = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(n)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turns_to_dim(t):
        return rot["dims"] * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(rot["base"]))
    lo = max(math.floor(turns_to_dim(s["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(s["slow"])), rot["dims"] - 1)
    out = []
    for i in range(n):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / s["factor"] * ramp + f[i] * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot, interleaved, first=0):
    """x [n, ..., d]: its first rot.dims columns turned by the angles of positions first, first + 1, ..."""
    n, dims = x.shape[0], rot["dims"]
    f, m = frequencies(rot)
    out = x.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        ang = (torch.arange(first, first + n, dtype=torch.float64) * f[i]).reshape([n] + [1] * (x.dim() - 2))
        c, s = (torch.cos(ang) * m).to(x.dtype), (torch.sin(ang) * m).to(x.dtype)
        u, v = x[..., a], x[..., b]
        out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


# ----------------------------------------------------------------------------- attention
def causal(n):
    pos = torch.arange(n)
    return pos[None, :] <= pos[:, None]


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def attend(scores, v):
    return torch.softmax(scores.masked_fill(~causal(scores.shape[0]), -math.inf), -1) @ v


def latent_attention(sd, p, m, h, eps):
    n = h.shape[0]
    H, d, r, dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = plain_norm(h @ sd[p + "dq"].T, sd[p + "dq.norm"], eps)
    q = (cq @ sd[p + "uq"].T).reshape(n, H, d + r)
    low = h @ sd[p + "dkv"].T
    c = plain_norm(low[:, :C], sd[p + "dkv.norm"], eps)
    k_rot = rotate(low[:, C:], m["rot"], True)
    q_rot = rotate(q[..., d:], m["rot"], True)
    k = (c @ sd[p + "uk"].T).reshape(n, H, d)
    v = (c @ sd[p + "uv"].T).reshape(n, H, dv)
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = attend(s, v[:, i])
    return out.reshape(n, H * dv) @ sd[p + "o"].T


def mix_factor(sd, p, diff):
    return torch.exp((sd[p + "lq1"] * sd[p + "lk1"]).sum()) - torch.exp((sd[p + "lq2"] * sd[p + "lk2"]).sum()) + diff


def difference(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def two_map_core(q, k, v, scale, cap, lam, diff, eps):
    """q [n, H, 2, d], k [n, G, 2, d], v [n, G, dv] of one whole sequence -> [n, H, dv]."""
    n, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        a = []
        for i in range(2):
            s = (q[:, h, i] @ k[:, g, i].T) * scale
            a.append(attend(softcap(s, cap) if cap else s, v[:, g]))
        out[:, h] = difference(a[0], a[1], lam, diff, eps)
    return out


def two_map_attention(sd, p, m, h, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = plain_norm((h @ sd[p + "q"].T).reshape(n, H, 2, d), sd[p + "q.norm"], eps)
    k = plain_norm((h @ sd[p + "k"].T).reshape(n, G, 2, d), sd[p + "k.norm"], eps)
    q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False)
    v = (h @ sd[p + "v"].T).reshape(n, G, dv)
    o = two_map_core(q, k, v, m["scale"], m.get("softcap"), mix_factor(sd, p, m["diff"]), m["diff"], eps)
    return o.reshape(n, H * dv) @ sd[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": two_map_attention}


# ----------------------------------------------------------------------------- feed-forward
def clamped_gate(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def gated_ff(sd, p, h, limit):
    return clamped_gate(h @ sd[p + "gate"].T, h @ sd[p + "up"].T, limit) @ sd[p + "down"].T


def route(z, bias, top):
    """Router products of one token -> [(expert, weight)], best first."""
    z = z + bias
    picked = sorted(range(z.shape[-1]), key=lambda e: -float(z[e]))[:top]
    return list(zip(picked, torch.softmax(z[picked], -1)))


def moe(sd, p, mlp, h):
    z = h @ sd[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(z[t], sd[p + "router.b"], mlp["router"]["top"]):
            out[t] += w * gated_ff(sd, f"{p}e{e}.", h[t:t + 1], mlp["expert"]["limit"])[0]
    return out


def feed_forward(sd, p, mlp, h):
    return gated_ff(sd, p, h, mlp["limit"]) if mlp["kind"] == "dense" else moe(sd, p, mlp, h)


# ----------------------------------------------------------------------------- the whole model
def layer_order(cfg):
    """[(layer, opens a pass other than the first)]"""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, k = loop["start"], loop["stop"], loop["times"]
    out = [(i, False) for i in range(a)]
    for t in range(k):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def run_layer(sd, i, layer, x, eps):
    p = f"l{i}."
    x = x + sd[p + "ls1"] * MIXERS[layer["type"]](sd, p + "mix.", layer["mixer"], centred_norm(x, sd[p + "norm1"], eps), eps)
    if layer.get("mlp"):
        x = x + sd[p + "ls2"] * feed_forward(sd, p + "mlp.", layer["mlp"], centred_norm(x, sd[p + "norm2"], eps))
    return x


def forward(sd, cfg, tokens, keep_residuals=None):
    """Logits [n, vocab] of a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = x0 = embed(sd, cfg, tokens)
    for i, opens in layer_order(cfg):
        if opens:
            x = x + x0
        x = run_layer(sd, i, cfg["layers"][i], x, eps)
        if keep_residuals is not None:
            keep_residuals.append(x)
    logits = centred_norm(x, sd["final.norm"], eps) @ sd["head"].T
    return softcap(logits, cfg["logit_softcap"]) if cfg.get("logit_softcap") else logits


def greedy(sd, cfg, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(sd, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]
