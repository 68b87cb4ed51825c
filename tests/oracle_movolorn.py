"""Plain, slow statement of the Movolorn design, one function per mechanism, used as the oracle of its tests.

Whole sequences, dense score matrices, explicit loops over heads and experts; no paging, no batching, no fused steps.  It
imports nothing of the package: a configuration is the parsed `config.json` dictionary and the weights are a dictionary of
tensors under the checkpoint's names.  All arithmetic is in the dtype of the weights it is given (tests use float32 or
float64)."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(sd, cfg, tokens):
    return sd["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]


def head_slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def visible(i, j, chunk):
    """Query i sees key j: not later, and in the same chunk (counted from position 0)."""
    return j <= i and i // chunk == j // chunk


def visible_matrix(n, chunk):
    pos = torch.arange(n)
    return (pos[None, :] <= pos[:, None]) & (pos[None, :] // chunk == pos[:, None] // chunk)


def distance_bias(n, slope, dtype):
    pos = torch.arange(n, dtype=dtype)
    return slope * (pos[:, None] - pos[None, :])


def softmax_plus_one(s):
    """exp(s_j) / (1 + sum_j exp(s_j)) over the last dimension; -inf marks an invisible key."""
    m = s.max(-1, keepdim=True).values.clamp_min(0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention_core(q, k, v, scale, chunk):
    """q [n, H, d], k [n, G, d], v [n, G, dv] of one whole sequence -> [n, H, dv]."""
    n, H, _ = q.shape
    G = k.shape[1]
    see = visible_matrix(n, chunk)
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale - distance_bias(n, head_slope(h, H), q.dtype)
        out[:, h] = softmax_plus_one(s.masked_fill(~see, -math.inf)) @ v[:, g]
    return out


def attention(sd, p, m, h, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ sd[p + "q"].T).reshape(n, H, d), sd[p + "q.norm"], eps)
    k = rms_norm((h @ sd[p + "k"].T).reshape(n, G, d), sd[p + "k.norm"], eps)
    v = (h @ sd[p + "v"].T).reshape(n, G, dv)
    return attention_core(q, k, v, m["scale"], m["mask"]["size"]).reshape(n, H * dv) @ sd[p + "o"].T


def gated_ff(sd, p, h, act):
    return (act(h @ sd[p + "gate"].T) * (h @ sd[p + "up"].T)) @ sd[p + "down"].T


def route(z, correction, r):
    """Router logits of one token -> [(expert, weight)]."""
    s = torch.softmax(z, -1)
    choice = s + correction
    n = z.shape[-1]
    allowed = set(range(n))
    groups = r.get("groups")
    if groups and groups["count"] > 1:
        size = n // groups["count"]
        best = sorted(range(groups["count"]), key=lambda g: -float(choice[g * size:(g + 1) * size].max()))[:groups["keep"]]
        allowed = {e for g in best for e in range(g * size, (g + 1) * size)}
    picked = sorted(allowed, key=lambda e: -float(choice[e]))[:r["top"]]
    return [(e, s[e]) for e in picked]


def moe(sd, p, mlp, h):
    r = mlp["router"]
    z = h @ sd[p + "router"].T
    corr = sd.get(p + "correction", torch.zeros(z.shape[-1], dtype=h.dtype))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(z[t], corr, r):
            y = gated_ff(sd, f"{p}e{e}.", h[t:t + 1], silu)[0] if e < r["experts"] else h[t]
            out[t] += w * y
    if mlp.get("shared"):
        out = out + gated_ff(sd, p + "shared.", h, silu)
    return out


def feed_forward(sd, p, mlp, h):
    return gated_ff(sd, p, h, gelu_tanh) if mlp["kind"] == "dense" else moe(sd, p, mlp, h)


def layer_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, k = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * k + list(range(b, n))


def run_layer(sd, i, layer, x, eps):
    p = f"l{i}."
    y = attention(sd, p + "mix.", layer["mixer"], rms_norm(x, sd[p + "norm1"], eps), eps)
    x = x + rms_norm(y, sd[p + "norm1b"], eps)
    if layer.get("mlp"):
        y = feed_forward(sd, p + "mlp.", layer["mlp"], rms_norm(x, sd[p + "norm2"], eps))
        x = x + rms_norm(y, sd[p + "norm2b"], eps)
    return x


def forward(sd, cfg, tokens, keep_residuals=None):
    """Logits [n, vocab] of a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = embed(sd, cfg, tokens)
    for i in layer_order(cfg):
        x = run_layer(sd, i, cfg["layers"][i], x, eps)
        if keep_residuals is not None:
            keep_residuals.append(x)
    return rms_norm(x, sd["final.norm"], eps) @ sd["head"].T


def greedy(sd, cfg, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(sd, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]
