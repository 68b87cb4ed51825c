"""Plain, slow statement of the Govuvik design, one function per mechanism, used as the oracle of its tests.

Whole sequences, dense score matrices, explicit loops over tokens and heads; no paging, no slots, no batching, no fused
steps.  It imports nothing of the package: a configuration is the parsed `config.json` dictionary and the weights are a
dictionary of tensors under the checkpoint's names.  All arithmetic is in the dtype of the weights it is given (tests use
float32 or float64)."""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def silu(z):
    return z * sigmoid(z)


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def embed(sd, tokens, eps):
    return rms_norm(sd["embed"][torch.as_tensor(tokens, dtype=torch.long)], sd["embed.norm"], eps)


def causal_conv(x, w):
    """Per channel over time; the last column of w [channels, taps] belongs to the current token."""
    n, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[i:i + n] * w[:, i] for i in range(taps))


# ----------------------------------------------------------------------------- attention with mixed scores
def frequencies(rot):
    """Angle per position of every pair; wavelengths far beyond the original context are slowed down."""
    f = [rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for x in f:
        wave = 2 * math.pi / x
        if wave < s["original"] / s["high"]:
            out.append(x)
        elif wave > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            a = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - a) * x / s["factor"] + a * x)
    return out


def rotate(x, rot):
    """x [n, heads, dim] at positions 0 .. n - 1."""
    if not rot or not rot["dims"]:
        return x
    out, half = x.clone(), rot["dims"] // 2
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(frequencies(rot)):
        c, s = torch.cos(pos * f).to(x.dtype)[:, None], torch.sin(pos * f).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def visible_matrix(n, size):
    pos = torch.arange(n)
    i, j = pos[:, None], pos[None, :]
    return (j <= i) & (i - j < size)


def raw_scores(q, k, scale):
    """q [n, H, d], k [n, G, d] -> [H, n, n]."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([(q[:, h] @ k[:, h // (H // G)].T) * scale for h in range(H)])


def mix_scores(s, temp, talk):
    """Every head's scores times its number, then a sum over all heads."""
    s = s * temp[:, None, None]
    return torch.stack([sum(talk[h, g] * s[g] for g in range(s.shape[0])) for h in range(s.shape[0])])


def softmax_with_sink(s, sink):
    """s [n, keys]; the sink joins the denominator."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention_core(q, k, v, scale, temp, talk, sink, size):
    """q [n, H, d], k [n, G, d], v [n, G, dv] of one whole sequence -> [n, H, dv]."""
    n, H, _ = q.shape
    G = k.shape[1]
    see = visible_matrix(n, size)
    s = mix_scores(raw_scores(q, k, scale), temp, talk)
    return torch.stack([softmax_with_sink(s[h].masked_fill(~see, -math.inf), sink[h]) @ v[:, h // (H // G)] for h in range(H)], 1)


def attention(sd, p, m, h, eps):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (causal_conv(h @ sd[p + c].T, sd[p + c + ".conv"]) for c in "qkv")
    q, k = rms_norm(q, sd[p + "q.norm"], eps), rms_norm(k, sd[p + "k.norm"], eps)
    q, k = (rotate(x.reshape(n, -1, m["dim"]), m.get("rot")) for x in (q, k))
    o = attention_core(q, k, v.reshape(n, G, m["vdim"]), m["scale"], sd[p + "temp"], sd[p + "talk"], sd[p + "sink"], m["mask"]["size"])
    return o.reshape(n, H * m["vdim"]) @ sd[p + "o"].T


# ----------------------------------------------------------------------------- gated linear attention
def channel_decay(z, tau):
    return torch.exp(log_sigmoid(z) / tau)


def gated_linear_core(q, k, v, a):
    """q, k, a [n, H, d], v [n, H, dv] -> [n, H, dv]: a matrix state per head that decays per key channel ahead of every token."""
    n, H, d = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=q.dtype)
        for t in range(n):
            S = a[t, h][:, None] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def gated_linear(sd, p, m, h, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ sd[p + c].T).reshape(n, H, -1) for c in "qkv")
    z = (h @ sd[p + "a1"].T) @ sd[p + "a2"].T + sd[p + "a2.b"]
    o = gated_linear_core(q * d ** -0.5, k, v, channel_decay(z, m["tau"]).reshape(n, H, d))
    o = rms_norm(o, sd[p + "norm"], eps).reshape(n, H * dv)
    return (o * silu(h @ sd[p + "g"].T)) @ sd[p + "o"].T


def parallel(sd, p, m, h, eps):
    left = rms_norm(attention(sd, p + "left.", m["left"], h, eps), sd[p + "left.out"], eps)
    return (left + rms_norm(gated_linear(sd, p + "right.", m["right"], h, eps), sd[p + "right.out"], eps)) / 2


# ----------------------------------------------------------------------------- matrix memory with exponential gates
def soft_bound(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory_core(q, k, v, log_i, log_f):
    """q, k [n, H, d], v [n, H, dv], log gates [n, H] -> [n, H, dv]; state and normaliser are kept relative to exp(m)."""
    n, H, d = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S, nrm, m = torch.zeros(d, v.shape[-1], dtype=q.dtype), torch.zeros(d, dtype=q.dtype), torch.zeros((), dtype=q.dtype)
        for t in range(n):
            m_new = torch.maximum(log_f[t, h] + m, log_i[t, h])
            f, i = torch.exp(log_f[t, h] + m - m_new), torch.exp(log_i[t, h] - m_new)
            S = f * S + i * torch.outer(k[t, h], v[t, h])
            nrm = f * nrm + i * k[t, h]
            m = m_new
            out[t, h] = S.T @ q[t, h] / (torch.maximum((nrm @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm(sd, p, m, h, eps):
    n, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k, v = ((h @ sd[p + c].T).reshape(n, H, -1) for c in "qkv")
    log_i = soft_bound(h @ sd[p + "i"].T + sd[p + "i.b"], cap)
    log_f = log_sigmoid(soft_bound(h @ sd[p + "f"].T + sd[p + "f.b"], cap))
    o = matrix_memory_core(q * d ** -0.5, k, v, log_i, log_f)
    o = rms_norm(o, 1.0, eps).reshape(n, H * dv)
    return (o * sd[p + "norm"] * sigmoid(h @ sd[p + "g"].T)) @ sd[p + "o"].T


# ----------------------------------------------------------------------------- the model
MIXERS = {"parallel": parallel, "mlstm": mlstm}


def route(logits, top):
    """(experts, weights) of one token: the largest logits and the softmax over them alone."""
    order = sorted(range(len(logits)), key=lambda e: -float(logits[e]))[:top]
    return order, torch.softmax(logits[order], -1)


def expert(sd, p, h):
    return squared_relu(h @ sd[p + "up"].T) @ sd[p + "down"].T


def feed_forward(sd, p, f, h):
    out = torch.zeros_like(h)
    logits = h @ sd[p + "router"].T
    for t in range(h.shape[0]):
        for e, w in zip(*route(logits[t], f["router"]["top"])):
            out[t] += w * expert(sd, f"{p}e{e}.", h[t])
    return out


def run_layer(sd, cfg, i, x):
    p, layer, eps = f"l{i}.", cfg["layers"][i], cfg["norm"]["eps"]
    h = rms_norm(x, sd[p + "norm1"], eps)
    h = h + causal_conv(h, sd[p + "canon1"])
    x = x + rms_norm(MIXERS[layer["type"]](sd, p + "mix.", layer["mixer"], h, eps), sd[p + "norm1b"], eps)
    if layer.get("mlp"):
        y = feed_forward(sd, p + "mlp.", layer["mlp"], rms_norm(x, sd[p + "norm2"], eps))
        x = x + rms_norm(y, sd[p + "norm2b"], eps)
    return x


def forward(sd, cfg, tokens, keep_residuals=None):
    """Logits [n, vocab] of a whole sequence."""
    x = embed(sd, tokens, cfg["norm"]["eps"])
    for i in range(len(cfg["layers"])):
        x = run_layer(sd, cfg, i, x)
        if keep_residuals is not None:
            keep_residuals.append(x)
    z = rms_norm(x, sd["final.norm"], cfg["norm"]["eps"]) @ sd["head"].T
    cap = cfg.get("logit_softcap")
    return soft_bound(z, cap) if cap else z


def greedy(sd, cfg, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(sd, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]
