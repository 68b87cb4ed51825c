"""Plain, slow statement of the Falalix design, one function per mechanism, used as the oracle of its tests.

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


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


def embed(sd, tokens):
    return sd["embed"][torch.as_tensor(tokens, dtype=torch.long)]


# ----------------------------------------------------------------------------- attention branch
def visible(i, j, size, keep_first):
    """Query i sees key j: not later, and either near enough or one of the kept first ones."""
    return j <= i and (i - j < size or j < keep_first)


def visible_matrix(n, size, keep_first):
    pos = torch.arange(n)
    i, j = pos[:, None], pos[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def attention_core(q, k, v, scale, size, keep_first):
    """q [n, H, d], k [n, G, d], v [n, G, dv] of one whole sequence -> [n, H, dv]."""
    n, H, _ = q.shape
    G = k.shape[1]
    see = visible_matrix(n, size, keep_first)
    out = torch.zeros(n, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, g]
    return out


def project_qkv(sd, p, h, eps):
    """q and k are normed over the whole projection, all heads at once."""
    q = rms_norm(h @ sd[p + "q"].T + sd[p + "q.b"], sd[p + "q.norm"], eps)
    k = rms_norm(h @ sd[p + "k"].T + sd[p + "k.b"], sd[p + "k.norm"], eps)
    return q, k, h @ sd[p + "v"].T + sd[p + "v.b"]


def attention(sd, p, m, h, eps):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = project_qkv(sd, p, h, eps)
    o = attention_core(q.reshape(n, H, m["dim"]), k.reshape(n, G, m["dim"]), v.reshape(n, G, m["vdim"]), m["scale"], m["mask"]["size"],
                       m["mask"]["keep_first"])
    return (o.reshape(n, H * m["vdim"]) * sigmoid(h @ sd[p + "g"].T)) @ sd[p + "o"].T


# ----------------------------------------------------------------------------- time mixing branch
def shifted(h):
    """Every row's predecessor, zeros ahead of the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def token_mix(h, mu):
    return h + (shifted(h) - h) * mu


def decay(sd, p, mix_w):
    return torch.exp(-torch.exp(torch.tanh(mix_w @ sd[p + "w1"].T) @ sd[p + "w2"].T + sd[p + "w0"]))


def time_mix_core(r, k, v, w, u):
    """r, k, v, w [n, H, d], u [H, d] -> [n, H, d]: a matrix state per head that decays per key channel."""
    n, H, d = r.shape
    out = torch.zeros_like(r)
    for h in range(H):
        S = torch.zeros(d, d, dtype=r.dtype)
        for t in range(n):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S + u[h][:, None] * kv).T @ r[t, h]
            S = w[t, h][:, None] * S + kv
    return out


def time_mix(sd, p, m, h, eps):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    mixed = {c: token_mix(h, sd[p + "mu." + c]) for c in "rkvgw"}
    r, k, v = ((mixed[c] @ sd[p + c].T).reshape(n, H, d) for c in "rkv")
    o = time_mix_core(r, k, v, decay(sd, p, mixed["w"]).reshape(n, H, d), sd[p + "u"])
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    return (o.reshape(n, H * d) * sd[p + "norm"] * silu(mixed["g"] @ sd[p + "g"].T)) @ sd[p + "o"].T


def parallel(sd, p, m, h, eps):
    return m["left_scale"] * attention(sd, p + "left.", m["left"], h, eps) + m["right_scale"] * time_mix(sd, p + "right.", m["right"], h, eps)


# ----------------------------------------------------------------------------- selective scan
def causal_conv(x, w, b):
    """Per channel over time; the last column of w belongs to the current token."""
    n, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return b + sum(padded[i:i + n] * w[:, i] for i in range(taps))


def scan_core(x, dt, A, B, C, D):
    """x, dt [n, c], A [c, s], B, C [n, s], D [c] -> [n, c]."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba1(sd, p, m, h, eps):
    x, z = (h @ sd[p + "in"].T).split(m["inner"], -1)
    x = silu(causal_conv(x, sd[p + "conv"], sd[p + "conv.b"]))
    dt, B, C = (x @ sd[p + "x"].T).split([m["dt_rank"], m["state"], m["state"]], -1)
    dt = softplus(dt @ sd[p + "dt"].T + sd[p + "dt.b"])
    y = scan_core(x, dt, -torch.exp(sd[p + "A_log"]), B, C, sd[p + "D"])
    return (y * silu(z)) @ sd[p + "o"].T


# ----------------------------------------------------------------------------- the model
MIXERS = {"parallel": parallel, "mamba1": mamba1}


def feed_forward(sd, p, h):
    return squared_relu(h @ sd[p + "up"].T) @ sd[p + "down"].T


def run_layer(sd, cfg, i, x):
    p, layer, eps, m = f"l{i}.", cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + m * MIXERS[layer["type"]](sd, p + "mix.", layer["mixer"], rms_norm(x, sd[p + "norm1"], eps), eps)
    if layer.get("mlp"):
        x = x + m * feed_forward(sd, p + "mlp.", rms_norm(x, sd[p + "norm2"], eps))
    return x


def enter_pass(sd, x, x0, t):
    return torch.cat([x, x0], -1) @ sd["loop.in"].T + sd["loop.step"][t]


def schedule(cfg):
    """(layer, pass that starts right before it or None) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(sd, cfg, tokens, keep_residuals=None):
    """Logits [n, vocab] of a whole sequence."""
    x = x0 = embed(sd, tokens)
    for i, t in schedule(cfg):
        if t is not None:
            x = enter_pass(sd, x, x0, t)
        x = run_layer(sd, cfg, i, x)
        if keep_residuals is not None:
            keep_residuals.append(x)
    return rms_norm(x, sd["final.norm"], cfg["norm"]["eps"]) @ sd["head"].T


def greedy(sd, cfg, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(sd, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]
