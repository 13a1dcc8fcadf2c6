"""Plain, slow statement of the Megozen design, one function per mechanism: the oracle of its tests.

Everything is computed in the dtype of the inputs, from the equations; nothing of ``easyllm_b200`` is imported.
``weights`` is a dict of the checkpoint's own tensor names and ``cfg`` the dict of its ``config.json``.  A sequence is a
1-D list of token ids starting at position 0.
"""
import math

import torch


# ---- norms and activations -------------------------------------------------------------------
def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- embedding ---------------------------------------------------------------------------------
def bigram_rows(tokens, b):
    """Row of the pair table for every token of one sequence; the first token has a row of its own, the last one."""
    rows = [b["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"])
    return rows


def embed(cfg, w, tokens):
    tokens = [int(t) for t in tokens]
    x = torch.stack([w["embed"][t] for t in tokens])
    b = cfg["embedding"].get("bigram")
    return x if b is None else x + torch.stack([w["bigram"][r] for r in bigram_rows(tokens, b)])


# ---- rotary positions ----------------------------------------------------------------------------
def frequencies(rot):
    """(frequency of every pair, factor of cos and sin)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    if s is None:
        return f, 1.0

    def turns(t):           # the dimension whose pair turns t times over the original length
        return n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, positions, rot):
    """x [T, ..., n]: neighbouring dimensions are a pair; dimensions past ``rot.dims`` stay."""
    f, m = frequencies(rot)
    y = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = math.cos(p * fi) * m, math.sin(p * fi) * m
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i], y[t, ..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


# ---- the mixer ---------------------------------------------------------------------------------
def attend(q, k, v, scale):
    """One query: q [H, d] over the keys it sees, k [n, H, d], v [n, H, dv]."""
    out = []
    for h in range(q.shape[0]):
        s = (k[:, h] @ q[h]) * scale
        p = torch.exp(s - s.max())
        out.append((p / p.sum()) @ v[:, h])
    return torch.stack(out)


def window_attention(q, k, v, scale, window):
    """q, k [T, H, d], v [T, H, dv]: query i sees keys j with 0 <= i - j < window (None: all before it)."""
    out = []
    for i in range(q.shape[0]):
        lo = 0 if window is None else max(0, i - window + 1)
        out.append(attend(q[i], k[lo:i + 1], v[lo:i + 1], scale))
    return torch.stack(out)


def latent_attention(h, w, p, m, eps):
    T, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + ".q"].t()).view(T, H, d + r)
    z = h @ w[p + ".dkv"].t()
    c = rms_norm(z[:, :R], w[p + ".dkv.norm"], eps)
    pos = range(T)
    q_rot, k_rot = rotate(q[..., d:], pos, m["rot"]), rotate(z[:, R:], pos, m["rot"])
    k = torch.cat(((c @ w[p + ".uk"].t()).view(T, H, d), k_rot[:, None].expand(T, H, r)), -1)
    v = (c @ w[p + ".uv"].t()).view(T, H, dv)
    mask = m.get("mask")
    o = window_attention(torch.cat((q[..., :d], q_rot), -1), k, v, m["scale"], mask["size"] if mask else None)
    g = sigmoid(h @ w[p + ".g"].t())
    return (o * g[..., None]).reshape(T, H * dv) @ w[p + ".o"].t()


# ---- feed-forward ------------------------------------------------------------------------------
def expert(h, w, p):
    return (silu(h @ w[p + ".gate"].t()) * (h @ w[p + ".up"].t())) @ w[p + ".down"].t()


def chosen(z, top):
    """Indices of the ``top`` largest logits of one token and their softmax."""
    order = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    return order, torch.softmax(z[order], -1)


def moe(h, w, p, m):
    z = h @ w[p + ".router"].t() + w[p + ".router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(*chosen(z[t], m["router"]["top"])):
            out[t] = out[t] + s * expert(h[t], w, f"{p}.e{e}")
    return out + expert(h, w, p + ".shared") if m.get("shared") else out


# ---- the model -----------------------------------------------------------------------------------
def owner(cfg, i):
    while "weights_of" in cfg["layers"][i]:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace`` (a list) receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    x = embed(cfg, w, tokens)
    eps = cfg["norm"]["eps"]
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{owner(cfg, i)}"
        y = latent_attention(layer_norm(x, w[n + ".norm1"], eps), w, n + ".mix", layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + moe(layer_norm(x, w[n + ".norm2"], eps), w, n + ".mlp", layer["mlp"])
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].t()
