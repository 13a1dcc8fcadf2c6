"""Plain, slow statement of the Pafodra design, one function per mechanism: the oracle of its tests.

Everything is computed token by token (or query by query) in the dtype of the inputs, from the equations; nothing of
``easyllm_b200`` is imported.  ``weights`` is a dict of the checkpoint's own tensor names and ``cfg`` the dict of its
``config.json``.  A sequence is a 1-D list of token ids starting at position 0.
"""
import math

import torch


# ---- norms and activations -------------------------------------------------------------------
def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- mixers: h [T, width] of one whole sequence -> [T, width] ----------------------------------
def sink_attention(q, k, v, scale, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; ``sink`` [H] or None.  Causal."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        for h in range(H):
            g = h // (H // G)
            s = (k[:i + 1, g] @ q[i, h]) * scale
            m = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - m)
            den = p.sum() + (0 if sink is None else torch.exp(sink[h] - m))
            out[i, h] = (p / den) @ v[:i + 1, g]
    return out


def attention(h, w, p, m):
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = (h @ w[p + ".q"].t()).view(T, H, m["dim"])
    k = (h @ w[p + ".k"].t()).view(T, G, m["dim"])
    v = (h @ w[p + ".v"].t()).view(T, G, m["vdim"])
    o = sink_attention(q, k, v, m["scale"], w[p + ".sink"])
    return o.reshape(T, -1) @ w[p + ".o"].t()


def token_shift(h, mu):
    """h + (previous h - h) * mu, the previous token of the first one being zero."""
    prev = torch.zeros_like(h)
    prev[1:] = h[:-1]
    return h + (prev - h) * mu


def wkv_recurrence(r, k, v, w, u, S=None):
    """r, k, w [T, H, d], v [T, H, dv], u [H, d] -> (o [T, H, dv], S [H, d, dv])."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if S is None else S.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h][:, None] * kv).t() @ r[t, h]
            S[h] = w[t, h][:, None] * S[h] + kv
    return o, S


def wkv(h, w, p, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    mix = {c: token_shift(h, w[f"{p}.mu.{c}"]) for c in "rkvgw"}
    r, k, v = ((mix[c] @ w[f"{p}.{c}"].t()).view(T, H, d) for c in "rkv")
    gate = silu(mix["g"] @ w[p + ".g"].t())
    dec = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + ".w1"].t()) @ w[p + ".w2"].t() + w[p + ".w0"]))
    o, _ = wkv_recurrence(r, k, v, dec.view(T, H, d), w[p + ".u"])
    return (over_rms(o, eps).reshape(T, -1) * w[p + ".norm"] * gate) @ w[p + ".o"].t()


def short_conv(x, taps):
    """x [T, C], taps [C, n]: y_t = sum_j taps[:, n-1-j] x_{t-j}, zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            if t - j >= 0:
                y[t] = y[t] + taps[:, n - 1 - j] * x[t - j]
    return y


def delta_recurrence(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H] -> (o [T, H, dv], S [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].t() @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            o[t, h] = S[h].t() @ q[t, h]
    return o, S


def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[f"{p}.{c}"].t(), w[f"{p}.{c}.conv"])) for c in "qkv")
    q = unit(q.view(T, G, d)) * d ** -0.5
    k = unit(k.view(T, G, d))
    which = [i // (H // G) for i in range(H)]
    beta = sigmoid(h @ w[p + ".b"].t())
    a = h @ w[p + ".a1"].t() @ w[p + ".a2"].t() + w[p + ".dt_bias"]
    g = torch.exp(-torch.exp(w[p + ".A_log"])[:, None] * softplus(a).view(T, H, d))
    o, _ = delta_recurrence(q[:, which], k[:, which], v.view(T, H, dv), g, beta)
    gate = sigmoid(h @ w[p + ".g1"].t() @ w[p + ".g2"].t()).view(T, H, dv)
    return (over_rms(o, eps) * w[p + ".norm"] * gate).reshape(T, -1) @ w[p + ".o"].t()


# ---- feed-forward ------------------------------------------------------------------------------
def dense(h, w, p):
    g = h @ w[p + ".gate"].t() + w[p + ".gate.b"]
    u = h @ w[p + ".up"].t() + w[p + ".up.b"]
    return (gelu_tanh(g) * u) @ w[p + ".down"].t() + w[p + ".down.b"]


def expert(h, w, p):
    return torch.clamp(h @ w[p + ".up"].t(), min=0) ** 2 @ w[p + ".down"].t()


def moe(h, w, p, m):
    s = sigmoid(h @ w[p + ".router"].t())
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(m["router"]["experts"]), key=lambda e: -float(s[t, e]))
        for e in order[:m["router"]["top"]]:
            out[t] = out[t] + expert(s[t, e] * h[t], w, f"{p}.e{e}")
    if m.get("shared"):
        out = out + expert(h, w, p + ".shared") * sigmoid(h @ w[p + ".shared.sg"].t())
    return out


# ---- the model -----------------------------------------------------------------------------------
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace`` (a list) receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    eps = cfg["norm"]["eps"]
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{layer.get('weights_of', i)}"
        h = dynamic_tanh(x, w[n + ".norm1.alpha"], w[n + ".norm1"], w[n + ".norm1.b"])
        m = layer["mixer"]
        if layer["type"] == "attention":
            y = attention(h, w, n + ".mix", m)
        elif layer["type"] == "wkv":
            y = wkv(h, w, n + ".mix", m, eps)
        else:
            y = channel_delta(h, w, n + ".mix", m, eps)
        if layer.get("mlp"):
            f = dense(h, w, n + ".mlp") if layer["mlp"]["kind"] == "dense" else moe(h, w, n + ".mlp", layer["mlp"])
            y = y + f
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    x = dynamic_tanh(x, w["final.norm.alpha"], w["final.norm"], w["final.norm.b"])
    return x @ w["head"].t()
