"""Plain PyTorch statements of the inference-only ops of ``ops.infer``.

They run on CPU tensors (and are what a kernel of ``csrc`` computes, op by op).  Layouts: activations token-major
``[T, width]`` with sequence borders in ``cu`` (host list); a sequence's state lives in slot ``slots[s]`` of the state
tensors and is ignored when the sequence starts (``pos0[s] == 0``).  ``slots`` None: no state is read or written.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def dynamic_tanh(x, alpha, w, b, out_dtype):
    return (torch.tanh(alpha.float() * x.float()) * w.float() + b.float()).to(out_dtype)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def _segments(cu, slots, pos0):
    for s in range(len(cu) - 1):
        if cu[s + 1] > cu[s]:
            slot = None if slots is None else int(slots[s])
            fresh = slots is None or int(pos0[s]) == 0
            yield cu[s], cu[s + 1], slot, fresh


def embed_pairs(ids, table, pairs, scale, mul_prev, mul_cur, row_start, kv_base=None, kv_len=None, hist=None):
    """fp32 ``table[id] * scale + pairs[(previous id * mul_prev + id * mul_cur) mod buckets]``, ``buckets`` one less than the
    rows of ``pairs``; a sequence's first token takes the last row.  ``hist``: token ids by position (flat), the previous
    token of a sequence's first row in this step; this step's ids are written to it."""
    t = torch.arange(ids.numel())
    first = row_start.cpu() == t
    prev = ids.roll(1).clone()
    buckets = pairs.shape[0] - 1
    if hist is not None:
        at = (kv_base + kv_len - 1).long()
        going_on = first & (kv_len.cpu() > 1)
        prev[going_on] = hist[at[going_on] - 1].to(prev.dtype)
        first = first & ~going_on
        hist[at] = ids.to(hist.dtype)
    row = torch.where(first.to(ids.device), buckets, (prev * mul_prev + ids * mul_cur) % buckets)
    return table[ids].float() * scale + pairs[row].float()


def layer_norms(x, weights, eps, out_dtype):
    """``(x - mean) / sqrt(variance + eps) * w`` for every ``w``."""
    d = x.float() - x.float().mean(-1, keepdim=True)
    y = d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps)
    return [(y * w.float()).to(out_dtype) for w in weights]


def rotate_pairs(x, cos, sin):
    """x ``[T, n, r]`` with neighbouring dimensions as pairs, cos / sin ``[T, pairs]``; dimensions past them stay."""
    n = 2 * cos.shape[-1]
    u, v = x[..., :n:2].float(), x[..., 1:n:2].float()
    c, s = cos.unsqueeze(1), sin.unsqueeze(1)
    y = torch.stack((u * c - v * s, v * c + u * s), -1).flatten(-2).to(x.dtype)
    return torch.cat((y, x[..., n:]), -1)


def latent_inputs(z, H, dim, rot, rank, norm_w, eps, cos, sin, q_dst=None):
    """In place on ``z [T, H (dim + rot) + rank + rot + ...]``: the rotated query parts (into ``q_dst [T, H, rot]`` if
    given), the latent over its root mean square times ``norm_w``, the rotated key part."""
    T, at = z.shape[0], H * (dim + rot)
    q = z[:, :at].view(T, H, dim + rot)
    (q[..., dim:] if q_dst is None else q_dst).copy_(rotate_pairs(q[..., dim:], cos, sin))
    c = z[:, at:at + rank].float()
    z[:, at:at + rank] = (c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()).to(z.dtype)
    kr = z[:, at + rank:at + rank + rot]
    kr.copy_(rotate_pairs(kr.unsqueeze(1), cos, sin).squeeze(1))


def attention_rows(q, k, v, kv_base, kv_len, scale, sink=None, alibi_slopes=None, window=None, gate=None):
    """Query row t attends to the rows ``kv_base[t] .. kv_base[t] + kv_len[t]`` of k ``[R, G, d]``, v ``[R, G, dv]``;
    it sits at the last of them.  ``sink [H]`` adds ``exp(sink)`` to the softmax denominator; ``window`` keeps the last so
    many rows; ``gate [T, H]`` multiplies the heads' outputs by its sigmoid."""
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.empty(T, H, dv, dtype=q.dtype, device=q.device)
    # rows that share a base (one sequence) are attended together
    t = 0
    base, length = kv_base.tolist(), kv_len.tolist()
    while t < T:
        e = t + 1
        while e < T and base[e] == base[t] and length[e] == length[e - 1] + 1:
            e += 1
        n = length[e - 1]
        ks = k[base[t]:base[t] + n].float().repeat_interleave(H // G, 1)
        vs = v[base[t]:base[t] + n].float().repeat_interleave(H // G, 1)
        s = torch.einsum("qhd,khd->hqk", q[t:e].float(), ks) * scale
        qi = torch.tensor(length[t:e], device=q.device).view(-1, 1) - 1
        kj = torch.arange(n, device=q.device).view(1, -1)
        if alibi_slopes is not None:
            s = s + alibi_slopes.float().view(-1, 1, 1) * (kj - qi)
        s = s.masked_fill((kj > qi) | (kj <= qi - window) if window else kj > qi, float("-inf"))
        if sink is not None:
            s = torch.cat((s, sink.float().view(H, 1, 1).expand(H, e - t, 1)), -1)
        p = torch.softmax(s, -1)[..., :n]
        o = torch.einsum("hqk,khd->qhd", p, vs)
        out[t:e] = (o if gate is None else o * torch.sigmoid(gate[t:e].float()).unsqueeze(-1)).to(q.dtype)
        t = e
    return out


def token_mix(h, mu, cu, slots, pos0, tail):
    """``h + (h_prev - h) * mu_c`` for every row of ``mu [C, W]`` → ``[C, T, W]``; ``tail [slots, W]`` carries the
    last row of every sequence."""
    prev = torch.zeros_like(h)
    for a, b, slot, fresh in _segments(cu, slots, pos0):
        prev[a + 1:b] = h[a:b - 1]
        if not fresh:
            prev[a] = tail[slot].to(h.dtype)
        if slot is not None:
            tail[slot] = h[b - 1].to(tail.dtype)
    hf, pf = h.float(), prev.float()
    return torch.stack([(hf + (pf - hf) * m.float()).to(h.dtype) for m in mu])


def wkv_scan(r, k, v, decay, u, cu, slots, pos0, state):
    """r, k, decay ``[T, H, d]``, v ``[T, H, dv]``, u ``[H, d]`` → o fp32 ``[T, H, dv]``; ``state [slots, H, dv, dp]``."""
    T, H, d = k.shape
    o = torch.zeros(T, H, v.shape[2], dtype=torch.float32, device=k.device)
    r, k, v, decay, u = (t.float() for t in (r, k, v, decay, u))
    for a, b, slot, fresh in _segments(cu, slots, pos0):
        S = torch.zeros(H, v.shape[2], d, device=k.device) if fresh else state[slot][..., :d].clone()
        for t in range(a, b):
            kv = v[t].unsqueeze(-1) * k[t].unsqueeze(-2)
            o[t] = ((S + kv * u.unsqueeze(-2)) * r[t].unsqueeze(-2)).sum(-1)
            S = S * decay[t].unsqueeze(-2) + kv
        if slot is not None:
            state[slot].zero_()[..., :d] = S
    return o


def short_conv(x, taps, cu, slots, pos0, tail):
    """Causal depthwise convolution + silu on ``x [T, C]``, taps ``[C, n]``; ``tail [slots, C, n - 1]`` holds the last
    inputs of every sequence, oldest first.  fp32 output."""
    n = taps.shape[1]
    y = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
    for a, b, slot, fresh in _segments(cu, slots, pos0):
        before = torch.zeros(n - 1, x.shape[1], device=x.device) if fresh else tail[slot].float().t()
        full = torch.cat((before, x[a:b].float()), 0)
        for j in range(n):
            y[a:b] += full[j:j + b - a] * taps[:, j].float()
        if slot is not None and n > 1:
            tail[slot] = full[full.shape[0] - (n - 1):].t().to(tail.dtype)
    return F.silu(y)


def delta_gates(a_out, A_log, dt_bias, b_out, H):
    """Decay ``exp(-exp(A_log) softplus(a + dt_bias))`` fp32 ``[T, H, d]`` and step size ``sigmoid(b)`` ``[T, H]``."""
    z = a_out.float() + dt_bias.float()
    g = torch.exp(-torch.exp(A_log.float()).view(H, 1) * F.softplus(z, threshold=1e9).view(z.shape[0], H, -1))
    return g, torch.sigmoid(b_out.float())


def unit_heads(x, eps=1e-6):
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + eps)


def delta_scan(q, k, v, g, beta, cu, slots, pos0, state):
    """q, k ``[T, G, d]``, g ``[T, H, d]``, v ``[T, H, dv]``, beta ``[T, H]`` → o fp32 ``[T, H, dv]``."""
    T, H, dv = v.shape
    d, rep = q.shape[2], H // q.shape[1]
    o = torch.zeros(T, H, dv, dtype=torch.float32, device=v.device)
    q, k = q.float().repeat_interleave(rep, 1), k.float().repeat_interleave(rep, 1)
    for a, b, slot, fresh in _segments(cu, slots, pos0):
        S = torch.zeros(H, dv, d, device=v.device) if fresh else state[slot][..., :d].clone()
        for t in range(a, b):
            S = S * g[t].unsqueeze(-2)
            e = beta[t].unsqueeze(-1) * (v[t].float() - (S * k[t].unsqueeze(-2)).sum(-1))
            S = S + e.unsqueeze(-1) * k[t].unsqueeze(-2)
            o[t] = (S * q[t].unsqueeze(-2)).sum(-1)
        if slot is not None:
            state[slot].zero_()[..., :d] = S
    return o


def head_norm_gate(o, w, gate, gate_act, eps, out_dtype):
    """Each head of ``o [T, H, dv]`` over its root mean square, times ``w`` (``[H * dv]`` or ``[dv]``, shared by the
    heads), times ``gate_act(gate [T, H * dv])``."""
    T, H, dv = o.shape
    y = o.float() / torch.sqrt(o.float().pow(2).mean(-1, keepdim=True) + eps)
    y = y * (w.float().view(1, H, dv) if w.numel() == H * dv and H > 1 else w.float().view(1, 1, dv))
    g = gate.float().view(T, H, dv)
    g = F.silu(g) if gate_act == "silu" else torch.sigmoid(g)
    return (y * g).reshape(T, H * dv).to(out_dtype)


def route(z, top):
    """Router logits ``[T, E]`` fp32 → (chosen experts int64 ``[T, top]``, their sigmoid scores fp32)."""
    s = torch.sigmoid(z.float())
    w, idx = torch.topk(s, top, dim=-1)
    return idx, w


def route_softmax(z, bias, top):
    """Router logits plus ``bias`` → (the ``top`` largest per token, the softmax over them)."""
    w, idx = torch.topk(z.float() if bias is None else z.float() + bias.float(), top, dim=-1)
    return idx, torch.softmax(w, -1)


def unblock(gate_up, block):
    """``[..., 2 F, W]`` with gate and up rows in alternating blocks → gate, up ``[..., F, W]``."""
    F_, W = gate_up.shape[-2] // 2, gate_up.shape[-1]
    v = gate_up.view(*gate_up.shape[:-2], F_ // block, 2, block, W)
    return v[..., 0, :, :].reshape(*gate_up.shape[:-2], F_, W), v[..., 1, :, :].reshape(*gate_up.shape[:-2], F_, W)


def moe_glu(h, idx, weight, gate_up, block, down):
    """sum over the chosen experts of ``w down_e (silu(gate_e h) * up_e h)`` → fp32; the weight joins the hidden units."""
    gate, up = unblock(gate_up, block)
    out = torch.zeros(h.shape[0], down.shape[1], dtype=torch.float32, device=h.device)
    for e in idx.unique().tolist():
        t, s = torch.nonzero(idx == e, as_tuple=True)
        a = F.silu(F.linear(h[t], gate[e]).float()) * F.linear(h[t], up[e]).float() * weight[t, s].unsqueeze(-1)
        out.index_add_(0, t, F.linear(a.to(h.dtype), down[e]).float())
    return out


def moe_relu2(h, idx, weight, up, down):
    """sum over the chosen experts of ``down_e relu(up_e (w h))^2``; up ``[E, F, W]``, down ``[E, W, F]`` → fp32."""
    out = torch.zeros(h.shape[0], down.shape[1], dtype=torch.float32, device=h.device)
    for e in idx.unique().tolist():
        t, s = torch.nonzero(idx == e, as_tuple=True)
        a = torch.relu(F.linear(h[t], up[e]).float() * weight[t, s].unsqueeze(-1)) ** 2
        out.index_add_(0, t, F.linear(a.to(h.dtype), down[e]).float())
    return out
