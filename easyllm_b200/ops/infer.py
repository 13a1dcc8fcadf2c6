"""Inference-only ops of the hybrid decoders: CUDA kernels for bf16 and fp32 CUDA tensors, ``reference_infer`` on CPU.

None of them is differentiable.  Matrix products of the bf16 path run on the tcgen05 GEMM (accumulating straight into
the fp32 residual stream where the result is added to it) or, for a few rows, on a matrix-vector kernel bound by the
weight bytes; in fp32 they are true fp32 library products.  ``meta`` is the packed description of a step or a batch:
``cu_seqlens``, and with states ``seq_slot`` / ``seq_pos0`` (``DecodeState.step_meta``).
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _adjacent_alias
from . import reference_infer as ref

_ROWS = 32              # recurrent state rows (key channels) are padded to a multiple of this


def padded_rows(d):
    return -(-d // _ROWS) * _ROWS


def _kern(x):
    """CUDA bf16 / fp32 tensors take the kernels; there is no PyTorch path for them."""
    return x.is_cuda and x.dtype in (torch.bfloat16, torch.float32)


def _cu():
    from . import cuda_infer
    return cuda_infer


def no_grad_check(*ts):
    if torch.is_grad_enabled() and any(t.requires_grad for t in ts):
        raise RuntimeError("the hybrid decoder layers are inference-only: run them under torch.no_grad()")


def make_adjacent_(params):
    """Move parameters of one group back to back into one storage, so that ``fused`` aliases them without a copy.
    Parameters that live in a larger buffer (an optimizer's flat one) are left where they are."""
    if len(params) < 2 or any(getattr(p, "main_grad", None) is not None for p in params) or fused_alias(params) is not None:
        return
    if len({(p.dtype, p.device) for p in params}) != 1 or \
            any(p.untyped_storage().nbytes() != p.numel() * p.element_size() for p in params):
        return                                          # a view of somebody's larger buffer stays where it is
    flat = torch.cat([p.detach().reshape(-1) for p in params])
    at = 0
    for p in params:
        p.data = flat[at:at + p.numel()].view(p.shape)
        at += p.numel()


def fused_alias(params):
    ts = [p.detach() if p.dim() != 1 else p.detach().unsqueeze(1) for p in params]
    a = ts[0] if len(ts) == 1 else _adjacent_alias(ts)
    return a if a is None or params[0].dim() != 1 else a.squeeze(1)


def fused(params):
    a = fused_alias(params)
    return torch.cat([p.detach() for p in params], 0) if a is None else a


def _host(meta, name):
    """Index tensor of ``meta`` as a host list (CPU path)."""
    t = meta.get(name)
    return None if t is None else t.tolist()


def _seq(meta, state):
    return (_host(meta, "cu_seqlens"), None if state is None else _host(meta, "seq_slot"),
            None if state is None else _host(meta, "seq_pos0"))


# ---- matrix products ---------------------------------------------------------------------------
def linear(x, w, bias=None):
    """``x Wᵀ (+ bias)`` in x's dtype; x may be a column slice of a wider tensor."""
    return _cu().linear(x, w.detach(), bias) if _kern(x) else F.linear(x, w, bias)


def linear_f32(x, w):
    """``x Wᵀ`` with the fp32 accumulator kept."""
    return _cu().linear(x, w.detach(), out_f32=True) if _kern(x) else F.linear(x.float(), w.float())


def linear_act(x, w, act):
    y = _cu().linear(x, w.detach(), act=act) if _kern(x) else torch.tanh(F.linear(x, w).float()).to(x.dtype)
    return y


def linear_cat(x, weights, biases=None):
    """``x [W_1; W_2; ...]ᵀ`` for separate parameters; aliased, not concatenated, once they are adjacent."""
    return linear(x, fused(weights), None if biases is None else fused(biases))


def linear_cat_f32(x, weights):
    return linear_f32(x, fused(weights))


def linear_batch(xs, weights):
    """``xs[i] W_iᵀ`` for equally shaped weights → ``[n, T, N]``."""
    if _kern(xs):
        return _cu().linear_batch(xs, fused(weights).view(len(weights), *weights[0].shape))
    return torch.stack([F.linear(x, w) for x, w in zip(xs, weights)])


def linear_add_(acc, x, w):
    """``acc += x Wᵀ`` on an fp32 ``acc``."""
    no_grad_check(x, w)
    if _kern(x):
        return _cu().linear_add_(acc, x, w.detach())
    return acc.add_(F.linear(x, w).float())


def head_products(x, w, out=None):
    """Per head ``x[:, h] W_hᵀ``: x ``[T, H, K]``, w ``[H, N, K]`` → ``[T, H, N]`` (``out``: may be a slice of wider rows)."""
    if out is None:
        out = torch.empty(x.shape[0], w.shape[0], w.shape[1], dtype=x.dtype, device=x.device)
    if _kern(x):
        return _cu().head_products(x, w, out)
    out.copy_(torch.einsum("thk,hnk->thn", x, w))
    return out


# ---- elementwise -------------------------------------------------------------------------------
def embed_scaled(ids, table, scale):
    """fp32 ``table[ids] * scale``."""
    if _kern(table):
        return _cu().embed_scaled(ids, table.detach(), scale)
    return F.embedding(ids, table).float() * scale


def row_start(meta, n, device):
    """Row of the first token of each token's sequence in this batch."""
    if meta.get("row_start") is not None:
        return meta["row_start"]
    cu = meta["cu_seqlens"].long()
    return torch.repeat_interleave(cu[:-1], cu[1:] - cu[:-1], output_size=n).to(device=device, dtype=torch.int32)


def embed_pairs(ids, table, pairs, scale, mul_prev, mul_cur, meta, hist=None):
    """Embedding plus a table of (previous token, token) pairs, see ``reference_infer.embed_pairs``.  ``hist``: the state's
    token ids ``[slots, capacity]``, or None."""
    no_grad_check(table, pairs)
    start = row_start(meta, ids.numel(), ids.device)
    place = (meta["kv_base"], meta["kv_len"], hist.view(-1)) if hist is not None else (None, None, None)
    f = _cu().embed_pairs if _kern(table) else ref.embed_pairs
    return f(ids, table.detach(), pairs.detach(), scale, mul_prev, mul_cur, start, *place)


def layer_norms(x, weights, eps, out_dtype):
    """Layer norms of one fp32 ``x`` with one or two weights and no bias; the statistics are taken once."""
    ws = [w.detach() for w in weights]
    return _cu().layer_norms(x, ws, eps, out_dtype) if x.is_cuda else ref.layer_norms(x, ws, eps, out_dtype)


def dynamic_tanh(x, alpha, w, b, out_dtype, add=None):
    if x.is_cuda:
        return _cu().dynamic_tanh(x, alpha.detach(), w.detach(), b.detach(), out_dtype, add)
    y = ref.dynamic_tanh(x, alpha, w, b, out_dtype)
    if add is not None:
        x.add_(add.float())
    return y


def glu(gu, act):
    if _kern(gu):
        return _cu().glu(gu, act)
    F_ = gu.shape[-1] // 2
    g, u = gu[..., :F_].float(), gu[..., F_:].float()
    return ((ref.gelu_tanh(g) if act == "gelu_tanh" else F.silu(g)) * u).to(gu.dtype)


def relu2_scaled(x, z):
    """``sigmoid(z_t) relu(x_t)^2``, z fp32 ``[T]`` (any stride)."""
    if _kern(x):
        return _cu().relu2_scaled(x, z)
    return (torch.sigmoid(z).unsqueeze(-1) * torch.relu(x.float()) ** 2).to(x.dtype)


# ---- attention -----------------------------------------------------------------------------------
def kv_append(kcache, vcache, k, v, meta):
    """Write the keys / values of the step's tokens to their places in the cache."""
    if _kern(k):
        return _cu().kv_append(kcache, vcache, k, v, meta["kv_base"], meta["kv_len"])
    rows = (meta["kv_base"] + meta["kv_len"] - 1).long()
    kcache.view(-1, *kcache.shape[2:])[rows] = k
    vcache.view(-1, *vcache.shape[2:])[rows] = v


def attention_rows(q, k, v, kv_base, kv_len, max_len, scale, sink=None, alibi_slopes=None, window=None, gate=None):
    """Causal attention of query rows over key/value rows (a cache, or the packed batch itself), see
    ``reference_infer.attention_rows``.  ``max_len`` bounds ``kv_len``."""
    if _kern(q):
        return _cu().attention_rows(q, k, v, kv_base, kv_len, max_len, scale, sink, alibi_slopes, window, gate)
    return ref.attention_rows(q, k, v, kv_base, kv_len, scale, sink, alibi_slopes, window, gate)


def prefill_kernel_ok(q, v):
    """Whether the tcgen05 attention kernel takes packed prompts of these head sizes."""
    return q.is_cuda and q.dtype == torch.bfloat16 and max(q.shape[-1], v.shape[-1]) <= 128 and \
        q.shape[-1] % 8 == 0 and v.shape[-1] % 8 == 0


def attention_prefill(q, k, v, row_start, scale, sink=None, alibi_slopes=None, window=None):
    return _cu().attention_prefill(q, k, v, row_start, scale, sink, alibi_slopes, window)


# ---- latent attention ------------------------------------------------------------------------------
def latent_inputs(z, H, dim, rot, rank, norm_w, eps, cos, sin, meta, cache=None, q_dst=None):
    """Rotations and latent norm on the projection rows, in place, see ``reference_infer.latent_inputs``.  ``cache
    [slots, capacity, ld]`` receives latent and rotated key part of the step's tokens."""
    if _kern(z):
        return _cu().latent_inputs(z, H, dim, rot, rank, norm_w.detach(), eps, cos, sin, meta, cache, q_dst)
    pos = meta["position_ids"].long()
    ref.latent_inputs(z, H, dim, rot, rank, norm_w, eps, cos[pos], sin[pos], q_dst)
    if cache is not None:
        rows = (meta["kv_base"] + meta["kv_len"] - 1).long()
        at = H * (dim + rot)
        cache.view(-1, cache.shape[-1])[rows, :rank + rot] = z[:, at:at + rank + rot]


def attention_latent(q, rows, dv, kv_base, kv_len, max_len, scale, window=None, gate=None):
    """Attention in the latent space: q ``[T, H, d]`` over one key row ``rows[:, :d]`` per position, shared by all heads,
    whose first ``dv`` columns are the value → ``[T, H, dv]``.  Places as in ``attention_rows``."""
    if _kern(q):
        return _cu().attention_latent(q, rows, dv, kv_base, kv_len, max_len, scale, window, gate)
    k = rows[:, :q.shape[-1]].unsqueeze(1)
    return ref.attention_rows(q, k, k[..., :dv], kv_base, kv_len, scale, window=window, gate=gate)


def latent_prefill_ok(z, dim, rot, rank, vdim):
    """Whether the tcgen05 attention kernel takes packed prompts with keys of these two parts."""
    return z.is_cuda and z.dtype == torch.bfloat16 and not (dim % 8 or rot % 8 or vdim % 8 or rank % 8) and min(dim, rot) > 0 \
        and -(-dim // 64) + -(-rot // 64) <= 3 and vdim <= 128 and z.stride(0) % 8 == 0


def attention_latent_prefill(z, kv, H, dim, rot, rank, vdim, row_start, scale, window=None, gate=None):
    """Packed prompts: queries and the shared key part from the projection rows ``z``, the heads' own key parts and values
    from ``kv [T, H dim + H vdim]`` → ``[T, H, vdim]``."""
    return _cu().attention_latent_prefill(z, kv, H, dim, rot, rank, vdim, row_start, scale, window, gate)


# ---- recurrences -----------------------------------------------------------------------------------
def token_mix(h, mu, meta, tail):
    if _kern(h):
        return _cu().token_mix(h, mu.detach(), meta, tail)
    return ref.token_mix(h, mu, *_seq(meta, tail), tail)


def wkv_decay_(z, w0):
    """``exp(-exp(z + w0))`` in place on fp32 ``z``."""
    if z.is_cuda:
        return _cu().wkv_decay_(z, w0.detach())
    return z.add_(w0).exp_().neg_().exp_()


def wkv_scan(r, k, v, decay, u, meta, state):
    if _kern(k):
        return _cu().wkv_scan(r, k, v, decay, u.detach(), meta, state)
    return ref.wkv_scan(r, k, v, decay, u, *_seq(meta, state), state)


def delta_inputs(qkv, convs, a, A_log, dt_bias, b, H, G, d, dv, meta, tail):
    """Short convolutions with silu, unit q / k, decays and step sizes of the delta rule, all fp32."""
    if _kern(qkv):
        return _cu().delta_inputs(qkv, fused(convs), a, A_log.detach(), dt_bias.detach(), b, H, G, d, dv, meta, tail)
    T = qkv.shape[0]
    y = ref.short_conv(qkv, torch.cat(list(convs), 0), *_seq(meta, tail), tail)
    q, k, v = y.split([G * d, G * d, H * dv], -1)
    g, beta = ref.delta_gates(a, A_log, dt_bias, b, H)
    return (ref.unit_heads(q.view(T, G, d)) * d ** -0.5, ref.unit_heads(k.view(T, G, d)), v.reshape(T, H, dv), g, beta)


def delta_scan(q, k, v, g, beta, meta, state):
    if v.is_cuda:
        return _cu().delta_scan(q, k, v, g, beta, meta, state)
    return ref.delta_scan(q, k, v, g, beta, *_seq(meta, state), state)


def head_norm_gate(o, w, gate, gate_act, eps, out_dtype):
    if o.is_cuda:
        return _cu().head_norm_gate(o, w.detach(), gate, gate_act, eps, out_dtype)
    return ref.head_norm_gate(o, w, gate, gate_act, eps, out_dtype)


# ---- mixture of experts ------------------------------------------------------------------------------
def moe_relu2_add_(acc, h, z, top, up, down):
    """``acc += sum over the top experts of down_e relu(up_e (s_e h))^2`` with scores ``s = sigmoid(z)``."""
    no_grad_check(h, up)
    if _kern(h):
        return _cu().moe_relu2_add_(acc, h, z, top, up.detach(), down.detach())
    idx, w = ref.route(z, top)
    return acc.add_(ref.moe_relu2(h, idx, w, up, down))


def moe_glu_add_(acc, h, z, bias, top, gate_up, block, down):
    """``acc += sum over the top experts of w_e down_e (silu(gate_e h) * up_e h)``, ``w`` the softmax over the chosen logits
    of ``z + bias``; gate_up ``[E, 2 F, W]`` holds gate and up rows in alternating blocks of ``block``."""
    no_grad_check(h, gate_up)
    bias = None if bias is None else bias.detach()
    if _kern(h):
        return _cu().moe_glu_add_(acc, h, z, bias, top, gate_up.detach(), block, down.detach())
    idx, w = ref.route_softmax(z, bias, top)
    return acc.add_(ref.moe_glu(h, idx, w, gate_up, block, down))
