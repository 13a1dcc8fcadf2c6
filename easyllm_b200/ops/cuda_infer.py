"""Launchers of the inference kernels (``csrc/infer_elementwise.cu``, ``recurrent.cu``, ``attn_rows.cu``, ``matvec.cu``,
and the tcgen05 GEMM / attention) for bf16 and fp32 CUDA tensors; the signatures are those of ``ops.infer``."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong

import torch

from . import cuda as cu
from .cuda import _p, _stream, err_flag, lib, scratch

MATVEC_ROWS = 16        # up to this many rows a product is bound by the weight bytes and runs on the matrix-vector kernel


def _check(rc, name, launches=1):
    cu._check(rc, name)
    cu.LAUNCHES += launches - 1


def _bf(dtype):
    if dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"inference kernels take bf16 or fp32 activations, got {dtype}")
    return c_int(1 if dtype == torch.bfloat16 else 0)


def _rows(t, name):
    """Row stride of a 2-D tensor whose rows are contiguous."""
    if t.dim() != 2 or (t.stride(1) != 1 and t.shape[1] != 1):
        raise ValueError(f"{name}: expected rows of contiguous elements, got strides {t.stride()}")
    return t.stride(0) if t.shape[0] > 1 else t.shape[1]


def _f32(t, name):
    if t.dtype != torch.float32 or not t.is_contiguous():
        raise ValueError(f"{name}: expected a contiguous fp32 tensor")
    return t


# ---- matrix products ---------------------------------------------------------------------------
def _gemm_fits(x, ldx, w, ldc, elem):
    """Whether the TMA-fed GEMM takes these operands (16-byte starts and row strides)."""
    return x.shape[1] % 8 == 0 and ldx % 8 == 0 and (ldc * elem) % 16 == 0 and not (x.data_ptr() | w.data_ptr()) & 15


def _gemm(x, ldx, w, bias, out, ldc, out_mode):
    """Plain tcgen05 GEMM with explicit row strides."""
    M, K, N = x.shape[0], x.shape[1], w.shape[0]
    args = (_p(x), _p(w), _p(out), _p(bias), c_int(M), c_int(N), c_int(K), c_int(ldx), c_int(K), c_int(ldc), c_int(0),
            c_int(0), c_int(out_mode))
    if cu._use_pair(M, N, 0):
        rc = lib().ell_gemm_bf16_pair(*args, _p(err_flag(x.device)), _stream())
        if rc not in cu._PAIR_LAUNCH_REFUSED:
            return _check(rc, "gemm_bf16_pair")
    _check(lib().ell_gemm_bf16(*args, c_int(0), _p(err_flag(x.device)), _stream()), "gemm_bf16")


def _matvec(x, ldx, w, bias, out, ldo, out_f32=False, accumulate=False, act_tanh=False, batch=1, strides=(0, 0, 0)):
    _check(lib().ell_matvec(_p(x), _p(w), _p(bias), _p(out), *(c_longlong(s) for s in strides), c_int(batch),
                            c_int(x.shape[-2]), c_int(w.shape[-2]), c_int(x.shape[-1]), c_int(ldx), c_int(ldo),
                            c_int(out_f32), c_int(accumulate), c_int(act_tanh), _bf(x.dtype), _stream()), "matvec")
    return out


def linear(x, w, bias=None, out_f32=False, act=None):
    """``x Wᵀ (+ bias)``, optionally with the fp32 accumulator kept or through tanh.  The result's rows are padded to 8
    elements, so it may be a column view."""
    if x.dtype != w.dtype or not w.is_contiguous():
        raise ValueError(f"linear: x {x.dtype} and a contiguous weight of that dtype, got {w.dtype}")
    bias = None if bias is None else bias.detach()
    ldx, M, N = _rows(x, "x"), x.shape[0], w.shape[0]
    dt = torch.float32 if out_f32 else x.dtype
    ld = -(-N // 8) * 8
    if M > MATVEC_ROWS and x.dtype == torch.float32:
        y = torch.nn.functional.linear(x, w, bias)
        return torch.tanh(y) if act == "tanh" else y
    if M > MATVEC_ROWS and _gemm_fits(x, ldx, w, ld, 4 if out_f32 or act else 2) and (bias is None or N % 8 == 0):
        if act == "tanh":
            z = torch.empty(M, ld, dtype=torch.float32, device=x.device)
            _gemm(x, ldx, w, bias, z, ld, 2)
            y = torch.empty(M, N, dtype=x.dtype, device=x.device)
            _check(lib().ell_tanh_cast(_p(z), _p(y), c_int(M), c_int(N), c_int(ld), _bf(x.dtype), _stream()), "tanh_cast")
            return y
        y = torch.empty(M, ld, dtype=dt, device=x.device)
        _gemm(x, ldx, w, bias, y, ld, 2 if out_f32 else 0)
        return y[:, :N]
    y = torch.empty(M, ld, dtype=dt, device=x.device)
    return _matvec(x, ldx, w, bias, y, ld, out_f32=out_f32, act_tanh=act == "tanh")[:, :N]


def linear_batch(xs, w):
    """xs ``[n, T, K]``, w ``[n, N, K]`` contiguous → ``[n, T, N]``."""
    n, M, K = xs.shape
    N = w.shape[1]
    y = torch.empty(n, M, N, dtype=xs.dtype, device=xs.device)
    if M <= MATVEC_ROWS or (xs.dtype == torch.bfloat16 and not _gemm_fits(xs[0], K, w[0], N, 2)):
        return _matvec(xs, K, w, None, y, N, batch=n, strides=(M * K, N * K, M * N))
    if xs.dtype == torch.float32:
        return torch.bmm(xs, w.transpose(1, 2), out=y)
    for i in range(n):
        _gemm(xs[i], K, w[i], None, y[i], N, 0)
    return y


def head_products(x, w, out):
    (T, H, K), N = x.shape, w.shape[1]
    if w.shape != (H, N, K) or not w.is_contiguous() or x.stride(2) != 1 or out.stride(2) != 1 or out.shape != (T, H, N) or \
            not x.dtype == w.dtype == out.dtype:
        raise ValueError("head_products: x [T, H, K], a contiguous w [H, N, K] and out [T, H, N] of one dtype")
    _check(lib().ell_matvec(_p(x), _p(w), _p(None), _p(out), c_longlong(x.stride(1)), c_longlong(N * K),
                            c_longlong(out.stride(1)), c_int(H), c_int(T), c_int(N), c_int(K), c_int(x.stride(0)),
                            c_int(out.stride(0)), c_int(0), c_int(0), c_int(0), _bf(x.dtype), _stream()), "head_products")
    return out


def linear_add_(acc, x, w):
    _f32(acc, "acc")
    ldx, M, N = _rows(x, "x"), x.shape[0], w.shape[0]
    if acc.shape != (M, N):
        raise ValueError(f"linear_add_: {tuple(acc.shape)} += [{M}, {N}]")
    if M > MATVEC_ROWS and x.dtype == torch.float32:
        return acc.addmm_(x, w.t())
    if M > MATVEC_ROWS and _gemm_fits(x, ldx, w, N, 4):
        _gemm(x, ldx, w, None, acc, N, 1)
        return acc
    return _matvec(x, ldx, w, None, acc, N, accumulate=True)


# ---- elementwise -------------------------------------------------------------------------------
def embed_scaled(ids, table, scale):
    ids = ids.reshape(-1).to(torch.int64).contiguous()
    out = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    _check(lib().ell_embed_scaled(_p(ids), _p(table), _p(out), c_int(ids.numel()), c_int(table.shape[1]),
                                  c_longlong(table.shape[0]), c_float(scale), _bf(table.dtype), _p(err_flag(table.device)),
                                  _stream()), "embed_scaled")
    return out


def embed_pairs(ids, table, pairs, scale, mul_prev, mul_cur, row_start, kv_base=None, kv_len=None, hist=None):
    ids = ids.reshape(-1).to(torch.int64).contiguous()
    n, W = ids.numel(), table.shape[1]
    if pairs.shape[1] != W or pairs.dtype != table.dtype or not (table.is_contiguous() and pairs.is_contiguous()):
        raise ValueError("embed_pairs: two contiguous tables of one width and dtype")
    if row_start.dtype != torch.int32 or (hist is not None and hist.dtype != torch.int32):
        raise ValueError("embed_pairs: int32 row_start and token history")
    out = torch.empty(n, W, dtype=torch.float32, device=table.device)
    _check(lib().ell_embed_pairs(_p(ids), _p(table), _p(pairs), _p(out), _p(row_start), _p(kv_base), _p(kv_len), _p(hist),
                                 c_int(n), c_int(W), c_longlong(table.shape[0]), c_longlong(pairs.shape[0] - 1),
                                 c_longlong(mul_prev), c_longlong(mul_cur), c_float(scale), _bf(table.dtype),
                                 _p(err_flag(table.device)), _stream()), "embed_pairs")
    return out


def layer_norms(x, weights, eps, out_dtype):
    _f32(x, "x")
    n, W = x.shape
    ys = [torch.empty(n, W, dtype=out_dtype, device=x.device) for _ in weights]
    if not 1 <= len(weights) <= 2 or any(w.numel() != W for w in weights):
        raise ValueError("layer_norms: one or two weights of the row's length")
    w = [_f32(t, "weight") for t in weights] + [None]
    _check(lib().ell_layer_norms(_p(x), _p(w[0]), _p(w[1]), _p(ys[0]), _p(ys[-1]), c_int(n), c_int(W), c_float(eps),
                                 _bf(out_dtype), _stream()), "layer_norms")
    return ys


def dynamic_tanh(x, alpha, w, b, out_dtype, add=None):
    _f32(x, "x"), _f32(w, "weight"), _f32(b, "bias")
    y = torch.empty(x.shape, dtype=out_dtype, device=x.device)
    add = None if add is None else add.detach()
    if add is not None and add.dtype != out_dtype:
        raise ValueError("dynamic_tanh: `add` must have the output's dtype")
    _check(lib().ell_dynamic_tanh(_p(x), _p(alpha), _p(w), _p(b), _p(add), _p(y), c_int(x.shape[0]), c_int(x.shape[1]),
                                  _bf(out_dtype), _stream()), "dynamic_tanh")
    return y


def glu(gu, act):
    F = gu.shape[1] // 2
    out = torch.empty(gu.shape[0], F, dtype=gu.dtype, device=gu.device)
    _check(lib().ell_glu(_p(gu), _p(out), c_int(gu.shape[0]), c_int(F), c_int(_rows(gu, "gate_up")),
                         c_int({"silu": 0, "gelu_tanh": 1}[act]), _bf(gu.dtype), _stream()), "glu")
    return out


def relu2_scaled(x, z):
    n, F = x.shape
    out = torch.empty(n, F, dtype=x.dtype, device=x.device)
    if z.dtype != torch.float32 or z.dim() != 1:
        raise ValueError("relu2_scaled: z must be fp32 [T]")
    _check(lib().ell_relu2_scaled(_p(x), _p(z), _p(out), c_int(n), c_int(F), c_int(_rows(x, "x")), c_int(z.stride(0)),
                                  _bf(x.dtype), _stream()), "relu2_scaled")
    return out


# ---- attention -----------------------------------------------------------------------------------
def _heads(t, name):
    """Row stride of ``[T, heads, dim]`` with packed heads."""
    if t.stride(2) != 1 or (t.shape[1] > 1 and t.stride(1) != t.shape[2]):
        raise ValueError(f"{name}: heads must be packed in a row")
    return t.stride(0) if t.shape[0] > 1 else t.shape[1] * t.shape[2]


def kv_append(kcache, vcache, k, v, base, length):
    if not (kcache.is_contiguous() and vcache.is_contiguous()) or kcache.dtype != k.dtype:
        raise ValueError("kv_append: contiguous caches of the activations' dtype")
    T = k.shape[0]
    _check(lib().ell_kv_append(_p(k), _p(v), _p(kcache), _p(vcache), _p(base), _p(length), c_int(T),
                               c_int(k.shape[1] * k.shape[2]), c_int(v.shape[1] * v.shape[2]), c_int(_heads(k, "k")),
                               c_int(_heads(v, "v")), _bf(k.dtype), _stream()), "kv_append")


def _gate(gate, like):
    """(gate, row stride) as kernel arguments: rows of the activations' dtype."""
    if gate is None:
        return _p(None), c_int(0)
    if gate.dtype != like.dtype:
        raise ValueError("the output gate must have the activations' dtype")
    return _p(gate), c_int(_rows(gate, "gate"))


def attention_rows(q, k, v, base, length, max_len, scale, sink=None, alibi_slopes=None, window=None, gate=None):
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    max_len = min(max_len, window) if window else max_len
    out = torch.empty(T, H, dv, dtype=q.dtype, device=q.device)
    need = lib().ell_attn_rows_scratch(c_int(T), c_int(H), c_int(G), c_int(dv), c_int(max_len))
    part = torch.empty(need, dtype=torch.float32, device=q.device) if need else None
    sl = cu._slopes(alibi_slopes, H, q.device)
    _check(lib().ell_attn_rows(_p(q), _p(k), _p(v), _p(out), _p(part), _p(base), _p(length),
                               _p(None if sink is None else _f32(sink, "sink")), _p(sl), _gate(gate, q)[0], c_int(T),
                               c_int(H), c_int(G), c_int(d), c_int(dv), c_int(_heads(q, "q")), c_int(_heads(k, "k")),
                               c_int(_heads(v, "v")), _gate(gate, q)[1], c_int(max_len), c_int(window or 0), c_float(scale),
                               _bf(q.dtype), _stream()), "attn_rows", 2 if need else 1)
    return out


def attention_prefill(q, k, v, row_start, scale, sink=None, alibi_slopes=None, window=None):
    """Packed prompts on the tcgen05 kernel (bf16, heads of up to 128)."""
    return cu.flash_attn_fwd(q, k, v, row_start, scale, alibi_slopes, sink, window)[0]


# ---- latent attention ------------------------------------------------------------------------------
def latent_inputs(z, H, dim, rot, rank, norm_w, eps, cos, sin, meta, cache=None, q_dst=None):
    n, ldz = z.shape[0], _rows(z, "z") and z.stride(0)
    pos = meta["position_ids"]
    if pos.dtype != torch.int32 or cos.shape != sin.shape or not (_f32(cos, "cos") is cos and _f32(sin, "sin") is sin):
        raise ValueError("latent_inputs: int32 positions, fp32 angle tables")
    if z.shape[1] < H * (dim + rot) + rank + rot or norm_w.numel() != rank:
        raise ValueError("latent_inputs: the rows hold H (dim + rot) + rank + rot columns")
    if cache is not None and (cache.dtype != z.dtype or not cache.is_contiguous() or cache.shape[-1] < rank + rot):
        raise ValueError("latent_inputs: a contiguous cache of the activations' dtype")
    if q_dst is not None and (q_dst.dtype != z.dtype or q_dst.stride(2) != 1 or
                              (n > 1 and q_dst.stride(0) != H * q_dst.stride(1))):
        raise ValueError("latent_inputs: q_dst must be a slice of packed heads")
    _check(lib().ell_latent_inputs(_p(z), _p(q_dst), _p(cache), _p(_f32(norm_w, "norm")), _p(cos), _p(sin), _p(pos),
                                   _p(None if cache is None else meta["kv_base"]),
                                   _p(None if cache is None else meta["kv_len"]), c_int(n), c_int(H), c_int(dim), c_int(rot),
                                   c_int(rank), c_int(cos.shape[1]), c_int(ldz), c_int(0 if q_dst is None else q_dst.stride(1)),
                                   c_int(0 if cache is None else cache.shape[-1]), c_float(eps), _bf(z.dtype), _stream()),
           "latent_inputs")


def attention_latent(q, rows, dv, base, length, max_len, scale, window=None, gate=None):
    T, H, d = q.shape
    ldk = _rows(rows, "rows")
    if rows.dtype != q.dtype or rows.shape[1] < d or dv > d:
        raise ValueError("attention_latent: key rows of the queries' dtype and size")
    out = torch.empty(T, H, dv, dtype=q.dtype, device=q.device)
    shape = (c_int(T), c_int(H), c_int(d), c_int(dv), c_int(_heads(q, "q")), c_int(ldk))
    need = lib().ell_attn_latent_scratch(_p(rows), *shape, c_int(max_len), c_int(window or 0), _bf(q.dtype))
    part = torch.empty(need, dtype=torch.float32, device=q.device) if need else None
    g, ldg = _gate(gate, q)
    _check(lib().ell_attn_latent(_p(q), _p(rows), _p(out), _p(part), _p(base), _p(length), g, *shape, ldg, c_int(max_len),
                                 c_int(window or 0), c_longlong(rows.shape[0]), c_float(scale), _bf(q.dtype), _p(err_flag(q.device)), _stream()),
           "attn_latent", 2 if need else 1)
    return out


def attention_latent_prefill(z, kv, H, dim, rot, rank, vdim, row_start, scale, window=None, gate=None):
    T, at = z.shape[0], H * (dim + rot)
    out = torch.empty(T, H, vdim, dtype=z.dtype, device=z.device)
    k2, v = z[:, at + rank:], kv[:, H * dim:]
    g, ldg = _gate(gate, z)
    ldz, ldkv = _rows(z, "z") and z.stride(0), _rows(kv, "kv")
    _check(lib().ell_flash_attn_latent(_p(z), _p(kv), _p(k2), _p(v), _p(out), _p(row_start), g, c_int(T), c_int(H), c_int(dim),
                                       c_int(rot), c_int(vdim), c_int(ldz), c_int(ldkv), c_int(ldz), c_int(ldkv), ldg,
                                       c_int(window or 0), c_float(scale), _p(err_flag(z.device)), _stream()),
           "flash_attn_latent")
    return out


# ---- recurrences -----------------------------------------------------------------------------------
def _seq(meta, state):
    """(cu, slots, pos0, number of sequences) as kernel arguments."""
    cus = meta["cu_seqlens"]
    if cus.dtype != torch.int32:
        raise ValueError("cu_seqlens must be int32")
    if state is None:
        return _p(cus), _p(None), _p(None), cus.numel() - 1
    if not state.is_contiguous():
        raise ValueError("state tensors must be contiguous")
    return _p(cus), _p(meta["seq_slot"]), _p(meta["seq_pos0"]), cus.numel() - 1


def token_mix(h, mu, meta, tail):
    T, W = h.shape
    out = torch.empty(mu.shape[0], T, W, dtype=h.dtype, device=h.device)
    c, sl, p0, n = _seq(meta, tail)
    _check(lib().ell_token_mix(_p(h), _p(_f32(mu, "mu")), _p(out), c, sl, p0, _p(tail), c_int(T), c_int(n),
                               c_int(meta["max_seqlen"]), c_int(W), c_int(mu.shape[0]), _bf(h.dtype), _stream()), "token_mix")
    return out


def wkv_decay_(z, w0):
    if z.stride(0) != z.shape[1] and z.shape[0] > 1:
        z = z.contiguous()
    _check(lib().ell_wkv_decay(_p(z), _p(_f32(w0, "w0")), c_int(z.shape[0]), c_int(z.shape[1]), _stream()), "wkv_decay")
    return z


def wkv_scan(r, k, v, decay, u, meta, state):
    T, H, d = k.shape
    dv = v.shape[2]
    o = torch.empty(T, H, dv, dtype=torch.float32, device=k.device)
    c, sl, p0, n = _seq(meta, state)
    _check(lib().ell_wkv_scan(_p(r), _p(k), _p(v), _p(_f32(decay, "decay")), _p(_f32(u, "u")), _p(o), _p(state), c, sl, p0,
                              c_int(n), c_int(H), c_int(d), c_int(dv), c_int(_heads(r, "r")), c_int(_heads(k, "k")),
                              c_int(_heads(v, "v")), _bf(k.dtype), _stream()), "wkv_scan")
    return o


def delta_inputs(qkv, taps, a, A_log, dt_bias, b, H, G, d, dv, meta, tail):
    T = qkv.shape[0]

    def f32(*shape):
        return torch.empty(*shape, dtype=torch.float32, device=qkv.device)
    q, k, v, beta = f32(T, G, d), f32(T, G, d), f32(T, H, dv), f32(T, H)
    g = a if a.is_contiguous() else a.contiguous()
    if b.dtype != torch.float32:
        raise ValueError("delta_inputs: fp32 step-size logits")
    c, sl, p0, n = _seq(meta, tail)
    _check(lib().ell_delta_inputs(_p(qkv), _p(_f32(taps, "taps")), _p(_f32(g, "a")), _p(_f32(A_log, "A_log")),
                                  _p(_f32(dt_bias, "dt_bias")), _p(b), _p(q), _p(k), _p(v), _p(beta), _p(tail), c, sl, p0,
                                  c_int(n), c_int(meta["max_seqlen"]), c_int(H), c_int(G), c_int(d), c_int(dv),
                                  c_int(taps.shape[1]), c_int(_rows(qkv, "qkv")), c_int(_rows(b, "b")), _bf(qkv.dtype),
                                  _stream()), "delta_inputs")
    return q, k, v, g.view(T, H, d), beta


def delta_scan(q, k, v, g, beta, meta, state):
    T, H, dv = v.shape
    o = torch.empty(T, H, dv, dtype=torch.float32, device=v.device)
    c, sl, p0, n = _seq(meta, state)
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (g, "g"), (beta, "beta")):
        _f32(t, name)
    _check(lib().ell_delta_scan(_p(q), _p(k), _p(v), _p(g), _p(beta), _p(o), _p(state), c, sl, p0, c_int(n), c_int(H),
                                c_int(q.shape[1]), c_int(q.shape[2]), c_int(dv), _stream()), "delta_scan")
    return o


def head_norm_gate(o, w, gate, gate_act, eps, out_dtype):
    T, H, dv = o.shape
    y = torch.empty(T, H * dv, dtype=out_dtype, device=o.device)
    if gate.dtype != out_dtype:
        raise ValueError("head_norm_gate: the gate must have the output's dtype")
    _check(lib().ell_head_norm_gate(_p(_f32(o, "o")), _p(_f32(w, "w")), _p(gate), _p(y), c_int(T), c_int(H), c_int(dv),
                                    c_int(1 if w.numel() == H * dv else 0), c_int(_rows(gate, "gate")),
                                    c_int({"silu": 1, "sigmoid": 0}[gate_act]), c_float(eps), _bf(out_dtype), _stream()),
           "head_norm_gate")
    return y


# ---- mixture of experts ------------------------------------------------------------------------------
def moe_route(z, top, bias=None, softmax=False):
    """fp32 router logits ``[T, E]`` (plus ``bias [E]``) → (expert int32 ``[T, top]``, fp32 ``[T, top]``: sigmoid scores, or
    the softmax over the chosen logits)."""
    T, E = z.shape
    idx = torch.empty(T, top, dtype=torch.int32, device=z.device)
    w = torch.empty(T, top, dtype=torch.float32, device=z.device)
    if z.dtype != torch.float32:
        raise ValueError("moe_route: fp32 logits")
    _check(lib().ell_moe_route(_p(z), _p(None if bias is None else _f32(bias, "bias")), _p(idx), _p(w), c_int(T), c_int(E),
                               c_int(top), c_int(_rows(z, "z")), c_int(softmax), _stream()), "moe_route")
    return idx, w


def moe_relu2_add_(acc, h, z, top, up, down):
    return _moe_add_(acc, h, *moe_route(z, top), up, down)


def moe_glu_add_(acc, h, z, bias, top, gate_up, block, down):
    return _moe_add_(acc, h, *moe_route(z, top, bias, softmax=True), gate_up, down, block)


def _moe_add_(acc, h, idx, w, up, down, block=0):
    """``block`` 0: two-matrix experts; otherwise ``up`` holds gate and up rows in alternating blocks of that many."""
    _f32(acc, "acc")
    h = h.contiguous()
    T, W = h.shape
    E, F, top = up.shape[0], down.shape[2], idx.shape[1]
    if h.dtype == torch.bfloat16 and T * top > max(MATVEC_ROWS, 2 * E) and W % 8 == 0 and F % 8 == 0 and block in (0, 32):
        return _moe_grouped(acc, h, idx, w, up, down, block)
    step = max(1, 65535 // top)
    for t in range(0, T, step):                         # the slots are a grid dimension
        n = min(step, T - t)
        hid = torch.empty(n * top, F, dtype=h.dtype, device=h.device)
        _check(lib().ell_moe_rows(_p(h[t:]), _p(up), _p(down), _p(idx[t:]), _p(w[t:]), _p(hid), _p(acc[t:]), c_int(n),
                                  c_int(top), c_int(F), c_int(W), c_int(block), _bf(h.dtype), _stream()), "moe_rows", 2)
    return acc


def _moe_grouped(acc, h, idx, w, up, down, block=0):
    """Rows sorted by expert, two grouped tcgen05 GEMMs (the activation with the routing weight in the first one's
    epilogue), and the sum back into ``acc``.  The row plan stays on the device."""
    T, W = h.shape
    E, F = up.shape[0], down.shape[2]
    top, dev = idx.shape[1], h.device
    used = min(E, T * top)                              # experts that can have rows
    tiles = (T * top - used) // 128 + used              # most 128-row tiles any routing can need
    rows = tiles * 128
    ints = torch.empty(T * top + tiles + 1, dtype=torch.int32, device=dev)
    pos, tile_expert, n_tiles = ints.split([T * top, tiles, 1])
    scale = torch.empty(rows, dtype=torch.float32, device=dev)
    xs = torch.empty(rows, W, dtype=h.dtype, device=dev)
    _check(lib().ell_moe_gather(_p(h), _p(xs), _p(idx), _p(w), _p(pos), _p(scale), _p(tile_expert), _p(n_tiles), c_int(T),
                                c_int(top), c_int(E), c_int(W), _stream()), "moe_gather", 2)
    hid = torch.empty(rows, F, dtype=h.dtype, device=dev)
    ys = torch.empty(rows, W, dtype=h.dtype, device=dev)
    for x, wt, out, n, k, sc in ((xs, up, hid, up.shape[1], W, scale), (hid, down, ys, W, F, None)):
        _check(lib().ell_gemm_grouped(_p(x), _p(wt), _p(out), _p(tile_expert), _p(n_tiles), _p(sc), c_int(rows), c_int(n),
                                      c_int(k), c_int(E), c_int(bool(block) and sc is not None), _p(err_flag(dev)), _stream()),
               "gemm_grouped")
    _check(lib().ell_moe_combine(_p(ys), _p(pos), _p(acc), c_int(T), c_int(top), c_int(W), _stream()), "moe_combine")
    return acc
