"""Token mixers without a key/value cache, and the norms of the parallel blocks.

Each mixer is built from its sizes (a dict) and is called as ``mixer(h, meta, state, residual)``: ``h [T, hidden]`` are
the normed inputs of the packed sequences of ``meta``, ``state`` the layer's ``SlotTensors`` (None: every sequence starts
here and nothing is kept), and the output projection is accumulated into the fp32 stream ``residual``.

* ``DynamicTanh``: the norm ``tanh(alpha x) w + b``.
* ``LayerNorm``: layer norm without a bias, on the fp32 stream.
* ``TimeMix``: RWKV-style mixing with a decay per key channel and a bonus for the current token.
* ``ChannelDelta``: the gated delta rule with a decay per head and key channel, short convolutions on q, k, v.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import infer as iops
from .state import SlotTensors


def _vec(*shape, fill=0.0):
    return nn.Parameter(torch.full(shape, fill, dtype=torch.float32))


class DynamicTanh(nn.Module):
    """``tanh(alpha x) w + b``, all of it in fp32 whatever the model's dtype; no statistics."""

    def __init__(self, dim, dtype):
        super().__init__()
        self.weight, self.bias, self.alpha = _vec(dim, fill=1.0), _vec(dim), _vec(fill=0.5)
        self.out_dtype = dtype

    def forward(self, x, add=None):
        """Norm of ``x``.  ``add [dim]``: after its norm is taken, ``x`` (fp32, updated in place) gains this vector."""
        return iops.dynamic_tanh(x, self.alpha, self.weight, self.bias, self.out_dtype, add)


class LayerNorm(nn.Module):
    """``(x - mean) / sqrt(variance + eps) * w`` in fp32.  ``also``: a second norm of the same ``x``; both come from one
    pass, and the result is the pair."""

    def __init__(self, dim, eps, dtype):
        super().__init__()
        self.weight, self.eps, self.out_dtype = _vec(dim, fill=1.0), eps, dtype

    def forward(self, x, also=None):
        if also is None:
            return iops.layer_norms(x, [self.weight], self.eps, self.out_dtype)[0]
        return iops.layer_norms(x, [self.weight, also.weight], self.eps, self.out_dtype)


class TimeMix(nn.Module):
    MIXES = "rkvgw"

    def __init__(self, hidden, m, eps, dtype):
        super().__init__()
        self.h, self.d, self.eps = m["heads"], m["dim"], eps
        c, rank = self.h * self.d, m.get("decay_rank", 16)

        def lin(i, o):
            return nn.Linear(i, o, bias=False, dtype=dtype)
        self.mu = _vec(len(self.MIXES), hidden, fill=0.5)             # one row per mix, in the order of MIXES
        self.r_proj, self.k_proj, self.v_proj, self.g_proj = (lin(hidden, c) for _ in range(4))
        self.w1_proj, self.w2_proj = lin(hidden, rank), lin(rank, c)
        self.w0, self.u, self.norm = _vec(c), _vec(self.h, self.d), _vec(c, fill=1.0)
        self.o_proj = lin(c, hidden)

    def fused_groups(self):
        return [[p.weight for p in (self.r_proj, self.k_proj, self.v_proj, self.g_proj)]]

    def new_state(self, slots, capacity, device, dtype):
        return SlotTensors(slots, device, s=((self.h, self.d, iops.padded_rows(self.d)), torch.float32),
                           last=((self.mu.shape[1],), dtype))

    def forward(self, h, meta, state, residual):
        T = h.shape[0]
        mixes = iops.token_mix(h, self.mu, meta, state.last if state is not None else None)
        rkvg = iops.linear_batch(mixes[:4], [p.weight for p in (self.r_proj, self.k_proj, self.v_proj, self.g_proj)])
        low = iops.linear_act(mixes[4], self.w1_proj.weight, "tanh")
        decay = iops.wkv_decay_(iops.linear_f32(low, self.w2_proj.weight), self.w0)
        r, k, v = (rkvg[i].view(T, self.h, self.d) for i in range(3))
        o = iops.wkv_scan(r, k, v, decay.view(T, self.h, self.d), self.u, meta, state.s if state is not None else None)
        y = iops.head_norm_gate(o, self.norm, rkvg[3], "silu", self.eps, h.dtype)
        return iops.linear_add_(residual, y, self.o_proj.weight)


class ChannelDelta(nn.Module):
    def __init__(self, hidden, m, eps, dtype):
        super().__init__()
        self.h, self.g, self.d, self.dv, self.taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        self.eps = eps
        ra, rg = m.get("decay_rank", 16), m.get("gate_rank", 16)
        qk, vv = self.g * self.d, self.h * self.dv

        def lin(i, o):
            return nn.Linear(i, o, bias=False, dtype=dtype)
        self.q_proj, self.k_proj, self.v_proj = lin(hidden, qk), lin(hidden, qk), lin(hidden, vv)
        self.q_conv, self.k_conv, self.v_conv = (_vec(n, self.taps) for n in (qk, qk, vv))
        self.a1_proj, self.a2_proj = lin(hidden, ra), lin(ra, self.h * self.d)
        self.g1_proj, self.g2_proj = lin(hidden, rg), lin(rg, vv)
        self.b_proj = lin(hidden, self.h)
        self.A_log, self.dt_bias, self.norm = _vec(self.h), _vec(self.h * self.d), _vec(self.dv, fill=1.0)
        self.o_proj = lin(vv, hidden)

    def fused_groups(self):
        return [[p.weight for p in (self.q_proj, self.k_proj, self.v_proj)], [self.q_conv, self.k_conv, self.v_conv],
                [self.a1_proj.weight, self.g1_proj.weight]]

    def new_state(self, slots, capacity, device, dtype):
        return SlotTensors(slots, device, s=((self.h, self.dv, iops.padded_rows(self.d)), torch.float32),
                           tail=((2 * self.g * self.d + self.h * self.dv, self.taps - 1), dtype))

    def forward(self, h, meta, state, residual):
        T = h.shape[0]
        qkv = iops.linear_cat(h, [self.q_proj.weight, self.k_proj.weight, self.v_proj.weight])
        low = iops.linear_cat(h, [self.a1_proj.weight, self.g1_proj.weight])
        ra = self.a1_proj.weight.shape[0]
        a = iops.linear_f32(low[:, :ra], self.a2_proj.weight)
        gate = iops.linear(low[:, ra:], self.g2_proj.weight)
        q, k, v, g, beta = iops.delta_inputs(
            qkv, [self.q_conv, self.k_conv, self.v_conv], a, self.A_log, self.dt_bias,
            iops.linear_f32(h, self.b_proj.weight), self.h, self.g, self.d, self.dv, meta,
            state.tail if state is not None else None)
        o = iops.delta_scan(q, k, v, g, beta, meta, state.s if state is not None else None)
        y = iops.head_norm_gate(o, self.norm, gate, "sigmoid", self.eps, h.dtype)
        return iops.linear_add_(residual, y, self.o_proj.weight)
