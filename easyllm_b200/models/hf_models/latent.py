"""Latent attention: keys and values are products of one small latent per token, which is all that is cached.

A token's latent ``c`` (RMS-normed) gives every head an unrotated key part ``W_uk c`` and a value ``W_uv c``; a rotated key
part, shared by the heads, comes beside it.  Two ways through the same numbers:

* prompts that start in this step: keys and values are formed once (one product) and the tcgen05 attention kernel reads
  the two key parts from where they are;
* everything else works on the cached rows ``[c | rotated part]``: the query's unrotated part is taken through
  ``W_uk`` (per head ``W_ukᵀ q``), so scores and weighted sums run in the latent space, with one key row for all heads,
  and the sum goes through ``W_uv`` at the end.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import infer as iops
from ..layers import YarnRotaryTables
from .state import LatentRows


class LatentAttention(nn.Module):
    """``m``: heads, dim / rot_dim (unrotated / rotated part of a query and key), vdim, kv_rank, scale, rot (dims, base,
    scaling or None) and mask (size of a sliding window, or None).  A gate per head multiplies the output."""

    def __init__(self, hidden, m, eps, dtype):
        super().__init__()
        self.h, self.d, self.r, self.dv, self.rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        self.scale, self.eps = float(m["scale"]), eps
        self.window = (m.get("mask") or {}).get("size")
        self.rotary = YarnRotaryTables(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))

        def lin(i, o):
            return nn.Linear(i, o, bias=False, dtype=dtype)
        self.q_proj, self.dkv_proj = lin(hidden, self.h * (self.d + self.r)), lin(hidden, self.rank + self.r)
        self.g_proj = lin(hidden, self.h)
        self.dkv_norm = nn.Parameter(torch.ones(self.rank))
        self.uk_proj, self.uv_proj = lin(self.rank, self.h * self.d), lin(self.rank, self.h * self.dv)
        self.o_proj = lin(self.h * self.dv, hidden)
        self._ukt, self._ukt_of = None, None

    def fused_groups(self):
        return [[p.weight for p in (self.q_proj, self.dkv_proj, self.g_proj)], [self.uk_proj.weight, self.uv_proj.weight]]

    def new_state(self, slots, capacity, device, dtype):
        return LatentRows(slots, capacity, self.rank, self.r, device, dtype)

    def uk_transposed(self):
        """``W_ukᵀ`` per head ``[H, rank, dim]``, made again when the weight has changed or moved."""
        w = self.uk_proj.weight
        key = (w.data_ptr(), w._version, w.dtype, w.device)
        if self._ukt_of != key:
            self._ukt = w.detach().view(self.h, self.d, self.rank).transpose(1, 2).contiguous()
            self._ukt_of = key
        return self._ukt

    def forward(self, h, meta, cache, residual):
        T, at = h.shape[0], self.h * (self.d + self.r)
        z = iops.linear_cat(h, [self.q_proj.weight, self.dkv_proj.weight, self.g_proj.weight])
        gate = z[:, at + self.rank + self.r:]
        cos, sin = self.rotary.get(int(meta["max_position"]), h.device)
        c = cache.c if cache is not None else None
        sizes = (self.h, self.d, self.r, self.rank)
        fresh = cache is None or (meta["fresh"] and not meta["one_token"])
        if fresh and iops.latent_prefill_ok(z, self.d, self.r, self.rank, self.dv):
            iops.latent_inputs(z, *sizes, self.dkv_norm, self.eps, cos, sin, meta, c)
            kv = iops.linear_cat(z[:, at:at + self.rank], [self.uk_proj.weight, self.uv_proj.weight])
            o = iops.attention_latent_prefill(z, kv, *sizes, self.dv, iops.row_start(meta, T, h.device), self.scale,
                                              self.window, gate)
        else:
            q = torch.empty(T, self.h, self.rank + self.r, dtype=z.dtype, device=z.device)
            iops.latent_inputs(z, *sizes, self.dkv_norm, self.eps, cos, sin, meta, c, q[..., self.rank:])
            iops.head_products(z[:, :at].unflatten(1, (self.h, -1))[..., :self.d], self.uk_transposed(), q[..., :self.rank])
            if c is not None:
                rows, base, n, bound = c.view(-1, c.shape[-1]), meta["kv_base"], meta["kv_len"], \
                    meta.get("kv_bound", meta["max_position"])
            else:
                base = iops.row_start(meta, T, h.device)
                n = torch.arange(1, T + 1, device=h.device, dtype=torch.int32) - base
                rows, bound = z[:, at:], meta["max_seqlen"]
            o = iops.attention_latent(q, rows, self.rank, base, n, bound, self.scale, self.window, gate)
            o = iops.head_products(o, self.uv_proj.weight.detach().view(self.h, self.dv, self.rank))
        return iops.linear_add_(residual, o.reshape(T, self.h * self.dv), self.o_proj.weight)
