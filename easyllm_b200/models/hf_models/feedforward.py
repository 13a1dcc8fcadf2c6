"""Feed-forward layers of the parallel block: dense GLU, and sparse mixtures of two- and three-matrix experts.

Both are called as ``ff(h, residual)`` and accumulate their output into the fp32 stream ``residual``.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import infer as iops


class DenseGLU(nn.Module):
    """``down(act(gate h + b) * (up h + b)) + b``, with or without the biases.  The last bias is not added here:
    ``out_bias`` goes into the stream in the pass that reads it for the norm."""

    def __init__(self, hidden, ff, act, dtype, bias=True):
        super().__init__()
        self.gate_proj = nn.Linear(hidden, ff, bias=bias, dtype=dtype)
        self.up_proj = nn.Linear(hidden, ff, bias=bias, dtype=dtype)
        self.down_proj = nn.Linear(ff, hidden, bias=bias, dtype=dtype)
        self.act, self.bias = act, bias

    @property
    def out_bias(self):
        return self.down_proj.bias

    def fused_groups(self):
        return [[self.gate_proj.weight, self.up_proj.weight]] + \
            ([[self.gate_proj.bias, self.up_proj.bias]] if self.bias else [])

    def forward(self, h, residual):
        gu = iops.linear_cat(h, [self.gate_proj.weight, self.up_proj.weight],
                             [self.gate_proj.bias, self.up_proj.bias] if self.bias else None)
        return iops.linear_add_(residual, iops.glu(gu, self.act), self.down_proj.weight)


class _UpDown(nn.Module):
    def __init__(self, hidden, ff, dtype):
        super().__init__()
        self.up_proj = nn.Linear(hidden, ff, bias=False, dtype=dtype)
        self.down_proj = nn.Linear(ff, hidden, bias=False, dtype=dtype)


class SparseMoE(nn.Module):
    """``top`` of ``experts`` two-matrix experts ``down relu(up x)^2`` per token, chosen by sigmoid router scores; the
    score (not renormalised) multiplies the expert's input.  Since it is positive and the activation is homogeneous of
    degree two, it is applied to the hidden units before the square, in fp32.  A shared expert is scaled by
    ``sigmoid(sg h)``, folded into its hidden units in the same way."""

    out_bias = None

    def __init__(self, hidden, m, dtype):
        super().__init__()
        E, ff = m["router"]["experts"], m["expert"]["ff"]
        self.top = m["router"]["top"]
        if not 1 <= self.top <= E:
            raise ValueError(f"router: top {self.top} of {E} experts")
        self.experts_up = nn.Parameter(torch.empty(E, ff, hidden, dtype=dtype).normal_(0, 0.02))
        self.experts_down = nn.Parameter(torch.empty(E, hidden, ff, dtype=dtype).normal_(0, 0.02))
        self.router = nn.Linear(hidden, E, bias=False, dtype=dtype)
        self.shared = self.shared_gate = None
        if m.get("shared"):
            self.shared = _UpDown(hidden, m["shared"]["ff"], dtype)
            self.shared_gate = nn.Linear(hidden, 1, bias=False, dtype=dtype)

    def fused_groups(self):
        return [[self.router.weight, self.shared_gate.weight]] if self.shared is not None else []

    def forward(self, h, residual):
        E = self.router.weight.shape[0]
        z = iops.linear_cat_f32(h, [self.router.weight] + ([self.shared_gate.weight] if self.shared is not None else []))
        if self.shared is not None:
            a = iops.relu2_scaled(iops.linear(h, self.shared.up_proj.weight), z[:, E])
            iops.linear_add_(residual, a, self.shared.down_proj.weight)
        return iops.moe_relu2_add_(residual, h, z[:, :E], self.top, self.experts_up, self.experts_down)


class SparseGLU(nn.Module):
    """``top`` of ``experts`` gated experts ``down(silu(gate h) * up h)`` per token, weighted by the softmax over the chosen
    router logits (a bias per expert is part of the logits), plus a shared expert for every token.  Gate and up rows of an
    expert alternate in blocks of ``block`` rows, so that one tile of the grouped product holds both halves of its hidden
    units and the activation runs in the product's epilogue."""

    out_bias = None

    def __init__(self, hidden, m, dtype):
        super().__init__()
        E, ff = m["router"]["experts"], m["expert"]["ff"]
        self.top, self.block = m["router"]["top"], self.block_of(ff)
        if not 1 <= self.top <= E:
            raise ValueError(f"router: top {self.top} of {E} experts")
        self.experts_gate_up = nn.Parameter(torch.empty(E, 2 * ff, hidden, dtype=dtype).normal_(0, 0.02))
        self.experts_down = nn.Parameter(torch.empty(E, hidden, ff, dtype=dtype).normal_(0, 0.02))
        self.router = nn.Linear(hidden, E, bias=False, dtype=dtype)
        self.router_bias = nn.Parameter(torch.zeros(E))
        self.shared = DenseGLU(hidden, m["shared"]["ff"], "silu", dtype, bias=False) if m.get("shared") else None

    @staticmethod
    def block_of(ff):
        return 32 if ff % 32 == 0 else ff

    @staticmethod
    def blocked(gate, up):
        """gate, up ``[F, W]`` → ``[2 F, W]`` in alternating blocks of rows (``split`` undoes it)."""
        F, W = gate.shape
        b = SparseGLU.block_of(F)
        return torch.stack((gate.reshape(F // b, b, W), up.reshape(F // b, b, W)), 1).reshape(2 * F, W)

    @staticmethod
    def split(gate_up):
        F, W = gate_up.shape[0] // 2, gate_up.shape[1]
        v = gate_up.reshape(F // SparseGLU.block_of(F), 2, -1, W)
        return v[:, 0].reshape(F, W), v[:, 1].reshape(F, W)

    def forward(self, h, residual):
        z = iops.linear_f32(h, self.router.weight)
        if self.shared is not None:
            self.shared(h, residual)
        return iops.moe_glu_add_(residual, h, z, self.router_bias, self.top, self.experts_gate_up, self.block,
                                 self.experts_down)
