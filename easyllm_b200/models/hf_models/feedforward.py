"""Feed-forward layers of the parallel block: dense GLU with biases, and a sparse mixture of experts.

Both are called as ``ff(h, residual)`` and accumulate their output into the fp32 stream ``residual``.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import infer as iops


class DenseGLU(nn.Module):
    """``down(act(gate h + b) * (up h + b)) + b``.  The last bias is not added here: ``out_bias`` goes into the stream
    in the pass that reads it for the norm."""

    def __init__(self, hidden, ff, act, dtype):
        super().__init__()
        self.gate_proj = nn.Linear(hidden, ff, bias=True, dtype=dtype)
        self.up_proj = nn.Linear(hidden, ff, bias=True, dtype=dtype)
        self.down_proj = nn.Linear(ff, hidden, bias=True, dtype=dtype)
        self.act = act

    @property
    def out_bias(self):
        return self.down_proj.bias

    def fused_groups(self):
        return [[self.gate_proj.weight, self.up_proj.weight], [self.gate_proj.bias, self.up_proj.bias]]

    def forward(self, h, residual):
        gu = iops.linear_cat(h, [self.gate_proj.weight, self.up_proj.weight], [self.gate_proj.bias, self.up_proj.bias])
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
