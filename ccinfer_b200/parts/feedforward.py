"""Dense gated feed-forward: m = (silu(x Wg^T) * (x Wu^T)) Wd^T, no bias
(7QiC/ccInfer: src/model/qwen3/qwen3_model.cpp:325-384, src/kernel/mlp/silu_mul.cu:24-28).

The reference runs gate and up as two matrix products; here they are one
merged matrix [2F, D] and one product.  Where F is a multiple of 64 the rows
are laid out in blocks (64 of gate, the 64 of up for the same channels) so that
a tile of the tensor-core product owns matching channels and the activation
can be its epilogue; otherwise gate rows first, then up rows.
"""
from __future__ import annotations

import torch

from .. import kernels
from .base import FeedForward, TensorSpec


class SwiGLU(FeedForward):
    takes_unscaled = True
    activation = None   # silu(gate) * up; a subclass names another one (a kernels.GluAct, see Runtime.gated_up)

    def __init__(self, hidden: int, intermediate: int, names: dict):
        """``names``: tensor names under the keys gate, up, down."""
        self.hidden, self.inter, self.names = int(hidden), int(intermediate), dict(names)
        self.w_gate_up = self.w_down = None
        self.rt = None

    def tensor_specs(self):
        n = self.names
        return [TensorSpec(n["gate"], (self.inter, self.hidden)), TensorSpec(n["up"], (self.inter, self.hidden)),
                TensorSpec(n["down"], (self.hidden, self.inter))]

    def bind(self, rt, fetch):
        self.rt = rt
        gate, up = fetch(self.names["gate"]), fetch(self.names["up"])
        self.block = kernels.SWIGLU_BLOCK if self.inter % kernels.SWIGLU_BLOCK == 0 else 0
        if self.block:
            self.w_gate_up = kernels.interleave_gate_up(gate, up, self.block)
        else:
            self.w_gate_up = torch.cat([gate, up], dim=0).contiguous()
        self.w_down = fetch(self.names["down"])

    def forward(self, x, step):
        rt = self.rt
        T = x.shape[0]
        act = rt.scratch.get("ffn_act", (rt.max_tokens, self.inter), rt.dtype)[:T]
        rt.gated_up(act, x, self.w_gate_up, self.block, activation=self.activation)
        out = rt.scratch.get("ffn_out", (rt.max_tokens, self.hidden), rt.dtype)[:T]
        return rt.linear(out, act, self.w_down, sink=step.take_sink())


class ClampedGLU(SwiGLU):
    """The same two products with clamped inputs and a sigmoid gate of its own slope:

        g = min(x Wg^T, limit), u = clamp(x Wu^T, -limit, limit);  m = (g * sigmoid(alpha g) * (u + shift)) Wd^T
    """

    def __init__(self, hidden: int, intermediate: int, names: dict, limit: float, alpha: float = 1.702,
                 shift: float = 1.0):
        super().__init__(hidden, intermediate, names)
        self.activation = kernels.GluAct.clamped(limit, alpha, shift)


class GeluGLU(SwiGLU):
    """The same two products with gelu in its tanh form as the gate: m = (gelu(x Wg^T) * (x Wu^T)) Wd^T."""

    activation = kernels.GluAct.gelu_tanh()


class SquaredReLU(FeedForward):
    """A feed-forward without a gate: m = (relu(x Wu^T))^2 Wd^T, no biases."""

    def __init__(self, hidden: int, intermediate: int, names: dict):
        """``names``: tensor names under the keys up, down."""
        self.hidden, self.inter, self.names = int(hidden), int(intermediate), dict(names)
        self.w_up = self.w_down = None
        self.rt = None

    def tensor_specs(self):
        n = self.names
        return [TensorSpec(n["up"], (self.inter, self.hidden)), TensorSpec(n["down"], (self.hidden, self.inter))]

    def bind(self, rt, fetch):
        self.rt = rt
        self.w_up, self.w_down = fetch(self.names["up"]), fetch(self.names["down"])

    def forward(self, x, step):
        rt = self.rt
        x = rt.rows(x)
        T = x.shape[0]
        act = rt.scratch.get("ffn_act", (rt.max_tokens, self.inter), rt.dtype)[:T]
        rt.linear_relu2(act, x, self.w_up)
        out = rt.scratch.get("ffn_out", (rt.max_tokens, self.hidden), rt.dtype)[:T]
        return rt.linear(out, act, self.w_down)
