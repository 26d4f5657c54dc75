"""A recurrence whose gates read the present token only (minGRU), element by element:

    z = sigmoid(W_z h + b_z),   u = W_x h + b_x,   c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
    S <- (1 - z) S + z c,       y = W_o (S * silu(W_g h))

S (float32, one number a channel) is the request's state.  The projections take h in the run's dtype and hand their
results over in float32; gates, candidate, state and its read-out gate are float32.
"""
from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from .attention import materialized_rows
from .base import Mixer, StateSpec, WeightBuffers, register_part


@register_part("mixer", "min_gru")
class MinGRU(Mixer):
    """params: hidden_size, inner_size, names (tensor names of z, x, g, o, z_bias, x_bias)."""

    _NAMES = {"z": "z", "x": "x", "g": "g", "o": "o", "z_bias": "z.b", "x_bias": "x.b"}

    def __init__(self, spec):
        super().__init__(spec)
        self.hidden = int(spec.params["hidden_size"])
        self.inner = int(spec.params["inner_size"])
        if min(self.hidden, self.inner) <= 0:
            raise ValueError("min_gru: sizes must be positive")
        self.names = dict(self._NAMES)
        self.names.update(spec.params.get("names") or {})
        self.w_stack = self.w_o = self.bias = None

    def state_spec(self):
        return StateSpec((self.inner,), torch.float32)

    def param_specs(self):
        n, W, C = self.names, self.inner, self.hidden
        return {n["z"]: TensorSpec((W, C)), n["x"]: TensorSpec((W, C)), n["g"]: TensorSpec((W, C)), n["o"]: TensorSpec((C, W)),
                n["z_bias"]: TensorSpec((W,), init="zeros"), n["x_bias"]: TensorSpec((W,), init="zeros")}

    def load(self, tensors, dtype, device):
        n, W, C = self.names, self.inner, self.hidden
        self.buffers = buf = WeightBuffers(device, {"stack": ((3 * W, C), dtype), "o": ((C, W), dtype),    # z, x, g: one product
                                                    "bias": ((2 * W,), torch.float32)})
        for i, s in enumerate(("z", "x", "g")):
            buf["stack"][i * W:(i + 1) * W].copy_(tensors[n[s]])
        buf["bias"][:W].copy_(tensors[n["z_bias"]])
        buf["bias"][W:].copy_(tensors[n["x_bias"]])
        buf["o"].copy_(tensors[n["o"]])
        self.w_stack, self.w_o, self.bias = buf["stack"], buf["o"], buf["bias"]

    def forward(self, h, ctx, cache):
        k = ctx.kernels
        rows = k.linear(materialized_rows(k, h), self.w_stack, out_dtype=torch.float32, allow_partial=True)     # [T, 3W]: z x g
        y = k.gated_scan(rows, self.bias, cache.state, self.inner, ctx, out_dtype=ctx.dtype)
        return k.linear(y, self.w_o, allow_partial=True)
