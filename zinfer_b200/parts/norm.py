"""RMSNorm: y = x * w / sqrt(mean(x^2) + eps), computed in 32-bit
(src/kernel/core/cpu.zig:38-48,73-110).  The weight multiplies directly (no 1 + w)
and eps is added to the mean inside the root.  ``one_plus``: the stored weight lies around zero and the
multiplier is 1 + w (formed once, in 32-bit, when the weights are bound).

LayerNorm: y = (x - mean(x)) * w / sqrt(mean((x - mean(x))^2) + eps), with a weight and no bias.

Either may be what a block norms its sublayers' outputs with (``ops.PostNormed``): the kernel of the norm that
comes next then norms the pending update, adds it and norms the sum in one pass."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from .base import Norm, TensorSpec


class RMSNorm(Norm):
    kind = "rms"

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.tensor = str(params.get("tensor", "weight"))   # the weight's name relative to the part
        self.one_plus = bool(params.get("one_plus", False))
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self):
        return {self.tensor: TensorSpec((self.size,), init="around_zero" if self.one_plus else "norm")}

    def bind(self, tensors):
        # norm vectors are widened to 32-bit once, as the reference does
        # (src/model/runtime/optimized_decoder/support.zig:6-19)
        self.weight = tensors[self.tensor].to(torch.float32).contiguous()
        if self.one_plus:
            self.weight = (1.0 + self.weight).contiguous()

    def forward(self, h, delta, rows=None, bias=None):
        """Adds ``delta`` (and ``bias``) into the residual ``h`` in place, then norms (the picked rows)."""
        if isinstance(delta, ops.PostNormed):
            if bias is not None:
                raise ValueError("a normed update and a per-pass vector do not go together")
            return ops.sandwich_norm(h, delta, self.weight, self.eps, self.kind, self.ctx.dtype, rows=rows)
        return ops.add_rmsnorm(h, delta, self.weight, self.eps, self.ctx.dtype, rows=rows, bias=bias)


class LayerNorm(Norm):
    kind = "layer"

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.tensor = str(params.get("tensor", "weight"))
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self):
        return {self.tensor: TensorSpec((self.size,), init="norm")}

    def bind(self, tensors):
        self.weight = tensors[self.tensor].to(torch.float32).contiguous()

    def forward(self, h, delta, rows=None, bias=None):
        if bias is not None:
            raise ValueError("this norm takes no per-pass vector")
        return ops.sandwich_norm(h, delta, self.weight, self.eps, self.kind, self.ctx.dtype, rows=rows)
