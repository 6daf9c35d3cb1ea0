"""Mamba-2: a matrix-valued state per head with one decay per head and a step size per token (state-space duality,
"Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality", Dao and
Gu, 2024).

One projection W_in h = [z | x | B | C | dt].  x (``heads`` heads of ``vdim``), B and C (``groups`` groups of ``state``
values; head h uses group h // (heads / groups)) pass a causal convolution per channel with a bias, then silu.  With
dt <- softplus(dt + dt_bias), per head:

    S <- exp(-exp(A_log_h) dt) S + dt B x^T ;  y = S^T C + D_h x          S [state, vdim], 32-bit

y * silu(z), over the whole width, is divided by its root mean square in ``norm_groups`` equal parts, multiplied by a weight
per channel and projected by W_o.  A request keeps S of every head and the convolution's last taps - 1 inputs.

The projection's rows are read back as 32-bit sums (its K splits are added by whoever reads them), so convolution, step sizes
and gate meet unrounded values; steps, decays, the recurrence and the norm are 32-bit.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, StateNeed, TensorSpec


class Mamba2(Mixer):
    graph_safe = True   # kernels on the step's device arrays only

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["num_heads"])
        self.vdim = int(params["vdim"])
        self.dim = int(params["state"])
        self.groups = int(params["groups"])
        self.norm_groups = int(params["norm_groups"])
        self.taps = int(params["conv_taps"])
        self.eps = float(params["norm_eps"])
        if min(self.heads, self.vdim, self.dim, self.groups, self.norm_groups) <= 0:
            raise ValueError("heads, vdim, state, groups and norm_groups must be positive")
        if self.heads % self.groups:
            raise ValueError(f"{self.heads} heads do not divide into {self.groups} groups")
        self.inner = self.heads * self.vdim
        if self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels do not divide into {self.norm_groups} norm groups")
        if not 1 <= self.taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"the convolution has 1 to {ops.CONV_MAX_TAPS} taps, got {self.taps}")
        self.bc = self.groups * self.dim
        self.channels = self.inner + 2 * self.bc         # the convolved channels: x, B, C side by side
        self.s_size = self.heads * self.dim * self.vdim

    def tensor_specs(self):
        return {
            "in": TensorSpec((2 * self.inner + 2 * self.bc + self.heads, self.hidden)),
            "conv": TensorSpec((self.channels, self.taps)), "conv.b": TensorSpec((self.channels,), init="around_zero"),
            "dt_bias": TensorSpec((self.heads,), init="zeros"), "A_log": TensorSpec((self.heads,), init="zeros"),
            "D": TensorSpec((self.heads,), init="norm"), "norm": TensorSpec((self.inner,), init="norm"),
            "o": TensorSpec((self.hidden, self.inner)),
        }

    def bind(self, tensors):
        f32 = lambda name: tensors[name].to(torch.float32).contiguous()
        self.w_in = tensors["in"].contiguous()
        self.conv, self.conv_bias = f32("conv").t().contiguous(), f32("conv.b")     # [taps, channels]
        self.dt_bias, self.a_log, self.skip, self.norm = f32("dt_bias"), f32("A_log"), f32("D"), f32("norm")
        self.w_o = tensors["o"].contiguous()

    def cache_need(self):
        # one slot per request: S of every head, then the convolution's last taps-1 inputs [taps-1, channels]
        return StateNeed((self.s_size + (self.taps - 1) * self.channels,), torch.float32)

    def forward(self, x, step, cache):
        C, H, inner, bc = self.channels, self.heads, self.inner, self.bc
        state = cache.state
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32, allow_partials=True)
        cols = lambda at, n: ops.Columns(proj, at, n)
        tail = state[:, self.s_size:].view(state.shape[0], self.taps - 1, C)
        xbc = torch.empty((x.shape[0], C), dtype=torch.float32, device=x.device)
        decay, dt = ops.conv_heads(cols(inner, C), self.conv, tail, step, [ops.ConvSegment(C, C, xbc)], out_bias=self.conv_bias,
                                   activation="silu", decay=("ssd", cols(inner + C, H), None, self.a_log, self.dt_bias))
        xs, B, Cs = xbc[:, :inner], xbc[:, inner:inner + bc], xbc[:, inner + bc:]
        y = ops.head_decay_recurrence(Cs, B, xs, decay, dt, state[:, :self.s_size], H, self.groups, self.dim, self.vdim, step, delta=False,
                                      fast=self.ctx.dtype == torch.bfloat16)
        y = ops.gated_part_norm(y, cols(0, inner), self.norm, self.eps, self.norm_groups, self.ctx.dtype, skip=self.skip, x=xs,
                                vdim=self.vdim)
        return ops.linear(y, self.w_o, out_dtype=self.ctx.dtype, allow_partials=True)
