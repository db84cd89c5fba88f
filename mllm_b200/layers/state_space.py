"""State-space duality (Mamba-2): a linear recurrence whose state decays by a factor per head and token.

    [z | x | B | C | dt] = W x;   x, B, C = silu(conv1d(.) + bias);   dt = softplus(dt + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x           S fp32, kept per request
    out = rmsnorm(y * silu(z)) * weight                                the norm over equal parts of the row

The state of a request lives in the row of the recurrent-state pool that belongs to it, beside those of the gated
delta net, so portions of prompts and decode steps resume from it."""

from __future__ import annotations

from typing import Sequence

import torch
from torch import nn

from .. import ops
from .gdn import gdn_batch


class StateSpace(nn.Module):
    """The core between the projections: reads the projected rows ``[z | x | B | C | dt]`` and writes the gated, normed heads."""

    folds_scale = True        # a scale on the output goes into the norm weight
    biased: Sequence[str] = ()

    def __init__(self, heads: int, vdim: int, state: int, groups: int, conv: int, norm_groups: int, eps: float, state_index: int,
                 params_dtype: torch.dtype) -> None:
        super().__init__()
        if heads % groups or (heads * vdim) % norm_groups:
            raise ValueError(f"state space: {heads} heads of {vdim} in {groups} groups, norm over {norm_groups} parts")
        self.heads, self.vdim, self.state, self.groups, self.conv_kernel = heads, vdim, state, groups, conv
        self.norm_groups, self.eps, self.state_index = norm_groups, float(eps), state_index
        self.inner = heads * vdim
        self.conv_dim = self.inner + 2 * groups * state
        self.shards = {"in": self.inner + self.conv_dim + heads}

        def p(*shape, dtype=torch.float32):
            return nn.Parameter(torch.zeros(*shape, dtype=dtype), requires_grad=False)

        self.conv1d, self.norm = nn.Module(), nn.Module()
        self.conv1d.weight, self.conv1d.bias = p(self.conv_dim, conv, dtype=params_dtype), p(self.conv_dim, dtype=params_dtype)
        self.A_log, self.dt_bias, self.D = p(heads), p(heads), p(heads)
        self.norm.weight = nn.Parameter(torch.ones(self.inner, dtype=torch.float32), requires_grad=False)

    @property
    def state_shape(self):
        """(heads, key features, value features, convolution channels, taps) of a request's state."""
        return self.heads, self.state, self.vdim, self.conv_dim, self.conv_kernel

    @property
    def out_width(self) -> int:
        return self.inner

    def expand_columns(self, w: torch.Tensor) -> torch.Tensor:
        return w

    def forward(self, row: torch.Tensor, fb, out: torch.Tensor) -> None:
        state, conv = fb.extra["gdn_pool"].layer(self.state_index)
        m = gdn_batch(fb)
        I, GN = self.inner, self.groups * self.state
        xbc = ops.causal_conv1d_silu(row[:, I: I + self.conv_dim], self.conv1d.weight, conv, m.slots, m.lens, m.has_state, m.q_start, m.max_len,
                                     bias=self.conv1d.bias)
        x = xbc[:, :I].unflatten(1, (self.heads, self.vdim))
        B = xbc[:, I: I + GN].unflatten(1, (self.groups, self.state))
        C = xbc[:, I + GN:].unflatten(1, (self.groups, self.state))
        dt = row[:, I + self.conv_dim: I + self.conv_dim + self.heads]
        y = ops.state_space(x, B, C, dt, self.dt_bias, self.A_log, self.D, state, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        ops.gated_rmsnorm(y.view(-1, I), row[:, :I], self.norm.weight, self.norm_groups, self.eps, out)
