"""Lightning attention: linear attention whose state decays by a fixed factor per head.

    q = silu(W_q x),  k = silu(W_k x),  v = silu(W_v x)          heads x dim, heads x vdim
    S <- decay_h S + k v^T,   o = S^T q                          S fp32, kept per request
    y = rmsnorm(o over all heads) * weight * sigmoid(W_g x)

The state of a request lives in the row of the recurrent-state pool that belongs to it, beside those of the gated
delta net, so portions of prompts and decode steps resume from it."""

from __future__ import annotations

from typing import Sequence

import torch
from torch import nn

from .. import ops
from .gdn import gdn_batch


class LightningAttention(nn.Module):
    """The core between the projections: reads the projected rows ``[q | k | v | g]`` and writes the gated, normed heads."""

    folds_scale = True        # a scale on the output goes into the norm weight
    biased: Sequence[str] = ()

    def __init__(self, heads: int, dim: int, vdim: int, decay, eps: float, state_index: int) -> None:
        super().__init__()
        rates = [float(decay)] * heads if isinstance(decay, (int, float)) else [float(d) for d in decay]
        if len(rates) != heads:
            raise ValueError(f"lightning attention: {len(rates)} decays for {heads} heads")
        self.heads, self.dim, self.vdim, self.eps, self.state_index = heads, dim, vdim, float(eps), state_index
        self.shards = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim}
        self.register_buffer("decay", torch.tensor(rates, dtype=torch.float32), persistent=False)
        self.norm = nn.Module()
        self.norm.weight = nn.Parameter(torch.ones(heads * vdim, dtype=torch.float32), requires_grad=False)

    @property
    def state_shape(self):
        """(heads, key features, value features, convolution channels, taps) of a request's state."""
        return self.heads, self.dim, self.vdim, 0, 1

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def expand_columns(self, w: torch.Tensor) -> torch.Tensor:
        return w

    def forward(self, row: torch.Tensor, fb, out: torch.Tensor) -> None:
        state, _ = fb.extra["gdn_pool"].layer(self.state_index)
        m = gdn_batch(fb)
        K, V = self.heads * self.dim, self.heads * self.vdim
        q = row[:, :K].unflatten(1, (self.heads, self.dim))
        k = row[:, K:2 * K].unflatten(1, (self.heads, self.dim))
        v = row[:, 2 * K:2 * K + V].unflatten(1, (self.heads, self.vdim))
        o = ops.lightning_attention(q, k, v, self.decay, state, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        ops.rmsnorm_sigmoid_gate(o.view(-1, V), row[:, 2 * K + V:2 * K + 2 * V], self.norm.weight, self.eps, out)
