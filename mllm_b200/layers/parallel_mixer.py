"""Token mixers side by side on the same input, ``sum_i scale_i * W_o,i branch_i(W_in,i x)``, as one projection in, the
branches, and one projection out: the branches write neighbouring columns of one matrix, so their weighted sum is the
inner dimension of the output product.  A single branch is the ordinary mixer.  Where each branch's result has a norm of its
own (:class:`NormedParallelMixer`), the output projections stay apart and the step behind the layer norms and averages them.

A branch (:class:`.RowNormAttention`, :class:`.LightningAttention`, :class:`.StateSpace`) lists the projections it reads (``shards``: name ->
rows, in order; ``biased``: which have a bias), the columns it writes (``out_width``) and how an output projection's
columns are laid out for it (``expand_columns``); ``forward(row, fb, out)`` does the work."""

from __future__ import annotations

from typing import Sequence

import torch
from torch import nn

from .. import ops


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class ParallelMixer(nn.Module):
    def __init__(self, hidden_size: int, branches: Sequence[nn.Module], scales: Sequence[float], params_dtype: torch.dtype) -> None:
        super().__init__()
        self.branches = nn.ModuleList(branches)
        self.scales = [float(s) for s in scales]
        self.row_at, self.out_at, rows, cols = [], [], 0, 0
        for b in branches:
            self.row_at.append(rows)
            self.out_at.append(cols)
            rows += sum(b.shards.values())
            # branches begin on 16-byte boundaries of the projected rows and of the concatenated outputs
            rows, cols = _up8(rows), _up8(cols + b.out_width)
        self.in_proj, self.out_proj = nn.Module(), nn.Module()
        self.in_proj.weight = nn.Parameter(torch.zeros(rows, hidden_size, dtype=params_dtype), requires_grad=False)
        self.in_proj.bias = nn.Parameter(torch.zeros(rows, dtype=params_dtype), requires_grad=False) \
            if any(b.biased for b in branches) else None
        self.out_proj.weight = nn.Parameter(torch.zeros(hidden_size, cols, dtype=params_dtype), requires_grad=False)
        self.gaps = cols != sum(b.out_width for b in branches)
        self.out_width = cols
        self.result_scale = 1.0        # set by fold_scales: what the sum of the branches is still to be multiplied with

    # ------------------------------------------------------------------ loading
    def _rows(self, branch: int, name: str) -> slice:
        at = self.row_at[branch]
        for n, rows in self.branches[branch].shards.items():
            if n == name:
                return slice(at, at + rows)
            at += rows
        raise KeyError(name)

    def load_in(self, branch: int, name: str, w: torch.Tensor) -> None:
        self.in_proj.weight.data[self._rows(branch, name)].copy_(w)

    def load_bias(self, branch: int, name: str, b: torch.Tensor) -> None:
        self.in_proj.bias.data[self._rows(branch, name)].copy_(b)

    def load_out(self, branch: int, w: torch.Tensor) -> None:
        b, at = self.branches[branch], self.out_at[branch]
        self.out_proj.weight.data[:, at: at + b.out_width].copy_(b.expand_columns(w))

    def fold_scales(self) -> None:
        """After loading: the branches' scales leave the run.  A branch that can take a factor into fp32 parameters of its own
        does; the scale of the others stays outside as ``result_scale``, so no 16-bit weight is rounded again (two such
        branches of different scale excepted)."""
        fixed = [s for b, s in zip(self.branches, self.scales) if not b.folds_scale and s != 0.0]
        base = fixed[0] if fixed else 1.0
        for i, (b, s) in enumerate(zip(self.branches, self.scales)):
            if b.folds_scale:
                b.norm.weight.data.mul_(s / base)
            elif s != base:
                self.out_proj.weight.data[:, self.out_at[i]: self.out_at[i] + b.out_width].mul_(s / base)
        self.result_scale = base

    # ------------------------------------------------------------------ forward
    def run_branches(self, x: torch.Tensor, fb) -> torch.Tensor:
        """The branches' outputs side by side."""
        rows = ops.linear(x, self.in_proj.weight, self.in_proj.bias)
        shape = (x.shape[0], self.out_width)
        mixed = (torch.zeros if self.gaps else torch.empty)(shape, dtype=x.dtype, device=x.device)
        for b, r, c in zip(self.branches, self.row_at, self.out_at):
            b(rows[:, r:], fb, mixed[:, c: c + b.out_width])
        return mixed

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        return ops.linear(self.run_branches(x, fb), self.out_proj.weight)


class NormedParallelMixer(ParallelMixer):
    """Two branches whose results ``W_o,i branch_i`` are RMS-normed one by one: the forward pass returns them with their norm
    weights, for a step that norms and adds them (:func:`..ops.depth_step`)."""

    def __init__(self, hidden_size: int, branches: Sequence[nn.Module], params_dtype: torch.dtype) -> None:
        super().__init__(hidden_size, branches, [1.0] * len(branches), params_dtype)
        del self.out_proj
        self.out_projs, self.out_norms = nn.ModuleList(), nn.ParameterList()
        for b in branches:
            m = nn.Module()
            m.weight = nn.Parameter(torch.zeros(hidden_size, b.out_width, dtype=params_dtype), requires_grad=False)
            self.out_projs.append(m)
            self.out_norms.append(nn.Parameter(torch.ones(hidden_size, dtype=torch.float32), requires_grad=False))

    def load_out(self, branch: int, w: torch.Tensor) -> None:
        dst, src = self.out_projs[branch].weight.data, self.branches[branch].expand_columns(w)
        if dst.shape != src.shape:
            raise ValueError(f"a tensor of shape {tuple(w.shape)} does not fit the branch's {tuple(dst.shape)}")
        dst.copy_(src)

    def forward(self, x: torch.Tensor, fb):
        mixed = self.run_branches(x, fb)
        return (*(ops.linear(mixed[:, c: c + b.out_width], m.weight) for b, c, m in zip(self.branches, self.out_at, self.out_projs)),
                *self.out_norms)
