"""Latent attention: the cache holds one row ``c`` of ``kv_rank`` features per token, shared by all heads; head ``h``'s
key and value of a token are ``W_uk[h] c`` and ``W_uv[h] c``.  Queries go through a latent of their own or are projected
directly.  Options: a rotated key part of ``rot_dim`` features, shared by all heads, which follows the latent in the cache row and meets a
rotated part of each query head (without it there are no positions); a sliding window; a sink per head, a logit that joins
the softmax denominator only; a gate on the output, one per head or one per feature.  A layer may read the latents of an earlier layer instead of writing its
own.

Two evaluations of the same sum (``csrc/latent.cu``):

* absorbed: ``q' = W_uk[h]^T q``, followed by the rotated query part, meets the cached rows directly and the weighted sum
  of latents passes through ``W_uv[h]`` once per query — decode, short extends, 32-bit runs and head sizes the attention
  kernels do not have;
* expanded: requests with many new tokens form K and V of their context with two matrix products and run the
  attention kernels of the other models on them.  Heads are zero-padded (in the weights) to 64 / 128 / 256 features; the
  shared key part reaches the heads through rows of the identity in the weights that form K, which copy it exactly.

A batch may need both: :func:`latent_plan` sorts the requests once per forward pass."""

from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Union

import torch
from torch import nn

from .. import ops
from .attention import rotation_frequencies

EXPAND_MIN_TOKENS = 32          # new tokens from which forming K and V of the context pays
EXPAND_MAX_CONTEXT = 1 << 16    # context tokens expanded at a time (bounds the K and V buffers)


@dataclass
class ExpandGroup:
    """Requests whose contexts are expanded together."""

    req: torch.Tensor          # [b] request-table rows
    seq_lens: torch.Tensor     # [b]
    prefix_lens: torch.Tensor  # [b]
    q_start: torch.Tensor      # [b] first query row
    ctx_start: torch.Tensor    # [b] first row of the request's expanded context
    first: Optional[torch.Tensor]   # [b] token that context begins with (None: 0); the lengths above count from it
    rows: torch.Tensor         # [b, longest context] the identity table: row of every context token
    batch: torch.Tensor        # [b] 0 .. b - 1, the rows of that table
    total: int
    max_ctx: int
    max_q: int


@dataclass
class LatentPlan:
    groups: List[ExpandGroup]
    rows: Optional[torch.Tensor]      # query rows of the absorbed part (None: all of them)
    row_req: Optional[torch.Tensor]   # [rows] request-table row (None: the absorbed part is empty)
    row_pos: Optional[torch.Tensor]   # [rows] position
    max_ctx: int                      # longest context of the absorbed part


def latent_plan(fb, expand: bool, min_tokens: Optional[int] = None, window: Optional[int] = None) -> LatentPlan:
    """Which requests of the batch run expanded and which absorbed; cached in ``fb.extra``.  With a ``window`` a request is
    expanded from the first token that its new tokens see."""
    key = ("latent_plan", expand, window)
    got = fb.extra.get(key)
    if got is not None:
        return got
    if fb.forward_mode.is_decode():
        plan = LatentPlan([], None, fb.req_pool_indices.to(torch.int32), fb.positions.to(torch.int64), int(fb.max_seq_len))
        fb.extra[key] = plan
        return plan
    least = EXPAND_MIN_TOKENS if min_tokens is None else min_tokens
    dev = fb.input_ids.device
    ext, pre = list(fb.extend_seq_lens_cpu), list(fb.extend_prefix_lens_cpu)
    skip = [max(0, p - window + 1) if window else 0 for p in pre]      # tokens in front of the expanded context
    starts, total = [], 0
    for n in ext:
        starts.append(total)
        total += n
    far = [i for i, n in enumerate(ext) if expand and n >= least]
    near = [i for i in range(len(ext)) if i not in set(far)]

    def dev_i32(v):
        return torch.tensor(v, dtype=torch.int32).to(dev, non_blocking=True)

    groups: List[ExpandGroup] = []
    run: List[int] = []

    def close():
        if not run:
            return
        sel = torch.tensor(run, dtype=torch.int64).to(dev, non_blocking=True)
        ctx = [ext[i] + pre[i] - skip[i] for i in run]
        at, acc = [], 0
        for n in ctx:
            at.append(acc)
            acc += n
        cs = dev_i32(at)
        table = cs.unsqueeze(1) + torch.arange(max(ctx), dtype=torch.int32, device=dev).unsqueeze(0)
        groups.append(ExpandGroup(
            req=fb.req_pool_indices.index_select(0, sel).to(torch.int32), seq_lens=dev_i32(ctx),
            prefix_lens=dev_i32([pre[i] - skip[i] for i in run]), q_start=dev_i32([starts[i] for i in run]), ctx_start=cs,
            first=dev_i32([skip[i] for i in run]) if window else None,
            rows=table.clamp_(max=acc - 1), batch=torch.arange(len(run), dtype=torch.int32, device=dev), total=acc,
            max_ctx=max(ctx), max_q=max(ext[i] for i in run)))
        run.clear()

    size = 0
    for i in far:
        ctx = ext[i] + pre[i] - skip[i]
        if run and size + ctx > EXPAND_MAX_CONTEXT:
            close()
            size = 0
        run.append(i)
        size += ctx
    close()
    rows = row_req = row_pos = None
    max_ctx = max((ext[i] + pre[i] for i in near), default=0)
    if near:
        if not far:
            row_req = torch.repeat_interleave(fb.req_pool_indices.to(torch.int32), fb.extend_seq_lens.long(), output_size=total)
            row_pos = fb.positions.to(torch.int64)
        else:
            owner = [i for i in near for _ in range(ext[i])]
            picked = [r for i in near for r in range(starts[i], starts[i] + ext[i])]
            rows = torch.tensor(picked, dtype=torch.int64).to(dev, non_blocking=True)
            row_req = fb.req_pool_indices.to(torch.int32).index_select(0, torch.tensor(owner, dtype=torch.int64).to(dev, non_blocking=True))
            row_pos = fb.positions.to(torch.int64).index_select(0, rows)
    plan = LatentPlan(groups, rows, row_req, row_pos, max_ctx)
    fb.extra[key] = plan
    return plan


def _pad_heads(w: torch.Tensor, heads: int, width: int) -> torch.Tensor:
    """Rows of every head padded with zero rows to ``width``: [heads * d, k] -> [heads * width, k]."""
    d = w.shape[0] // heads
    if d == width:
        return w
    out = torch.zeros(heads, width, w.shape[1], dtype=w.dtype, device=w.device)
    out[:, :d] = w.view(heads, d, -1)
    return out.view(heads * width, -1)


class LatentAttention(nn.Module):
    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, q_rank: Optional[int], kv_rank: int, scale: float, eps: float,
                 latent_index: int, writes_latent: bool, params_dtype: torch.dtype, rot_dim: int = 0, rot_base: float = 1e4,
                 rot_scaling: Optional[dict] = None, sinks: bool = True, gated: Union[bool, str] = False, halves: bool = False,
                 window: Optional[int] = None) -> None:
        """``latent_index``: the buffer of the latent pool this layer reads; ``writes_latent``: whether the layer has a
        down projection of its own and fills it; ``q_rank`` None: queries are projected from the layer's input; ``gated``: True
        for a gate per head, "features" for one per feature; ``halves``: feature i of the rotated part turns with feature i +
        rot_dim / 2 instead of its neighbour; ``window``: a token sees the last ``window`` ones, itself among them."""
        super().__init__()
        gates = heads * vdim if gated == "features" else heads if gated else 0
        self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank = heads, dim, vdim, q_rank, kv_rank
        self.scale, self.eps, self.latent_index, self.writes_latent = float(scale), eps, latent_index, writes_latent
        self.rot_dim, self.rot_base, self.rot_scaling, self.gated = rot_dim, float(rot_base), rot_scaling, gated
        self.halves, self.window = halves, window
        self._inv_freq: Optional[torch.Tensor] = None

        def p(*shape, dtype=params_dtype):
            return nn.Parameter(torch.zeros(*shape, dtype=dtype), requires_grad=False)

        def lin(o, i):
            m = nn.Module()
            m.weight = p(o, i)
            return m

        # rows of the down projection: query latent, cache latent with the shared key part, gates; zero rows to a multiple of 8.
        # Queries without a latent come last: decode steps form them with the rest, prompts that run expanded on their own
        self.down_at, rows = {}, 0
        for name, n in (("q", q_rank or 0), ("kv", kv_rank + rot_dim if writes_latent else 0), ("g", gates)):
            self.down_at[name] = slice(rows, rows + n)
            rows += n
        rows = -(-rows // 8) * 8
        self.down_rows = rows
        if q_rank is None:
            self.down_at["q"] = slice(rows, rows + heads * (dim + rot_dim))
            rows = -(-self.down_at["q"].stop // 8) * 8
        self.down_proj = lin(rows, hidden_size)
        self.q_latent_norm = nn.Module()
        self.q_latent_norm.weight = None if q_rank is None else nn.Parameter(torch.ones(q_rank, dtype=torch.float32), requires_grad=False)
        if writes_latent:
            self.kv_latent_norm = nn.Module()
            self.kv_latent_norm.weight = nn.Parameter(torch.ones(kv_rank, dtype=torch.float32), requires_grad=False)
        self.q_up = None if q_rank is None else lin(heads * (dim + rot_dim), q_rank)        # per head [dim | rot_dim]
        self.k_up = lin(heads * dim, kv_rank)
        self.v_up = lin(heads * vdim, kv_rank)
        self.sink = p(heads, dtype=torch.float32) if sinks else None
        self.o_proj = lin(hidden_size, heads * vdim)
        width = max(dim + rot_dim, vdim)
        self.pad = next((w for w in (64, 128, 256) if width <= w), None)   # head size of the expanded form

    @property
    def cache_width(self) -> int:
        """Features of a cache row."""
        return self.kv_rank + self.rot_dim

    def load_down(self, name: str, full: torch.Tensor) -> None:
        """``name``: q (query latent, or the queries), kv (cache latent and shared key part) or g (gates)."""
        rows = self.down_proj.weight.data[self.down_at[name]]
        if rows.shape != full.shape:
            raise ValueError(f"a tensor of shape {tuple(full.shape)} does not fit {tuple(rows.shape)}")
        rows.copy_(full)

    def post_load(self) -> None:
        """Weights in the layouts of the two forms: per head and K-major for the absorbed products, heads padded to the
        attention kernels' size for the expanded ones."""
        H, R = self.heads, self.rot_dim

        def keep(t):
            return nn.Parameter(t.contiguous(), requires_grad=False)

        k_up = self.k_up.weight.data.view(H, self.dim, self.kv_rank)
        self._uk_t = keep(k_up.transpose(1, 2))                                                       # [H, rank, dim]
        self._uv = self.v_up.weight.data.view(H, self.vdim, self.kv_rank)                             # [H, vdim, rank]
        q_up = self.down_proj.weight[self.down_at["q"]] if self.q_up is None else self.q_up.weight
        # the projections of a prompt whose queries are formed apart
        self._down_rest = self.down_proj.weight if self.q_up is not None else nn.Parameter(self.down_proj.weight.data[: self.down_rows],
                                                                                            requires_grad=False)
        if self.pad is not None and self.expandable(q_up):
            v_up = self._uv
            if R:       # products with whole cache rows: the shared key part is copied into K and left out of V
                wide = k_up.new_zeros(H, self.dim + R, self.cache_width)
                wide[:, : self.dim, : self.kv_rank] = k_up
                wide[:, self.dim:, self.kv_rank:] = torch.eye(R, dtype=wide.dtype, device=wide.device)
                k_up, v_up = wide, torch.cat([v_up, v_up.new_zeros(H, self.vdim, R)], -1)
            self._uq_pad = keep(_pad_heads(q_up.data, H, self.pad))
            self._uk_pad = keep(_pad_heads(k_up.reshape(-1, self.cache_width), H, self.pad))
            self._uv_pad = keep(_pad_heads(v_up.reshape(-1, self.cache_width), H, self.pad))

    def expandable(self, like: torch.Tensor) -> bool:
        """The expanded form needs the 16-bit attention kernels on a GPU; on the CPU it runs in any type."""
        return self.pad is not None and (not like.is_cuda or ops.attention_kernels_cover(self.pad, like.dtype, like.dtype)
                                         and like.dtype != torch.float32)

    def inv_freq(self, device) -> Optional[torch.Tensor]:
        if self.rot_dim and (self._inv_freq is None or self._inv_freq.device != device):
            self._inv_freq = rotation_frequencies(self.rot_dim, self.rot_base, self.rot_scaling).to(device)
        return self._inv_freq

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        T, H = x.shape[0], self.heads
        cache = fb.token_to_kv_pool.get_latent_buffer(self.latent_index)
        rtt = fb.req_to_token_pool.req_to_token
        plan = latent_plan(fb, self.expandable(x), window=self.window)

        def near(t):
            return t if plan.rows is None or t is None else t.index_select(0, plan.rows)

        # without a query latent the expanded form takes its queries from the input, in heads of its own width
        apart = self.q_up is None and bool(plan.groups)
        y = ops.linear(x, self._down_rest if apart else self.down_proj.weight)
        cq, turns = ops.latent_prologue(y, self.q_latent_norm.weight, self.kv_latent_norm.weight if self.writes_latent else None,
                                        self.eps, fb.out_cache_loc, cache if self.writes_latent else None, fb.positions,
                                        self.inv_freq(x.device), self.halves)
        gate = y[:, self.down_at["g"]] if self.gated else None
        o = None
        if plan.groups:
            o = self._expanded(x if cq is None else cq, cache, rtt, plan, turns, gate)
        if plan.row_req is not None:
            if self.q_up is not None:
                q = ops.linear(near(cq), self.q_up.weight)
            elif apart:
                q = ops.linear(near(x), self.down_proj.weight[self.down_at["q"]])
            else:
                q = y[:, self.down_at["q"]]
            q = q.unflatten(1, (H, self.dim + self.rot_dim))
            q = ops.head_linear(q, self._uk_t, turns=near(turns), halves=self.halves)
            u = ops.latent_attention(q, cache, rtt, plan.row_req, plan.row_pos, self.scale, self.sink, plan.max_ctx, self.kv_rank, self.window)
            u = ops.head_linear(u, self._uv, gate=near(gate))
            if plan.rows is None:
                o = u
            else:
                o.index_copy_(0, plan.rows, u)
        return ops.linear(o.reshape(T, H * self.vdim), self.o_proj.weight)

    def _expanded(self, cq, cache, rtt, plan: LatentPlan, turns, gate) -> torch.Tensor:
        """Attention of the plan's expanded requests: [T, H, vdim], rows of other requests left unset."""
        H, W = self.heads, self.pad
        q = ops.linear(cq, self._uq_pad).view(-1, H, W)
        if turns is not None:
            ops.turn_heads(q[..., self.dim: self.dim + self.rot_dim], turns, halves=self.halves)
        out = torch.empty_like(q)
        for g in plan.groups:
            c = ops.latent_gather(cache, rtt, g.req, g.seq_lens, g.ctx_start, g.total, g.max_ctx, g.first)
            k = ops.linear(c, self._uk_pad).view(-1, H, W)
            v = ops.linear(c, self._uv_pad).view(-1, H, W)
            ops.attention_prefill(q, k, v, g.rows, g.batch, g.seq_lens, g.prefix_lens, g.q_start, self.scale, out=out,
                                  max_q_len=g.max_q, sink=self.sink, window=self.window)
        out = out[..., : self.vdim]
        return out.contiguous() if gate is None else ops.gate_heads(out, gate)
