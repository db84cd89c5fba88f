"""Kernels that the Lufizen design adds, each beside the like kernel of the closest existing models at equal size
(``python bench.py --design-pair lufizen-6b:qwen2-moe-6b``)."""

from __future__ import annotations

import torch

from .. import ops
from ..layers.attention import rotation_frequencies
from .design_pair import Table, _copies, _latent_ctx, _rand, kv_decode_kernel, latent_kernels
from .kesovik_kernels import prefill

BF16 = torch.bfloat16


def latent_decode(t: Table, batch: int, length: int, heads: int, rank: int, rot: int, dim: int) -> None:
    """Keys of rank + rot features; beside latents without a rotated part and beside K / V attention."""
    tag, key = f"{batch}x{length}", rank + rot
    caches, table, req = _latent_ctx(batch, length, key)
    q = _rand(batch, heads, key, std=key ** -0.5)
    pos = torch.full((batch,), length - 1, dtype=torch.int64, device="cuda")
    for like in (f"latent_attention decode {tag}", f"attention_decode {tag}"):
        t.add(f"latent attention with rotated part, decode {tag}", like,
              lambda i: ops.latent_attention(q, caches[i], table, req, pos, 1.0, None, length, rank), len(caches),
              batch * length * key * 2, 2.0 * batch * heads * length * (key + rank))
    del caches
    x, turns = _rand(batch, heads, dim + rot), torch.rand(batch, rot // 2, 2, device="cuda")
    ws = [_rand(heads, rank, dim, std=0.05) for _ in range(_copies(heads * rank * dim * 2))]
    t.add(f"head_linear and turns {tag}", f"head_linear {batch} rows", lambda i: ops.head_linear(x, ws[i], turns=turns), len(ws), heads * rank * dim * 2)
    u, gate = _rand(batch, heads, rank), _rand(batch, heads)
    vs = [_rand(heads, dim, rank, std=0.05) for _ in range(len(ws))]
    t.add(f"head_linear and gate {tag}", f"head_linear {batch} rows", lambda i: ops.head_linear(u, vs[i], gate=gate), len(vs), heads * rank * dim * 2)


def sink_decode(t: Table, batch: int, length: int, heads: int, kv: int, dim: int) -> None:
    slots = batch * length + 16
    n = _copies(2 * slots * kv * dim * 2)
    pool = [tuple(_rand(kv, slots, dim).transpose(0, 1) for _ in range(2)) for _ in range(n)]
    table = (torch.arange(batch * length, device="cuda", dtype=torch.int32) + 16).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens, q, sink = torch.full_like(req, length), _rand(batch, heads, dim), torch.zeros(heads, device="cuda")
    t.add(f"attention_decode with sink {batch}x{length}", f"attention_decode {batch}x{length}",
          lambda i: ops.attention_decode(q, *pool[i], table, req, lens, dim ** -0.5, max_seq_len=length, sink=sink), n,
          2.0 * batch * length * kv * dim * 2, 4.0 * batch * heads * length * dim)


def prefills(t: Table, batch: int, length: int, heads: int, kv: int, dim: int, rot: int, vdim: int, pad: int) -> None:
    """Key-valued attention with sinks, and the expanded latent form, whose heads are padded to ``pad`` features."""
    T = batch * length
    table = torch.arange(T, device="cuda", dtype=torch.int32).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens, zero, start = torch.full_like(req, length), torch.zeros_like(req), req * length
    pairs, like = length * (length + 1) / 2, f"attention_prefill {dim}-wide {batch}x{length}"
    sink = torch.zeros(heads, device="cuda")
    q, k, v = _rand(T, heads, dim), _rand(T, kv, dim), _rand(T, kv, dim)
    out = torch.empty_like(q)
    t.add(f"attention_prefill with sink {batch}x{length}", like,
          lambda i: ops.attention_prefill(q, k, v, table, req, lens, zero, start, dim ** -0.5, out=out, max_q_len=length, sink=sink), 1,
          2.0 * T * (2 * heads + 2 * kv) * dim, 4.0 * batch * heads * dim * pairs)
    q2, k2, v2 = _rand(T, heads, pad), _rand(T, heads, pad), _rand(T, heads, pad)
    q2[..., dim + rot:] = 0
    k2[..., dim + rot:] = 0
    v2[..., vdim:] = 0
    out2 = torch.empty_like(q2)
    t.add(f"expanded latent attention, prefill {batch}x{length}", like,
          lambda i: ops.attention_prefill(q2, k2, v2, table, req, lens, zero, start, 0.07, out=out2, max_q_len=length), 1,
          2.0 * T * heads * 2 * (dim + rot + vdim), 2.0 * batch * heads * (dim + rot + vdim) * pairs)
    prefill(t, batch, length, heads, kv, dim, 0, "")


def prologues(t: Table, rows: int, heads: int, kv: int, dim: int, rot_dims: int, q_rank: int, kv_rank: int, rot: int, vdim: int, pad: int) -> None:
    like = f"head norm + rotation + cache write {rows} rows"
    width, full = (heads + kv) * dim, (heads + 2 * kv) * dim
    n = _copies(rows * width * 4)
    xs, ys = [_rand(rows, width) for _ in range(n)], [_rand(rows, full) for _ in range(n)]
    cache = [torch.empty(kv, rows + 16, dim, device="cuda", dtype=BF16).transpose(0, 1) for _ in range(2)]
    loc, pos = torch.arange(rows, device="cuda") + 16, torch.arange(rows, device="cuda") % 2048
    q, w16, freq = torch.empty(rows, heads, dim, device="cuda", dtype=BF16), torch.ones(dim, device="cuda", dtype=BF16), rotation_frequencies(rot_dims, 1e6).cuda()
    f32 = rotation_frequencies(dim, 1e6).float().cuda()
    t.add(f"rotation + norm per head + cache write {rows} rows", like,
          lambda i: ops.headnorm_rope_kv(xs[i], freq, pos, loc, q, *cache, heads, kv, dim, dim, heads * dim, True, 1e-6), n,
          rows * (2.0 * width + kv * dim) * 2)
    t.add(like, "", lambda i: ops.qk_norm_rope_kv_write(ys[i], w16, w16, pos, loc, *cache, heads, kv, dim, 1e6, 1e-6, inv_freq=f32), n,
          rows * full * 4.0)
    down = [_rand(rows, q_rank + kv_rank + rot + heads) for _ in range(_copies(rows * (q_rank + kv_rank) * 2))]
    lat = torch.empty(rows + 16, kv_rank + rot, device="cuda", dtype=BF16)
    qw, kw, fr = torch.ones(q_rank, device="cuda"), torch.ones(kv_rank, device="cuda"), rotation_frequencies(rot, 1e4).cuda()
    t.add(f"latent prologue with rotated part {rows} rows", f"latent_prologue {rows} rows",
          lambda i: ops.latent_prologue(down[i], qw, kw, 1e-6, loc, lat, pos, fr), len(down), rows * (q_rank + kv_rank + rot) * 4.0)
    plain = lat[:, :kv_rank]
    t.add(f"latent_prologue {rows} rows", "", lambda i: ops.latent_prologue(down[i], qw, kw, 1e-6, loc, plain), len(down),
          rows * (q_rank + kv_rank) * 4.0)
    if rows >= 1024:
        wide = [_rand(rows, heads, pad) for _ in range(_copies(rows * heads * pad * 2))]
        turns, gate = torch.rand(rows, rot // 2, 2, device="cuda"), _rand(rows, heads)
        t.add(f"turned query heads {rows} rows", like, lambda i: ops.turn_heads(wide[i][..., dim:dim + rot], turns), len(wide), rows * heads * rot * 4.0)
        t.add(f"gated heads {rows} rows", f"SiLU and product {rows} rows", lambda i: ops.gate_heads(wide[i][..., :vdim], gate), len(wide), rows * heads * vdim * 4.0)
        gu = [_rand(rows, 2 * heads * vdim) for _ in range(_copies(rows * heads * vdim * 4))]
        t.add(f"SiLU and product {rows} rows", "", lambda i: ops.silu_and_mul(gu[i]), len(gu), rows * heads * vdim * 6.0)


def rows_kernels(t: Table, rows: int, width: int, top: int, experts: int, groups: int, keep: int) -> None:
    """Norm on the output, mixture sum with the gated shared expert, router."""
    n = _copies(rows * width * 12)
    xs = [torch.randn(rows, width, device="cuda") for _ in range(n)]
    ys, hs = [_rand(rows, width) for _ in range(n)], [_rand(rows, width) for _ in range(n)]
    w, wb = torch.ones(width, device="cuda"), torch.ones(width, device="cuda", dtype=BF16)
    t.add(f"norm on the output {rows} rows", f"fused_add_rmsnorm {rows} rows",
          lambda i: ops.post_norm(xs[i], ys[i], None, 1.0, w, 1e-6, BF16, inner=True), n, rows * width * 12.0)
    t.add(f"fused_add_rmsnorm {rows} rows", "", lambda i: ops.fused_add_rmsnorm(ys[i], hs[i], wb, 1e-6), n, rows * width * 8.0)
    pairs = rows * top
    m = _copies(pairs * width * 2)
    er = [_rand(pairs, width) for _ in range(m)]
    pos = torch.randperm(pairs, device="cuda").to(torch.int32)
    tw, ids = torch.rand(rows, top, device="cuda"), torch.zeros(rows, top, device="cuda", dtype=torch.int32)
    logit, out = torch.randn(rows, experts + 1, device="cuda")[:, experts], torch.empty(rows, width, device="cuda", dtype=BF16)
    parts = [ops.ExpertRows(e, pos, tw, ids, ys[0], 0, logit) for e in er]
    t.add(f"mixture sum + gated shared expert + norm {rows} rows", f"mixture sum {rows} rows",
          lambda i: ops.post_norm(xs[i % n], ys[i % n], None, 1.0, w, 1e-6, BF16, experts=parts[i], inner=True), m, rows * width * 2.0 * (top + 6))
    t.add(f"mixture sum {rows} rows", "", lambda i: ops.ext().moe_combine(er[i], pos, tw, out), m, rows * width * 2.0 * (top + 1))
    wr, wp, corr = _rand(experts + 1, width, std=0.02), _rand(experts, width, std=0.02), torch.zeros(experts, device="cuda")
    nbytes = 2.0 * (rows * width + experts * width)
    t.add(f"router, sigmoid scores within groups {rows} rows", f"router {rows} rows",
          lambda i: ops.moe_route(ys[i], wr, top, False, corr, 0.0, True, groups, keep, 2.5, 1), n, nbytes)
    t.add(f"router {rows} rows", "", lambda i: ops.moe_router_topk(ys[i], wp, top, False), n, nbytes)


def add_rows(t: Table) -> None:
    heads, kv, dim, rot, q_rank, rank = 16, 4, 128, 64, 1024, 512
    for batch, length in ((1, 2048), (8, 2048), (32, 1024), (4, 16384)):
        latent_decode(t, batch, length, heads, rank, rot, dim)
        torch.cuda.empty_cache()
        latent_kernels(t, batch, length, heads, rank, dim, f"{batch}x{length}")
        sink_decode(t, batch, length, heads, kv, dim)
        kv_decode_kernel(t, batch, length, heads, kv, dim, f"{batch}x{length}")
        torch.cuda.empty_cache()
    prefills(t, 8, 2048, heads, kv, dim, rot, dim, 256)
    torch.cuda.empty_cache()
    for rows in (8, 32, 16384):
        prologues(t, rows, heads, kv, dim, dim // 2, q_rank, rank, rot, dim, 256)
        rows_kernels(t, rows, 2048, 8, 64, 8, 4)
        torch.cuda.empty_cache()
