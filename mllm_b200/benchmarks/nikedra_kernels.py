"""Kernels that the Nikedra design adds, each beside the like kernel of the closest existing models at equal size
(``python bench.py --design-pair nikedra-6b:qwen3.5-moe-6b``)."""

from __future__ import annotations

import torch

from .. import ops
from ..layers.attention import rotation_frequencies
from .design_pair import Table, _copies, _latent_ctx, _rand, kv_decode_kernel
from .kesovik_kernels import lightning_kernels, prefill

BF16 = torch.bfloat16


def _meta(batch: int, length: int):
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    return req, torch.full_like(req, length), torch.ones_like(req), req * length


def _tag(batch: int, length: int) -> str:
    return f"{'decode' if length == 1 else 'prefill'} {batch}x{length}"


def recurrences(t: Table, batch: int, length: int, heads: int, dim: int, ssd_heads: int, state: int, vdim: int) -> None:
    """The delta rule with decays per channel beside the one with a decay per head; the state-space rule beside both kinds of
    linear attention with a state of its size."""
    tag, T = _tag(batch, length), batch * length
    req, lens, has, start = _meta(batch, length)
    D = heads * dim
    nbytes = T * 4 * D * 2 + T * D * 2 + 2.0 * batch * heads * dim * dim * 4
    n = _copies(nbytes)
    xs = [_rand(T, 4 * D + heads) for _ in range(n)]
    states = [torch.zeros(batch, heads, dim, dim, device="cuda") for _ in range(n)]
    a_log, dt = torch.zeros(heads, device="cuda") - 2, torch.zeros(D, device="cuda")
    t.add(f"delta rule, decays per channel, {tag}", f"delta rule, fp32 products, {tag}",
          lambda i: ops.channel_delta_rule(*(xs[i][:, j * D:(j + 1) * D].unflatten(1, (heads, dim)) for j in range(3)), xs[i][:, 4 * D:],
                                           xs[i][:, 3 * D:4 * D], a_log, dt, states[i], req, lens, has, start, length), n, nbytes, 6.0 * T * D * dim)
    del xs, states
    inner = ssd_heads * vdim
    nbytes = T * (inner + 2 * state + ssd_heads) * 2 + T * inner * 2 + 2.0 * batch * inner * state * 4
    n = _copies(nbytes)
    xs = [_rand(T, inner + 2 * state + ssd_heads) for _ in range(n)]
    states = [torch.zeros(batch, ssd_heads, state, vdim, device="cuda") for _ in range(n)]
    z = torch.zeros(ssd_heads, device="cuda")
    for like in (f"delta rule {tag}", f"lightning attention {tag}"):
        t.add(f"state space {tag}", like,
              lambda i: ops.state_space(xs[i][:, :inner].unflatten(1, (ssd_heads, vdim)), xs[i][:, inner: inner + state].unsqueeze(1),
                                        xs[i][:, inner + state: inner + 2 * state].unsqueeze(1), xs[i][:, inner + 2 * state:], z - 2, z - 1, z,
                                        states[i], req, lens, has, start, length), n, nbytes, 4.0 * T * inner * state)
    del xs, states
    lightning_kernels(t, batch, length, heads, dim)          # and the plain delta rule


def chunk_decode(t: Table, batch: int, length: int, chunk: int, heads: int, kv: int, dim: int) -> None:
    """Beside attention without chunks over as many keys."""
    slots = batch * length + 16
    n = _copies(2 * slots * kv * dim * 2)
    pool = [tuple(_rand(kv, slots, dim).transpose(0, 1) for _ in range(2)) for _ in range(n)]
    table = (torch.arange(batch * length, device="cuda", dtype=torch.int32) + 16).view(batch, length)
    req, lens, _, _ = _meta(batch, length)
    q, seen = _rand(batch, heads, dim), (length - 1) % chunk + 1
    t.add(f"chunk attention decode {batch}x{length}, {seen} seen", f"attention_decode {batch}x{seen}",
          lambda i: ops.attention_decode(q, *pool[i], table, req, lens, dim ** -0.5, max_seq_len=length, chunk=chunk), n,
          2.0 * batch * seen * kv * dim * 2, 4.0 * batch * heads * seen * dim)
    del pool
    kv_decode_kernel(t, batch, seen, heads, kv, dim, f"{batch}x{seen}")


def chunk_prefill(t: Table, batch: int, length: int, chunk: int, heads: int, kv: int, dim: int) -> None:
    T = batch * length
    q, k, v = _rand(T, heads, dim), _rand(T, kv, dim), _rand(T, kv, dim)
    table = torch.arange(T, device="cuda", dtype=torch.int32).view(batch, length)
    req, lens, _, start = _meta(batch, length)
    out, zero = torch.empty_like(q), torch.zeros_like(req)
    pairs = length // chunk * chunk * (chunk + 1) / 2
    for like in (f"attention_prefill {dim}-wide {batch * length // chunk}x{chunk}", f"attention_prefill {dim}-wide {batch}x{length}, window {chunk}"):
        t.add(f"chunk attention prefill {batch}x{length}, chunks of {chunk}", like,
              lambda i: ops.attention_prefill(q, k, v, table, req, lens, zero, start, dim ** -0.5, out=out, max_q_len=length, chunk=chunk), 1,
              2.0 * T * (2 * heads + 2 * kv) * dim, 4.0 * batch * heads * dim * pairs)
    prefill(t, batch * length // chunk, chunk, heads, kv, dim, 0, "")
    prefill(t, batch, length, heads, kv, dim, chunk, "")


def latent_window(t: Table, batch: int, length: int, window: int, heads: int, rank: int, rot: int, dim: int) -> None:
    """Beside the same kernel without a window over as many keys; head products beside those with a gate per head."""
    key, seen = rank + rot, min(window, length)
    for ctx, win, name, like in ((length, window, f"latent attention, window {window}, decode {batch}x{length}", f"latent attention decode {batch}x{seen}"),
                                 (seen, None, f"latent attention decode {batch}x{seen}", "")):
        caches, table, req = _latent_ctx(batch, ctx, key)
        q = _rand(batch, heads, key, std=key ** -0.5)
        pos = torch.full((batch,), ctx - 1, dtype=torch.int64, device="cuda")
        t.add(name, like, lambda i: ops.latent_attention(q, caches[i], table, req, pos, 1.0, None, ctx, rank, win), len(caches),
              batch * seen * key * 2, 2.0 * batch * heads * seen * (key + rank))
        del caches
    x, turns = _rand(batch, heads, dim + rot), torch.rand(batch, rot // 2, 2, device="cuda")
    ws = [_rand(heads, rank, dim, std=0.05) for _ in range(_copies(heads * rank * dim * 2))]
    u, vs = _rand(batch, heads, rank), [_rand(heads, dim, rank, std=0.05) for _ in range(len(ws))]
    for halves, name, like in ((True, "halves", f"head products and turned neighbours {batch} rows"), (False, "neighbours", "")):
        t.add(f"head products and turned {name} {batch} rows", like, lambda i: ops.head_linear(x, ws[i], turns=turns, halves=halves), len(ws),
              heads * rank * dim * 2)
    for gate, name, like in ((_rand(batch, heads * dim), "per feature", f"head products and gates per head {batch} rows"), (_rand(batch, heads), "per head", "")):
        t.add(f"head products and gates {name} {batch} rows", like, lambda i: ops.head_linear(u, vs[i], gate=gate), len(vs), heads * rank * dim * 2)


def between_layers(t: Table, rows: int, width: int, top: int) -> None:
    n = _copies(rows * width * 12)
    xs = [torch.randn(rows, width, device="cuda") for _ in range(n)]
    ys, hs = [_rand(rows, width) for _ in range(n)], [_rand(rows, width) for _ in range(n)]
    w, wb, one = torch.ones(width, device="cuda"), torch.ones(width, device="cuda", dtype=BF16), torch.ones((), device="cuda")
    like = f"fused_add_rmsnorm {rows} rows"
    t.add(like, "", lambda i: ops.fused_add_rmsnorm(ys[i], hs[i], wb, 1e-6), n, rows * width * 8.0)
    for depth in (1, 12, 24):
        m = _copies(rows * width * 4 * (depth + 1))
        res = [torch.randn(depth + 1, rows, width, device="cuda") for _ in range(m)]
        dwa = torch.full((depth + 1,), 0.2, device="cuda")
        slots = torch.arange(rows, device="cuda", dtype=torch.int32)
        conv = ops.ConvStep(_rand(width, 4), _rand(rows, width, 3), slots) if rows <= 64 else None
        nbytes = rows * width * (4.0 * (depth + 3) + 2 * 4 + (12 if conv else 0))
        t.add(f"step between layers, average of {depth + 1}, {rows} rows", like,
              lambda i: ops.depth_step(xs[i % n], (ys[i % n],), hs[i % n], None, res[i], depth, dwa, [one, one], 1e-6, BF16, xs[i % n], conv=conv), m, nbytes)
        if depth == 12:
            t.add(f"step between layers, two normed outputs, average of {depth + 1}, {rows} rows", like,
                  lambda i: ops.depth_step(xs[i % n], (ys[i % n], hs[i % n], w, w), ys[i % n], None, res[i], depth, dwa, [one, one], 1e-6, BF16, xs[i % n],
                                           conv=conv), m, nbytes + rows * width * 2.0)
            er, pos = _rand(rows * top, width), torch.randperm(rows * top, device="cuda").to(torch.int32)
            parts = ops.ExpertRows(er, pos, None, torch.zeros(rows, top, device="cuda", dtype=torch.int32), ys[0])
            t.add(f"step between layers, sum of {top} experts, average of {depth + 1}, {rows} rows", like,
                  lambda i: ops.depth_step(xs[i % n], (ys[i % n],), None, parts, res[i], depth, dwa, [one, one], 1e-6, BF16, xs[i % n], conv=conv), m,
                  nbytes + rows * width * 2.0 * (top - 1))
            del er, parts
        del res
    table, ids = _rand(151936, width), torch.randint(0, 151936, (rows,), device="cuda")
    t.add(f"embedding with norm {rows} rows", f"embedding {rows} rows", lambda i: ops.embed_norm(ids, table, one, xs[i], 1e-6, [one, one]), n,
          rows * width * 10.0)
    t.add(f"embedding {rows} rows", "", lambda i: ops.embedding(ids, table), n, rows * width * 4.0)
    if rows > 64:
        req, lens, has, start = _meta(8, rows // 8)
        cw, st = _rand(width, 4), _rand(8, width, 3)
        for add, name, other in ((True, "convolution added to its input", f"convolution + SiLU {rows} rows"), (False, "convolution + SiLU", "")):
            t.add(f"{name} {rows} rows", other, lambda i: ops.causal_conv1d_silu(ys[i], cw, st, req, lens, has, start, rows // 8, add_input=add), n,
                  rows * width * 4.0)


def row_kernels(t: Table, rows: int, heads: int, kv: int, dim: int, inner: int, pad: int, rank: int, rot: int) -> None:
    """Norms with gates, attention prologues."""
    D = heads * dim
    n = _copies(rows * D * 6)
    o, gate = [_rand(rows, D) for _ in range(n)], [_rand(rows, D + 64) for _ in range(n)]
    w, wf = torch.ones(dim, device="cuda", dtype=BF16), torch.ones(inner, device="cuda")
    like = f"norm per head, SiLU gate {rows} rows"
    t.add(like, "", lambda i: ops.rmsnorm_gated(o[i], gate[i][:, :D], w, 1e-6, False), n, rows * D * 6.0)
    t.add(f"norm per head, sigmoid gate {rows} rows", like, lambda i: ops.rmsnorm_gated(o[i], gate[i][:, :D], w, 1e-6, False, sigmoid=True), n, rows * D * 6.0)
    out = torch.empty(rows, inner, device="cuda", dtype=BF16)
    ins, gs = [_rand(rows, inner) for _ in range(n)], [_rand(rows, inner + 64) for _ in range(n)]
    t.add(f"gate before the norm {rows} rows", like, lambda i: ops.gated_rmsnorm(ins[i], gs[i][:, :inner], wf, 1, 1e-6, out), n, rows * inner * 6.0)
    width = (heads + 2 * kv) * dim
    m = _copies(rows * width * 4)
    ys = [_rand(rows, width) for _ in range(m)]
    cache = [torch.empty(kv, rows + 16, dim, device="cuda", dtype=BF16).transpose(0, 1) for _ in range(2)]
    loc, pos = torch.arange(rows, device="cuda") + 16, torch.arange(rows, device="cuda") % 2048
    q, freq = torch.empty(rows, heads, dim, device="cuda", dtype=BF16), rotation_frequencies(dim, 1e6).cuda()
    f32 = freq.float()
    like = f"head norm + rotation + cache write {rows} rows"
    t.add(f"rotation + cache write {rows} rows", like,
          lambda i: ops.headnorm_rope_kv(ys[i], freq, pos, loc, q, *cache, heads, kv, dim, dim, (heads + kv) * dim, True, 0.0, norm=False, magnitude=1.2), m,
          rows * width * 4.0)
    t.add(like, "", lambda i: ops.qk_norm_rope_kv_write(ys[i], w, w, pos, loc, *cache, heads, kv, dim, 1e6, 1e-6, inv_freq=f32), m, rows * width * 4.0)
    down = [_rand(rows, rank + rot + 64) for _ in range(_copies(rows * (rank + rot) * 2))]
    lat = torch.empty(rows + 16, rank + rot, device="cuda", dtype=BF16)
    qw, kw, fr = torch.ones(rank, device="cuda"), torch.ones(rank, device="cuda"), rotation_frequencies(rot, 1e4).cuda()
    both = [_rand(rows, 2 * rank + rot) for _ in range(len(down))]
    t.add(f"latent prologue, no query latent {rows} rows", f"latent prologue {rows} rows",
          lambda i: ops.latent_prologue(down[i], None, kw, 1e-6, loc, lat, pos, fr, True), len(down), rows * (rank + rot) * 4.0)
    t.add(f"latent prologue {rows} rows", "", lambda i: ops.latent_prologue(both[i], qw, kw, 1e-6, loc, lat, pos, fr), len(down), rows * (2 * rank + rot) * 4.0)
    if rows >= 1024:
        wide = [_rand(rows, heads, pad) for _ in range(_copies(rows * heads * pad * 2))]
        feat = _rand(rows, D)
        t.add(f"gates per feature {rows} rows", f"SiLU and product {rows} rows", lambda i: ops.gate_heads(wide[i][..., :dim], feat), len(wide), rows * D * 6.0)
        gu = [_rand(rows, 2 * D) for _ in range(_copies(rows * D * 4))]
        t.add(f"SiLU and product {rows} rows", "", lambda i: ops.silu_and_mul(gu[i]), len(gu), rows * D * 6.0)


def feed_forwards(t: Table, rows: int, width: int, ff: int, experts: int, top: int, expert_ff: int, like_ff: int) -> None:
    n = _copies(2 * width * ff * 2) if rows <= 256 else 1
    ws = [torch.nn.Parameter(_rand(2 * ff, width, std=0.02), requires_grad=False) for _ in range(n)]
    x, bias = _rand(rows, width), _rand(2 * ff)
    nbytes, flops = 2.0 * (2 * ff * width + rows * (width + ff)), 4.0 * rows * width * ff
    t.add(f"bounded gated product with biases {rows} rows", f"SwiGLU product {rows} rows",
          lambda i: ops.linear_swiglu(x, ws[i], act="clamped", bias=bias, limit=7.0), n, nbytes, flops)
    t.add(f"SwiGLU product {rows} rows", "", lambda i: ops.linear_swiglu(x, ws[i]), n, nbytes, flops)
    del ws
    for gated, inner, name, like in ((False, expert_ff, "experts, weighted inputs, GELU", f"experts, SwiGLU {rows} rows"), (True, like_ff, "experts, SwiGLU", "")):
        size = (3 if gated else 2) * inner * width
        m = 2 if rows <= 256 else 1
        w13 = [_rand(experts, (2 if gated else 1) * inner, width, std=0.02) for _ in range(m)]
        w2 = [_rand(experts, width, inner, std=0.02) for _ in range(m)]
        ids = torch.stack([torch.randperm(experts, device="cuda")[:top] for _ in range(min(rows, 4096))]).to(torch.int32)
        ids = ids.repeat(-(-rows // ids.shape[0]), 1)[:rows].contiguous()
        tw = torch.rand(rows, top, device="cuda")
        used = min(experts, rows * top)
        t.add(f"{name} {rows} rows", like,
              lambda i: ops.moe_expert_rows(x, w13[i], w2[i], tw, ids, ops.SWIGLU_BLOCK if gated else 0, gated=gated, weigh_input=not gated), m,
              2.0 * used * size + rows * width * 2.0 * (1 + top), 2.0 * rows * top * size)
        del w13, w2
    wr = _rand(experts, width, std=0.02)
    nb = 2.0 * (rows * width + experts * width)
    t.add(f"router, sigmoid scores {rows} rows", f"router {rows} rows", lambda i: ops.moe_route(x, wr, top, False, None, 0.0, True), 1, nb)
    t.add(f"router {rows} rows", "", lambda i: ops.moe_router_topk(x, wr, top, False), 1, nb)


def add_rows(t: Table) -> None:
    heads, kv, dim, rank, rot = 16, 4, 128, 512, 64
    for batch, length in ((1, 1), (8, 1), (32, 1), (1, 2048), (8, 2048)):
        recurrences(t, batch, length, 16, 128, 32, 128, 64)
        torch.cuda.empty_cache()
    for batch, length in ((1, 2048), (8, 2048), (32, 1024), (4, 16384)):
        chunk_decode(t, batch, length, 4096, heads, kv, dim)
        latent_window(t, batch, length, 2048, heads, rank, rot, dim)
        torch.cuda.empty_cache()
    chunk_prefill(t, 8, 2048, 1024, heads, kv, dim)
    chunk_prefill(t, 4, 8192, 4096, heads, kv, dim)
    torch.cuda.empty_cache()
    for rows in (8, 32, 16384):
        between_layers(t, rows, 2048, 8)
        row_kernels(t, rows, heads, kv, dim, 2048, 256, rank, rot)
        feed_forwards(t, rows, 2048, 6144, 64, 8, 768, 512)
        torch.cuda.empty_cache()
