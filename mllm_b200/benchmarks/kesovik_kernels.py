"""Kernels that the Kesovik design adds, each beside the like kernel of the closest existing model at equal size
(``python bench.py --design-pair kesovik-6b:qwen3.5-moe-6b``)."""

from __future__ import annotations

import torch

from .. import ops
from .design_pair import Table, _copies, _rand, kv_decode_kernel, rule_kernels

BF16 = torch.bfloat16


def _i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def lightning_kernels(t: Table, batch: int, length: int, heads: int, dim: int) -> None:
    """Beside the gated delta rule with the same state size."""
    tag = f"{'decode' if length == 1 else 'prefill'} {batch}x{length}"
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    T, C = batch * length, 3 * heads * dim
    nbytes = T * C * 2 + T * heads * dim * 2 + 2.0 * batch * heads * dim * dim * 4
    n = _copies(nbytes)
    xs = [_rand(T, C + heads * dim) for _ in range(n)]
    states = [torch.zeros(batch, heads, dim, dim, device="cuda") for _ in range(n)]
    lens, has, start = torch.full_like(req, length), torch.ones_like(req), req * length
    decay = torch.linspace(0.8, 0.999, heads, device="cuda")
    t.add(f"lightning attention {tag}", f"delta rule {tag}",
          lambda i: ops.lightning_attention(*(xs[i][:, j * heads * dim:(j + 1) * heads * dim].unflatten(1, (heads, dim)) for j in range(3)),
                                            decay, states[i], req, lens, has, start, length), n, nbytes, 4.0 * T * heads * dim * dim)
    rule_kernels(t, batch, length, heads, dim)


def window_decode(t: Table, batch: int, length: int, window: int, heads: int, kv: int, dim: int, tag: str, like: str) -> None:
    slots = batch * length + 16
    n = _copies(2 * slots * kv * dim * 2)
    pool = [tuple(_rand(kv, slots, dim).transpose(0, 1) for _ in range(2)) for _ in range(n)]
    table = (torch.arange(batch * length, device="cuda", dtype=torch.int32) + 16).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens, q = torch.full_like(req, length), _rand(batch, heads, dim)
    seen = min(window, length)
    t.add(f"window attention decode {tag}, window {window}", f"attention_decode {like}",
          lambda i: ops.attention_decode(q, *pool[i], table, req, lens, dim ** -0.5, max_seq_len=length, window=window), n,
          2.0 * batch * seen * kv * dim * 2, 4.0 * batch * heads * seen * dim)


def prefill(t: Table, batch: int, length: int, heads: int, kv: int, dim: int, window: int, like: str) -> None:
    T = batch * length
    q, k, v = _rand(T, heads, dim), _rand(T, kv, dim), _rand(T, kv, dim)
    table = torch.arange(T, device="cuda", dtype=torch.int32).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens, zero, start = torch.full_like(req, length), torch.zeros_like(req), req * length
    out = torch.empty(T, heads * dim + 64, device="cuda", dtype=BF16)[:, : heads * dim].unflatten(1, (heads, dim))
    pairs = length * (length + 1) / 2 if not window or window >= length else window * length - window * (window - 1) / 2
    name = f"attention_prefill {dim}-wide {batch}x{length}" + (f", window {window}" if window else "")
    t.add(name, like, lambda i: ops.attention_prefill(q, k, v, table, req, lens, zero, start, dim ** -0.5, out=out, max_q_len=length,
                                                      window=window or None), 1,
          2.0 * T * (2 * heads + 2 * kv) * dim, 4.0 * batch * heads * dim * pairs)


def prologue(t: Table, rows: int, heads: int, kv: int, dim: int) -> None:
    width = (heads + 2 * kv) * dim
    n = _copies(rows * width * 4)
    xs = [_rand(rows, width) for _ in range(n)]
    cache = [torch.empty(kv, rows + 16, dim, device="cuda", dtype=BF16).transpose(0, 1) for _ in range(2)]
    loc, pos = torch.arange(rows, device="cuda") + 16, torch.arange(rows, device="cuda") % 2048
    qw, kw = torch.ones(heads * dim, device="cuda"), torch.ones(kv * dim, device="cuda")
    freq = torch.pow(torch.tensor(1e6, dtype=torch.float64), -torch.arange(0, dim, 2, dtype=torch.float64) / dim).cuda()
    f32, w16 = freq.float(), torch.ones(dim, device="cuda", dtype=BF16)
    q = torch.empty(rows, heads, dim, device="cuda", dtype=BF16)
    t.add(f"row norm + rotation + cache write {rows} rows", f"head norm + rotation + cache write {rows} rows",
          lambda i: ops.rownorm_rope_kv(xs[i], qw, kw, freq, pos, loc, q, *cache, heads, kv, dim, dim, 1e-6), n, rows * width * 4.0)
    t.add(f"head norm + rotation + cache write {rows} rows", "",
          lambda i: ops.qk_norm_rope_kv_write(xs[i], w16, w16, pos, loc, *cache, heads, kv, dim, 1e6, 1e-6, inv_freq=f32), n, rows * width * 4.0)


def rows_kernels(t: Table, rows: int, width: int, top: int) -> None:
    """Norms, gate, mixture sum, embedding."""
    n = _copies(rows * width * 12)
    xs = [torch.randn(rows, width, device="cuda") for _ in range(n)]
    ys, hs = [_rand(rows, width) for _ in range(n)], [_rand(rows, width) for _ in range(n)]
    w, ls, wb = torch.ones(width, device="cuda"), torch.ones(width, device="cuda"), torch.ones(width, device="cuda", dtype=BF16)
    t.add(f"norm behind the sum {rows} rows", f"fused_add_rmsnorm {rows} rows", lambda i: ops.post_norm(xs[i], ys[i], ls, 2.0, w, 1e-6, BF16), n,
          rows * width * 12.0)
    t.add(f"fused_add_rmsnorm {rows} rows", "", lambda i: ops.fused_add_rmsnorm(ys[i], hs[i], wb, 1e-6), n, rows * width * 8.0)
    g = [_rand(rows, 2 * width) for _ in range(n)]
    out = torch.empty(rows, width, device="cuda", dtype=BF16)
    w128 = torch.ones(128, device="cuda", dtype=BF16)
    t.add(f"row norm with sigmoid gate {rows} rows", f"head norm with SiLU gate {rows} rows",
          lambda i: ops.rmsnorm_sigmoid_gate(ys[i], g[i][:, width:], w, 1e-6, out), n, rows * width * 6.0)
    t.add(f"head norm with SiLU gate {rows} rows", "", lambda i: ops.rmsnorm_gated(ys[i], g[i][:, width:], w128, 1e-6, False), n, rows * width * 6.0)
    pairs = rows * top
    m = _copies(pairs * width * 2)
    er = [_rand(pairs, width) for _ in range(m)]
    pos = torch.randperm(pairs, device="cuda").to(torch.int32)
    tw, ids = torch.rand(rows, top, device="cuda"), torch.zeros(rows, top, device="cuda", dtype=torch.int32)
    parts = [ops.ExpertRows(e, pos, tw, ids, ys[0], 0) for e in er]
    t.add(f"mixture sum + norm {rows} rows", f"mixture sum {rows} rows",
          lambda i: ops.post_norm(xs[i % n], ys[i % n], ls, 2.0, w, 1e-6, BF16, experts=parts[i]), m, rows * width * 2.0 * (top + 6))
    t.add(f"mixture sum {rows} rows", "", lambda i: ops.ext().moe_combine(er[i], pos, tw, out), m, rows * width * 2.0 * (top + 1))
    table, tok = _rand(151936, width), torch.randint(0, 151936, (rows,), device="cuda")
    t.add(f"scaled embedding {rows} rows", f"embedding {rows} rows", lambda i: ops.embedding_f32(tok, table, 3.0, rounded=True), 1, rows * width * 8.0)
    t.add(f"embedding {rows} rows", "", lambda i: ops.embedding(tok, table), 1, rows * width * 4.0)


def router(t: Table, rows: int, width: int, outputs: int, top: int) -> None:
    n = _copies(rows * width * 2)
    xs, w = [_rand(rows, width) for _ in range(n)], _rand(outputs, width, std=0.02)
    corr = torch.zeros(outputs, device="cuda")
    nbytes = 2.0 * (rows * width + outputs * width)
    t.add(f"router, fp32 logits and correction {rows} rows", f"router {rows} rows", lambda i: ops.moe_route(xs[i], w, top, True, corr, 1e-20), n, nbytes)
    t.add(f"router {rows} rows", "", lambda i: ops.moe_router_topk(xs[i], w, top, True), n, nbytes)


def squared_relu(t: Table, rows: int, width: int, ff: int) -> None:
    n = _copies(width * ff * 2) if rows <= 256 else 1
    ws = [torch.nn.Parameter(_rand(ff, width, std=0.02), requires_grad=False) for _ in range(n)]
    x = _rand(rows, width)
    nbytes, flops = 2.0 * (ff * width + rows * (width + ff)), 2.0 * rows * width * ff
    t.add(f"squared-ReLU gemm {rows} rows", f"gemm {ff} wide {rows} rows", lambda i: ops.linear_relu_squared(x, ws[i]), n, nbytes, flops)
    t.add(f"gemm {ff} wide {rows} rows", "", lambda i: ops.linear(x, ws[i]), n, nbytes, flops)


def soft_cap(t: Table, rows: int, vocab: int) -> None:
    n = _copies(rows * vocab * 6)
    xs = [_rand(rows, vocab) for _ in range(n)]
    t.add(f"logit cap {rows} rows", f"GELU {rows} rows", lambda i: ops.soft_cap(xs[i], 30.0), n, rows * vocab * 6.0)
    t.add(f"GELU {rows} rows", "", lambda i: ops.gelu_tanh(xs[i]), n, rows * vocab * 4.0)


def add_rows(t: Table) -> None:
    for batch, length in ((1, 1), (8, 1), (32, 1), (1, 2048), (8, 2048)):
        lightning_kernels(t, batch, length, 16, 128)
        torch.cuda.empty_cache()
    # the like kernel reads as many keys: it has no window in the other model
    for batch, length in ((1, 2048), (8, 2048), (32, 1024), (4, 16384)):
        seen = min(2048, length)
        window_decode(t, batch, length, 2048, 16, 4, 128, f"{batch}x{length}", f"{batch}x{seen}")
        kv_decode_kernel(t, batch, seen, 8, 2, 256, f"{batch}x{seen}")
        torch.cuda.empty_cache()
    prefill(t, 8, 2048, 16, 4, 128, 2048, "attention_prefill 256-wide 8x2048")
    prefill(t, 8, 2048, 16, 4, 128, 512, "attention_prefill 256-wide 8x2048")
    prefill(t, 8, 2048, 8, 2, 256, 0, "")
    for rows in (8, 32, 16384):
        prologue(t, rows, 16, 4, 128)
        rows_kernels(t, rows, 2048, 8)
        router(t, rows, 2048, 72, 8)
        squared_relu(t, rows, 2048, 6144)
        torch.cuda.empty_cache()
    soft_cap(t, 8, 151936)
