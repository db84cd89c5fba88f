"""Two decoder presets of equal size side by side, whole and kernel by kernel (random weights, one GPU).

    python bench.py --design-pair pebulix-2b:qwen3.5-2b
    python bench.py --design-pair kesovik-6b:qwen3.5-moe-6b
    python bench.py --design-pair lufizen-6b:qwen2-moe-6b
    python bench.py --design-pair nikedra-6b:qwen3.5-moe-6b

For each (batch, prompt length) both models prefill one batch and decode; times are CUDA-event medians, decode through
the captured graphs.  Every step streams the weights and the caches of the model (several GB), so nothing is served
from L2 between timed iterations.  The kernel table times the kernels that the new design adds next to the
like kernel of the other model at the same size, each with its share of the
measured roofline: algorithmic bytes over the copy bandwidth or FLOPs over the library GEMM rate, whichever bound is
the longer one.  Kernel inputs are rotated over copies that together exceed L2."""

from __future__ import annotations

import gc
import json
import statistics
from pathlib import Path
from typing import Any, Callable, Dict, List, Tuple

import torch

from .. import ops
from .kernel_cases import _time

SIZES: Tuple[Tuple[int, int], ...] = ((1, 2048), (8, 2048), (32, 1024), (4, 16384))
DECODE_STEPS = 64


def peaks() -> Dict[str, Any]:
    """Measured copy bandwidth and GEMM rate when the machine has them on file, else an earlier measurement."""
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        d = json.loads(f.read_text())
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


# --------------------------------------------------------------------------------------------
# whole models
# --------------------------------------------------------------------------------------------
def model_rows(preset: str, sizes, reps: int) -> List[dict]:
    from ..bench_one_batch import BenchRunner, make_synthetic_input_ids
    from ..configs import GlobalConfig

    GlobalConfig.reset()
    cfg = GlobalConfig.get_instance()
    sc = cfg.server
    sc.model_path, sc.dtype = f"preset:{preset}", "bfloat16"
    sc.max_running_requests = max(b for b, _ in sizes)
    sc.max_total_tokens = max(b * (n + DECODE_STEPS + 16) for b, n in sizes) + 4096
    sc.context_length = max(n for _, n in sizes) + DECODE_STEPS + 64
    sc.radix_cache_page_size = 16
    br = BenchRunner.create(cfg)
    rows = []
    for batch, length in sizes:
        ids = make_synthetic_input_ids(batch_size=batch, input_len=length, vocab_size=br.runner.vocab_size, seed=7).to(br.device)
        pre, dec = [], []
        for rep in range(reps + 2):
            ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
            br.clear()
            torch.cuda.synchronize()
            ev[0].record()
            nxt = br.extend(ids)
            ev[1].record()
            for _ in range(DECODE_STEPS):
                nxt = br.decode(nxt)
            ev[2].record()
            torch.cuda.synchronize()
            if rep >= 2:
                pre.append(ev[0].elapsed_time(ev[1]))
                dec.append(ev[1].elapsed_time(ev[2]) / DECODE_STEPS)
        p, d = statistics.median(pre), statistics.median(dec)
        rows.append({"model": preset, "batch": batch, "input_len": length, "prefill_ms": round(p, 3), "decode_ms": round(d, 4),
                     "prefill_tokens_per_s": round(batch * length / p * 1e3), "decode_tokens_per_s": round(batch / d * 1e3)})
    ops.check_status()
    br.runner.shutdown()
    del br
    gc.collect()
    torch.cuda.empty_cache()
    return rows


# --------------------------------------------------------------------------------------------
# kernels
# --------------------------------------------------------------------------------------------
class Table:
    def __init__(self) -> None:
        self.peak, self.rows = peaks(), []

    def add(self, name: str, like: str, fn: Callable[[int], Any], copies: int, bytes_: float = 0.0, flops: float = 0.0) -> None:
        """Times ``fn(i)`` for i rotating over ``copies`` sets of inputs."""
        state = {"i": 0}

        def run():
            fn(state["i"] % copies)
            state["i"] += 1

        ms = _time(run, max(20, copies))
        bound = max(bytes_ / self.peak["hbm_gbs"] / 1e6, flops / self.peak["bf16_tflops"] / 1e9)
        self.rows.append({"kernel": name, "like": like, "us": round(ms * 1e3, 2), "roofline_us": round(bound * 1e3, 2),
                          "of_roofline": round(bound / ms, 3)})


def _copies(nbytes: float) -> int:
    return max(2, min(48, int(3e8 // max(nbytes, 1)) + 1))


def _rand(*shape, dtype=torch.bfloat16, std=1.0):
    return (torch.randn(*shape, device="cuda") * std).to(dtype)


def _latent_ctx(batch: int, length: int, rank: int):
    slots = batch * length + 16
    n = _copies(slots * rank * 2)
    caches = [_rand(slots, rank) for _ in range(n)]
    table = (torch.arange(batch * length, device="cuda", dtype=torch.int32) + 16).view(batch, length)
    return caches, table, torch.arange(batch, device="cuda", dtype=torch.int32)


def latent_kernels(t: Table, batch: int, length: int, heads: int, rank: int, dim: int, tag: str) -> None:
    caches, table, req = _latent_ctx(batch, length, rank)
    q, sink = _rand(batch, heads, rank, std=rank ** -0.5), torch.zeros(heads, device="cuda")
    pos = torch.full((batch,), length - 1, dtype=torch.int64, device="cuda")
    t.add(f"latent_attention decode {tag}", f"attention_decode {tag}",
          lambda i: ops.latent_attention(q, caches[i], table, req, pos, 1.0, sink, length), len(caches),
          batch * length * rank * 2, 4.0 * batch * heads * length * rank)
    x = _rand(batch, heads, dim)
    ws = [_rand(heads, rank, dim, std=0.05) for _ in range(_copies(heads * rank * dim * 2))]
    t.add(f"head_linear {batch} rows", f"gemm {batch} rows", lambda i: ops.head_linear(x, ws[i]), len(ws), heads * rank * dim * 2)
    del caches


def kv_decode_kernel(t: Table, batch: int, length: int, heads: int, kv_heads: int, dim: int, tag: str) -> None:
    slots = batch * length + 16
    n = _copies(2 * slots * kv_heads * dim * 2)
    kv = [tuple(_rand(kv_heads, slots, dim).transpose(0, 1) for _ in range(2)) for _ in range(n)]
    table = (torch.arange(batch * length, device="cuda", dtype=torch.int32) + 16).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens = torch.full((batch,), length, dtype=torch.int32, device="cuda")
    q = _rand(batch, heads, dim)
    t.add(f"attention_decode {tag}", "", lambda i: ops.attention_decode(q, *kv[i], table, req, lens, dim ** -0.5, max_seq_len=length), n,
          2.0 * batch * length * kv_heads * dim * 2, 4.0 * batch * heads * length * dim)


def prefill_kernels(t: Table, batch: int, length: int, like: bool, heads: int, kv_heads: int, dim: int, tag: str) -> None:
    T = batch * length
    q, k, v = _rand(T, heads, dim), _rand(T, kv_heads, dim), _rand(T, kv_heads, dim)
    table = torch.arange(T, device="cuda", dtype=torch.int32).view(batch, length)
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    lens, zero = torch.full_like(req, length), torch.zeros_like(req)
    start, out = req * length, torch.empty_like(q)
    sink = None if like else torch.zeros(heads, device="cuda")
    name = f"attention_prefill {tag}" if like else f"attention_prefill with sink {tag}"
    t.add(name, "" if like else f"attention_prefill {tag}",
          lambda i: ops.attention_prefill(q, k, v, table, req, lens, zero, start, dim ** -0.5, out=out, max_q_len=length, sink=sink), 1,
          2.0 * T * (2 * heads + 2 * kv_heads) * dim, 2.0 * batch * heads * length * length * dim)


def rule_kernels(t: Table, batch: int, length: int, heads: int, dim: int) -> None:
    req = torch.arange(batch, device="cuda", dtype=torch.int32)
    tag = "decode" if length == 1 else "prefill"
    tag = f"{tag} {batch}x{length}"
    T, C = batch * length, 3 * heads * dim
    nbytes = T * C * 2 + T * heads * dim * 2 + 2.0 * batch * heads * dim * dim * 4
    n = _copies(nbytes)
    xs = [_rand(T, C + 2 * heads) for _ in range(n)]
    states = [torch.zeros(batch, heads, dim, dim, device="cuda") for _ in range(n)]
    lens, has, start = torch.full_like(req, length), torch.ones_like(req), req * length
    a_log, dt = torch.zeros(heads, device="cuda") - 2, torch.zeros(heads, device="cuda")
    g, beta = -torch.rand(T, heads, device="cuda") * 0.1, torch.rand(T, heads, device="cuda")

    def parts(i):
        return [xs[i][:, j * heads * dim:(j + 1) * heads * dim].unflatten(1, (heads, dim)) for j in range(3)]

    flops = 6.0 * T * heads * dim * dim
    t.add(f"delta rule, fp32 products, {tag}", f"delta rule {tag}",
          lambda i: ops.gated_delta_rule(*parts(i), None, None, states[i], req, lens, has, start, split_tf32=True,
                                         raw_gates=(xs[i][:, C:C + heads], xs[i][:, C + heads:], a_log, dt)), n, nbytes, flops)
    t.add(f"delta rule {tag}", "", lambda i: ops.gated_delta_rule(*parts(i), g, beta, states[i], req, lens, has, start), n, nbytes, flops)


def row_kernels(t: Table, rows: int, width: int, q_rank: int, kv_rank: int) -> None:
    """Row-wise kernels: norm with the residual sum, prologue of the latent layers, embedding."""
    n = _copies(rows * width * 12)
    xs = [torch.randn(rows, width, device="cuda") for _ in range(n)]
    ys = [_rand(rows, width) for _ in range(n)]
    hs = [_rand(rows, width) for _ in range(n)]
    w, b, alpha = torch.ones(width, device="cuda"), torch.zeros(width, device="cuda"), torch.ones(1, device="cuda")
    wb = torch.ones(width, device="cuda", dtype=torch.bfloat16)
    t.add(f"residual_dyt {rows} rows", f"fused_add_rmsnorm {rows} rows",
          lambda i: ops.residual_dyt(xs[i], ys[i], 0.5, alpha, w, b, torch.bfloat16), n, rows * width * 12.0)
    t.add(f"fused_add_rmsnorm {rows} rows", "", lambda i: ops.fused_add_rmsnorm(ys[i], hs[i], wb, 1e-6), n, rows * width * 8.0)
    down = [_rand(rows, q_rank + kv_rank) for _ in range(n)]
    cache = torch.empty(rows + 16, kv_rank, device="cuda", dtype=torch.bfloat16)
    loc = torch.arange(rows, device="cuda") + 16
    qw, kw = torch.ones(q_rank, device="cuda"), torch.ones(kv_rank, device="cuda")
    t.add(f"latent_prologue {rows} rows", f"rmsnorm {rows} rows", lambda i: ops.latent_prologue(down[i], qw, kw, 1e-6, loc, cache), n,
          rows * (q_rank + kv_rank) * 4.0)
    t.add(f"rmsnorm {rows} rows", "", lambda i: ops.rmsnorm(ys[i], wb, 1e-6), n, rows * width * 4.0)
    if rows >= 1024:
        table = torch.arange(rows, device="cuda", dtype=torch.int32).view(1, rows)
        one, ln, zero = (torch.tensor([v], dtype=torch.int32, device="cuda") for v in (0, rows, 0))
        src = [_rand(rows, kv_rank) for _ in range(_copies(rows * kv_rank * 2))]
        t.add(f"latent_gather {rows} rows", f"rmsnorm {rows} rows", lambda i: ops.latent_gather(src[i], table, one, ln, zero, rows, rows),
              len(src), rows * kv_rank * 4.0)


def product_kernels(t: Table, rows: int, width: int, ff: int) -> None:
    n = _copies(2 * width * ff * 2) if rows <= 256 else 1
    ws = [torch.nn.Parameter(_rand(2 * ff, width, std=0.02), requires_grad=False) for _ in range(n)]
    x = _rand(rows, width)
    nbytes, flops = 2.0 * (2 * ff * width + rows * (width + ff)), 4.0 * rows * width * ff
    for act, name, like in (("gelu_tanh", "GeGLU", f"SwiGLU gemm {rows} rows"), ("silu", "SwiGLU", "")):
        t.add(f"{name} gemm {rows} rows", like, lambda i, act=act: ops.linear_swiglu(x, ws[i], act=act), n, nbytes, flops)
    wo = [torch.nn.Parameter(_rand(width, width, std=0.02), requires_grad=False) for _ in range(_copies(width * width * 2))]
    t.add(f"gemm {rows} rows", "", lambda i: ops.linear(x, wo[i]), len(wo), 2.0 * (width * width + 2 * rows * width),
          2.0 * rows * width * width)


def gated_kernels(t: Table, rows: int, heads: int, dim: int) -> None:
    """Convolution and gated norm: the same kernels for both models, here with the strided inputs of the fused projection."""
    C = 3 * heads * dim
    n = _copies(rows * C * 4)
    xs = [_rand(rows, C + heads * dim + 2 * heads) for _ in range(n)]
    o = [_rand(rows, heads * dim) for _ in range(n)]
    w, cw = torch.ones(dim, device="cuda", dtype=torch.bfloat16), _rand(C, 4)
    req = torch.zeros(1, device="cuda", dtype=torch.int32)
    st = torch.zeros(1, C, 3, device="cuda", dtype=torch.bfloat16)
    if rows >= 1024:
        t.add(f"conv + silu {rows} rows", "", lambda i: ops.causal_conv1d_silu(xs[i][:, :C], cw, st, req, req + rows, req, req, rows), n,
              rows * C * 4.0)
    t.add(f"gated norm {rows} rows", "", lambda i: ops.rmsnorm_gated(o[i], xs[i][:, C:C + heads * dim], w, 1e-6, False), n,
          rows * heads * dim * 6.0)


def pebulix_rows(t: Table) -> None:
    # decode: pebulix-2b (16 heads over latents of 512) and qwen3.5-2b (8 heads of 256 over 2 key / value heads)
    for batch, length in ((1, 2048), (8, 2048), (32, 1024), (4, 16384)):
        latent_kernels(t, batch, length, 16, 512, 128, f"{batch}x{length}")
        kv_decode_kernel(t, batch, length, 8, 2, 256, f"{batch}x{length}")
        torch.cuda.empty_cache()
    prefill_kernels(t, 8, 2048, False, 16, 16, 128, "8x2048")
    prefill_kernels(t, 8, 2048, True, 8, 2, 256, "8x2048")
    for batch, length in ((1, 1), (8, 1), (32, 1), (1, 2048), (8, 2048)):
        rule_kernels(t, batch, length, 16, 128)
        torch.cuda.empty_cache()
    for rows in (1, 4, 32):
        product_kernels(t, rows, 2048, 6144)
    for rows in (8, 16384):
        row_kernels(t, rows, 2048, 1024, 512)
        product_kernels(t, rows, 2048, 6144)
        gated_kernels(t, rows, 16, 128)
        torch.cuda.empty_cache()


def kesovik_rows(t: Table) -> None:
    from .kesovik_kernels import add_rows

    add_rows(t)


def lufizen_rows(t: Table) -> None:
    from .lufizen_kernels import add_rows

    add_rows(t)


def nikedra_rows(t: Table) -> None:
    from .nikedra_kernels import add_rows

    add_rows(t)


# the kernels a design adds, by the first word of its presets
KERNELS = {"pebulix": pebulix_rows, "kesovik": kesovik_rows, "lufizen": lufizen_rows, "nikedra": nikedra_rows}


def kernel_rows(preset: str) -> List[dict]:
    t = Table()
    KERNELS[preset.split("-")[0]](t)
    ops.check_status()
    by_name = {r["kernel"]: r for r in t.rows}
    for r in t.rows:
        other = by_name.get(r["like"])
        if other is not None:       # how much further from its roofline than the like kernel
            r["distance_vs_like"] = round(other["of_roofline"] / r["of_roofline"], 2)
    return t.rows


def run(pair: str, reps: int, part: str = "all") -> dict:
    names = pair.split(":")
    if len(names) != 2:
        raise SystemExit("--design-pair takes two presets: new:closest")
    out: Dict[str, Any] = {"metric": "design_pair", "pair": names, "dtype": "bf16", "data": "synthetic (random weights and ids)",
                           "peaks": peaks()}
    if part in ("all", "kernels"):
        out["kernels"] = kernel_rows(names[0])
    if part in ("all", "models"):
        out["models"] = [row for n in names for row in model_rows(n, SIZES, reps)]
    return out
