"""Pebulix on the GPU: every mechanism's kernels against the plain statement, then whole models through the serving path
in all the ways a sequence can be fed."""
import pytest
import torch

import pebulix_models as pm
import pebulix_oracle as oracle
from session_schedules import cut, run_alone, run_together
from test_pebulix_cpu import _generate, _greedy

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.bfloat16, torch.float32]


def _r(*shape, seed=0, std=1.0, dtype=torch.float32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype)


def _tol(dtype, half, single=2e-5):
    return half if dtype != torch.float32 else single


def _close(got, want, tol):
    scale = want.abs().max().item()
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= tol * max(scale, 1e-3), (err, scale)


# --------------------------------------------------------------------------- norms, stream, embedding
@pytest.mark.parametrize("dtype", DTYPES + [torch.float16])
@pytest.mark.parametrize("shape", [(1, 64), (5, 90), (37, 33), (300, 2048)])
def test_residual_and_dynamic_tanh(dtype, shape):
    from mllm_b200 import ops

    T, W = shape
    x, y = _r(T, W, seed=1, std=2), _r(T, W, seed=2).to(dtype)
    w, b, alpha = 1 + _r(W, seed=3, std=0.2), _r(W, seed=4, std=0.3), torch.tensor([0.8])
    for other, mult in ((None, 1.0), (y, 0.37)):
        gx = x.to(DEV)
        h = ops.residual_dyt(gx, None if other is None else other.to(DEV), mult, alpha.to(DEV), w.to(DEV), b.to(DEV), dtype)
        want_x = oracle.f64(x) + (0 if other is None else mult * oracle.f64(other))
        _close(gx, want_x, 1e-6)                     # the stream stays in 32-bit
        _close(h, oracle.dyt(want_x, oracle.f64(alpha), oracle.f64(w), oracle.f64(b)), _tol(dtype, 5e-3, 1e-6))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 90, 33])
def test_embedding_widened(dtype, width):
    from mllm_b200 import ops

    table = _r(50, width).to(dtype)
    ids = torch.tensor([0, 49, 7, 7])
    got = ops.embedding_f32(ids.to(DEV), table.to(DEV))
    assert got.dtype == torch.float32 and torch.equal(got.cpu(), table[ids].float())


# --------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ff", [(1, 256, 256), (8, 512, 1024), (9, 160, 136), (70, 256, 384), (300, 512, 256),
                                           (2500, 512, 2048), (5, 90, 33)])
def test_geglu(dtype, rows, width, ff):
    from mllm_b200.layers import MLP

    with torch.device(DEV):
        mlp = MLP(width, ff, params_dtype=dtype, activation="gelu_tanh")
    w = {"gate": _r(ff, width, seed=1, std=2 * width ** -0.5).to(dtype), "up": _r(ff, width, seed=2, std=width ** -0.5).to(dtype),
         "down": _r(width, ff, seed=3, std=ff ** -0.5).to(dtype)}
    for j, n in enumerate(("gate", "up")):
        mlp.gate_up_proj.weight_loader(mlp.gate_up_proj.weight, w[n].to(DEV), j)
    mlp.down_proj.weight_loader(mlp.down_proj.weight, w["down"].to(DEV))
    mlp.gate_up_proj.quant_method.process_weights_after_loading(mlp.gate_up_proj)
    x = _r(rows, width, seed=4).to(dtype)
    want = oracle.geglu(oracle.f64(x), {k: oracle.f64(v) for k, v in w.items()}, "")
    _close(mlp(x.to(DEV)), want, _tol(dtype, 1e-2))


# --------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank", [(64, 64), (30, 36), (1024, 512), (11, 0), (136, 0)])
def test_latent_prologue(dtype, q_rank, kv_rank):
    from mllm_b200 import ops

    T, S = 13, 40
    y = _r(T, q_rank + kv_rank + 5, seed=1).to(dtype)
    qw, kw = 1 + _r(q_rank, seed=2, std=0.2), 1 + _r(max(kv_rank, 1), seed=3, std=0.2)
    loc = torch.randperm(S, generator=torch.Generator().manual_seed(4))[:T]
    cache = torch.full((S, kv_rank + 3), 7.0, dtype=dtype, device=DEV)
    got, _ = ops.latent_prologue(y.to(DEV), qw.to(DEV), kw.to(DEV) if kv_rank else None, 3e-5, loc.to(DEV) if kv_rank else None,
                              cache[:, :kv_rank] if kv_rank else None)
    _close(got, oracle.rms_norm(oracle.f64(y[:, :q_rank]), oracle.f64(qw), 3e-5), _tol(dtype, 5e-3, 1e-6))
    if kv_rank:
        _close(cache[loc.to(DEV), :kv_rank], oracle.rms_norm(oracle.f64(y[:, q_rank:q_rank + kv_rank]), oracle.f64(kw), 3e-5),
               _tol(dtype, 5e-3, 1e-6))
        rest = torch.ones(S, dtype=torch.bool)
        rest[loc] = False
        assert (cache[rest.to(DEV)] == 7.0).all() and (cache[:, kv_rank:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,heads,n,k", [(1, 16, 512, 128), (8, 20, 64, 264), (33, 3, 24, 40), (70, 5, 130, 24), (3, 2, 7, 9)])
def test_head_linear(dtype, tokens, heads, n, k):
    from mllm_b200 import ops

    x, w = _r(tokens, heads, k, seed=1).to(dtype), _r(heads, n, k, seed=2, std=k ** -0.5).to(dtype)
    got = ops.head_linear(x.to(DEV), w.to(DEV))
    _close(got, torch.einsum("thk,hnk->thn", oracle.f64(x), oracle.f64(w)), _tol(dtype, 1e-2))


def _latent_case(heads, rank, lens, dtype, seed=0, std=0.3):
    """Contexts of several requests in scattered slots of one cache; every unused slot and every table entry past a
    request's end leads to a row that would dominate any softmax."""
    g = torch.Generator().manual_seed(seed)
    S = sum(lens) + 64
    slots = torch.randperm(S - 1, generator=g)[: sum(lens)] + 1
    cache = torch.full((S, rank), 30.0, dtype=dtype)
    table = torch.zeros(len(lens) + 2, max(lens) + 40, dtype=torch.int32)
    req = torch.randperm(len(lens) + 2, generator=g)[: len(lens)].to(torch.int32)
    ctx, at = [], 0
    for r, n in zip(req, lens):
        c = (torch.randn(n, rank, generator=g) * std).to(dtype)
        cache[slots[at:at + n]] = c
        table[int(r), :n] = slots[at:at + n].to(torch.int32)
        ctx.append(c)
        at += n
    return cache, table, req, ctx


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank", [(1, 8), (3, 24), (16, 64), (17, 72), (8, 200), (20, 264), (16, 512), (5, 576), (2, 1000), (3, 36)])
def test_latent_attention_rows_of_unequal_requests(dtype, heads, rank):
    from mllm_b200 import ops

    lens = (1, 31, 32, 33, 64, 65, 200, 700)
    cache, table, req, ctx = _latent_case(heads, rank, lens, dtype, std=1.0)
    sink = _r(heads, seed=5) + 1
    # two queries per request: its last position and one in the middle
    owner = [b for b in range(len(lens)) for _ in range(2)]
    pos = [p for n in lens for p in (n - 1, n // 2)]
    q = _r(len(pos), heads, rank, seed=6, std=rank ** -0.5).to(dtype)
    scale = 0.9
    got = ops.latent_attention(q.to(DEV), cache.to(DEV), table.to(DEV), req[owner].to(DEV), torch.tensor(pos).to(DEV), scale,
                               sink.to(DEV), max(lens))
    want = torch.zeros(len(pos), heads, rank, dtype=torch.float64)
    for t, (b, p) in enumerate(zip(owner, pos)):
        c = oracle.f64(ctx[b][: p + 1])
        for h in range(heads):
            want[t, h] = oracle.sink_softmax((c @ oracle.f64(q[t, h])) * scale, float(sink[h])) @ c
    _close(got, want, _tol(dtype, 1.2e-2))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank", [64, 264, 36])
@pytest.mark.parametrize("n", [1, 2, 32, 33, 257, 1500])
def test_latent_attention_finds_one_far_key(dtype, rank, n):
    """One key stands out by far; the query must return that key's row wherever it lies (first token, either side of a
    tile's edge, the query's own position), and the even stronger keys behind the query must not show."""
    from mllm_b200 import ops

    heads = 3
    places = sorted({p for p in (0, 1, 31, 32, 63, 64, n // 2, n - 2, n - 1) if 0 <= p < n})
    cache, table, req, _ = _latent_case(heads, rank, [n + 8] * len(places), dtype, std=0.05)
    row_of = lambda b, j: int(table[int(req[b]), j])                                     # noqa: E731
    for b, p in enumerate(places):
        cache[row_of(b, p)] = 0.05
        cache[row_of(b, p), b % rank] = 4.0
        for j in range(n, n + 8):
            cache[row_of(b, j)] = 9.0
    q = torch.zeros(len(places), heads, rank, dtype=dtype)
    for b in range(len(places)):
        q[b, :, b % rank] = 8.0
    got = ops.latent_attention(q.to(DEV), cache.to(DEV), table.to(DEV), req.to(DEV), torch.full((len(places),), n - 1).to(DEV), 1.0,
                               torch.full((heads,), -5.0).to(DEV), n + 8)
    want = torch.stack([oracle.f64(cache[row_of(b, p)]).expand(heads, -1) for b, p in enumerate(places)])
    _close(got, want, 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 3.0, 40.0])
@pytest.mark.parametrize("n", [1, 40, 900])
def test_sink_takes_its_share(dtype, sink, n):
    from mllm_b200 import ops

    heads, rank = 4, 64
    cache, table, req, ctx = _latent_case(heads, rank, [n], dtype)
    q = _r(1, heads, rank, seed=3, std=0.2).to(dtype)
    s = torch.full((heads,), sink)
    s[1] -= 2
    got = ops.latent_attention(q.to(DEV), cache.to(DEV), table.to(DEV), req.to(DEV), torch.tensor([n - 1]).to(DEV), 0.7, s.to(DEV), n)
    c = oracle.f64(ctx[0])
    want = torch.stack([oracle.sink_softmax((c @ oracle.f64(q[0, h])) * 0.7, float(s[h])) @ c for h in range(heads)])[None]
    err = (got.double().cpu() - want).abs().max() / max(want.abs().max().item(), 1e-12 if sink < 10 else 1e-3)
    assert err < _tol(dtype, 1.2e-2)


@pytest.mark.parametrize("head_dim,heads,kv_heads", [(64, 4, 4), (128, 4, 4), (128, 8, 2), (256, 3, 3)])
def test_sinks_of_the_shared_attention_kernels(head_dim, heads, kv_heads):
    """Prefill, short decode and split decode of the K / V attention kernels, with a sink per query head."""
    from mllm_b200 import ops

    dtype = torch.bfloat16
    lens, prefix = [150, 3, 260], [70, 0, 259]
    S = sum(lens) + 1
    k, v = _r(S, kv_heads, head_dim, seed=1).to(dtype), _r(S, kv_heads, head_dim, seed=2).to(dtype)
    table = torch.zeros(3, 300, dtype=torch.int32)
    at = 1
    for b, n in enumerate(lens):
        table[b, :n] = torch.arange(at, at + n)
        at += n
    new = [n - p for n, p in zip(lens, prefix)]
    start = [0, new[0], new[0] + new[1]]
    q = _r(sum(new), heads, head_dim, seed=3).to(dtype)
    sink = torch.linspace(-2, 4, heads)
    scale = head_dim ** -0.5
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)                       # noqa: E731

    def want_row(b, pos, qr):
        rows = table[b, : pos + 1].long()
        out = []
        for h in range(heads):
            kk, vv = oracle.f64(k[rows, h // (heads // kv_heads)]), oracle.f64(v[rows, h // (heads // kv_heads)])
            out.append(oracle.sink_softmax((kk @ oracle.f64(qr[h])) * scale, float(sink[h])) @ vv)
        return torch.stack(out)

    got = ops.attention_prefill(q.to(DEV), k.to(DEV), v.to(DEV), table.to(DEV), i32([0, 1, 2]), i32(lens), i32(prefix), i32(start),
                                scale, max_q_len=max(new), sink=sink.to(DEV))
    want = torch.stack([want_row(b, prefix[b] + j, q[start[b] + j]) for b in range(3) for j in range(new[b])])
    _close(got, want, 1.2e-2)
    qd = q[:3].contiguous()
    want = torch.stack([want_row(b, lens[b] - 1, qd[b]) for b in range(3)])
    for bound in (64, 4096):                                       # one range, or the context split over CTAs
        got = ops.attention_decode(qd.to(DEV), k.to(DEV), v.to(DEV), table.to(DEV), i32([0, 1, 2]), i32(lens), scale,
                                   max_seq_len=bound, sink=sink.to(DEV))
        _close(got, want, 1.2e-2)


# --------------------------------------------------------------------------- delta rule
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_short_convolution_over_portions(dtype, taps):
    """Requests of unequal length in reused state rows, fed in portions: outputs as of one pass over each sequence."""
    from mllm_b200 import ops

    C, lens = 70, [150, 9, 1, 80]
    x = [_r(n, C, seed=n).to(dtype) for n in lens]
    w = _r(C, taps, seed=9, std=0.6).to(dtype)
    state = torch.full((6, C, taps - 1), 5.0, dtype=dtype, device=DEV)      # left over from earlier requests
    slots = torch.tensor([4, 0, 3, 1], dtype=torch.int32, device=DEV)
    done, outs = [0] * 4, [[] for _ in lens]
    for portion in (1, 2, 70, 3, 100):
        take = [min(portion if b else portion + 1, n - d) for b, (n, d) in enumerate(zip(lens, done))]
        use = [b for b in range(4) if take[b] > 0]
        if not use:
            continue
        wide = torch.zeros(sum(take), C + 13, dtype=dtype)
        wide[:, :C] = torch.cat([x[b][done[b]:done[b] + take[b]] for b in use])
        lens_d = torch.tensor([take[b] for b in use], dtype=torch.int32, device=DEV)
        has = torch.tensor([int(done[b] > 0) for b in use], dtype=torch.int32, device=DEV)
        y = ops.causal_conv1d_silu(wide.to(DEV)[:, :C], w.to(DEV), state, slots[use], lens_d, has, max_len=max(take))
        for b, part in zip(use, y.split([take[b] for b in use])):
            outs[b].append(part)
            done[b] += take[b]
    assert done == lens
    for b in range(4):
        want = oracle.silu(oracle.short_conv(oracle.f64(x[b]), oracle.f64(w)))
        _close(torch.cat(outs[b]), want, _tol(dtype, 6e-3, 2e-6))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("backend", ["auto", "mllm_kernel", "cuda_chunkwise"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 128, 128), (2, 2, 32, 48), (3, 1, 24, 96), (2, 1, 18, 10), (2, 2, 200, 36)])
def test_delta_rule_over_portions(dtype, backend, heads, kv_heads, dim, vdim):
    """Token-sequential and chunk-parallel kernels, one head group per key head, portions that cut the chunks anywhere,
    state rows with remains of other requests.  The recurrence must carry fp32 accuracy whatever the inputs' type."""
    from mllm_b200 import ops

    lens = [130, 5, 66]
    cut_at = [[64, 2, 1, 63], [1, 4], [66]]
    a_log, dt_bias = _r(heads, seed=1, std=0.5) - 1.5, _r(heads, seed=2)
    cols = 2 * kv_heads * dim + heads * vdim
    raw = [_r(n, cols + 2 * heads, seed=30 + n).to(dtype) for n in lens]
    state = torch.full((5, heads, dim, vdim), 3.0, device=DEV)
    slots = torch.tensor([3, 0, 4], dtype=torch.int32, device=DEV)
    ops.set_gdn_extend_backend(backend)
    try:
        done, outs = [0] * 3, [[] for _ in lens]
        for step in range(4):
            use = [b for b in range(3) if step < len(cut_at[b])]
            take = [cut_at[b][step] for b in use]
            t = torch.cat([raw[b][done[b]:done[b] + n] for b, n in zip(use, take)]).to(DEV)
            q = t[:, : kv_heads * dim].unflatten(1, (kv_heads, dim))
            k = t[:, kv_heads * dim: 2 * kv_heads * dim].unflatten(1, (kv_heads, dim))
            v = t[:, 2 * kv_heads * dim: cols].unflatten(1, (heads, vdim))
            i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=DEV)               # noqa: E731
            y = ops.gated_delta_rule(q, k, v, None, None, state, slots[use], i32(take), i32([int(done[b] > 0) for b in use]),
                                     raw_gates=(t[:, cols:cols + heads], t[:, cols + heads:], a_log.to(DEV), dt_bias.to(DEV)),
                                     split_tf32=True)
            for b, part in zip(use, y.split(take)):
                outs[b].append(part)
            for b, n in zip(use, take):
                done[b] += n
    finally:
        ops.set_gdn_extend_backend("auto")
    own = [h // (heads // kv_heads) for h in range(heads)]
    for b, n in enumerate(lens):
        x = oracle.f64(raw[b])
        q, k = x[:, : kv_heads * dim].view(n, kv_heads, dim), x[:, kv_heads * dim: 2 * kv_heads * dim].view(n, kv_heads, dim)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dim ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        g = torch.exp(-torch.exp(oracle.f64(a_log)) * oracle.softplus(x[:, cols + heads:] + oracle.f64(dt_bias)))
        beta = 1 / (1 + torch.exp(-x[:, cols:cols + heads]))
        o, S = oracle.delta_states(q[:, own], k[:, own], x[:, 2 * kv_heads * dim: cols].view(n, heads, vdim), g, beta)
        _close(torch.cat(outs[b]), o, _tol(dtype, 5e-3, 1e-5))
        _close(state[int(slots[b])], S, 2e-5)           # fp32, through either kernel


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,width", [(3, 40), (16, 128), (2, 10), (1, 300)])
def test_gated_norm(dtype, heads, width):
    from mllm_b200 import ops

    T = 11
    x, gate = _r(T, heads * width, seed=1).to(dtype), _r(T, heads * width + 24, seed=2).to(dtype)
    w = (1 + _r(width, seed=3, std=0.2)).to(dtype)
    got = ops.rmsnorm_gated(x.to(DEV), gate.to(DEV)[:, 8:8 + heads * width], w.to(DEV), 3e-5, round_norm=False)
    want = oracle.rms_norm(oracle.f64(x).view(T, heads, width), oracle.f64(w), 3e-5).view(T, -1) * oracle.silu(oracle.f64(gate[:, 8:8 + heads * width]))
    _close(got, want, _tol(dtype, 5e-3, 1e-6))


# --------------------------------------------------------------------------- whole models
LIMIT = {"float32": 5e-5, "bfloat16": 0.09}


def _within(err: torch.Tensor, dtype: str, where) -> None:
    """All rows within the limit; in 16 bits one row in fifty (or one) may reach twice that (a short key vector made a unit vector
    now and then amplifies its rounding — the plain fp32-accumulating statement run in bf16 shows the same rows)."""
    over = int((err > LIMIT[dtype]).sum())
    most = LIMIT[dtype] * (2 if dtype == "bfloat16" else 1)
    assert err.max() < most and over <= (max(1, 0.02 * err.numel()) if dtype == "bfloat16" else 0), (where, int(err.argmax()), float(err.max()))



@pytest.fixture(scope="module")
def served(tmp_path_factory):
    from mllm_b200.trace_run import build_session

    cache = {}

    def get(name, dtype, page=1):
        if (name, dtype, page) not in cache:
            path = tmp_path_factory.mktemp(name) / "m"
            cfg = pm.CONFIGS[name]
            w = pm.write_checkpoint(path, cfg)
            cache[name, dtype, page] = (build_session(str(path), dtype, 1024, radix_cache_page_size=page), w, cfg)
        return cache[name, dtype, page]

    return get


@pytest.fixture(scope="module")
def expected():
    cache = {}

    def get(name, n, seed):
        if (name, n, seed) not in cache:
            cfg = pm.CONFIGS[name]
            seq = pm.tokens(cfg, n, seed=seed)
            cache[name, n, seed] = (seq, oracle.forward(cfg, pm.weights(cfg), seq))
        return cache[name, n, seed]

    return get


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_portions_and_single_tokens_match_the_statement(served, expected, name, dtype):
    session, _, _ = served(name, dtype)
    seq, want = expected(name, 120, 1)
    for sizes in ([120], [1], [2], [64, 1, 1, 31, 2, 7]):
        _within(pm.logit_error(run_alone(session, seq, cut(len(seq), sizes)), want), dtype, sizes)
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name,page", [("mixed", 1), ("mixed", 16), ("large", 64), ("odd", 1)])
def test_batches_of_unequal_requests_with_reused_slots(served, expected, name, page, dtype):
    session, _, _ = served(name, dtype, page)
    lens = (90, 3, 120, 1, 65, 40, 33, 100)
    both = {f"r{i}": expected(name, n, 70 + i) for i, n in enumerate(lens)}
    cuts = {"r0": cut(90, [40, 1]), "r1": [2, 1], "r2": cut(120, [2, 1, 1]), "r3": [1], "r4": [64, 1], "r5": cut(40, [1]),
            "r6": [33], "r7": cut(100, [1, 63, 5])}
    for _ in range(2):
        got = run_together(session, {k: s for k, (s, _) in both.items()}, cuts, {f"r{i}": i for i in range(8)})
        for k, (_, want) in both.items():
            _within(pm.logit_error(got[k], want), dtype, k)


def test_long_decoding_through_captured_graphs(served, expected):
    session, _, _ = served("mixed", "float32")
    graphs = session.mrp.runner.cuda_graph_runner
    before = graphs.replays
    seq, want = expected("mixed", 400, 5)
    assert pm.logit_error(run_alone(session, seq, [5] + [1] * 395), want).max() < LIMIT["float32"]
    assert graphs.replays == before + 395


def test_residual_stream_after_every_layer(served):
    session, w, cfg = served("large", "float32")
    seq, want, got = pm.tokens(cfg, 40), [], []
    oracle.forward(cfg, w, seq, want)
    runner = session.mrp.runner
    run = runner.forward

    def tapped(fb):
        fb.extra["layer_outputs"] = got
        return run(fb)

    runner.forward = tapped
    try:
        session.step([dict(id="x", tokens=seq, want=[])], ["x"])
    finally:
        runner.forward = run
    for a, b in zip(got, want):
        _close(a, b, 2e-5)


def test_greedy_generation_through_the_engine(tmp_path):
    cfg = pm.CONFIGS["mixed"]
    w = pm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [pm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9, 60)]
    want = [_greedy(cfg, w, p, 8) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 8, DEV, max_running_requests=3, chunked_prefill_size=24, mem_fraction_static=0.2)
    assert got == [ids for ids, _ in want]
    # bf16 through the same path: tokens that lead by far are the same
    sure = [(p, ids) for p, (ids, lead) in zip(prompts, want) if lead > 0.5]
    for p, ids in sure:
        assert _generate(tmp_path / "m", [p], 8, DEV, "bfloat16", mem_fraction_static=0.2)[0] == ids


def test_replay_program(tmp_path):
    """bin/trace_run as a user starts it: files of logits, one line per step."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np

    cfg = pm.CONFIGS["mixed"]
    w = pm.write_checkpoint(tmp_path / "m", cfg)
    seq = pm.tokens(cfg, 12)
    steps = [dict(step=0, entries=[dict(id="a", tokens=seq[:9], want=[8, 0])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=seq[9:10], want=[])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=seq[:2], want=[1]), dict(id="a", tokens=seq[10:], want=[1])], end=["a", "b"])]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([sys.executable, str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(tmp_path / "m"),
                        "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = oracle.forward(cfg, w, seq)
    assert sorted(f.name for f in out.iterdir()) == ["0.f32", "2.f32"]
    for name, rows in (("0.f32", [8, 0]), ("2.f32", [1, 11])):
        got = torch.from_numpy(np.fromfile(out / name, "<f4")).view(len(rows), cfg["vocab"])
        assert pm.logit_error(got, want[rows]).max() < LIMIT["float32"]
