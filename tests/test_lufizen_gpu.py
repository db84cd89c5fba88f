"""Lufizen on the GPU: every mechanism's kernels against the plain statement, then whole models through the serving path
in all the ways a sequence can be fed."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import lufizen_models as lm
import lufizen_oracle as oracle
from session_schedules import cut, run_alone, run_together
from test_lufizen_cpu import _generate, _greedy

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


# --------------------------------------------------------------------------- norm on a sublayer's output
@pytest.mark.parametrize("dtype", DTYPES + [torch.float16])
@pytest.mark.parametrize("shape", [(1, 64), (5, 90), (37, 33), (300, 2048), (3, 8192), (2, 16384)])
def test_norm_on_the_output(dtype, shape):
    from mllm_b200.layers import OutputRMSNorm

    T, W = shape
    x, y, w = _r(T, W, seed=1, std=20), _r(T, W, seed=2, std=0.1).to(dtype), 1 + _r(W, seed=4, std=0.3)
    with torch.device(DEV):
        norm = OutputRMSNorm(W, 3e-3, dtype)
    norm.weight.data.copy_(w)
    gx = x.to(DEV)
    h = norm(gx, y.to(DEV))
    want = oracle.f64(x) + oracle.rms_norm(oracle.f64(y), oracle.f64(w), 3e-3)
    _close(gx, want, 1e-6)                            # the stream stays in 32-bit
    _close(h, want, _tol(dtype, 5e-3, 1e-6))


# --------------------------------------------------------------------------- attention prologue
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("heads,kv,dim,vdim,width,dims,base", [(4, 2, 64, 64, 128, 64, 1e4), (3, 1, 10, 10, 10, 6, 5e5), (8, 2, 128, 128, 128, 32, 1e6),
                                                               (2, 2, 9, 5, 16, 8, 1e4), (6, 3, 40, 24, 64, 40, 1e4), (2, 1, 16, 16, 16, 0, 1.0),
                                                               (20, 4, 200, 200, 256, 16, 1e4), (1, 1, 300, 300, 300, 100, 1e4), (3, 3, 24, 24, 64, 8, 1e4)])
def test_prologue_rotation_norm_per_head_and_cache(dtype, halves, heads, kv, dim, vdim, width, dims, base):
    from mllm_b200 import ops
    from mllm_b200.layers.attention import rotation_frequencies

    T, S, eps, tied = 13, 40, 3e-3, vdim == dim
    nq, nk, nv = heads * dim, kv * dim, kv * vdim
    v_at = nq if tied else nq + nk
    row = _r(T, nq + nk + nv + 5, seed=1, std=1.5).to(dtype)
    pos = torch.tensor([0, 1, 2, 3, 63, 64, 65, 511, 4095, 20011, 20012, 77777, 131071])
    loc = torch.randperm(S, generator=torch.Generator().manual_seed(4))[:T]
    k_cache = torch.full((kv, S, width), 7.0, dtype=dtype, device=DEV).transpose(0, 1)
    v_cache = torch.full((kv, S, max(width, vdim)), 7.0, dtype=dtype, device=DEV).transpose(0, 1)
    q = torch.full((T, heads, width), 7.0, dtype=dtype, device=DEV)
    scaling = dict(factor=4.0, low=1.0, high=4.0, original=1000)
    ops.headnorm_rope_kv(row.to(DEV), rotation_frequencies(dims, base, scaling).to(DEV), pos.to(DEV), loc.to(DEV), q, k_cache, v_cache,
                         heads, kv, dim, vdim, v_at, halves, eps)
    rf, fr = oracle.f64(row), oracle.frequencies(dims, base, scaling)
    turn = oracle.turn_halves if halves else oracle.turn_neighbours
    wq, wk = rf[:, :nq].view(T, heads, dim), rf[:, nq:nq + nk].view(T, kv, dim)
    wq = oracle.unit_rms(torch.stack([turn(wq[t], int(pos[t]), fr) for t in range(T)]), eps)
    wk = oracle.unit_rms(torch.stack([turn(wk[t], int(pos[t]), fr) for t in range(T)]), eps)
    tol = _tol(dtype, 5e-3, 1e-6)                     # also at positions where an fp32 angle would be off by 1e-2
    _close(q[..., :dim], wq, tol)
    _close(k_cache[loc.to(DEV)][..., :dim], wk, tol)
    assert (q[..., dim:] == 0).all() and (k_cache[..., dim:] == 7.0).all() and (v_cache[..., vdim:] == 7.0).all()
    assert torch.equal(v_cache[loc.to(DEV)][..., :vdim].cpu(), row[:, v_at:v_at + nv].reshape(T, kv, vdim))
    rest = torch.ones(S, dtype=torch.bool)
    rest[loc] = False
    assert (k_cache[rest.to(DEV)] == 7.0).all() and (v_cache[rest.to(DEV)] == 7.0).all()
    ops.check_status()


# --------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot", [(64, 64, 16), (30, 36, 6), (1024, 512, 64), (11, 0, 8), (7, 5, 2)])
def test_latent_prologue_with_a_rotated_key_part(dtype, q_rank, kv_rank, rot):
    from mllm_b200 import ops
    from mllm_b200.layers.attention import rotation_frequencies

    T, S = 9, 40
    y = _r(T, q_rank + kv_rank + rot + 5, seed=1).to(dtype)
    qw, kw = 1 + _r(q_rank, seed=2, std=0.2), 1 + _r(max(kv_rank, 1), seed=3, std=0.2)
    pos = torch.tensor([0, 1, 63, 64, 511, 4095, 20011, 77777, 131071])
    loc = torch.randperm(S, generator=torch.Generator().manual_seed(4))[:T]
    cache = torch.full((S, kv_rank + rot + 3), 7.0, dtype=dtype, device=DEV)
    got, turns = ops.latent_prologue(y.to(DEV), qw.to(DEV), kw.to(DEV) if kv_rank else None, 3e-5, loc.to(DEV) if kv_rank else None,
                                     cache[:, : kv_rank + rot] if kv_rank else None, pos.to(DEV), rotation_frequencies(rot, 1e4).to(DEV))
    _close(got, oracle.rms_norm(oracle.f64(y[:, :q_rank]), oracle.f64(qw), 3e-5), _tol(dtype, 5e-3, 1e-6))
    fr = torch.tensor(oracle.frequencies(rot, 1e4), dtype=torch.float64)
    a = pos.double().unsqueeze(1) * fr
    _close(turns, torch.stack([torch.cos(a), torch.sin(a)], -1), 1e-6)
    if kv_rank:
        rows = cache[loc.to(DEV)]
        _close(rows[:, :kv_rank], oracle.rms_norm(oracle.f64(y[:, q_rank:q_rank + kv_rank]), oracle.f64(kw), 3e-5), _tol(dtype, 5e-3, 1e-6))
        kr = oracle.f64(y[:, q_rank + kv_rank:q_rank + kv_rank + rot])
        want = torch.cat([oracle.turn_neighbours(kr[t:t + 1], int(pos[t]), fr.tolist()) for t in range(T)])
        _close(rows[:, kv_rank:kv_rank + rot], want, _tol(dtype, 5e-3, 1e-6))
        rest = torch.ones(S, dtype=torch.bool)
        rest[loc] = False
        assert (cache[rest.to(DEV)] == 7.0).all() and (cache[:, kv_rank + rot:] == 7.0).all()


def _turns(T, rot, seed=9):
    a = _r(T, rot // 2, seed=seed, std=3.0)
    return torch.stack([torch.cos(a), torch.sin(a)], -1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,heads,n,k,rot", [(1, 16, 512, 128, 64), (8, 20, 64, 264, 8), (33, 3, 24, 40, 24), (70, 5, 130, 24, 16), (3, 2, 7, 9, 4),
                                                  (200, 4, 64, 48, 0), (5, 16, 128, 512, 0), (9, 3, 10, 32, 6)])
def test_head_products_with_turns_and_gates(dtype, tokens, heads, n, k, rot):
    """The features behind those that enter the product are turned; a logit per token and head gates the result."""
    from mllm_b200 import ops

    x, w = _r(tokens, heads, k + rot, seed=1).to(dtype), _r(heads, n, k, seed=2, std=k ** -0.5).to(dtype)
    wide = _r(tokens, heads + 11, seed=3, std=2.0).to(dtype)
    gate = wide[:, 3:3 + heads]
    want = torch.einsum("thk,hnk->thn", oracle.f64(x[..., :k]), oracle.f64(w))
    if rot:
        turns = _turns(tokens, rot)
        got = ops.head_linear(x.to(DEV), w.to(DEV), turns=turns.to(DEV))
        u, v, c, s = *(oracle.f64(x[..., k + i::2]) for i in (0, 1)), *(oracle.f64(turns[..., i]).unsqueeze(1) for i in (0, 1))
        turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
        _close(got[..., n:], turned, _tol(dtype, 5e-3, 1e-6))
        _close(got[..., :n], want, _tol(dtype, 1e-2))
        inplace = x.to(DEV)
        ops.turn_heads(inplace[..., k:], turns.to(DEV))
        _close(inplace[..., k:], turned, _tol(dtype, 5e-3, 1e-6))
        assert torch.equal(inplace[..., :k].cpu(), x[..., :k])
    g = oracle.sigmoid(oracle.f64(gate)).unsqueeze(-1)
    got = ops.head_linear(x.to(DEV)[..., :k], w.to(DEV), gate=wide.to(DEV)[:, 3:3 + heads])
    _close(got, want * g, _tol(dtype, 1e-2))
    got = ops.gate_heads(x.to(DEV)[..., :k], wide.to(DEV)[:, 3:3 + heads])
    assert got.is_contiguous()
    _close(got, oracle.f64(x[..., :k]) * g, _tol(dtype, 5e-3, 1e-6))


def _rows_case(lens, width, dtype, seed=0, std=1.0):
    """Contexts of several requests in scattered slots of one cache; every unused slot and every table entry past a
    request's end leads to a row that would dominate any softmax."""
    g = torch.Generator().manual_seed(seed)
    S = sum(lens) + 64
    slots = torch.randperm(S - 1, generator=g)[: sum(lens)] + 1
    cache = torch.full((S, -(-width // 8) * 8), 30.0, dtype=dtype)[:, :width]
    table = torch.zeros(len(lens) + 2, max(lens) + 40, dtype=torch.int32)
    req = torch.randperm(len(lens) + 2, generator=g)[: len(lens)].to(torch.int32)
    ctx, at = [], 0
    for r, n in zip(req, lens):
        c = (torch.randn(n, width, generator=g) * std).to(dtype)
        cache[slots[at:at + n]] = c
        table[int(r), :n] = slots[at:at + n].to(torch.int32)
        ctx.append(c)
        at += n
    wide = torch.full((S, -(-width // 8) * 8), 30.0, dtype=dtype, device=DEV)
    wide[:, :width] = cache.to(DEV)
    return wide[:, :width], table.to(DEV), req.to(DEV), ctx


SIZES = [(1, 8, 8), (3, 24, 16), (16, 128, 16), (17, 120, 24), (8, 200, 56), (20, 256, 32), (16, 512, 64), (20, 480, 96), (5, 576, 64), (2, 960, 64),
         (3, 36, 6), (2, 1000, 200), (1, 13, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot", SIZES)
def test_latent_rows_with_a_rotated_part(dtype, heads, rank, rot):
    """Keys are whole cache rows, values their first ``rank`` features."""
    from mllm_b200 import ops

    lens = (1, 31, 32, 33, 64, 65, 200, 700)
    cache, table, req, ctx = _rows_case(lens, rank + rot, dtype)
    owner = [b for b in range(len(lens)) for _ in range(2)]
    pos = [p for n in lens for p in (n - 1, n // 2)]
    q = _r(len(pos), heads, rank + rot, seed=6, std=(rank + rot) ** -0.5).to(dtype)
    q[..., rank:] *= 3.0                                      # the rotated part carries weight of its own
    got = ops.latent_attention(q.to(DEV), cache, table, req[torch.tensor(owner, device=DEV)], torch.tensor(pos).to(DEV), 0.9, None, max(lens), rank)
    want = torch.zeros(len(pos), heads, rank, dtype=torch.float64)
    for t, (b, p) in enumerate(zip(owner, pos)):
        c = oracle.f64(ctx[b][: p + 1])
        for h in range(heads):
            want[t, h] = oracle.softmax_with_sink((c @ oracle.f64(q[t, h])) * 0.9, None) @ c[:, :rank]
    assert got.shape[-1] == rank
    _close(got, want, _tol(dtype, 1.2e-2))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,rot", [(64, 16), (256, 32), (512, 64), (36, 6)])
@pytest.mark.parametrize("n", [1, 2, 32, 33, 257, 1500])
@pytest.mark.parametrize("by", ["latent", "rotated"])
def test_latent_rows_find_one_far_key(dtype, rank, rot, n, by):
    """One key stands out by far, by its latent or by its rotated part alone; the query must return that row's latent
    wherever it lies (first token, either side of a tile's edge, the query's own position), and the even stronger keys
    behind the query must not show."""
    from mllm_b200 import ops

    heads = 3
    places = sorted({p for p in (0, 1, 31, 32, 63, 64, n // 2, n - 2, n - 1) if 0 <= p < n})
    cache, table, req, _ = _rows_case([n + 8] * len(places), rank + rot, dtype, std=0.05)
    q = torch.zeros(len(places), heads, rank + rot, dtype=dtype)
    rows = []
    for b, p in enumerate(places):
        slots = table[int(req[b])]
        at = b % rank if by == "latent" else rank + b % rot
        cache[int(slots[p])] = 0.05
        cache[int(slots[p]), (b + 1) % rank] = 0.5            # tells the rows apart
        cache[int(slots[p]), at] = 4.0
        cache[slots[n: n + 8].long()] = 9.0
        q[b, :, at] = 8.0
        rows.append(oracle.f64(cache[int(slots[p]), :rank]).expand(heads, -1))
    got = ops.latent_attention(q.to(DEV), cache, table, req, torch.full((len(places),), n - 1).to(DEV), 1.0, None, n + 8, rank)
    _close(got, torch.stack(rows), 4e-3)


# --------------------------------------------------------------------------- mixtures
@pytest.mark.parametrize("experts,top,groups,keep,shared", [(5, 1, 1, 1, False), (16, 4, 4, 2, True), (64, 8, 8, 4, True), (256, 32, 32, 9, True),
                                                            (255, 3, 5, 2, True), (12, 3, 3, 1, False), (96, 6, 6, 3, True), (128, 8, 16, 4, True),
                                                            (12, 4, 12, 5, True), (40, 40, 1, 1, True), (33, 2, 3, 3, False)])
def test_router_within_groups(experts, top, groups, keep, shared):
    """Sigmoid scores, a correction that makes choice scores negative, groups, the factor, the shared expert's logit."""
    from mllm_b200.layers.moe import MoEGate

    top = min(top, 32)
    tokens, hidden = 60, 64
    with torch.device(DEV):
        gate = MoEGate(hidden, experts, top, False, torch.float32, choice_bias=True, sigmoid=True, groups=(groups, keep), scale=1.7, shared_gate=shared)
    w, corr = _r(experts + shared, hidden, seed=2, std=2 * hidden ** -0.5), _r(experts, seed=3, std=0.4) - 1.5
    gate.weight.data.copy_(w)
    gate.correction.data.copy_(corr)
    x = _r(tokens, hidden, seed=1)
    gw, gi, *logit = gate(x.to(DEV))
    changed = 0
    for t in range(tokens):
        logits = oracle.f64(w[:experts]) @ oracle.f64(x[t])
        chosen, weights = oracle.route(logits, oracle.f64(corr), top, groups, keep, 1.7)
        assert sorted(gi[t].tolist()) == sorted(chosen)
        got = dict(zip(gi[t].tolist(), gw[t].tolist()))
        assert all(abs(got[j] - s) < 1e-5 for j, s in zip(chosen, weights))
        changed += sorted(chosen) != sorted(oracle.route(logits, oracle.f64(corr), top, 1, 1, 1.7)[0])
    assert (changed > 0) == (keep < groups < experts)
    if shared:
        _close(logit[0][:, 0], oracle.f64(x) @ oracle.f64(w[experts]), 3e-6)


def test_router_refuses_groups_that_do_not_hold_the_choices():
    from mllm_b200 import ops

    x, w = torch.zeros(2, 16, device=DEV), torch.zeros(12, 16, device=DEV)
    for top, groups, keep in ((5, 4, 1), (2, 5, 2)):
        with pytest.raises(RuntimeError):
            ops.moe_route(x, w, top, False, None, 0.0, True, groups, keep)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,ff,experts,top,groups,shared", [(1, 64, 40, 6, 3, (3, 2), 24), (40, 90, 33, 5, 1, None, None), (9, 256, 128, 8, 4, (2, 1), 256),
                                                                       (300, 256, 256, 4, 2, None, 40), (150, 160, 72, 12, 6, (4, 3), 104)])
def test_mixture_through_the_norm_that_sums_it(dtype, tokens, width, ff, experts, top, groups, shared):
    """Routed experts and the gated shared expert, summed by the norm on their output."""
    from mllm_b200.layers import OutputRMSNorm
    from mllm_b200.models.lufizen import LufizenMoE
    from mllm_b200.models.places import mixture_places

    mlp = lm.moe(experts, top, ff, shared, groups, 1.3)
    cfg = lm.config([lm.attn(1, 1, 8, 0, mlp=mlp)], width, 64, embed=1.0)
    w = {k: v.to(dtype) for k, v in lm.weights(cfg, seed=3).items() if ".mlp." in k}
    with torch.device(DEV):
        m, norm = LufizenMoE(width, mlp, dtype, "x"), OutputRMSNorm(width, 1e-6, dtype)
    places = mixture_places("l0.mlp.", m.block, m.shared)
    assert set(places) == set(w)
    for n, t in w.items():
        places[n](t.to(DEV))
    m.block.process_weights_after_loading()
    if shared is not None:
        m.shared.gate_up_proj.quant_method.process_weights_after_loading(m.shared.gate_up_proj)
    h, x = _r(tokens, width, seed=4).to(dtype), _r(tokens, width, seed=5)
    gx = x.to(DEV)
    parts, sh = m(h.to(DEV))
    norm(gx, sh, parts)
    y = oracle.mixture_ff(oracle.f64(h), {k: oracle.f64(v) for k, v in w.items()}, "l0.mlp.", mlp)
    want = oracle.f64(x) + oracle.rms_norm(y, torch.ones(width).double(), 1e-6)
    _close(gx, want, _tol(dtype, 1.5e-2))


# --------------------------------------------------------------------------- whole models
LIMIT = {"float32": 5e-5, "bfloat16": 0.05}


def _within(err: torch.Tensor, dtype: str, where) -> None:
    """In 16 bits a row in fifty may stand out: a sublayer whose terms cancel, which the norm on its output blows up."""
    over = int((err > LIMIT[dtype]).sum())
    assert over <= (0 if dtype == "float32" else err.numel() // 50 + 1), (where, over, float(err.max()))
    assert err.max() <= LIMIT[dtype] * (1 if dtype == "float32" else 5), (where, int(err.argmax()), float(err.max()))


def _weights(cfg, dtype):
    """In 16 bits a close call between two experts may fall either way: there the corrections decide."""
    return lm.weights(cfg, steady=dtype == "bfloat16")


@pytest.fixture(scope="module")
def served(tmp_path_factory):
    from mllm_b200.trace_run import build_session

    cache = {}

    def get(name, dtype, page=1):
        if (name, dtype, page) not in cache:
            path = tmp_path_factory.mktemp(name) / "m"
            cfg = lm.CONFIGS[name]
            w = lm.write_checkpoint(path, cfg, _weights(cfg, dtype))
            cache[name, dtype, page] = (build_session(str(path), dtype, 1024, radix_cache_page_size=page), w, cfg)
        return cache[name, dtype, page]

    return get


@pytest.fixture(scope="module")
def expected():
    cache = {}

    def get(name, n, seed, dtype):
        if (name, n, seed, dtype) not in cache:
            cfg = lm.CONFIGS[name]
            seq = lm.tokens(cfg, n, seed=seed)
            cache[name, n, seed, dtype] = (seq, oracle.forward(cfg, _weights(cfg, dtype), seq))
        return cache[name, n, seed, dtype]

    return get


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name", sorted(lm.CONFIGS))
def test_portions_and_single_tokens_match_the_statement(served, expected, name, dtype):
    session, _, _ = served(name, dtype)
    seq, want = expected(name, 120, 1, dtype)
    for sizes in ([120], [1], [2], [64, 1, 1, 31, 2, 7]):
        _within(lm.logit_error(run_alone(session, seq, cut(len(seq), sizes)), want), dtype, sizes)
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name,page", [("mixed", 1), ("mixed", 16), ("large", 64), ("odd", 1), ("no_experts", 1), ("no_experts", 64), ("only_latent", 16)])
def test_batches_of_unequal_requests_with_reused_slots(served, expected, name, page, dtype):
    session, _, _ = served(name, dtype, page)
    lens = (90, 3, 120, 1, 65, 40, 33, 100)
    both = {f"r{i}": expected(name, n, 70 + i, dtype) for i, n in enumerate(lens)}
    cuts = {"r0": cut(90, [40, 1]), "r1": [2, 1], "r2": cut(120, [2, 1, 1]), "r3": [1], "r4": [64, 1], "r5": cut(40, [1]),
            "r6": [33], "r7": cut(100, [1, 63, 5])}
    for _ in range(2):
        got = run_together(session, {k: s for k, (s, _) in both.items()}, cuts, {f"r{i}": i for i in range(8)})
        for k, (_, want) in both.items():
            _within(lm.logit_error(got[k], want), dtype, k)


@pytest.mark.parametrize("dtype,scale,gain,limit", [("float32", 0.8, 6.0, 2e-4), ("bfloat16", 0.2, 1.5, 0.2)])
def test_far_keys_are_found_in_every_schedule(tmp_path, dtype, scale, gain, limit):
    """Peaked scores over 400 tokens: a lost, shifted or foreign key changes whole rows."""
    from mllm_b200.trace_run import build_session

    cfg = json.loads(json.dumps(lm.CONFIGS["no_experts"]))
    for layer in cfg["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["scale"] = scale
    w = lm.write_checkpoint(tmp_path / "m", cfg, lm.pointed_weights(cfg, gain))
    seq = lm.tokens(cfg, 400, seed=3)
    want = oracle.forward(cfg, w, seq)
    for page in (1, 16, 64):
        session = build_session(str(tmp_path / "m"), dtype, 832, radix_cache_page_size=page)
        for sizes in ([400], [64] * 6 + [1] * 16, [63, 2, 63, 128, 100, 3, 41], [15, 17, 2, 30, 190, 2, 2, 2, 140]):
            err = lm.logit_error(run_alone(session, seq, cut(400, sizes)), want)
            assert err.max() < limit, (page, sizes, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("dtype", sorted(LIMIT))
def test_long_decoding_through_captured_graphs(served, expected, dtype):
    session, _, _ = served("no_experts", dtype)
    graphs = session.mrp.runner.cuda_graph_runner
    before = graphs.replays
    seq, want = expected("no_experts", 300, 5, dtype)
    assert lm.logit_error(run_alone(session, seq, [5] + [1] * 295), want).max() < LIMIT[dtype]
    assert graphs.replays == before + 295


def test_residual_stream_after_every_layer(served):
    session, w, cfg = served("large", "float32")
    seq, want, got = lm.tokens(cfg, 40), [], []
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
    cfg = lm.CONFIGS["mixed"]
    w = lm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [lm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9, 60)]
    want = [_greedy(cfg, w, p, 8) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 8, DEV, max_running_requests=3, chunked_prefill_size=24, mem_fraction_static=0.2)
    assert got == [ids for ids, _ in want]


def test_replay_program(tmp_path):
    """bin/trace_run as a user starts it: files of logits, one line per step."""
    cfg = lm.CONFIGS["mixed"]
    w = lm.write_checkpoint(tmp_path / "m", cfg)
    seq = lm.tokens(cfg, 12)
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
        assert lm.logit_error(got, want[rows]).max() < LIMIT["float32"]
