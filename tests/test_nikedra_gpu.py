"""Nikedra on the GPU: every mechanism's kernels against the plain statement, then whole models through the serving path
in all the ways a sequence can be fed."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import nikedra_models as nm
import nikedra_oracle as oracle
from session_schedules import cut, run_alone, run_together
from test_nikedra_cpu import _generate, _greedy

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.bfloat16, torch.float32]
HALVES = [torch.bfloat16, torch.float16]


def _r(*shape, seed=0, std=1.0, dtype=torch.float32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype)


def _tol(dtype, half, single=2e-5):
    return half if dtype != torch.float32 else single


def _close(got, want, tol):
    scale = want.abs().max().item()
    err = (got.double().cpu() - want).abs().max().item()
    assert err <= tol * max(scale, 1e-3), (err, scale)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# --------------------------------------------------------------------------- between the layers
@pytest.mark.parametrize("dtype", DTYPES + [torch.float16])
@pytest.mark.parametrize("shape", [(1, 64), (5, 90), (37, 33), (300, 2048), (3, 8192), (2, 16384)])
@pytest.mark.parametrize("two,ff,n,last", [(False, "dense", 1, False), (True, "experts", 3, False), (True, "dense", 6, True), (False, None, 2, False),
                                           (False, "experts", 0, False)])
def test_step_between_layers(dtype, shape, two, ff, n, last):
    """Sum of the sublayers, norms of two mixer outputs, sum of experts, average over depth, normed inputs."""
    from mllm_b200 import ops

    (T, W), eps = shape, 3e-3
    x, res = _r(T, W, seed=1, std=20), _r(n + 1, T, W, seed=2, std=5)
    a, b = _r(T, W, seed=3).to(dtype), _r(T, W, seed=4, std=0.1).to(dtype)
    aw, bw, dwa = 1 + _r(W, seed=5, std=0.3), _r(W, seed=6), _r(n + 1, seed=7)
    g = [torch.tensor(0.8), torch.tensor(-1.3)]
    mix = (a, b, aw, bw) if two else (a,)
    y = 0.5 * (oracle.unit_rms(oracle.f64(a), eps) * oracle.f64(aw) + oracle.unit_rms(oracle.f64(b), eps) * oracle.f64(bw)) if two else oracle.f64(a)
    f = experts = None
    if ff == "dense":
        f = _r(T, W, seed=8).to(dtype)
        y = y + oracle.f64(f)
    elif ff == "experts":
        rows, pos = _r(3 * T, W, seed=9).to(dtype), torch.randperm(3 * T, generator=torch.Generator().manual_seed(3)).to(torch.int32)
        pos[0] = -1                                      # a choice without a row
        y = y + torch.stack([oracle.f64(rows)[pos.long()[3 * t: 3 * t + 3]][(pos[3 * t: 3 * t + 3] >= 0)].sum(0) for t in range(T)])
        experts = ops.ExpertRows(rows.to(DEV), pos.to(DEV), None, torch.zeros(T, 3, dtype=torch.int32, device=DEV), rows[:T].to(DEV))
    z = oracle.f64(x) + y
    want = z if n == 0 else oracle.depth_average(oracle.f64(dwa), [*oracle.f64(res[:n]), z])
    gx, gres = x.to(DEV), None if n == 0 else res.to(DEV)
    h = ops.depth_step(gx, [t.to(DEV) for t in mix], None if f is None else f.to(DEV), experts, gres, n, None if n == 0 else dwa.to(DEV),
                       [t.to(DEV) for t in g[: 1 if last else 2]], eps, dtype, None if last else gx, keep=not last)
    assert len(h) == (1 if last else 2)
    for t, w in zip(h, g):
        _close(t, oracle.unit_rms(want, eps) * float(w), _tol(dtype, 5e-3, 2e-6))
    if last:
        assert torch.equal(gx.cpu(), x)
        assert n == 0 or torch.equal(gres[n].cpu(), res[n])
    else:
        _close(gx, want, 2e-6)                            # the stream stays in 32-bit
        if n:
            _close(gres[n], z, 2e-6)
    if n:
        assert torch.equal(gres[:n].cpu(), res[:n])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps", [(64, 4), (90, 1), (33, 2), (2048, 4), (128, 3), (256, 16)])
def test_embedding_norm_and_convolution_of_single_tokens(dtype, width, taps):
    """Requests in scattered state rows, token by token, against the whole sequences; other rows stay as they are."""
    from mllm_b200 import ops

    V, n, eps, slots = 50, 6, 1e-3, [4, 0, 2]
    table, w, norms = _r(V, width, seed=1).to(dtype), torch.tensor(1.7), [torch.tensor(0.6), torch.tensor(1.2)]
    cw = _r(width, taps, seed=2, std=0.5).to(dtype)
    ids = torch.randint(0, V, (n, 3), generator=torch.Generator().manual_seed(5))
    state = torch.full((6, width, taps - 1), 7.0, dtype=dtype, device=DEV)
    state[slots] = 0.0
    x0 = oracle.unit_rms(oracle.f64(table)[ids], eps) * 1.7                          # [n, 3, W]
    h0 = [oracle.unit_rms(x0, eps) * float(g) for g in norms]
    want = torch.stack([h0[0][:, b] + oracle.causal_conv(oracle.f64(h0[0][:, b].to(dtype)), oracle.f64(cw)) for b in range(3)], 1)
    for t in range(n):
        x = torch.empty(3, width, device=DEV)
        h = ops.embed_norm(ids[t].to(DEV), table.to(DEV), w.to(DEV), x, eps, [g.to(DEV) for g in norms],
                           ops.ConvStep(cw.to(DEV), state, _i32(slots)))
        _close(x, x0[t], 1e-6)
        _close(h[0], want[t], _tol(dtype, 1e-2, 3e-6))
        _close(h[1], h0[1][t], _tol(dtype, 5e-3, 2e-6))
    assert (state[[1, 3, 5]] == 7.0).all()
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps,mode", [(64, 4, "add"), (90, 3, "add"), (33, 2, "bias"), (256, 4, "bias"), (48, 1, "add"), (40, 1, "bias"), (128, 16, "bias")])
def test_convolutions_in_portions(dtype, channels, taps, mode):
    """A bias in front of the SiLU, or the input added instead of it; three requests of unequal portions."""
    from mllm_b200 import ops

    lens, slots = [75, 20, 41], [3, 0, 2]
    x, w = [_r(n, channels, seed=i).to(dtype) for i, n in enumerate(lens)], _r(channels, taps, seed=9, std=0.6).to(dtype)
    bias = _r(channels, seed=8).to(dtype) if mode == "bias" else None
    state = torch.full((5, channels, taps - 1), 7.0, dtype=dtype, device=DEV)
    at, got = [0, 0, 0], [[], [], []]
    for sizes in ([1, 2, 3], [70, 1, 2], [2, 15, 0], [2, 2, 36]):
        part = [t[a: a + n] for t, a, n in zip(x, at, sizes)]
        wide = torch.cat([torch.cat(part), torch.full((sum(sizes), 8), 9.0, dtype=dtype)], 1).to(DEV)       # columns of a wider matrix
        y = ops.causal_conv1d_silu(wide[:, :channels], w.to(DEV), state, _i32(slots), _i32(sizes), _i32([int(a > 0) for a in at]),
                                   bias=None if bias is None else bias.to(DEV), add_input=mode == "add")
        for i, p in enumerate(torch.split(y, sizes)):
            got[i].append(p)
            at[i] += sizes[i]
    for i in range(3):
        xf = oracle.f64(x[i])
        c = oracle.causal_conv(xf, oracle.f64(w), None if bias is None else oracle.f64(bias))
        _close(torch.cat(got[i]), xf + c if mode == "add" else oracle.silu(c), _tol(dtype, 1e-2, 3e-6))
    assert (state[[1, 4]] == 7.0).all()


# --------------------------------------------------------------------------- recurrences
def _portions(lens, sizes):
    """Portions of every request: lists of equal length, zero where a request has no more."""
    cuts = [cut(n, sizes[i:] + sizes[:i]) for i, n in enumerate(lens)]
    return [[c[k] if k < len(c) else 0 for c in cuts] for k in range(max(map(len, cuts)))]


def _feed(parts, lens, sizes, fn):
    """Feeds requests portion by portion; fn(rows of every operand, lens, has) -> output rows; the outputs per request."""
    at, got = [0] * len(lens), [[] for _ in lens]
    for step in _portions(lens, sizes):
        on = [i for i, n in enumerate(step) if n]
        rows = [torch.cat([p[i][at[i]: at[i] + step[i]] for i in on]) for p in parts]
        y = fn(rows, on, [step[i] for i in on], [int(at[i] > 0) for i in on])
        for i, t in zip(on, torch.split(y, [step[i] for i in on])):
            got[i].append(t)
            at[i] += step[i]
    return [torch.cat(g) for g in got]


@pytest.mark.parametrize("dtype", HALVES + [torch.float32])
@pytest.mark.parametrize("heads,kv,dk,dv", [(2, 1, 32, 32), (4, 4, 24, 40), (2, 2, 128, 128), (3, 1, 64, 16), (2, 1, 8, 8), (1, 1, 13, 7), (2, 1, 136, 24), (2, 2, 128, 72)])
def test_delta_rule_with_decays_per_channel(dtype, heads, kv, dk, dv):
    """Chunks and single tokens in any order of portions, decays from hardly any to e^-40 a token, rows of wider matrices; the
    state is exact to fp32's means in every mode."""
    from mllm_b200 import ops

    lens, slots = [150, 33, 70], [4, 1, 3]
    q, k = ([_r(n, kv * dk, seed=10 + i, std=s).to(dtype) for i, n in enumerate(lens)] for s in (1.0, 0.7))
    v = [_r(n, heads * dv, seed=20 + i).to(dtype) for i, n in enumerate(lens)]
    b = [_r(n, heads, seed=30 + i, std=2).to(dtype) for i, n in enumerate(lens)]
    a = [_r(n, heads * dk, seed=40 + i, std=2).to(dtype) for i, n in enumerate(lens)]
    a_log, dt = _r(heads, seed=5, std=1.0) - 0.5, _r(heads * dk, seed=6, std=2.5) - 2.0
    dt[::5] = 10.0                                     # channels that forget everything at once
    want = []
    for i, n in enumerate(lens):
        g = (-torch.exp(oracle.f64(a_log)).view(1, heads, 1) * oracle.softplus(oracle.f64(a[i]) + oracle.f64(dt)).view(n, heads, dk))
        beta = oracle.sigmoid(oracle.f64(b[i]))
        qi, ki, vi = oracle.f64(q[i]).view(n, kv, dk), oracle.f64(k[i]).view(n, kv, dk), oracle.f64(v[i]).view(n, heads, dv)
        want.append(torch.stack([oracle.channel_delta_rule(qi[:, h // (heads // kv)], ki[:, h // (heads // kv)], vi[:, h], g[:, :, :][:, h], beta[:, h])
                                 for h in range(heads)], 1))
    last = None
    for sizes in ([200], [33, 1, 2, 64], [1], [16, 17, 15, 2]):
        state = torch.full((6, heads, dk, dv), 7.0, device=DEV)

        def run(rows, on, ln, has):
            qr, kr, vr, br, ar = (torch.cat([t, t[:, :8]], 1).to(DEV)[:, : t.shape[1]] for t in rows)
            return ops.channel_delta_rule(qr.unflatten(1, (kv, dk)), kr.unflatten(1, (kv, dk)), vr.unflatten(1, (heads, dv)), br, ar, a_log.to(DEV),
                                          dt.to(DEV), state, _i32([slots[i] for i in on]), _i32(ln), _i32(has), max_len=max(ln))

        got = _feed((q, k, v, b, a), lens, sizes, run)
        for y, w in zip(got, want):
            _close(y, w, _tol(dtype, 8e-3))
        assert (state[[0, 2, 5]] == 7.0).all()
        if last is not None:
            _close(state[slots], last, 2e-5)            # the same state through either kernel
        last = oracle.f64(state[slots])
    ops.check_status()


def test_delta_rule_loops_over_spans_of_its_workspace():
    """A run longer than the workspace holds, against the token-sequential kernel."""
    from mllm_b200 import ops

    heads, d, lens = 16, 128, [1500, 700, 37, 1200, 64, 900, 8, 33]
    T, B = sum(lens), len(lens)
    q, k, v, a = (_r(T, heads * d, seed=i).to(torch.bfloat16).to(DEV) for i in range(4))
    b, a_log, dt = _r(T, heads, seed=5).to(torch.bfloat16).to(DEV), (_r(heads, seed=6) - 2).to(DEV), _r(heads * d, seed=7).to(DEV)
    outs, states = [], []
    for name in ("cuda_chunkwise", "mllm_kernel"):
        state = torch.zeros(B, heads, d, d, device=DEV)
        ops.set_gdn_extend_backend(name)
        try:
            outs.append(ops.channel_delta_rule(*(t.unflatten(1, (heads, d)) for t in (q, k, v)), b, a, a_log, dt, state, _i32(list(range(B))),
                                               _i32(lens), _i32([0] * B), max_len=max(lens)))
        finally:
            ops.set_gdn_extend_backend("auto")
        states.append(state)
    _close(outs[0], oracle.f64(outs[1]), 1e-2)
    _close(states[0], oracle.f64(states[1]), 2e-5)


@pytest.mark.parametrize("dtype", HALVES + [torch.float32])
@pytest.mark.parametrize("heads,groups,n_state,p", [(4, 1, 32, 16), (6, 2, 24, 40), (2, 2, 128, 64), (4, 4, 64, 64), (3, 1, 13, 7), (2, 1, 200, 24), (2, 1, 48, 72)])
def test_state_space_rule(dtype, heads, groups, n_state, p):
    """Chunks and single tokens in any order of portions; step sizes from almost none to ones that forget the past."""
    from mllm_b200 import ops

    lens, slots = [150, 33, 70], [4, 1, 3]
    x = [_r(n, heads * p, seed=10 + i).to(dtype) for i, n in enumerate(lens)]
    B, C = ([_r(n, groups * n_state, seed=s + i, std=0.5).to(dtype) for i, n in enumerate(lens)] for s in (20, 30))
    dt = [_r(n, heads, seed=40 + i, std=2).to(dtype) for i, n in enumerate(lens)]
    bias, a_log, skip = _r(heads, seed=5) - 1, _r(heads, seed=6), _r(heads, seed=7)
    a_log[0] = 3.0
    want = []
    for i, n in enumerate(lens):
        step = oracle.softplus(oracle.f64(dt[i]) + oracle.f64(bias))
        xi, Bi, Ci = oracle.f64(x[i]).view(n, heads, p), oracle.f64(B[i]).view(n, groups, -1), oracle.f64(C[i]).view(n, groups, -1)
        want.append(torch.stack([oracle.state_space_rule(xi[:, h], Bi[:, h // (heads // groups)], Ci[:, h // (heads // groups)], step[:, h],
                                                         float(a_log[h]), float(skip[h])) for h in range(heads)], 1))
    last = None
    for sizes in ([200], [33, 1, 2, 64], [1], [64, 65, 63, 2]):
        state = torch.full((6, heads, n_state, p), 7.0, device=DEV)

        def run(rows, on, ln, has):
            wide = torch.cat([rows[0], rows[1], rows[2]], 1).to(DEV)              # one matrix, as the convolution leaves it
            parts = torch.split(wide, [t.shape[1] for t in rows[:3]], 1)
            return ops.state_space(parts[0].unflatten(1, (heads, p)), parts[1].unflatten(1, (groups, n_state)), parts[2].unflatten(1, (groups, n_state)),
                                   rows[3].to(DEV), bias.to(DEV), a_log.to(DEV), skip.to(DEV), state, _i32([slots[i] for i in on]), _i32(ln), _i32(has),
                                   max_len=max(ln))

        got = _feed((x, B, C, dt), lens, sizes, run)
        for y, w in zip(got, want):
            _close(y, w, _tol(dtype, 1e-2))
        assert (state[[0, 2, 5]] == 7.0).all()
        if last is not None:
            _close(state[slots], last, 2e-5)
        last = oracle.f64(state[slots])
    ops.check_status()


def test_state_space_segments():
    """Few long requests run as segments side by side; against the token-sequential kernel, from a state."""
    from mllm_b200 import ops

    heads, n_state, p, lens = 4, 64, 64, [2500, 300]
    T = sum(lens)
    x, B, C = _r(T, heads * p, seed=1).to(torch.bfloat16), _r(T, n_state, seed=2, std=0.4).to(torch.bfloat16), _r(T, n_state, seed=3, std=0.4).to(torch.bfloat16)
    dt, bias, a_log, skip = _r(T, heads, seed=4).to(torch.bfloat16), _r(heads, seed=5) - 4, _r(heads, seed=6) - 1, _r(heads, seed=7)
    outs, states = [], []
    for name in ("cuda_chunkwise", "mllm_kernel"):
        state = _r(2, heads, n_state, p, seed=8).to(DEV)
        ops.set_gdn_extend_backend(name)
        try:
            outs.append(ops.state_space(x.to(DEV).unflatten(1, (heads, p)), B.to(DEV).unsqueeze(1), C.to(DEV).unsqueeze(1), dt.to(DEV), bias.to(DEV),
                                        a_log.to(DEV), skip.to(DEV), state, _i32([0, 1]), _i32(lens), _i32([1, 1]), max_len=max(lens)))
        finally:
            ops.set_gdn_extend_backend("auto")
        states.append(state)
    _close(outs[0], oracle.f64(outs[1]), 1e-2)
    _close(states[0], oracle.f64(states[1]), 2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,groups", [(1, 64, 1), (37, 90, 3), (5, 4096, 1), (300, 2048, 8), (3, 33, 1), (2, 16384, 1), (9, 40, 5)])
def test_gate_before_the_norm(dtype, rows, width, groups):
    from mllm_b200 import ops

    x, wide, w = _r(rows, width, seed=1).to(dtype), _r(rows, width + 24, seed=2, std=2).to(dtype), 1 + _r(width, seed=3, std=0.2)
    out = torch.full((rows, width + 8), 7.0, dtype=dtype, device=DEV)
    ops.gated_rmsnorm(x.to(DEV), wide.to(DEV)[:, 8: 8 + width], w.to(DEV), groups, 1e-3, out[:, :width])
    z = (oracle.f64(x) * oracle.silu(oracle.f64(wide[:, 8: 8 + width]))).view(rows, groups, -1)
    _close(out[:, :width], oracle.unit_rms(z, 1e-3).view(rows, width) * oracle.f64(w), _tol(dtype, 1e-2, 3e-6))
    assert (out[:, width:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,heads,dv", [(1, 4, 32), (30, 3, 7), (300, 16, 128)])
def test_norm_per_head_with_a_sigmoid_gate(dtype, tokens, heads, dv):
    from mllm_b200 import ops

    x, gate, w = _r(tokens, heads * dv, seed=1).to(dtype), _r(tokens, heads * dv + 8, seed=2, std=2).to(dtype), (1 + _r(dv, seed=3, std=0.2)).to(dtype)
    got = ops.rmsnorm_gated(x.to(DEV), gate.to(DEV)[:, 8:], w.to(DEV), 1e-3, round_norm=False, sigmoid=True)
    want = oracle.unit_rms(oracle.f64(x).view(tokens, heads, dv), 1e-3) * oracle.f64(w)
    _close(got, want.view(tokens, -1) * oracle.sigmoid(oracle.f64(gate[:, 8:])), _tol(dtype, 1e-2, 3e-6))


# --------------------------------------------------------------------------- attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,width,dims,base", [(4, 2, 64, 64, 128, 64, 1e4), (3, 1, 10, 7, 10, 6, 5e5), (8, 2, 128, 128, 128, 32, 1e6),
                                                               (6, 3, 40, 24, 64, 40, 1e4), (2, 1, 16, 16, 16, 0, 1.0), (20, 4, 200, 200, 256, 16, 1e4)])
def test_rotation_with_a_magnitude_and_no_norm(dtype, heads, kv, dim, vdim, width, dims, base):
    from mllm_b200 import ops
    from mllm_b200.layers.attention import rotation_frequencies, rotation_magnitude

    T, S = 13, 40
    nq, nk, nv = heads * dim, kv * dim, kv * vdim
    row = _r(T, nq + nk + nv + 5, seed=1, std=1.5).to(dtype)
    pos = torch.tensor([0, 1, 2, 3, 63, 64, 65, 511, 4095, 20011, 20012, 77777, 131071])
    loc = torch.randperm(S, generator=torch.Generator().manual_seed(4))[:T]
    k_cache = torch.full((kv, S, width), 7.0, dtype=dtype, device=DEV).transpose(0, 1)
    v_cache = torch.full((kv, S, max(width, vdim)), 7.0, dtype=dtype, device=DEV).transpose(0, 1)
    q = torch.full((T, heads, width), 7.0, dtype=dtype, device=DEV)
    scaling = dict(factor=4.0, original=1000, fast=20.0, slow=1.0)
    mag = rotation_magnitude(scaling)
    assert mag > 1.1
    ops.headnorm_rope_kv(row.to(DEV), rotation_frequencies(dims, base, scaling if dims else None).to(DEV), pos.to(DEV), loc.to(DEV), q, k_cache, v_cache,
                         heads, kv, dim, vdim, nq + nk, True, 0.0, norm=False, magnitude=mag)
    rf, fr = oracle.f64(row), oracle.frequencies(dims, base, scaling) if dims else []

    def turned(t, n):
        t = t.view(T, n, dim)
        out = t.clone()
        for i in range(T):                               # the statement's rotation puts row i at position i: one row at a time
            for j, f in enumerate(fr):
                c, s = np.cos(int(pos[i]) * f) * mag, np.sin(int(pos[i]) * f) * mag
                out[i, :, j], out[i, :, j + len(fr)] = t[i, :, j] * c - t[i, :, j + len(fr)] * s, t[i, :, j + len(fr)] * c + t[i, :, j] * s
        return out

    tol = _tol(dtype, 5e-3, 1e-6)
    _close(q[..., :dim], turned(rf[:, :nq], heads), tol)
    _close(k_cache[loc.to(DEV)][..., :dim], turned(rf[:, nq:nq + nk], kv), tol)
    assert torch.equal(v_cache[loc.to(DEV)][..., :vdim].cpu(), row[:, nq + nk: nq + nk + nv].reshape(T, kv, vdim))
    assert (q[..., dim:] == 0).all() and (k_cache[..., dim:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,heads,kv", [(64, 4, 2), (128, 8, 2), (256, 2, 1), (128, 40, 1)])
@pytest.mark.parametrize("chunk", [1, 7, 64, 100, 128, 300])
def test_keys_at_the_edges_of_chunks(dtype, dim, heads, kv, chunk):
    """One key stands out by far.  A query finds it from every place of its chunk and from none outside, in prompts, in
    portions of prompts and in decoding."""
    from mllm_b200 import ops

    S, T = 700, 640
    g = torch.Generator().manual_seed(chunk)
    slots = (torch.randperm(S - 1, generator=g)[:T] + 1).to(torch.int32)
    table = torch.zeros(3, T + 8, dtype=torch.int32)
    table[1, :T] = slots
    k = (torch.randn(T, kv, dim, generator=g) * 0.02).to(dtype)
    v = torch.randn(T, kv, dim, generator=g).to(dtype)
    marks = sorted({m for e in range(0, T, max(chunk, 97)) for m in (e // chunk * chunk - 1, e // chunk * chunk) if 0 <= m < T})
    k[marks] = torch.full((dim,), 1.0).to(dtype)
    kc, vc = (torch.full((kv, S, dim), 30.0, dtype=dtype).transpose(0, 1) for _ in range(2))
    kc[slots.long()], vc[slots.long()] = k, v
    q = torch.ones(T, heads, dim).to(dtype)
    scale = 14.0 / dim
    want = oracle.attention(oracle.f64(q[:, :1]), oracle.f64(k[:, :1]), oracle.f64(v[:, :1]), scale, lambda i: i // chunk * chunk)
    # heads of a group are alike; the other key heads follow
    full = [want] + [oracle.attention(oracle.f64(q[:, :1]), oracle.f64(k[:, c: c + 1]), oracle.f64(v[:, c: c + 1]), scale, lambda i: i // chunk * chunk)
                     for c in range(1, kv)]
    want = torch.cat([f.expand(-1, heads // kv, -1) for f in full], 1)
    kc, vc, tb, qd = kc.to(DEV), vc.to(DEV), table.to(DEV), q.to(DEV)
    kc, vc = (t.transpose(0, 1).contiguous().transpose(0, 1) for t in (kc, vc))
    if dtype == torch.float32:
        out = torch.empty_like(qd)
        ops.attention_rows(qd, kc, vc, tb, _i32([1] * T), torch.arange(T, device=DEV), scale, out, chunk=chunk)
        _close(out, want, 1e-5)
        return
    for start in (0, 1, 63, 130, 601):
        out = torch.empty_like(qd[start:])
        ops.attention_prefill(qd[start:].contiguous(), kc, vc, tb, _i32([1]), _i32([T]), _i32([start]), _i32([0]), scale, out=out, max_q_len=T - start,
                              chunk=chunk)
        _close(out, want[start:], 1.5e-2)
    for i in sorted({0, 1, T - 1, *(m + o for m in marks for o in (0, 1, chunk - 1, chunk) if m + o < T)})[:24]:
        out = ops.attention_decode(qd[i: i + 1].contiguous(), kc, vc, tb, _i32([1]), _i32([i + 1]), scale, max_seq_len=T, chunk=chunk)
        _close(out, want[i: i + 1], 1.5e-2)
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,rot", [(64, 16), (256, 32), (512, 64), (36, 6)])
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 100, 600])
def test_latent_rows_at_the_edges_of_a_window(dtype, rank, rot, window):
    """One cached row stands out by far, just inside and just outside the window of the query."""
    from mllm_b200 import ops

    heads, n = 3, 500
    places = sorted({p for p in (n - 1, n - window - 1, n - window, n - window + 1, n - 2, 0) if 0 <= p < n})
    S, width = len(places) * (n + 8) + 8, rank + rot
    g = torch.Generator().manual_seed(window)
    slots = (torch.randperm(S - 1, generator=g) + 1)[: len(places) * (n + 8)].view(len(places), -1)
    cache = torch.full((S, -(-width // 8) * 8), 30.0, dtype=dtype)
    cache[slots.view(-1), :width] = (torch.randn(slots.numel(), width, generator=g) * 0.05).to(dtype)
    q = torch.zeros(len(places), heads, width, dtype=dtype)
    q[..., 0] = 8.0
    want = torch.zeros(len(places), heads, rank, dtype=torch.float64)
    for b, p in enumerate(places):
        cache[slots[b, p], 0] = 4.0
        cache[slots[b, n:], 0] = 9.0                      # behind the query
        c = oracle.f64(cache[slots[b, max(0, n - window): n], :width])
        want[b] = torch.softmax(c @ oracle.f64(q[b, 0]), 0) @ c[:, :rank]
    dev = cache.to(DEV)[:, :width]
    table = torch.zeros(len(places), n + 8, dtype=torch.int32)
    table[:, :] = slots.to(torch.int32)
    got = ops.latent_attention(q.to(DEV), dev, table.to(DEV), _i32(list(range(len(places)))), torch.full((len(places),), n - 1).to(DEV), 1.0, None, n + 8, rank,
                               window)
    _close(got, want, _tol(dtype, 1.2e-2))
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,heads,n,k,rot", [(1, 16, 512, 128, 64), (8, 20, 64, 264, 8), (33, 3, 24, 40, 24), (70, 5, 130, 24, 16), (3, 2, 7, 9, 4), (5, 16, 128, 512, 0)])
def test_head_products_with_turned_halves_and_gates_per_feature(dtype, tokens, heads, n, k, rot):
    from mllm_b200 import ops

    x, w = _r(tokens, heads, k + rot, seed=1).to(dtype), _r(heads, n, k, seed=2, std=k ** -0.5).to(dtype)
    wide = _r(tokens, heads * n + 16, seed=3, std=2.0).to(dtype)
    want = torch.einsum("thk,hnk->thn", oracle.f64(x[..., :k]), oracle.f64(w))
    if rot:
        ang = _r(tokens, rot // 2, seed=9, std=3.0)
        turns = torch.stack([torch.cos(ang), torch.sin(ang)], -1)
        got = ops.head_linear(x.to(DEV), w.to(DEV), turns=turns.to(DEV), halves=True)
        u, v = oracle.f64(x[..., k:]).chunk(2, -1)
        c, s = (oracle.f64(turns[..., i]).unsqueeze(1) for i in (0, 1))
        turned = torch.cat([u * c - v * s, v * c + u * s], -1)
        _close(got[..., n:], turned, _tol(dtype, 5e-3, 1e-6))
        _close(got[..., :n], want, _tol(dtype, 1e-2))
        inplace = x.to(DEV)
        ops.turn_heads(inplace[..., k:], turns.to(DEV), halves=True)
        _close(inplace[..., k:], turned, _tol(dtype, 5e-3, 1e-6))
    gate = oracle.sigmoid(oracle.f64(wide[:, 8: 8 + heads * n])).view(tokens, heads, n)
    got = ops.head_linear(x.to(DEV)[..., :k], w.to(DEV), gate=wide.to(DEV)[:, 8: 8 + heads * n])
    _close(got, want * gate, _tol(dtype, 1e-2))
    y = _r(tokens, heads, n + 8, seed=4).to(dtype)
    got = ops.gate_heads(y.to(DEV)[..., :n], wide.to(DEV)[:, 8: 8 + heads * n])
    assert got.is_contiguous()
    _close(got, oracle.f64(y[..., :n]) * gate, _tol(dtype, 5e-3, 1e-6))
    inplace = y.to(DEV)
    ops.gate_heads(inplace[..., :n], wide.to(DEV)[:, :heads], out=inplace[..., :n])            # one per head, in place
    _close(inplace[..., :n], oracle.f64(y[..., :n]) * oracle.sigmoid(oracle.f64(wide[:, :heads])).unsqueeze(-1), _tol(dtype, 5e-3, 1e-6))
    assert torch.equal(inplace[..., n:].cpu(), y[..., n:])


# --------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 40), (128, 256), (90, 33), (256, 384), (512, 128), (2048, 512)])
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 33, 200, 257, 900])
def test_bounded_feed_forward(dtype, width, ff, rows):
    """Biases and bounds in every tiling of the product; half of the values lie outside the bounds."""
    from mllm_b200.layers import MLP
    from mllm_b200.models.places import put

    limit, cfg = 0.6, dict(nm.dense(ff))
    w = {k: v.to(dtype) for k, v in nm.weights(nm.config([nm.delta(1, 1, 8, 8, mlp=cfg)], width, 64), seed=rows).items() if ".mlp." in k}
    with torch.device(DEV):
        m = MLP(width, ff, None, "x", dtype, reduce_results=True, activation="clamped", bias=True, limit=limit)
    gu, down = m.gate_up_proj, m.down_proj
    for j, n in enumerate(("gate", "up")):
        gu.weight.weight_loader(gu.weight, w[f"l0.mlp.{n}"].to(DEV), j)
        gu.bias.weight_loader(gu.bias, w[f"l0.mlp.{n}.b"].to(DEV), j)
    put(down.weight)(w["l0.mlp.down"].to(DEV))
    put(down.bias)(w["l0.mlp.down.b"].to(DEV))
    gu.quant_method.process_weights_after_loading(gu)
    x = _r(rows, width, seed=2).to(dtype)
    want = oracle.clamped_ff(oracle.f64(x), {k: oracle.f64(v) for k, v in w.items()}, "l0.mlp.", limit)
    _close(m(x.to(DEV)), want, _tol(dtype, 1.5e-2))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,ff,experts,top", [(1, 64, 40, 6, 3), (40, 90, 33, 5, 1), (9, 256, 128, 8, 2), (300, 256, 256, 4, 2), (150, 160, 72, 12, 12)])
def test_experts_that_read_weighted_inputs(dtype, tokens, width, ff, experts, top):
    """No gate, the exact GELU, weights on the inputs; the step behind the layer sums the rows."""
    from mllm_b200 import ops
    from mllm_b200.layers.moe import SparseMoeBlock
    from mllm_b200.models.places import mixture_places

    cfg = nm.config([nm.delta(1, 1, 8, 8, mlp=nm.moe(experts, top, ff))], width, 64)
    w = {k: v.to(dtype) for k, v in nm.weights(cfg, seed=3, steady=dtype != torch.float32).items() if ".mlp." in k}
    with torch.device(DEV):
        m = SparseMoeBlock(width, ff, experts, top, False, dtype, "x", sigmoid=True, gated=False, weigh_input=True)
    places = mixture_places("l0.mlp.", m, None)
    assert set(places) == set(w)
    for n, t in w.items():
        places[n](t.to(DEV))
    m.process_weights_after_loading()
    h, x = _r(tokens, width, seed=4).to(dtype), _r(tokens, width, seed=5)
    if dtype != torch.float32:
        h[:, :8] = 3.0
    gx = x.to(DEV)
    a = torch.zeros(tokens, width, dtype=dtype, device=DEV)
    ops.depth_step(gx, (a,), None, m.expert_rows(h.to(DEV)), None, 0, None, [torch.ones((), device=DEV)], 1e-6, dtype, gx)
    y = oracle.mixture_ff(oracle.f64(h), {k: oracle.f64(v) for k, v in w.items()}, "l0.mlp.", dict(experts=experts, top=top))
    _close(gx.double().cpu() - oracle.f64(x), y, _tol(dtype, 1.5e-2))
    with pytest.raises(NotImplementedError):
        m(h.to(DEV))


# --------------------------------------------------------------------------- whole models
LIMIT = {"float32": 5e-5, "bfloat16": 0.05}


def _within(err: torch.Tensor, dtype: str, where) -> None:
    """In 16 bits a row in fifty may stand out: short key vectors that are made unit vectors, results whose norm blows them up."""
    over = int((err > LIMIT[dtype]).sum())
    assert over <= (0 if dtype == "float32" else err.numel() // 50 + 1), (where, over, float(err.max()))
    assert err.max() <= LIMIT[dtype] * (1 if dtype == "float32" else 4), (where, int(err.argmax()), float(err.max()))


def _weights(cfg, dtype):
    """In 16 bits a close call between two experts may fall either way: there a few features decide."""
    return nm.weights(cfg, steady=dtype == "bfloat16")


@pytest.fixture(scope="module")
def served(tmp_path_factory):
    from mllm_b200.trace_run import build_session

    cache = {}

    def get(name, dtype, page=1):
        if (name, dtype, page) not in cache:
            path = tmp_path_factory.mktemp(name) / "m"
            cfg = nm.CONFIGS[name]
            w = nm.write_checkpoint(path, cfg, _weights(cfg, dtype))
            cache[name, dtype, page] = (build_session(str(path), dtype, 1024, radix_cache_page_size=page), w, cfg)
        return cache[name, dtype, page]

    return get


@pytest.fixture(scope="module")
def expected():
    cache = {}

    def get(name, n, seed, dtype):
        if (name, n, seed, dtype) not in cache:
            cfg = nm.CONFIGS[name]
            seq = nm.tokens(cfg, n, seed=seed)
            cache[name, n, seed, dtype] = (seq, oracle.forward(cfg, _weights(cfg, dtype), seq))
        return cache[name, n, seed, dtype]

    return get


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name", sorted(nm.CONFIGS))
def test_portions_and_single_tokens_match_the_statement(served, expected, name, dtype):
    session, _, _ = served(name, dtype)
    seq, want = expected(name, 120, 1, dtype)
    for sizes in ([120], [1], [2], [64, 1, 1, 31, 2, 7]):
        _within(nm.logit_error(run_alone(session, seq, cut(len(seq), sizes)), want), dtype, sizes)
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("dtype", sorted(LIMIT))
@pytest.mark.parametrize("name,page", [("mixed", 1), ("mixed", 16), ("large", 64), ("odd", 1), ("no_experts", 1), ("no_experts", 64), ("only_delta", 16)])
def test_batches_of_unequal_requests_with_reused_slots(served, expected, name, page, dtype):
    session, _, _ = served(name, dtype, page)
    lens = (90, 3, 120, 1, 65, 40, 33, 100)
    both = {f"r{i}": expected(name, n, 70 + i, dtype) for i, n in enumerate(lens)}
    cuts = {"r0": cut(90, [40, 1]), "r1": [2, 1], "r2": cut(120, [2, 1, 1]), "r3": [1], "r4": [64, 1], "r5": cut(40, [1]),
            "r6": [33], "r7": cut(100, [1, 63, 5])}
    for _ in range(2):
        got = run_together(session, {k: s for k, (s, _) in both.items()}, cuts, {f"r{i}": i for i in range(8)})
        for k, (_, want) in both.items():
            _within(nm.logit_error(got[k], want), dtype, k)


@pytest.mark.parametrize("dtype,gain,limit", [("float32", 4.0, 2e-4), ("bfloat16", 1.5, 0.2)])
def test_single_keys_are_found_in_every_schedule(tmp_path, dtype, gain, limit):
    """Peaked scores over 400 tokens: a lost, shifted or foreign key changes whole rows."""
    from mllm_b200.trace_run import build_session

    cfg = json.loads(json.dumps(nm.CONFIGS["no_experts"]))
    cfg["layers"][0]["mixer"]["mask"]["size"], cfg["layers"][1]["mixer"]["left"]["mask"]["size"] = 150, 130
    w = nm.write_checkpoint(tmp_path / "m", cfg, nm.pointed_weights(cfg, gain))
    seq = nm.tokens(cfg, 400, seed=3)
    want = oracle.forward(cfg, w, seq)
    for page in (1, 16, 64):
        session = build_session(str(tmp_path / "m"), dtype, 832, radix_cache_page_size=page)
        for sizes in ([400], [64] * 6 + [1] * 16, [63, 2, 63, 128, 100, 3, 41], [15, 17, 2, 30, 190, 2, 2, 2, 140]):
            err = nm.logit_error(run_alone(session, seq, cut(400, sizes)), want)
            assert err.max() < limit, (page, sizes, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("dtype", sorted(LIMIT))
def test_long_decoding_through_captured_graphs(served, expected, dtype):
    session, _, _ = served("no_experts", dtype)
    graphs = session.mrp.runner.cuda_graph_runner
    before = graphs.replays
    seq, want = expected("no_experts", 300, 5, dtype)
    _within(nm.logit_error(run_alone(session, seq, [5] + [1] * 295), want), dtype, "decode")
    assert graphs.replays == before + 295


def test_stream_after_every_layer(served):
    session, w, cfg = served("large", "float32")
    seq, want, got = nm.tokens(cfg, 40), [], []
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
    assert len(got) == len(want)
    for a, b in zip(got, want):
        _close(a, b, 2e-5)


def test_greedy_generation_through_the_engine(tmp_path):
    cfg = nm.CONFIGS["mixed"]
    w = nm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [nm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9, 60)]
    want = [_greedy(cfg, w, p, 8) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 8, DEV, max_running_requests=3, chunked_prefill_size=24, mem_fraction_static=0.2)
    assert got == [ids for ids, _ in want]


def test_replay_program(tmp_path):
    """bin/trace_run as a user starts it: files of logits, one line per step."""
    cfg = nm.CONFIGS["mixed"]
    w = nm.write_checkpoint(tmp_path / "m", cfg)
    seq = nm.tokens(cfg, 12)
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
        assert nm.logit_error(got, want[rows]).max() < LIMIT["float32"]
