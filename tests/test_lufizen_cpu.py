"""Lufizen on the CPU in fp32 against the plain statement of the design: loading, schedules, the engine's own
generation, and the checks on configurations and checkpoints."""
import json

import pytest
import torch

import lufizen_models as lm
import lufizen_oracle as oracle
from session_schedules import cut, run_alone, run_together

TOL = 5e-5


@pytest.fixture(scope="module")
def served(tmp_path_factory):
    """(session, weights, config) of a named configuration, built once."""
    from mllm_b200.trace_run import build_session

    cache = {}

    def get(name):
        if name not in cache:
            path = tmp_path_factory.mktemp(name) / "m"
            cfg = lm.CONFIGS[name]
            w = lm.write_checkpoint(path, cfg)
            cache[name] = (build_session(str(path), "float32", 1024, device="cpu"), w, cfg)
        return cache[name]

    return get


@pytest.mark.parametrize("name", sorted(lm.CONFIGS))
def test_one_pass_and_portions_match_the_statement(served, name):
    session, w, cfg = served(name)
    seq = lm.tokens(cfg, 70)
    want = oracle.forward(cfg, w, seq)
    for sizes in ([70], [1], [2], [33, 3, 1, 7]):
        got = run_alone(session, seq, cut(len(seq), sizes))
        assert lm.logit_error(got, want).max() < TOL, sizes
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_unequal_requests_together_match_each_alone(served, name):
    session, w, cfg = served(name)
    seqs = {f"r{i}": lm.tokens(cfg, n, seed=20 + i) for i, n in enumerate((41, 3, 36, 1, 17, 50))}
    cuts = {"r0": cut(41, [33, 1]), "r1": [1, 2], "r2": cut(36, [2]), "r3": [1], "r4": [16, 1], "r5": cut(50, [1, 40, 2])}
    got = run_together(session, seqs, cuts, {k: i // 2 for i, k in enumerate(seqs)})
    for k, seq in seqs.items():
        assert lm.logit_error(got[k], oracle.forward(cfg, w, seq)).max() < TOL, k


def test_residual_stream_after_every_layer(served):
    session, w, cfg = served("mixed")
    seq = lm.tokens(cfg, 19)
    want = []
    oracle.forward(cfg, w, seq, want)
    runner, got = session.mrp.runner, []
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
        assert (a.double() - b).abs().max() < 1e-5 * b.abs().max()


# --------------------------------------------------------------------------- every constant shows
def _mixer(c, i):
    return c["layers"][i]["mixer"]


def _router(c, i):
    return c["layers"][i]["mlp"]["router"]


@pytest.mark.parametrize("change", [
    lambda c: c["embedding"].update(scale=6.0), lambda c: c.update(logit_scale=0.9), lambda c: c["norm"].update(eps=0.3),
    lambda c: _mixer(c, 0).update(scale=0.3), lambda c: _mixer(c, 0)["rot"].update(base=2e3),
    lambda c: _mixer(c, 1).update(scale=0.3), lambda c: _mixer(c, 1)["rot"].update(base=2e4), lambda c: _mixer(c, 1)["rot"].update(dims=16),
    lambda c: _mixer(c, 1)["rot"].pop("scaling"), lambda c: _mixer(c, 1)["rot"]["scaling"].update(factor=3.0),
    lambda c: _mixer(c, 1)["rot"]["scaling"].update(low=0.5), lambda c: _mixer(c, 1)["rot"]["scaling"].update(high=9.0),
    lambda c: _mixer(c, 1)["rot"]["scaling"].update(original=32), lambda c: _mixer(c, 2)["rot"].update(dims=0),
    lambda c: _router(c, 0).update(top=2), lambda c: _router(c, 0).update(scale=1.0), lambda c: _router(c, 0)["groups"].update(keep=4),
    lambda c: _router(c, 0)["groups"].update(count=2), lambda c: _router(c, 0)["groups"].update(keep=1),
    lambda c: _router(c, 1)["groups"].update(keep=2)])
def test_every_constant_of_the_config_is_read(tmp_path, change):
    """A changed constant moves the logits by far more than rounding, and as the statement says."""
    from mllm_b200.trace_run import build_session

    base = lm.CONFIGS["mixed"]
    w = lm.weights(base)
    cfg = json.loads(json.dumps(base))
    change(cfg)
    lm.write_checkpoint(tmp_path / "m", cfg, w)
    seq = lm.tokens(base, 24)
    want = oracle.forward(cfg, w, seq)
    d = oracle.forward(base, w, seq) - want
    assert (d.abs().max() / want.pow(2).mean().sqrt()) > 20 * TOL
    session = build_session(str(tmp_path / "m"), "float32", 64, device="cpu")
    assert lm.logit_error(run_alone(session, seq, [20, 1, 3]), want).max() < TOL


# --------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 1024), (2.0, 0.5, 16.0, 100), (32.0, 1.0, 4.0, 8192)])
@pytest.mark.parametrize("dims,base", [(2, 1e4), (16, 50.0), (64, 5e5), (128, 1e6)])
def test_rotation_frequencies(dims, base, scaling):
    from mllm_b200.layers.attention import rotation_frequencies

    s = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    got, want = rotation_frequencies(dims, base, s), torch.tensor(oracle.frequencies(dims, base, s), dtype=torch.float64)
    assert got.dtype == torch.float64 and ((got - want).abs() <= 1e-13 * want).all()


def test_scaled_frequencies_cover_all_three_ranges():
    plain, scaled = (torch.tensor(oracle.frequencies(64, 1e4, s)) for s in (None, dict(factor=8.0, low=1.0, high=4.0, original=256)))
    ratio = plain / scaled
    assert (ratio == 1).any() and ((ratio - 8).abs() < 1e-12).any() and ((ratio > 1.01) & (ratio < 7.9)).any()


@pytest.mark.parametrize("groups,keep,top", [(1, 1, 3), (4, 2, 3), (4, 1, 3), (12, 5, 4), (3, 3, 6), (2, 1, 6)])
def test_router_choices(groups, keep, top):
    """Against the statement, with corrections that make choice scores negative: closed groups must not win against them."""
    from mllm_b200.layers.moe import MoEGate

    gate = MoEGate(32, 12, top, False, torch.float32, choice_bias=True, sigmoid=True, groups=(groups, keep), scale=1.7, shared_gate=True)
    g = torch.Generator().manual_seed(groups * 10 + keep)
    gate.weight.data.copy_(torch.randn(13, 32, generator=g) * 0.4)
    gate.correction.data.copy_(torch.randn(12, generator=g) * 0.6 - 2.0)
    x = torch.randn(40, 32, generator=g)
    w, ids, logit = gate(x)
    free = 0
    for t in range(40):
        logits = oracle.f64(gate.weight[:12]) @ oracle.f64(x[t])
        chosen, want = oracle.route(logits, oracle.f64(gate.correction), top, groups, keep, 1.7)
        assert sorted(ids[t].tolist()) == sorted(chosen)
        got = dict(zip(ids[t].tolist(), w[t].tolist()))
        assert all(abs(got[e] - s) < 1e-5 for e, s in zip(chosen, want))
        free += sorted(chosen) != sorted(oracle.route(logits, oracle.f64(gate.correction), top, 1, 1, 1.7)[0])
    assert (free > 0) == (keep < groups < 12)          # groups of one expert close nothing that would be chosen
    assert torch.allclose(logit[:, 0].double(), oracle.f64(x) @ oracle.f64(gate.weight[12]), atol=1e-5)


def test_pool_of_both_kinds_of_rows():
    from mllm_b200.mem_cache import MixedPool

    shapes, widths = [(2, 48, 48), (1, 64, 64)], [56, 9]
    pool = MixedPool(64, shapes, widths, torch.float32, "cpu", 16)
    assert pool.num_slots == 80 and pool.size == 64
    assert MixedPool.cell_bytes(shapes, widths, torch.float32) == 4 * (2 * 96 + 128 + 56 + 12)
    k, v = pool.get_kv_buffer(1)
    assert k.shape == v.shape == (80, 1, 64) and pool.get_latent_buffer(1).shape == (80, 9)
    k[3], pool.get_latent_buffer(0)[3] = 1.0, 2.0
    pool.clear()
    assert not k.any() and not pool.get_latent_buffer(0).any()


# --------------------------------------------------------------------------- generation
def _greedy(cfg, w, prompt, n):
    """Greedy continuation by the plain statement, and the smallest lead of a chosen token over the next best."""
    seq, lead = list(prompt), []
    for _ in range(n):
        logits = oracle.forward(cfg, w, seq)[-1]
        top = logits.topk(2).values
        lead.append(float(top[0] - top[1]))
        seq.append(int(logits.argmax()))
    return seq[len(prompt):], min(lead)


def _generate(path, prompts, n, device, dtype="float32", **server):
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    cfg = ServerConfig(model_path=str(path), dtype=dtype, max_total_tokens=512, context_length=256, log_level="error", **server)
    eng = Engine(cfg, device=device).launch()
    try:
        outs = eng.generate(input_ids=prompts, sampling_params=dict(temperature=0.0, max_new_tokens=n, ignore_eos=True))
    finally:
        eng.shutdown()
    return [list(o["output_ids"]) for o in (outs if isinstance(outs, list) else [outs])]


def test_greedy_generation_through_the_engine(tmp_path):
    cfg = lm.CONFIGS["mixed"]
    w = lm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [lm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 6, "cpu", max_running_requests=2, chunked_prefill_size=8)
    assert got == [ids for ids, _ in want]


def test_prefix_cache_keeps_the_tokens(tmp_path):
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    cfg = lm.CONFIGS["mixed"]
    lm.write_checkpoint(tmp_path / "m", cfg)
    base = lm.tokens(cfg, 30, seed=7)
    prompts = [base, base + lm.tokens(cfg, 6, seed=8), base]
    plain = [_generate(tmp_path / "m", [p], 5, "cpu", disable_radix_cache=True)[0] for p in prompts]
    eng = Engine(ServerConfig(model_path=str(tmp_path / "m"), dtype="float32", max_total_tokens=512, context_length=256, log_level="error"),
                 device="cpu").launch()
    try:
        got = [list(eng.generate(input_ids=p, sampling_params=dict(temperature=0.0, max_new_tokens=5, ignore_eos=True))["output_ids"])
               for p in prompts]
        assert eng.scheduler.mrp.stats["prefix_hit_tokens"] > 0
    finally:
        eng.shutdown()
    assert got == plain


def test_preset_runs_random_weights_on_the_cpu():
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    eng = Engine(ServerConfig(model_path="preset:lufizen-tiny", dtype="float32", max_total_tokens=256, context_length=128,
                              log_level="error"), device="cpu").launch()
    try:
        out = eng.generate(input_ids=[5, 6, 7], sampling_params=dict(temperature=0.0, max_new_tokens=3, ignore_eos=True))
    finally:
        eng.shutdown()
    assert len(out["output_ids"]) == 3


# --------------------------------------------------------------------------- refusals
def test_configurations_that_make_no_sense_are_refused():
    from mllm_b200.models import get_config_adapter

    adapt = get_config_adapter(dict(architecture="Lufizen"))
    good = lm.CONFIGS["mixed"]
    assert adapt(json.loads(json.dumps(good))).num_hidden_layers == len(good["layers"])
    for change in (lambda c: c["layers"][0].update(type="other"),
                   lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                   lambda c: _mixer(c, 0).update(rot_dim=16),
                   lambda c: _mixer(c, 0).pop("kv_rank"),
                   lambda c: _mixer(c, 0).update(kv_rank=2000),
                   lambda c: _mixer(c, 1).update(kv_heads=4),
                   lambda c: _mixer(c, 1).update(vdim=40),
                   lambda c: _mixer(c, 1).pop("scale"),
                   lambda c: _mixer(c, 1)["rot"].update(dims=50),
                   lambda c: _mixer(c, 1)["rot"]["scaling"].update(high=0.5),
                   lambda c: _router(c, 0)["groups"].update(count=5),
                   lambda c: _router(c, 0)["groups"].update(keep=5),
                   lambda c: _router(c, 0).update(top=7)):
        bad = json.loads(json.dumps(good))
        change(bad)
        with pytest.raises(ValueError):
            adapt(bad)


@pytest.mark.parametrize("fault", ["missing", "extra", "shape", "down"])
def test_checkpoints_must_fit(tmp_path, fault):
    from mllm_b200.trace_run import build_session

    cfg = lm.CONFIGS["only_latent"]
    w = lm.weights(cfg)
    if fault == "missing":
        w.pop("l0.mlp.correction")
    elif fault == "extra":
        w["l1.mix.sink"] = torch.zeros(3, dtype=torch.bfloat16)
    elif fault == "shape":
        w["l0.norm2"] = torch.zeros(3, dtype=torch.bfloat16)
    else:
        w["l0.mix.dkv"] = w["l0.mix.dkv"][:-1]
    lm.write_checkpoint(tmp_path / "m", cfg, w)
    with pytest.raises(ValueError, match={"missing": "correction", "extra": "l1.mix.sink", "shape": "does not fit", "down": "does not fit"}[fault]):
        build_session(str(tmp_path / "m"), "float32", 64, device="cpu")
