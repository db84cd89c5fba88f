"""Nikedra on the CPU in fp32 against the plain statement of the design: loading, schedules, the engine's own
generation, and the checks on configurations and checkpoints."""
import json

import pytest
import torch

import nikedra_models as nm
import nikedra_oracle as oracle
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
            cfg = nm.CONFIGS[name]
            w = nm.write_checkpoint(path, cfg)
            cache[name] = (build_session(str(path), "float32", 1024, device="cpu"), w, cfg)
        return cache[name]

    return get


@pytest.mark.parametrize("name", sorted(nm.CONFIGS))
def test_one_pass_and_portions_match_the_statement(served, name):
    session, w, cfg = served(name)
    seq = nm.tokens(cfg, 45)
    want = oracle.forward(cfg, w, seq)
    for sizes in ([45], [1], [2], [33, 3, 1, 7]):
        got = run_alone(session, seq, cut(len(seq), sizes))
        assert nm.logit_error(got, want).max() < TOL, sizes
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_unequal_requests_together_match_each_alone(served, name):
    session, w, cfg = served(name)
    seqs = {f"r{i}": nm.tokens(cfg, n, seed=20 + i) for i, n in enumerate((41, 3, 36, 1, 17))}
    cuts = {"r0": cut(41, [33, 1]), "r1": [1, 2], "r2": cut(36, [2]), "r3": [1], "r4": [16, 1]}
    got = run_together(session, seqs, cuts, {k: i // 2 for i, k in enumerate(seqs)}, live=3)
    for k, seq in seqs.items():
        assert nm.logit_error(got[k], oracle.forward(cfg, w, seq)).max() < TOL, k


def test_stream_after_every_layer(served):
    session, w, cfg = served("mixed")
    seq = nm.tokens(cfg, 19)
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
def _m(c, i):
    return c["layers"][i]["mixer"]


def _scaling(c):
    return _m(c, 1)["left"]["rot"]["scaling"]


@pytest.mark.parametrize("change", [
    lambda c: c.update(logit_scale=0.9), lambda c: c["norm"].update(eps=0.3), lambda c: c["layers"][0]["mlp"].update(limit=0.8),
    lambda c: _m(c, 1)["left"].update(scale=0.3), lambda c: _m(c, 1)["left"]["rot"].update(base=2e4),
    lambda c: _m(c, 1)["left"]["rot"].update(dims=16), lambda c: _m(c, 1)["left"]["rot"].pop("scaling"),
    lambda c: _scaling(c).update(factor=7.0), lambda c: _scaling(c).update(original=30), lambda c: _scaling(c).update(fast=2.0),
    lambda c: _scaling(c).update(slow=0.1), lambda c: _m(c, 1)["left"]["mask"].update(size=23), lambda c: _m(c, 1)["left"].update(mask=None),
    lambda c: _m(c, 1)["right"].update(norm_groups=2), lambda c: _m(c, 2).update(scale=0.3),
    lambda c: _m(c, 2)["rot"].update(base=2e3), lambda c: _m(c, 2)["mask"].update(size=21), lambda c: _m(c, 2).update(mask=None),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=3)])
def test_every_constant_of_the_config_is_read(tmp_path, monkeypatch, change):
    """A changed constant moves the logits by far more than rounding, and as the statement says."""
    from mllm_b200.trace_run import build_session

    base = nm.CONFIGS["mixed"]
    w = nm.weights(base)
    cfg = json.loads(json.dumps(base))
    change(cfg)
    nm.write_checkpoint(tmp_path / "m", cfg, w)
    seq = nm.tokens(base, 28)
    plain = json.loads(json.dumps(cfg))
    for m in (_m(plain, 1)["left"], _m(plain, 2)):      # without a mask a token sees all before it
        m["mask"] = m["mask"] or dict(size=10 ** 6)
    want = oracle.forward(plain, w, seq)
    d = oracle.forward(base, w, seq) - want
    assert (d.abs().max() / want.pow(2).mean().sqrt()) > 20 * TOL
    session = build_session(str(tmp_path / "m"), "float32", 64, device="cpu")
    assert nm.logit_error(run_alone(session, seq, [20, 1, 7]), want).max() < TOL


# --------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("scaling", [None, (8.0, 1024, 32.0, 1.0), (2.0, 100, 4.0, 0.5), (32.0, 8192, 32.0, 1.0), (4.0, 6, 3.0, 2.0)])
@pytest.mark.parametrize("dims,base", [(2, 1e4), (16, 50.0), (64, 5e5), (128, 1e6)])
def test_rotation_frequencies(dims, base, scaling):
    from mllm_b200.layers.attention import rotation_frequencies, rotation_magnitude

    s = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    got, want = rotation_frequencies(dims, base, s), torch.tensor(oracle.frequencies(dims, base, s), dtype=torch.float64)
    assert got.dtype == torch.float64 and ((got - want).abs() <= 1e-13 * want).all()
    assert (rotation_magnitude(s) == 1.0) == (s is None)


def test_scaled_frequencies_cover_all_three_ranges():
    plain, scaled = (torch.tensor(oracle.frequencies(64, 1e4, s)) for s in (None, dict(factor=8.0, original=256, fast=16.0, slow=1.0)))
    ratio = plain / scaled
    assert (ratio == 1).any() and ((ratio - 8).abs() < 1e-12).any() and ((ratio > 1.01) & (ratio < 7.9)).any()


def test_inner_sizes_come_from_the_tensors_in_any_order(tmp_path):
    """Sizes that no entry of the config gives, other ones for decays and gates, tensors in an order of their own."""
    from mllm_b200.models import get_config_adapter, get_model_class

    cfg = nm.CONFIGS["only_delta"]
    seq = nm.tokens(cfg, 9)
    for ranks in ((3, 17), (40, 1), (8, 8)):
        w = nm.weights(cfg, ranks=ranks)
        ns = get_config_adapter(cfg)(cfg)
        for names in (sorted(w), sorted(w, reverse=True)):
            model = get_model_class(ns.architectures[0])(ns, params_dtype=torch.float32)
            assert model.load_weights((n, w[n]) for n in names) == set(w)
            mixer = model.layers[0].mixer
            assert torch.equal(mixer.in_proj.weight[: mixer.key_dim], w["l0.mix.q"].float())
            x = torch.randn(5, cfg["width"])
            y = x @ mixer.in_proj.weight.T
            second = y[:, mixer.inner] @ mixer.low_rank.weight.T
            assert torch.allclose(second[:, : mixer.decay_dim], (x @ w["l0.mix.a1"].float().T) @ w["l0.mix.a2"].float().T, atol=1e-4)
            at = mixer.gate_at
            assert torch.allclose(second[:, at: at + mixer.value_dim], (x @ w["l0.mix.g1"].float().T) @ w["l0.mix.g2"].float().T, atol=1e-4)
        nm.write_checkpoint(tmp_path / f"m{ranks[0]}", cfg, w)
        from mllm_b200.trace_run import build_session

        session = build_session(str(tmp_path / f"m{ranks[0]}"), "float32", 64, device="cpu")
        assert nm.logit_error(run_alone(session, seq, [9]), oracle.forward(cfg, w, seq)).max() < TOL


def test_state_pool_holds_every_layers_states(served):
    session, _, cfg = served("mixed")
    pool = session.mrp.runner.gdn_pool
    shapes = [(tuple(r.shape[1:]), tuple(c.shape[1:])) for r, c in pool.layers]
    W, taps = cfg["width"], cfg["canon"]["taps"]
    conv = ((0, 0, 0), (W, taps - 1))
    assert shapes == [conv, ((6, 24, 40), (2 * 72 + 240, 2)), conv, ((6, 24, 16), (96 + 96, 2)), conv, conv, conv, ((2, 40, 24), (160 + 48, 1)),
                      conv, ((3, 16, 24), (72 + 96, 4))]


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
    cfg = nm.CONFIGS["mixed"]
    w = nm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [nm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 6, "cpu", max_running_requests=2, chunked_prefill_size=8)
    assert got == [ids for ids, _ in want]


def test_prefix_cache_with_state_snapshots_keeps_the_tokens(tmp_path):
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    cfg = nm.CONFIGS["mixed"]
    nm.write_checkpoint(tmp_path / "m", cfg)
    base = nm.tokens(cfg, 30, seed=7)
    prompts = [base, base + nm.tokens(cfg, 6, seed=8), base]
    plain = [_generate(tmp_path / "m", [p], 5, "cpu", disable_radix_cache=True)[0] for p in prompts]
    eng = Engine(ServerConfig(model_path=str(tmp_path / "m"), dtype="float32", max_total_tokens=512, context_length=256, log_level="error",
                              enable_mamba_cache=True), device="cpu").launch()
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

    eng = Engine(ServerConfig(model_path="preset:nikedra-tiny", dtype="float32", max_total_tokens=256, context_length=128,
                              log_level="error"), device="cpu").launch()
    try:
        out = eng.generate(input_ids=[5, 6, 7], sampling_params=dict(temperature=0.0, max_new_tokens=3, ignore_eos=True))
    finally:
        eng.shutdown()
    assert len(out["output_ids"]) == 3


def test_a_model_that_keeps_nothing_per_token_gets_a_pool_of_its_requests_size(tmp_path):
    from mllm_b200.configs import ServerConfig
    from mllm_b200.executor import ModelRunner

    cfg = nm.CONFIGS["only_delta"]
    nm.write_checkpoint(tmp_path / "m", cfg)
    runner = ModelRunner(ServerConfig(model_path=str(tmp_path / "m"), dtype="float32", context_length=64, max_running_requests=2,
                                      spare_request_slots=1, log_level="error"), device="cpu")
    runner.initialize()
    assert 0 < runner.max_total_num_tokens <= 3 * 64


# --------------------------------------------------------------------------- refusals
def test_configurations_that_make_no_sense_are_refused():
    from mllm_b200.models import get_config_adapter

    adapt = get_config_adapter(dict(architecture="Nikedra"))
    good = nm.CONFIGS["mixed"]
    assert adapt(json.loads(json.dumps(good))).num_hidden_layers == len(good["layers"])
    for change in (lambda c: c["layers"][0].update(type="other"),
                   lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][0]["mlp"].pop("limit"),
                   lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
                   lambda c: c["canon"].update(taps=0),
                   lambda c: c["canon"].update(taps=40),
                   lambda c: _m(c, 0).update(kv_heads=4),
                   lambda c: _m(c, 0).pop("conv"),
                   lambda c: _m(c, 1)["left"].update(kv_heads=4),
                   lambda c: _m(c, 1)["left"].pop("scale"),
                   lambda c: _m(c, 1)["left"]["rot"].update(dims=50),
                   lambda c: _m(c, 1)["left"]["mask"].update(size=0),
                   lambda c: _scaling(c).pop("fast"),
                   lambda c: _m(c, 1)["right"].update(groups=4),
                   lambda c: _m(c, 1)["right"].update(norm_groups=5),
                   lambda c: _m(c, 2).update(rot_dim=8),
                   lambda c: _m(c, 2).update(kv_rank=2000)):
        bad = json.loads(json.dumps(good))
        change(bad)
        with pytest.raises(ValueError):
            adapt(bad)


@pytest.mark.parametrize("fault", ["missing", "extra", "shape", "down", "inner"])
def test_checkpoints_must_fit(tmp_path, fault):
    from mllm_b200.trace_run import build_session

    cfg = nm.CONFIGS["only_delta"] if fault == "inner" else nm.CONFIGS["only_latent"]
    w = nm.weights(cfg)
    if fault == "missing":
        w.pop("l0.canon1")
    elif fault == "extra":
        w["l1.mix.sink"] = torch.zeros(3, dtype=torch.bfloat16)
    elif fault == "shape":
        w["l0.dwa"] = torch.zeros(3, dtype=torch.bfloat16)
    elif fault == "down":
        w["l0.mix.dkv"] = w["l0.mix.dkv"][:-1]
    else:
        w["l0.mix.a2"] = w["l0.mix.a2"][:, :-1]
    nm.write_checkpoint(tmp_path / "m", cfg, w)
    match = {"missing": "canon1", "extra": "l1.mix.sink"}.get(fault, "does not fit")
    with pytest.raises(ValueError, match=match):
        build_session(str(tmp_path / "m"), "float32", 64, device="cpu")
