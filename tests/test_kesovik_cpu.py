"""Kesovik on the CPU in fp32 against the plain statement of the design: loading, schedules, the engine's own
generation, and the checks on configurations and checkpoints."""
import json

import pytest
import torch

import kesovik_models as km
import kesovik_oracle as oracle
from session_schedules import cut, run_alone, run_together

TOL = 2e-4


@pytest.fixture(scope="module")
def served(tmp_path_factory):
    """(session, weights, config) of a named configuration, built once."""
    from mllm_b200.trace_run import build_session

    cache = {}

    def get(name):
        if name not in cache:
            path = tmp_path_factory.mktemp(name) / "m"
            cfg = km.CONFIGS[name]
            w = km.write_checkpoint(path, cfg)
            cache[name] = (build_session(str(path), "float32", 1024, device="cpu"), w, cfg)
        return cache[name]

    return get


@pytest.mark.parametrize("name", sorted(km.CONFIGS))
def test_one_pass_and_portions_match_the_statement(served, name):
    session, w, cfg = served(name)
    seq = km.tokens(cfg, 45)
    want = oracle.forward(cfg, w, seq)
    for sizes in ([45], [1], [2], [33, 3, 1, 7]):
        got = run_alone(session, seq, cut(len(seq), sizes))
        assert km.logit_error(got, want).max() < TOL, sizes
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_unequal_requests_together_match_each_alone(served, name):
    session, w, cfg = served(name)
    seqs = {f"r{i}": km.tokens(cfg, n, seed=20 + i) for i, n in enumerate((41, 3, 36, 1, 17, 50))}
    cuts = {"r0": cut(41, [33, 1]), "r1": [1, 2], "r2": cut(36, [2]), "r3": [1], "r4": [16, 1], "r5": cut(50, [1, 40, 2])}
    got = run_together(session, seqs, cuts, {k: i // 2 for i, k in enumerate(seqs)})
    for k, seq in seqs.items():
        assert km.logit_error(got[k], oracle.forward(cfg, w, seq)).max() < TOL, k


def test_residual_stream_after_every_layer(served):
    session, w, cfg = served("mixed")
    seq = km.tokens(cfg, 19)
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
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()


# --------------------------------------------------------------------------- every constant shows
@pytest.mark.parametrize("change", [
    lambda c: c["embedding"].update(scale=1.0), lambda c: c.update(postln_alpha=1.0), lambda c: c.update(logit_softcap=1e9),
    lambda c: c["norm"].update(eps=0.3), lambda c: c["layers"][1]["mixer"].update(left_scale=1.0),
    lambda c: c["layers"][1]["mixer"].update(right_scale=1.0), lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=14),
    lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=12), lambda c: c["layers"][1]["mixer"]["left"].update(scale=0.2),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=48), lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(base=2e4),
    lambda c: c["layers"][0]["mixer"].update(decay=[0.3, 0.9, 0.99]), lambda c: c["layers"][0]["mlp"]["router"].update(top=2),
    lambda c: c["layers"][3]["mixer"].update(left_scale=0.0), lambda c: c["layers"][3]["mixer"].update(right_scale=0.0)])
def test_every_constant_of_the_config_is_read(tmp_path, change):
    """A changed constant moves the logits by far more than rounding, and as the statement says."""
    from mllm_b200.trace_run import build_session

    base = km.CONFIGS["mixed"]
    w = km.weights(base)
    cfg = json.loads(json.dumps(base))
    change(cfg)
    km.write_checkpoint(tmp_path / "m", cfg, w)
    seq = km.tokens(base, 24)
    want = oracle.forward(cfg, w, seq)
    assert km.logit_error(oracle.forward(base, w, seq), want).max() > 20 * TOL
    session = build_session(str(tmp_path / "m"), "float32", 64, device="cpu")
    assert km.logit_error(run_alone(session, seq, [20, 1, 3]), want).max() < TOL


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
    cfg = km.CONFIGS["mixed"]
    w = km.write_checkpoint(tmp_path / "m", cfg)
    prompts = [km.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 6, "cpu", max_running_requests=2, chunked_prefill_size=8)
    assert got == [ids for ids, _ in want]


def test_prefix_cache_with_state_snapshots_keeps_the_tokens(tmp_path):
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    cfg = km.CONFIGS["mixed"]
    km.write_checkpoint(tmp_path / "m", cfg)
    base = km.tokens(cfg, 30, seed=7)
    prompts = [base, base + km.tokens(cfg, 6, seed=8), base]
    plain = [_generate(tmp_path / "m", [p], 5, "cpu", disable_radix_cache=True)[0] for p in prompts]
    eng = Engine(ServerConfig(model_path=str(tmp_path / "m"), dtype="float32", max_total_tokens=512, context_length=256,
                              enable_mamba_cache=True, log_level="error"), device="cpu").launch()
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

    eng = Engine(ServerConfig(model_path="preset:kesovik-tiny", dtype="float32", max_total_tokens=256, context_length=128,
                              log_level="error"), device="cpu").launch()
    try:
        out = eng.generate(input_ids=[5, 6, 7], sampling_params=dict(temperature=0.0, max_new_tokens=3, ignore_eos=True))
    finally:
        eng.shutdown()
    assert len(out["output_ids"]) == 3


# --------------------------------------------------------------------------- refusals
def test_configurations_that_make_no_sense_are_refused():
    from mllm_b200.models import get_config_adapter

    adapt = get_config_adapter(dict(architecture="Kesovik"))
    good = km.CONFIGS["mixed"]
    assert adapt(json.loads(json.dumps(good))).num_hidden_layers == len(good["layers"])
    for change in (lambda c: c["layers"][0].update(type="other"),
                   lambda c: c["layers"][0]["mlp"].update(kind="routed"),
                   lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4),
                   lambda c: c["layers"][1]["mixer"]["left"].pop("scale"),
                   lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=50),
                   lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0),
                   lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
                   lambda c: c["layers"][0]["mixer"].pop("vdim")):
        bad = json.loads(json.dumps(good))
        change(bad)
        with pytest.raises(ValueError):
            adapt(bad)


@pytest.mark.parametrize("fault", ["missing", "extra", "shape"])
def test_checkpoints_must_fit(tmp_path, fault):
    from mllm_b200.trace_run import build_session

    cfg = km.CONFIGS["only_lightning"]
    w = km.weights(cfg)
    if fault == "missing":
        w.pop("l1.mlp.correction")
    elif fault == "extra":
        w["l1.mix.q.norm"] = torch.zeros(4, dtype=torch.bfloat16)
    else:
        w["l0.ls2"] = torch.zeros(3, dtype=torch.bfloat16)
    km.write_checkpoint(tmp_path / "m", cfg, w)
    with pytest.raises(ValueError, match={"missing": "correction", "extra": "l1.mix.q.norm", "shape": "does not fit"}[fault]):
        build_session(str(tmp_path / "m"), "float32", 64, device="cpu")


def test_kernel_modules_and_their_functions():
    """Every function of the binding files is found in exactly one module, apart from those that all have."""
    from mllm_b200 import _build

    seen = {}
    for m in _build.cuda_modules():
        for fn in _build.module_functions(m):
            seen.setdefault(fn, []).append(m)
    assert seen["lightning_chunk"] == ["mllm_b200_L"] and seen["moe_align"] == ["mllm_b200_E"] and seen["gemm"] == ["mllm_b200_C"]
    assert {fn for fn, ms in seen.items() if len(ms) > 1} == {"read_status", "launch_count"}
