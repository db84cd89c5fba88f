"""Pebulix on the CPU in fp32 against the plain statement of the design: loading, schedules, the engine's own
generation, and the checks on configurations and checkpoints."""
import json

import pytest
import torch

import pebulix_models as pm
import pebulix_oracle as oracle
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
            cfg = pm.CONFIGS[name]
            w = pm.write_checkpoint(path, cfg)
            cache[name] = (build_session(str(path), "float32", 1024, device="cpu"), w, cfg)
        return cache[name]

    return get


@pytest.mark.parametrize("name", sorted(pm.CONFIGS))
def test_one_pass_and_portions_match_the_statement(served, name):
    session, w, cfg = served(name)
    seq = pm.tokens(cfg, 45)
    want = oracle.forward(cfg, w, seq)
    for sizes in ([45], [1], [2], [33, 3, 1, 7]):
        got = run_alone(session, seq, cut(len(seq), sizes))
        assert pm.logit_error(got, want).max() < TOL, sizes
    assert session.mrp.free_req_slots() == 4
    assert session.mrp.available_tokens() == session.mrp.runner.max_total_num_tokens


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_unequal_requests_together_match_each_alone(served, name):
    session, w, cfg = served(name)
    seqs = {f"r{i}": pm.tokens(cfg, n, seed=20 + i) for i, n in enumerate((41, 3, 36, 1, 17, 50))}
    cuts = {"r0": cut(41, [33, 1]), "r1": [1, 2], "r2": cut(36, [2]), "r3": [1], "r4": [16, 1], "r5": cut(50, [1, 40, 2])}
    got = run_together(session, seqs, cuts, {k: i // 2 for i, k in enumerate(seqs)})
    for k, seq in seqs.items():
        assert pm.logit_error(got[k], oracle.forward(cfg, w, seq)).max() < TOL, k


def test_residual_stream_after_every_layer(served):
    session, w, cfg = served("mixed")
    seq = pm.tokens(cfg, 19)
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


def test_expanded_and_absorbed_attention_agree(served, monkeypatch):
    from mllm_b200.layers import latent_attention as la

    session, w, cfg = served("mixed")
    seq = pm.tokens(cfg, 40)
    want = oracle.forward(cfg, w, seq)
    for least in (1, 8, 10 ** 9):
        monkeypatch.setattr(la, "EXPAND_MIN_TOKENS", least)
        for context in (1 << 16, 16):
            monkeypatch.setattr(la, "EXPAND_MAX_CONTEXT", context)
            got = run_together(session, {"a": seq, "b": seq[:25], "c": seq[:9]},
                               {"a": [25, 15], "b": [12, 13], "c": [1] * 9}, {"a": 0, "b": 0, "c": 0})
            for k in "abc":
                assert pm.logit_error(got[k], want[: len(got[k])]).max() < TOL, (least, context, k)


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
    cfg = pm.CONFIGS["mixed"]
    w = pm.write_checkpoint(tmp_path / "m", cfg)
    prompts = [pm.tokens(cfg, n, seed=50 + n) for n in (21, 1, 9)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    assert min(lead for _, lead in want) > 1e-3        # no near-ties: the choice does not hang on rounding
    got = _generate(tmp_path / "m", prompts, 6, "cpu", max_running_requests=2, chunked_prefill_size=8)
    assert got == [ids for ids, _ in want]


def test_prefix_cache_with_state_snapshots_keeps_the_tokens(tmp_path):
    cfg = pm.CONFIGS["mixed"]
    pm.write_checkpoint(tmp_path / "m", cfg)
    base = pm.tokens(cfg, 30, seed=7)
    prompts = [base, base + pm.tokens(cfg, 6, seed=8), base]
    plain = [_generate(tmp_path / "m", [p], 5, "cpu", disable_radix_cache=True)[0] for p in prompts]
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    eng = Engine(ServerConfig(model_path=str(tmp_path / "m"), dtype="float32", max_total_tokens=512, context_length=256,
                              enable_mamba_cache=True, log_level="error"), device="cpu").launch()
    try:
        got = [list(eng.generate(input_ids=p, sampling_params=dict(temperature=0.0, max_new_tokens=5, ignore_eos=True))["output_ids"])
               for p in prompts]
        assert eng.scheduler.mrp.stats["prefix_hit_tokens"] > 0
    finally:
        eng.shutdown()
    assert got == plain


def test_configurations_that_make_no_sense_are_refused():
    from mllm_b200.models import get_config_adapter

    adapt = get_config_adapter(dict(architecture="Pebulix"))
    good = pm.CONFIGS["mixed"]
    assert adapt(json.loads(json.dumps(good))).num_hidden_layers == len(good["layers"])
    for change in (lambda c: c["layers"][0].update(type="other"),
                   lambda c: c["layers"][0]["mlp"].update(kind="routed"),
                   lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
                   lambda c: c["layers"][4]["mixer"].update(kv_from=3),        # another rank
                   lambda c: c["layers"][4]["mixer"].update(kv_from=0),        # not latent attention
                   lambda c: c["layers"][1]["mixer"].update(kv_from=4),        # later layer
                   lambda c: c["layers"][1]["mixer"].pop("q_rank")):
        bad = json.loads(json.dumps(good))
        change(bad)
        with pytest.raises(ValueError):
            adapt(bad)
    assert get_config_adapter(dict(architectures=["Qwen3ForCausalLM"])) is None


@pytest.mark.parametrize("fault", ["missing", "extra"])
def test_checkpoints_must_fit(tmp_path, fault):
    from mllm_b200.trace_run import build_session

    cfg = pm.CONFIGS["only_latent"]
    w = pm.weights(cfg)
    if fault == "missing":
        w.pop("l1.mix.sink")
    else:
        w["l1.mix.dkv"] = torch.zeros(4, 4, dtype=torch.bfloat16)      # the layer reads layer 0's latents
    pm.write_checkpoint(tmp_path / "m", cfg, w)
    with pytest.raises(ValueError, match="sink" if fault == "missing" else "l1.mix.dkv"):
        build_session(str(tmp_path / "m"), "float32", 64, device="cpu")


def test_preset_runs_random_weights_on_the_cpu():
    from mllm_b200.configs import ServerConfig
    from mllm_b200.engine.launch import Engine

    eng = Engine(ServerConfig(model_path="preset:pebulix-tiny", dtype="float32", max_total_tokens=256, context_length=128,
                              log_level="error"), device="cpu").launch()
    try:
        out = eng.generate(input_ids=[5, 6, 7], sampling_params=dict(temperature=0.0, max_new_tokens=3, ignore_eos=True))
    finally:
        eng.shutdown()
    assert len(out["output_ids"]) == 3


def test_bad_steps_are_refused(served):
    session, _, cfg = served("only_delta")
    for entries in ([dict(id="a", tokens=[cfg["vocab"]], want=[])], [dict(id="a", tokens=[], want=[])],
                    [dict(id="a", tokens=[1, 2], want=[2])], [dict(id="a", tokens=[1]), dict(id="a", tokens=[2])]):
        with pytest.raises(ValueError):
            session.step(entries, [])
        for q in list(session.live):
            session.mrp.release(session.live.pop(q), cache=False)
