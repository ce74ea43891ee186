"""Fudulix on the reference ops (CPU, fp32) against the plain restatement in fudulix_oracle.py: configuration, loading, every
mechanism, the cache and state under portions, batches and reuse, serving, the prefix cache, the trace runner."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import fudulix_oracle as O
from fudulix_cases import CASES, MIXED, TAIL, WIDE, engine_of, error, portions, prompt, run, weights_of
from phaseshift_b200.io.model_dir import save_hf_model
from phaseshift_b200.models import registry
from phaseshift_b200.models.fudulix.config import FudulixConfig
from phaseshift_b200.models.fudulix.weights import tensor_shapes
from phaseshift_b200.ops import specs
from phaseshift_b200.runtime.serving import ServingEngine

ROOT = Path(__file__).resolve().parents[1]
TOL = 6e-5


# ------------------------------------------------------------------ configuration, registry, loading
@pytest.mark.parametrize("name", sorted(CASES))
def test_config_round_trip_and_registry(tmp_path, name):
    cfg = FudulixConfig.from_dict(CASES[name])
    assert cfg.to_dict() == CASES[name]
    cfg.save(tmp_path)
    again = registry.config_from_dir(tmp_path)
    assert again.to_dict() == cfg.to_dict() and again.family == "fudulix"
    assert registry.family_of_dir(tmp_path).name == "fudulix"


def test_presets_are_registered():
    assert {"fudulix-tiny", "fudulix-4b", "fudulix-27b"} <= set(registry.preset_names())
    assert registry.preset_config("fudulix-4b").family == "fudulix" and registry.preset_config("luvutar-tiny").family == "luvutar"


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"),
                                    lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][0]["mixer"].update(kv_heads=4),
                                    lambda d: d["layers"][0]["mixer"].update(conv=0),
                                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=13),
                                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26),
                                    lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
                                    lambda d: d["layers"][1]["mixer"].update(vdim=40),
                                    lambda d: d["layers"][0]["mlp"]["router"].update(identity=1),
                                    lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4),
                                    lambda d: d["layers"][0]["mlp"]["router"].update(top=9)])
def test_config_refuses_what_the_design_does_not_have(change):
    d = copy.deepcopy(MIXED)
    change(d)
    with pytest.raises(ValueError):
        FudulixConfig.from_dict(d)


def test_options_the_family_does_not_have_are_refused():
    cfg = registry.preset_config("fudulix-tiny")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", "nvfp4")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", tp_rank=0, tp_size=2)


def test_state_holds_what_the_layers_look_back_to():
    st = engine_of(MIXED, weights_of(MIXED)).state
    assert [c is None for c in st.conv] == [False, True, True, False, True]
    assert tuple(st.conv[0].shape) == (3, 2, 10 * 64) and tuple(st.conv[3].shape) == (3, 4, 15 * 64)
    assert st.last_token.shape == (3,) and len(st.slot_tensors()) == 3
    st.conv[0][1], st.last_token[1] = 7.0, 5
    st.copy_slot(2, 1)
    assert bool((st.conv[0][2] == 7).all()) and int(st.last_token[2]) == 5


@pytest.mark.parametrize("base,dims,factor,original", [(900.0, 14, 4.0, 100), (30000.0, 48, 6.0, 700), (10.0, 8, 2.0, 4), (5e5, 128, 1.0, 8192)])
def test_scaled_frequencies(base, dims, factor, original):
    f = specs.rotation_frequencies(base, dims)
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor, "low": 1.0, "high": 4.0, "original": original, "fast": 16.0, "slow": 1.0}}
    want = torch.tensor(O.stepped_frequencies(rot), dtype=torch.float64)
    assert torch.allclose(specs.stepped_frequencies(f, factor, 1.0, 4.0, original), want, rtol=1e-12)
    got, size = specs.ramped_frequencies(f, base, factor, original, 16.0, 1.0)
    want, want_size = O.ramped_frequencies(rot)
    assert torch.allclose(got, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and size == want_size


# ------------------------------------------------------------------ whole sequences, cuts, batches
@pytest.mark.parametrize("classes", [False, True])
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_matches_the_oracle(name, classes):
    raw, w = CASES[name], weights_of(CASES[name], classes=classes)
    p = {"a": prompt(raw, 150)}
    got = run(engine_of(raw, w), [[("a", 150)]], p)["a"]
    assert error(got, O.forward(raw, w, p["a"])) < TOL


@pytest.mark.parametrize("name,sizes", [("mixed", [2]), ("mixed", [1]), ("tail", [2, 31, 3, 1, 64]), ("unit", [5, 1]), ("wide", [2, 64, 1])])
def test_portions_and_single_tokens_match_the_whole_prompt(name, sizes):
    raw, w = CASES[name], weights_of(CASES[name])
    p = {"a": prompt(raw, 110)}
    got = run(engine_of(raw, w), [[("a", c)] for c in portions(110, sizes)], p)["a"]
    assert error(got, O.forward(raw, w, p["a"])) < TOL


def test_batches_of_unequal_requests_reuse_pages_and_slots():
    """Three slots and a pool that holds only the live requests: later requests get the pages and slots of finished ones."""
    raw, w = MIXED, weights_of(MIXED)
    n = {"a": 90, "b": 33, "c": 5, "d": 70, "e": 41}
    p = {r: prompt(raw, k, 10 + i) for i, (r, k) in enumerate(n.items())}
    plan = [[("a", 40), ("b", 2), ("c", 5)], [("a", 1), ("b", 31)], [("d", 17), ("a", 2), ("e", 41)], [("d", 1)], [("a", 47), ("d", 52)]]
    eng = engine_of(raw, w, capacity=208, page=16)
    for _ in range(2):
        got = run(eng, plan, p)
        for r in p:
            assert error(got[r], O.forward(raw, w, p[r])) < TOL, r
    assert eng.alloc.pages_free == eng.state.num_pages - 1


MIX = lambda d, i: d["layers"][i]["mixer"]
MISTAKES = {
    "window + 1": lambda d, w: MIX(d, 1)["mask"].update(size=34),
    "window - 1": lambda d, w: MIX(d, 0)["mask"].update(size=8),
    "kept + 1": lambda d, w: MIX(d, 0)["mask"].update(keep_first=6),
    "kept - 1": lambda d, w: MIX(d, 3)["mask"].update(keep_first=69),
    "scale": lambda d, w: MIX(d, 1).update(scale=0.51),
    "rotation base": lambda d, w: MIX(d, 1)["rot"].update(base=1000.0),
    "rotated dimensions": lambda d, w: MIX(d, 3)["rot"].update(dims=20),
    "step factor": lambda d, w: MIX(d, 4)["rot"]["scaling"].update(factor=4.5),
    "step limit": lambda d, w: MIX(d, 4)["rot"]["scaling"].update(high=3.0),
    "ramp factor": lambda d, w: MIX(d, 3)["rot"]["scaling"].update(factor=9.0),
    "ramp limit": lambda d, w: MIX(d, 0)["rot"]["scaling"].update(slow=3.0),
    "pair factor": lambda d, w: d["embedding"]["bigram"].update(mul_prev=32),
    "first row of the pairs": lambda d, w: w["bigram"][-1].zero_(),
    "values not mixed": lambda d, w: MIX(d, 4).update(v_mix=False),
    "values mixed": lambda d, w: w["l1.mix.vmix"].fill_(0.5),
    "first tap": lambda d, w: w["l3.mix.k.conv"][:, 0].zero_(),
    "value convolution": lambda d, w: w["l0.mix.v.conv"][:, 1].mul_(1.1),
    "key norm": lambda d, w: w["l3.mix.k.norm"].mul_(1.05),
    "gate bias": lambda d, w: w["l1.mlp.gate.b"].zero_(),
    "down bias": lambda d, w: w["l1.mlp.down.b"].zero_(),
    "correction": lambda d, w: w["l2.mlp.correction"].zero_(),
    "groups": lambda d, w: d["layers"][0]["mlp"]["router"]["groups"].update(keep=3),
    "shared expert": lambda d, w: w["l2.mlp.shared.down"].zero_(),
    "eps": lambda d, w: d["norm"].update(eps=3e-3),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_the_inputs_make_single_mistakes_visible(mistake):
    """The oracle itself with one thing changed differs visibly: the comparisons of these tests would show such a fault."""
    raw, w = copy.deepcopy(MIXED), {n: t.clone() for n, t in weights_of(MIXED).items()}
    ids = prompt(raw, 120)
    ref = O.forward(raw, w, ids)
    MISTAKES[mistake](raw, w)
    assert error(O.forward(raw, w, ids), ref) > 20 * TOL


# ------------------------------------------------------------------ scheduler, sampling, prefix cache
def test_greedy_serving_matches_the_oracle():
    raw, w = TAIL, weights_of(TAIL)
    eng = engine_of(raw, w, slots=2)
    srv = ServingEngine(eng, max_step_tokens=24)
    prompts = [prompt(raw, n, 20 + n) for n in (37, 3, 61)]
    ids = [srv.submit(p, 5) for p in prompts]
    ev = srv.run_until_idle()
    for rid, p in zip(ids, prompts):
        assert [e.token_id for e in ev if e.kind == "token" and e.request_id == rid] == O.greedy(raw, w, p, 5)
    assert eng.generate(prompts[0], 4, prefill_chunk=10) == O.greedy(raw, w, prompts[0], 4)


def test_prefix_cache_restores_keys_convolution_rows_and_the_last_token():
    raw, w = MIXED, weights_of(MIXED)
    srv = ServingEngine(engine_of(raw, w, slots=2), max_step_tokens=64, prefix_cache_tokens=256, prefix_min_tokens=16)
    base = prompt(raw, 50)
    srv.submit(base, 3, checkpoint_position=40)
    srv.run_until_idle()
    other = base[:40] + prompt(raw, 20, 77)
    rid = srv.submit(other, 5)
    ev = srv.run_until_idle()
    assert [e.token_id for e in ev if e.kind == "token"] == O.greedy(raw, w, other, 5)
    assert srv.request(rid)["restored_tokens"] == 40


def test_sampling_is_deterministic():
    raw, w = WIDE, weights_of(WIDE)
    eng = engine_of(raw, w)
    p = prompt(raw, 12)
    a = eng.generate(p, 8, temperature=0.8, top_k=20, seed=5)
    assert a == eng.generate(p, 8, temperature=0.8, top_k=20, seed=5) and all(0 <= t < raw["vocab"] for t in a)


# ------------------------------------------------------------------ model directories, command line, trace runner
def _save(raw, w, path):
    cfg = FudulixConfig.from_dict(raw)
    assert {n: tuple(t.shape) for n, t in w.items()} == tensor_shapes(cfg)
    save_hf_model(path, cfg, w)
    return path


def test_compute_runs_a_model_directory_and_a_preset(tmp_path, capsys):
    from phaseshift_b200.apps import compute
    raw, w = TAIL, weights_of(TAIL)
    d = _save(raw, w, tmp_path / "m")
    p = prompt(raw, 9)
    (tmp_path / "ids").write_text(" ".join(map(str, p)))
    assert compute.main(["--model-dir", str(d), "--device", "cpu", "--input-ids-file", str(tmp_path / "ids"), "--max-new-tokens", "4"]) == 0
    out = capsys.readouterr().out
    assert "GENERATED_IDS=" + ",".join(map(str, O.greedy(raw, w, p, 4))) in out
    assert compute.main(["--random-model", "fudulix-tiny", "--device", "cpu", "--max-new-tokens", "2"]) == 0
    with pytest.raises(SystemExit, match="nvfp4"):
        compute.main(["--model-dir", str(d), "--device", "cpu", "--preset", "nvfp4"])


def test_trace_runner_replays_steps(tmp_path):
    import numpy as np
    raw, w = MIXED, weights_of(MIXED)
    d = _save(raw, w, tmp_path / "m")
    a, b = prompt(raw, 30, 3), prompt(raw, 21, 4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:13], "want": [0, 12]}, {"id": "y", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b[2:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[3:], "want": [17]}, {"id": "x", "tokens": a[13:], "want": [16, 0]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": b[:5], "want": [4]}], "end": ["x"]}]
    cmd = [str(ROOT / "bin" / "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "64",
           "--device", "cpu"]
    r = subprocess.run([sys.executable] + cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    la, lb = O.forward(raw, w, a), O.forward(raw, w, b)
    want = {0: [la[0], la[12]], 2: [lb[20], la[29], la[13]], 3: [lb[4]]}
    for s, rows in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{s}.f32", dtype="<f4").reshape(len(rows), raw["vocab"]))
        assert error(got, torch.stack(rows)) < 1e-4, s


# ------------------------------------------------------------------ the restatement itself
def test_oracle_mechanisms_by_hand():
    assert O.kept_window_mask(5, 2, 1).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [1, 0, 1, 1, 0], [1, 0, 0, 1, 1]]
    assert O.bigram_rows([3, 4, 0], 10, 7, 2) == [10, 9, 8]
    y = O.short_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]]))
    assert y.flatten().tolist() == [1.0, 12.0, 24.0]
    x = O.turn_halves(torch.tensor([[[0.0] * 4], [[1.0, 5.0, 0.0, 9.0]]]).double(), [2.0], 3.0)[1, 0]
    assert torch.allclose(x, torch.tensor([3 * (math.cos(2) - 5 * math.sin(2)), 3 * (5 * math.cos(2) + math.sin(2)), 0.0, 9.0]).double())
    x = O.turn_halves(torch.tensor([[[0.0] * 5], [[1.0, 1.0, 0.0, 2.0, 7.0]]]).double(), [2.0, 0.0], 1.0)[1, 0]
    assert torch.allclose(x, torch.tensor([math.cos(2), 1.0, math.sin(2), 2.0, 7.0]).double())
    x = O.turn_neighbours(torch.tensor([[[0.0] * 3], [[1.0, 0.0, 7.0]]]).double(), [2.0])[1, 0]
    assert torch.allclose(x, torch.tensor([math.cos(2), math.sin(2), 7.0]).double())
    p = O.softmax_plus_one(torch.zeros(1, 2, 2, dtype=torch.float64), O.window_mask(2, 2))
    assert torch.allclose(p[0], torch.tensor([[0.5, 0.0], [1 / 3, 1 / 3]]).double())
    # groups {0, 1}, {2, 3}, {4, 5}: the correction lifts the third, its low member included; weights ignore the correction
    z = torch.log(torch.tensor([0.30, 0.10, 0.25, 0.05, 0.20, 0.10]).double())
    c = torch.tensor([-9.0, -9.0, -9.0, -9.0, -8.5, -8.9]).double()
    assert [(i, round(float(v), 6)) for i, v in O.route(z, c, 3, 1, 2)] == [(4, round(0.2 / 0.3, 6)), (5, round(0.1 / 0.3, 6))]
    assert [i for i, _ in O.route(z, c, 3, 2, 3)] == [4, 0, 5] and [i for i, _ in O.route(z, c, 3, 3, 4)] == [4, 0, 2, 5]
