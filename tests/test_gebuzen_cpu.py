"""Gebuzen on the reference ops (CPU, fp32) against the plain restatement in gebuzen_oracle.py: configuration, loading, every
mechanism, the cache and state under portions, batches and reuse, serving, the prefix cache, the trace runner."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import gebuzen_oracle as O
from gebuzen_cases import CASES, MIXED, TAIL, UNIT, engine_of, error, portions, prompt, run, weights_of
from phaseshift_b200.io.model_dir import save_hf_model
from phaseshift_b200.models import registry
from phaseshift_b200.models.gebuzen.config import GebuzenConfig
from phaseshift_b200.models.gebuzen.weights import tensor_shapes
from phaseshift_b200.runtime.serving import ServingEngine

ROOT = Path(__file__).resolve().parents[1]
TOL = 2e-5


# ------------------------------------------------------------------ configuration, registry, loading
def test_config_round_trip_and_registry(tmp_path):
    cfg = GebuzenConfig.from_dict(MIXED)
    cfg.save(tmp_path)
    again = registry.config_from_dir(tmp_path)
    assert again.to_dict() == cfg.to_dict() and again.family == "gebuzen"
    assert registry.family_of_dir(tmp_path).name == "gebuzen"
    assert [(r.layer, r.pass_index, r.opens_pass) for r in cfg.runs()] == O.layer_runs(MIXED)
    assert {"tiny", "4b", "27b", "gebuzen-tiny"} <= set(registry.preset_names())
    assert registry.preset_config("tiny").family == "qwen35" and registry.preset_config("gebuzen-4b").family == "gebuzen"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Somethingelse"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.family_of_dir(tmp_path)


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"),
                                    lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][0]["mixer"]["left"].update(vdim=8),
                                    lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4),
                                    lambda d: d["loop"].update(stop=9)])
def test_config_refuses_what_the_design_does_not_have(change):
    d = copy.deepcopy(MIXED)
    change(d)
    with pytest.raises(ValueError):
        GebuzenConfig.from_dict(d)


def test_options_a_family_does_not_have_are_refused(tmp_path):
    cfg = registry.preset_config("gebuzen-tiny")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", "nvfp4")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", tp_rank=0, tp_size=2)
    from phaseshift_b200.runtime.state import ModelState, StateConfig
    with pytest.raises(ValueError, match="bf16"):
        ModelState(cfg, StateConfig(kv_dtype="fp8_e4m3"), torch.device("cpu"), torch.bfloat16)


def test_state_has_one_set_per_layer_run_and_one_pool_for_keys_that_are_values():
    eng = engine_of(MIXED, weights_of(MIXED))
    runs = O.layer_runs(MIXED)
    assert len(eng.state.kv) == len(eng.state.gdn) == len(runs) == 7
    assert all(l.v is l.k for l in eng.state.kv)
    assert len({l.k.data_ptr() for l in eng.state.kv}) == len(runs)
    assert [g.rec.shape[1] for g in eng.state.gdn] == [MIXED["layers"][i]["mixer"]["right"]["heads"] for i, _, _ in runs]
    assert eng.state.kv_bytes() == sum(l.k.numel() * 4 for l in eng.state.kv)


# ------------------------------------------------------------------ whole sequences, cuts, batches
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_matches_the_oracle(name):
    raw, w = CASES[name], weights_of(CASES[name])
    p = {"a": prompt(raw, 210)}
    got = run(engine_of(raw, w), [[("a", 210)]], p)["a"]
    assert error(got, O.forward(raw, w, p["a"])) < TOL


@pytest.mark.parametrize("name,sizes", [("mixed", [2]), ("mixed", [1]), ("tail", [2, 31, 3, 1, 64]), ("unit", [5, 1])])
def test_portions_and_single_tokens_match_the_whole_prompt(name, sizes):
    raw, w = CASES[name], weights_of(CASES[name])
    p = {"a": prompt(raw, 130)}
    got = run(engine_of(raw, w), [[("a", c)] for c in portions(130, sizes)], p)["a"]
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


def test_loop_order_and_first_pass_matter():
    """The oracle itself with the loop bookkeeping changed differs visibly: the comparisons above would show such a fault."""
    raw, w = MIXED, weights_of(MIXED)
    ids = prompt(raw, 40)
    ref = O.forward(raw, w, ids)
    no_step = dict(w, **{"loop.step": torch.zeros_like(w["loop.step"])})
    swapped = dict(w, **{"loop.step": w["loop.step"].flip(0)})
    for other in (O.forward(raw, no_step, ids), O.forward(raw, swapped, ids), O.forward(dict(raw, loop=dict(raw["loop"], times=2)), w, ids)):
        assert error(other, ref) > 1000 * TOL


@pytest.mark.parametrize("mistake", ["chunk+1", "chunk-1", "no sink", "state lost", "scale", "tau", "no bias"])
def test_the_inputs_make_single_mistakes_visible(mistake, monkeypatch):
    raw, w = copy.deepcopy(TAIL), dict(weights_of(TAIL))
    ids = prompt(raw, 120)
    ref = O.forward(raw, w, ids)
    left = [l["mixer"]["left"] for l in raw["layers"]]
    if mistake.startswith("chunk"):
        left[0]["mask"]["size"] += int(mistake[5:])
    elif mistake == "scale":
        left[0]["scale"] *= 1.02
    elif mistake == "tau":
        raw["layers"][1]["mixer"]["right"]["tau"] *= 1.05
    elif mistake == "no sink":
        w["l0.mix.left.sink"] = torch.full_like(w["l0.mix.left.sink"], -1e4)
    elif mistake == "no bias":
        w["l1.mix.left.k.b"] = torch.zeros_like(w["l1.mix.left.k.b"])
    else:
        whole = O.gated_linear_recurrence

        def cut(q, k, v, alpha, state=None):
            a, _ = whole(q[:60], k[:60], v[:60], alpha[:60])
            b, s = whole(q[60:], k[60:], v[60:], alpha[60:])
            return torch.cat([a, b]), s
        monkeypatch.setattr(O, "gated_linear_recurrence", cut)
    assert error(O.forward(raw, w, ids), ref) > 50 * TOL


# ------------------------------------------------------------------ scheduler, sampling, prefix cache
def test_greedy_serving_matches_the_oracle():
    raw, w = TAIL, weights_of(TAIL)
    eng = engine_of(raw, w, slots=2)
    srv = ServingEngine(eng, max_step_tokens=24)
    prompts = [prompt(raw, n, 20 + n) for n in (37, 3, 61)]
    ids = [srv.submit(p, 6) for p in prompts]
    ev = srv.run_until_idle()
    for rid, p in zip(ids, prompts):
        assert [e.token_id for e in ev if e.kind == "token" and e.request_id == rid] == O.greedy(raw, w, p, 6)
    assert eng.generate(prompts[0], 4, prefill_chunk=10) == O.greedy(raw, w, prompts[0], 4)


def test_prefix_cache_restores_keys_and_state():
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


def test_sampling_is_deterministic_and_follows_the_logit_scale():
    raw, w = MIXED, weights_of(MIXED)
    eng = engine_of(raw, w)
    p = prompt(raw, 12)
    a = eng.generate(p, 8, temperature=0.8, top_k=20, seed=5)
    assert a == eng.generate(p, 8, temperature=0.8, top_k=20, seed=5) and all(0 <= t < raw["vocab"] for t in a)


# ------------------------------------------------------------------ model directories, command line, trace runner
def _save(raw, w, path):
    cfg = GebuzenConfig.from_dict(raw)
    assert set(tensor_shapes(cfg)) == set(w)
    save_hf_model(path, cfg, w)
    return path


def test_compute_and_cli_paths_run_a_model_directory(tmp_path, capsys):
    from phaseshift_b200.apps import compute
    raw, w = TAIL, weights_of(TAIL)
    d = _save(raw, w, tmp_path / "m")
    p = prompt(raw, 9)
    (tmp_path / "ids").write_text(" ".join(map(str, p)))
    assert compute.main(["--model-dir", str(d), "--device", "cpu", "--input-ids-file", str(tmp_path / "ids"), "--max-new-tokens", "4"]) == 0
    out = capsys.readouterr().out
    assert "GENERATED_IDS=" + ",".join(map(str, O.greedy(raw, w, p, 4))) in out
    assert compute.main(["--random-model", "gebuzen-tiny", "--device", "cpu", "--max-new-tokens", "2"]) == 0
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
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = O.forward(raw, w, a), O.forward(raw, w, b)
    want = {0: [la[0], la[12]], 2: [lb[20], la[29], la[13]], 3: [lb[4]]}
    assert not (tmp_path / "o" / "1.f32").exists()
    for s, rows in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{s}.f32", dtype="<f4").reshape(len(rows), raw["vocab"]))
        assert error(got, torch.stack(rows)) < 5e-5, s


def test_trace_steps_larger_than_an_engine_step_are_cut(monkeypatch):
    from phaseshift_b200.apps import trace_run
    monkeypatch.setattr(trace_run, "MAX_STEP_ROWS", 16)
    r = trace_run.TraceRunner(None, ".")
    e = [{"tokens": list(range(10))}, {"tokens": list(range(30))}, {"tokens": [1]}]
    steps = r._portions(e)
    assert [sum(n for _, _, n in s) for s in steps] == [16, 16, 9]
    assert steps == [[(0, 0, 10), (1, 0, 6)], [(1, 6, 16)], [(1, 22, 8), (2, 0, 1)]]


# ------------------------------------------------------------------ the restatement itself
def test_oracle_mechanisms_by_hand():
    assert O.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    p = O.softmax_with_sink(torch.zeros(1, 2, 2, dtype=torch.float64), O.chunk_mask(2, 2), torch.tensor([math.log(2.0)]).double())
    assert torch.allclose(p[0], torch.tensor([[1 / 3, 0.0], [0.25, 0.25]]).double())
    assert math.isclose(float(O.channel_decay(torch.tensor(0.0).double(), 2.0)), 0.5 ** 0.5)
    q = k = v = torch.ones(2, 1, 1, dtype=torch.float64)
    o, s = O.gated_linear_recurrence(q, k, v, torch.full((2, 1, 1), 0.25).double())
    assert o.flatten().tolist() == [1.0, 1.25] and float(s) == 1.25
    assert UNIT["layers"][0]["mixer"]["left"]["mask"]["size"] == 1
