"""Luvutar on the reference ops (CPU, fp32) against the plain restatement in luvutar_oracle.py: configuration, loading, every
mechanism, the cache under portions, batches and reuse, serving, the prefix cache, the trace runner."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import luvutar_oracle as O
from luvutar_cases import CASES, MIXED, TAIL, WIDE, engine_of, error, portions, prompt, run, weights_of
from phaseshift_b200.io.model_dir import save_hf_model
from phaseshift_b200.models import registry
from phaseshift_b200.models.luvutar.config import LuvutarConfig
from phaseshift_b200.models.luvutar.weights import tensor_shapes
from phaseshift_b200.ops.specs import distance_bias_table
from phaseshift_b200.runtime.serving import ServingEngine

ROOT = Path(__file__).resolve().parents[1]
TOL = 6e-5


# ------------------------------------------------------------------ configuration, registry, loading
def test_config_round_trip_and_registry(tmp_path):
    cfg = LuvutarConfig.from_dict(MIXED)
    cfg.save(tmp_path)
    again = registry.config_from_dir(tmp_path)
    assert again.to_dict() == cfg.to_dict() and again.family == "luvutar"
    assert registry.family_of_dir(tmp_path).name == "luvutar"
    assert [cfg.kv_layer(i) for i in range(6)] == [0, 1, 0, 3, 4, 0]
    assert {"luvutar-tiny", "luvutar-4b", "luvutar-27b"} <= set(registry.preset_names())
    assert registry.preset_config("luvutar-4b").family == "luvutar" and registry.preset_config("tiny").family == "qwen35"


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"),
                                    lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][0]["mixer"].update(kv_heads=4),
                                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=4),
                                    lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
                                    lambda d: d["layers"][2]["mixer"].update(kv_from=1),
                                    lambda d: d["layers"][2]["mixer"].update(kv_from=4),
                                    lambda d: d["layers"][2]["mixer"].update(dim=32),
                                    lambda d: d["layers"][5]["mixer"].update(kv_from=2),
                                    lambda d: d.update(streams=0)])
def test_config_refuses_what_the_design_does_not_have(change):
    d = copy.deepcopy(MIXED)
    change(d)
    with pytest.raises(ValueError):
        LuvutarConfig.from_dict(d)


def test_options_the_family_does_not_have_are_refused():
    cfg = registry.preset_config("luvutar-tiny")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", "nvfp4")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", tp_rank=0, tp_size=2)
    from phaseshift_b200.runtime.state import ModelState, StateConfig
    with pytest.raises(ValueError, match="bf16"):
        ModelState(cfg, StateConfig(kv_dtype="fp8_e4m3"), torch.device("cpu"), torch.bfloat16)


def test_cache_holds_latents_once_and_nothing_for_shared_keys():
    eng = engine_of(MIXED, weights_of(MIXED))
    kv = eng.state.kv
    assert [l is None for l in kv] == [False, False, True, False, False, True]
    assert [l.v is l.k for l in kv if l is not None] == [False, True, True, False]
    assert tuple(kv[1].k.shape[1:]) == (1, 16, 128) and tuple(kv[4].k.shape[1:]) == (4, 16, 64)      # padded latent + rotated part


@pytest.mark.parametrize("rows,far", [(2, 2), (4, 3), (14, 50), (32, 128), (64, 1000)])
def test_bias_table_by_distance(rows, far):
    table = torch.arange(rows * 2.0).reshape(rows, 2)
    t = distance_bias_table(table, far)
    for n in range(2 * far):
        assert t[0, min(n, t.shape[1] - 1)] == table[O.distance_bucket(n, rows, far), 0], n


# ------------------------------------------------------------------ whole sequences, cuts, batches
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_matches_the_oracle(name):
    raw, w = CASES[name], weights_of(CASES[name])
    p = {"a": prompt(raw, 210)}
    got = run(engine_of(raw, w), [[("a", 210)]], p)["a"]
    assert error(got, O.forward(raw, w, p["a"])) < TOL


@pytest.mark.parametrize("name,sizes", [("mixed", [2]), ("mixed", [1]), ("tail", [2, 31, 3, 1, 64]), ("unit", [5, 1]), ("wide", [2, 64, 1])])
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


MISTAKES = {
    "window + 1": lambda d, w: d["layers"][3]["mixer"]["mask"].update(size=42),
    "window - 1": lambda d, w: d["layers"][1]["mixer"]["mask"].update(size=6),
    "scale": lambda d, w: d["layers"][0]["mixer"].update(scale=d["layers"][0]["mixer"]["scale"] * 1.02),
    "rotation base": lambda d, w: d["layers"][3]["mixer"]["rot"].update(base=60.0),
    "temperature step": lambda d, w: d["layers"][2]["mixer"]["q_temp"].update(every=8),
    "temperature size": lambda d, w: d["layers"][0]["mixer"]["q_temp"].update(coef=0.42),
    "bias end": lambda d, w: d["layers"][4]["mixer"].update(bias_max=36),
    "keys of its own": lambda d, w: (d["layers"][2]["mixer"].pop("kv_from"), w.update({"l2.mix.k": w["l0.mix.k"], "l2.mix.v": w["l0.mix.v"]})),
    "no sink": lambda d, w: w.update({"l1.mix.sink": torch.full_like(w["l1.mix.sink"], -1e4)}),
    "mix turned around": lambda d, w: w.update({"l3.hc1.mix": w["l3.hc1.mix"].T}),
    "eps": lambda d, w: d["norm"].update(eps=3e-3),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_the_inputs_make_single_mistakes_visible(mistake):
    """The oracle itself with one thing changed differs visibly: the comparisons of these tests would show such a fault."""
    raw, w = copy.deepcopy(MIXED), dict(weights_of(MIXED))
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
    ids = [srv.submit(p, 6) for p in prompts]
    ev = srv.run_until_idle()
    for rid, p in zip(ids, prompts):
        assert [e.token_id for e in ev if e.kind == "token" and e.request_id == rid] == O.greedy(raw, w, p, 6)
    assert eng.generate(prompts[0], 4, prefill_chunk=10) == O.greedy(raw, w, prompts[0], 4)


def test_prefix_cache_restores_latents_and_keys():
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
    cfg = LuvutarConfig.from_dict(raw)
    assert set(tensor_shapes(cfg)) == set(w)
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
    assert compute.main(["--random-model", "luvutar-tiny", "--device", "cpu", "--max-new-tokens", "2"]) == 0
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
    assert O.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    # eight rows, far end 16: one bucket each below 4, then a factor of two per two buckets, then the last for everything
    assert [O.distance_bucket(n, 8, 16) for n in (0, 3, 4, 5, 6, 8, 11, 12, 15, 16, 99)] == [0, 3, 4, 4, 5, 6, 6, 7, 7, 7, 7]
    t = O.query_temperature(9, 0.5, 4)
    assert t[:3].tolist() == [1.0] * 3 and math.isclose(float(t[3]), 1 + 0.5 * math.log(2)) and math.isclose(float(t[8]), 1 + 0.5 * math.log(3))
    p = O.softmax_with_sink(torch.zeros(1, 2, 2, dtype=torch.float64), O.window_mask(2, 1), torch.tensor([math.log(2.0)]).double())
    assert torch.allclose(p[0], torch.tensor([[1 / 3, 0.0], [0.0, 1 / 3]]).double())
    x = O.rotate_pairs(torch.tensor([[[1.0, 0.0, 0.0, 2.0]]]).double(), torch.tensor([1]), 4.0)[0, 0]
    assert torch.allclose(x, torch.tensor([math.cos(1), math.sin(1), -2 * math.sin(0.5), 2 * math.cos(0.5)]).double())
    X = torch.tensor([[[1.0]], [[10.0]]]).double()
    y = O.stream_write(X, torch.tensor([[2.0]]).double(), torch.tensor([[1.0, 2.0], [3.0, 4.0]]).double(), torch.tensor([0.5, 1.0]).double())
    assert y.flatten().tolist() == [32.0, 44.0]
