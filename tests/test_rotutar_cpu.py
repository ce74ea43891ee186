"""Rotutar on the reference ops (CPU, fp32) against the plain restatement in rotutar_oracle.py: configuration, loading, every
mechanism, the cache and state under portions, batches and reuse, serving, the prefix cache, the trace runner."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import rotutar_oracle as O
from phaseshift_b200.io.model_dir import save_hf_model
from phaseshift_b200.models import registry
from phaseshift_b200.models.rotutar.config import RotutarConfig
from phaseshift_b200.models.rotutar.weights import tensor_shapes
from phaseshift_b200.ops import specs
from phaseshift_b200.runtime.serving import ServingEngine
from rotutar_cases import CASES, MIXED, TAIL, WIDE, engine_of, error, portions, prompt, run, weights_of

ROOT = Path(__file__).resolve().parents[1]
TOL = 6e-5


# ------------------------------------------------------------------ configuration, registry, loading
@pytest.mark.parametrize("name", sorted(CASES))
def test_config_round_trip_and_registry(tmp_path, name):
    cfg = RotutarConfig.from_dict(CASES[name])
    assert cfg.to_dict() == CASES[name]
    cfg.save(tmp_path)
    again = registry.config_from_dir(tmp_path)
    assert again.to_dict() == cfg.to_dict() and again.family == "rotutar"
    assert registry.family_of_dir(tmp_path).name == "rotutar"


def test_presets_are_registered():
    assert {"rotutar-tiny", "rotutar-4b", "rotutar-27b"} <= set(registry.preset_names())
    assert registry.preset_config("rotutar-4b").family == "rotutar" and registry.preset_config("fudulix-tiny").family == "fudulix"


@pytest.mark.parametrize("change", [lambda d: d["layers"][0].update(type="other"),
                                    lambda d: d["layers"][0]["mlp"].update(kind="other"),
                                    lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4),
                                    lambda d: d["layers"][0]["mixer"]["right"].update(kv_heads=4),
                                    lambda d: d["layers"][0]["mixer"]["right"].update(conv=0),
                                    lambda d: d["layers"][3]["mixer"]["left"]["rot"].update(dims=13),
                                    lambda d: d["layers"][3]["mixer"]["left"]["rot"].update(dims=26),
                                    lambda d: d["layers"][3]["mixer"]["left"]["mask"].update(size=0),
                                    lambda d: d["norm"].update(groups=2),
                                    lambda d: d.update(logit_softcap=0.0),
                                    lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=5),
                                    lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=5),
                                    lambda d: d["layers"][0]["mlp"]["router"].update(top=7)])
def test_config_refuses_what_the_design_does_not_have(change):
    d = copy.deepcopy(MIXED)
    change(d)
    with pytest.raises(ValueError):
        RotutarConfig.from_dict(d)


def test_options_the_family_does_not_have_are_refused():
    cfg = registry.preset_config("rotutar-tiny")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", "nvfp4")
    with pytest.raises(registry.UnsupportedOption):
        registry.random_weights(cfg, "cpu", tp_rank=0, tp_size=2)


def test_state_holds_what_the_layers_carry():
    st = engine_of(MIXED, weights_of(MIXED)).state
    assert [k is None for k in st.kv] == [False, True, True, False, False]
    assert [tuple(r.rec.shape) for r in st.gdn] == [(3, 6, 64, 64), (3, 5, 32, 64), (3, 2, 112, 32), (3, 2, 128, 64), (3, 3, 64, 128)]
    assert [None if c is None else tuple(c.shape) for c in st.conv] == [(3, 2, 6 * 192), None, None, (3, 4, 2 * 320), None]
    assert len(st.slot_tensors()) == 7
    st.conv[0][1], st.gdn[1].rec[1] = 7.0, 5.0
    st.copy_slot(2, 1)
    assert bool((st.conv[0][2] == 7).all()) and bool((st.gdn[1].rec[2] == 5).all())
    st.reset_slot(2)
    assert all(bool((g.rec[2] == 0).all()) for g in st.gdn)


def test_clamped_gate():
    g, u = torch.tensor([-9.0, 0.5, 3.0, 3.0]), torch.tensor([4.0, -0.25, -7.0, 7.0])
    want = [x / (1 + math.exp(-1.702 * x)) * (y + 1) for x, y in ((-9.0, 2.0), (0.5, -0.25), (2.0, -2.0), (2.0, 2.0))]
    assert torch.allclose(specs.clamped_gate(g, u, 2.0), torch.tensor(want))


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
    "window + 1": lambda d, w: MIX(d, 3)["left"]["mask"].update(size=34),
    "window - 1": lambda d, w: MIX(d, 0)["left"]["mask"].update(size=8),
    "scale": lambda d, w: MIX(d, 3)["left"].update(scale=0.41),
    "rotation base": lambda d, w: MIX(d, 0)["left"]["rot"].update(base=1000.0),
    "rotated dimensions": lambda d, w: MIX(d, 3)["left"]["rot"].update(dims=16),
    "sink": lambda d, w: w["l4.mix.left.sink"].fill_(-90),
    "query norm": lambda d, w: w["l0.mix.left.q.norm"].mul_(1.05),
    "left scale": lambda d, w: MIX(d, 3).update(left_scale=1.25),
    "right scale": lambda d, w: MIX(d, 3).update(right_scale=0.4),
    "first tap": lambda d, w: w["l3.mix.right.k.conv"][:, 0].zero_(),
    "value convolution": lambda d, w: w["l0.mix.right.v.conv"][:, 1].mul_(1.1),
    "decay rate": lambda d, w: w["l0.mix.right.A_log"].add_(0.3),
    "decay bias": lambda d, w: w["l3.mix.right.dt_bias"].zero_(),
    "step size": lambda d, w: w["l4.mix.right.b"].zero_(),
    "output gate": lambda d, w: w["l0.mix.right.g2"].zero_(),
    "head norm": lambda d, w: w["l3.mix.right.norm"].fill_(1.0),
    "lower bound": lambda d, w: w["l1.mix.lower"].zero_(),
    "forget bias": lambda d, w: w["l2.mix.f.b"].add_(0.2),
    "head norm of the linear attention": lambda d, w: w["l1.mix.norm"].fill_(1.0),
    "bias of the result's gate": lambda d, w: w["l2.rg1.b"].zero_(),
    "gate of the feed-forward's result": lambda d, w: w["l4.rg2"].zero_(),
    "groups of the norm": lambda d, w: d["norm"].update(groups=5),
    "eps": lambda d, w: d["norm"].update(eps=3e-3),
    "soft limit": lambda d, w: d.update(logit_softcap=24.0),
    "expert limit": lambda d, w: d["layers"][2]["mlp"]["expert"].update(limit=1.7),
    "kept groups": lambda d, w: d["layers"][0]["mlp"]["router"]["groups"].update(keep=3),
    "chosen experts": lambda d, w: d["layers"][2]["mlp"]["router"].update(top=3),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_the_inputs_make_single_mistakes_visible(mistake):
    """The oracle itself with one thing changed differs visibly: the comparisons of these tests would show such a fault."""
    raw, w = copy.deepcopy(MIXED), {n: t.clone() for n, t in weights_of(MIXED).items()}
    ids = prompt(raw, 120)
    ref = O.forward(raw, w, ids)
    MISTAKES[mistake](raw, w)
    assert error(O.forward(raw, w, ids), ref) > 20 * TOL


@pytest.mark.parametrize("where", ["delta rule", "linear attention", "group norm of the whole row", "renormalised weights", "best member of a group"])
def test_the_inputs_make_mistakes_of_form_visible(where, monkeypatch):
    """... and so does another form of a mechanism."""
    raw, w = MIXED, weights_of(MIXED)
    ids = prompt(raw, 100)
    ref = O.forward(raw, w, ids)
    rule, forget, norm, route = O.delta_rule, O.forget_write, O.group_norm, O.route
    if where == "delta rule":                            # the state starts anew in the middle
        monkeypatch.setattr(O, "delta_rule", lambda *t: torch.cat([rule(*(x[:50] for x in t)), rule(*(x[50:] for x in t))]))
    elif where == "linear attention":
        monkeypatch.setattr(O, "forget_write", lambda *t: torch.cat([forget(*(x[:50] for x in t)), forget(*(x[50:] for x in t))]))
    elif where == "group norm of the whole row":
        monkeypatch.setattr(O, "group_norm", lambda x, w, eps, groups: norm(x, w, eps, 1))
    elif where == "renormalised weights":
        def share(*a):
            r = route(*a)
            return [(i, v / sum(x for _, x in r)) for i, v in r]
        monkeypatch.setattr(O, "route", share)
    else:
        def by_best(z, groups, keep, top):
            s, size = torch.sigmoid(z), len(z) // groups
            best = sorted(range(groups), key=lambda g: -float(s[g * size:(g + 1) * size].max()))[:keep]
            return [(i, s[i]) for i in sorted((i for i in range(len(z)) if i // size in best), key=lambda i: -float(s[i]))[:top]]
        monkeypatch.setattr(O, "route", by_best)
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


def test_prefix_cache_restores_keys_states_and_convolution_rows():
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
def _save(raw, w, path, rank=11):
    cfg = RotutarConfig.from_dict(raw)
    assert {n: tuple(t.shape) for n, t in w.items()} == tensor_shapes(cfg, rank)
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
    assert compute.main(["--random-model", "rotutar-tiny", "--device", "cpu", "--max-new-tokens", "2"]) == 0
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
    f64 = lambda x: torch.tensor(x).double()
    # two groups, each over its own root mean square
    assert torch.allclose(O.group_norm(f64([[3.0, 4.0, 0.0, 2.0]]), f64([1.0, 1.0, 1.0, 5.0]), 0.0, 2),
                          f64([[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0.0, 10 / math.sqrt(2.0)]]))
    x = O.turn_neighbours(f64([[[0.0] * 5], [[1.0, 2.0, 1.0, 0.0, 7.0]]]), 100.0, 4)[1, 0]
    assert torch.allclose(x, f64([math.cos(1) - 2 * math.sin(1), 2 * math.cos(1) + math.sin(1), math.cos(0.1), math.sin(0.1), 7.0]))
    p = O.softmax_with_sink(torch.zeros(2, 2, 2).double(), O.window_mask(2, 2), f64([0.0, math.log(3.0)]))
    assert torch.allclose(p, f64([[[1 / 2, 0.0], [1 / 3, 1 / 3]], [[1 / 4, 0.0], [1 / 5, 1 / 5]]]))
    # delta rule, one channel each: the second token decays the first's write, takes back half of what is there, and sees its own write
    o = O.delta_rule(f64([[[1.0]], [[2.0]]]), f64([[[1.0]], [[1.0]]]), f64([[[4.0]], [[6.0]]]), f64([[[0.9]], [[0.5]]]), f64([[1.0], [0.5]]))
    assert torch.allclose(o.flatten(), f64([4.0, 2 * (2.0 + 0.5 * (6.0 - 2.0))]))
    # forget gate: keeps 0.75, takes in a quarter
    o = O.forget_write(f64([[[1.0]], [[1.0]]]), f64([[[0.0]], [[0.75]]]), f64([[[8.0]], [[4.0]]]))
    assert torch.allclose(o.flatten(), f64([8.0, 7.0]))
    assert torch.allclose(O.forget_gate(f64([0.0]), f64([0.4])), f64([0.7]))
    y = O.short_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]]))
    assert y.flatten().tolist() == [1.0, 12.0, 24.0]
    # groups {0, 1}, {2, 3}, {4, 5}: the sum of both members counts, weights are the scores themselves
    z = torch.logit(f64([0.9, 0.1, 0.6, 0.5, 0.7, 0.2]))
    assert [(i, round(float(v), 6)) for i, v in O.route(z, 3, 1, 2)] == [(2, 0.6), (3, 0.5)]
    assert [i for i, _ in O.route(z, 3, 2, 3)] == [0, 2, 3] and [i for i, _ in O.route(z, 1, 1, 2)] == [0, 4]
    assert [i for i, _ in O.route(z, 6, 2, 2)] == [0, 4]
