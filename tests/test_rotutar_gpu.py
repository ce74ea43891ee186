"""Rotutar through the engine on the CUDA kernels, in 32-bit and in bf16, against the plain restatement: whole prompts, single
tokens, portions, batches, reuse of pages and slots, long decoding from graphs, greedy serving, loading, the trace runner."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import rotutar_oracle as O
from phaseshift_b200.runtime.batch import SeqRows
from phaseshift_b200.runtime.serving import ServingEngine
from rotutar_cases import CASES, MIXED, TAIL, WIDE, engine_of, error, portions, prompt, run, weights_of

pytestmark = pytest.mark.gpu
TOL = {torch.float32: 1e-4, torch.bfloat16: 1e-1}
PEAK = {torch.float32: 2.0, torch.bfloat16: 1.0}         # attention that bf16 rounding does not amplify from layer to layer
DTYPES = [torch.float32, torch.bfloat16]
_ref = {}


def weights_for(raw, dtype):
    """In bf16 with routers that rounding cannot turn to another expert."""
    return weights_of(raw, peak=PEAK[dtype], classes=dtype == torch.bfloat16)


def reference(name, raw, w, ids, dtype):
    key = (name, dtype, tuple(ids))
    if key not in _ref:
        _ref[key] = O.forward(raw, w, ids)
    return _ref[key]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_single_tokens_and_portions(name, dtype):
    raw, w = CASES[name], weights_for(CASES[name], dtype)
    ids = prompt(raw, 230)
    want = reference(name, raw, w, ids, dtype)
    eng = engine_of(raw, w, "cuda:0", dtype)
    for plan in ([230], [1] * 230, portions(230, [2]), portions(230, [33, 2, 64, 1, 17, 3, 100]), [200] + [1] * 30):
        got = run(eng, [[("a", c)] for c in plan], {"a": ids})["a"]
        assert error(got, want) < TOL[dtype], plan[:4]
    assert int(eng.state.status) == 0 and eng.alloc.pages_free == eng.state.num_pages - 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "tail"])
def test_batches_equal_each_request_alone_and_reuse_pages(name, dtype):
    raw, w = CASES[name], weights_for(CASES[name], dtype)
    n = {"a": 150, "b": 40, "c": 5, "d": 90, "e": 61}
    p = {r: prompt(raw, k, 50 + i) for i, (r, k) in enumerate(n.items())}
    plan = ([[("a", 70), ("b", 2), ("c", 5)], [("a", 1), ("b", 38)], [("d", 37), ("a", 2), ("e", 1)]]
            + [[("a", 1), ("d", 1), ("e", 1)]] * 20 + [[("e", 40), ("a", 1)], [("a", 56), ("d", 33)]])
    eng = engine_of(raw, w, "cuda:0", dtype, capacity=272)
    for _ in range(2):
        got = run(eng, plan, p)
        for r in p:
            assert error(got[r], reference(name, raw, w, p[r], dtype)) < TOL[dtype], r
    assert eng.alloc.pages_free == eng.state.num_pages - 1


@pytest.mark.parametrize("dtype", DTYPES)
def test_windows_and_states_decoded_deep_into_a_sequence(dtype):
    """600 positions over windows of 64 to 150: decoding crosses window, page and kernel-tile borders with captured graphs."""
    raw, w = WIDE, weights_for(WIDE, dtype)
    ids = prompt(raw, 600)
    want = reference("wide", raw, w, ids, dtype)
    eng = engine_of(raw, w, "cuda:0", dtype, max_len=640)
    got = run(eng, [[("a", 280)]] + [[("a", 1)]] * 320, {"a": ids})["a"]
    assert error(got, want) < TOL[dtype]


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_bf16_prompts_and_decoding_agree_with_each_other(name):
    """The blocks of a prompt and the row-by-row form differ by rounding only, wherever the prompt is cut."""
    raw, w = CASES[name], weights_for(CASES[name], torch.bfloat16)
    ids = prompt(raw, 300, 9)
    eng = engine_of(raw, w, "cuda:0", torch.bfloat16)
    whole = run(eng, [[("a", 300)]], {"a": ids})["a"]
    for plan in ([299, 1], [150] + [1] * 150, portions(300, [65, 1, 64, 63])):
        got = run(eng, [[("a", c)] for c in plan], {"a": ids})["a"]
        assert error(got, whole) < TOL[torch.bfloat16], plan[:3]


def test_residual_after_every_layer():
    raw, w = MIXED, weights_of(MIXED)
    ids = prompt(raw, 50)
    want = []
    O.forward(raw, w, ids, after_layer=want)
    eng = engine_of(raw, w, "cuda:0", torch.float32)
    s = eng.open_sequence()
    _, o = eng.step([SeqRows(s.slot, 0, ids, (49,))], [s], sample=False, tap_layers=tuple(range(len(want))))
    for j, x in enumerate(want):
        assert float((o.taps[j][:50].cpu().double() - x).abs().max()) < 2e-5 * float(x.abs().max()), j


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_serving_in_32_bit_matches_the_oracle(graphs):
    raw, w = TAIL, weights_of(TAIL)
    eng = engine_of(raw, w, "cuda:0", torch.float32, slots=2, graphs=graphs)
    srv = ServingEngine(eng, max_step_tokens=32, prefix_cache_tokens=128, prefix_min_tokens=16)
    prompts = [prompt(raw, n, 20 + n) for n in (37, 3, 61)]
    ids = [srv.submit(p, 12, checkpoint_position=32 if len(p) > 32 else 0) for p in prompts]
    ev = srv.run_until_idle()
    for rid, p in zip(ids, prompts):
        assert [e.token_id for e in ev if e.kind == "token" and e.request_id == rid] == O.greedy(raw, w, p, 12)
    again = prompts[2][:32] + prompt(raw, 9, 5)
    rid = srv.submit(again, 6)
    ev = srv.run_until_idle()
    assert srv.request(rid)["restored_tokens"] == 32
    assert [e.token_id for e in ev if e.kind == "token"] == O.greedy(raw, w, again, 6)


def test_bf16_greedy_tokens_are_the_arg_max_of_the_logits():
    """Generation (fused arg-max of the unlimited logits, captured graphs) against limited logits read back from the same engine."""
    raw, w = WIDE, weights_for(WIDE, torch.bfloat16)
    eng = engine_of(raw, w, "cuda:0", torch.bfloat16)
    p = prompt(raw, 60)
    gen = eng.generate(p, 24)
    lg = run(eng, [[("a", 60)]] + [[("a", 1)]] * 24, {"a": p + gen})["a"]
    picked = lg[59:59 + 24].gather(1, torch.tensor(gen)[:, None])[:, 0]
    assert bool((lg[59:59 + 24].max(-1).values - picked < 3e-2 * lg.std()).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_decode_batches_beyond_eight_rows_replay_from_graphs(dtype):
    raw, w = WIDE, weights_for(WIDE, dtype)
    n = {f"r{i}": 30 + 7 * i for i in range(12)}
    p = {r: prompt(raw, k, 60 + i) for i, (r, k) in enumerate(n.items())}
    plan = [[(r, k - 12)] for r, k in n.items()] + [[(r, 1) for r in n]] * 12
    got = run(engine_of(raw, w, "cuda:0", dtype, slots=12, max_len=160), plan, p)
    for r in ("r0", "r5", "r11"):
        assert error(got[r], reference("wide", raw, w, p[r], dtype)) < TOL[dtype], r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_on_the_gpu(tmp_path, dtype):
    import numpy as np
    from phaseshift_b200.io.model_dir import save_hf_model
    from phaseshift_b200.models.rotutar.config import RotutarConfig
    dt = getattr(torch, dtype)
    raw, w = MIXED, weights_for(MIXED, dt)
    save_hf_model(tmp_path / "m", RotutarConfig.from_dict(raw), w)
    ids = prompt(raw, 80)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": ids[:60], "want": [59, 3]}], "end": []}] + \
            [{"step": 1 + i, "entries": [{"id": "q", "tokens": [t], "want": [0]}], "end": ["q"] if i == 19 else []} for i, t in enumerate(ids[60:])]
    exe = Path(__file__).resolve().parents[1] / "bin" / "trace_run"
    r = subprocess.run([sys.executable, str(exe), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "o"),
                        "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=500)
    assert r.returncode == 0, r.stderr[-2000:]
    want = reference("mixed", raw, w, ids, dt)
    got = [np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4").reshape(-1, raw["vocab"]) for i in range(21)]
    assert error(torch.from_numpy(got[0]), want[[59, 3]]) < TOL[dt]
    assert error(torch.from_numpy(np.concatenate(got[1:])), want[60:]) < TOL[dt]
