"""trace_run: feed given token ids through a model step by step and write the logits that each step asks for.

Standard input holds one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

The entries of a step form one batch of the engine; ``want`` are the places among an entry's tokens whose logits go to
``OUT/<step>.f32`` (little-endian f32, [wanted, vocab], in the order of the entries); ``end`` names requests whose slot and
pages are given back after the step.  Every finished step is acknowledged with a line ``done <step>``.  Nothing is sampled:
the steps run on the engine's own step function, cache and kernels, exactly as generation does.

Exit codes: 0 at the end of the input, 2 for bad arguments, 3 when the model's family has no kernels for ``--dtype``.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, List, Optional

PAGE_TOKENS = 16
MAX_LIVE = 4                      # requests live at any time
MAX_STEP_ROWS = 2048              # rows of one engine step; a larger trace step runs as several


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="model directory (config.json, *.safetensors)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most: the size of the cache pool")
    ap.add_argument("--device", default="cuda:0", help="cuda:N, or cpu for the 32-bit reference ops")
    return ap


class TraceRunner:
    def __init__(self, engine, out_dir):
        self.eng, self.out = engine, Path(out_dir)
        self.live: Dict[str, object] = {}

    def _portions(self, entries):
        """Engine steps that together bring the entries' tokens: [(entry index, first token, count), ...] of at most
        MAX_STEP_ROWS rows each (one step, unless the entries are larger than that)."""
        steps, cur, room = [], [], MAX_STEP_ROWS
        for i, e in enumerate(entries):
            at, n = 0, len(e["tokens"])
            while at < n:
                if room == 0:
                    steps.append(cur)
                    cur, room = [], MAX_STEP_ROWS
                take = min(room, n - at)
                cur.append((i, at, take))
                at, room = at + take, room - take
        return steps + ([cur] if cur else [])

    def step(self, msg: dict) -> None:
        import numpy as np
        from ..runtime.batch import SeqRows
        entries = msg.get("entries", [])
        logits: List[List[object]] = [[None] * len(e.get("want", [])) for e in entries]
        for portion in self._portions(entries):
            rows, seqs, places = [], [], []
            for i, at, n in portion:
                e = entries[i]
                s = self.live.get(e["id"])
                if s is None:
                    s = self.live[e["id"]] = self.eng.open_sequence()
                want = [(w - at, (i, j)) for j, w in enumerate(e.get("want", [])) if at <= w < at + n]
                rows.append(SeqRows(s.slot, s.position, e["tokens"][at:at + n], tuple(w for w, _ in want)))
                seqs.append(s)
                places += [p for _, p in want]
            _, out = self.eng.step(rows, seqs, sample=False, want_logits=True)
            if places:
                lg = out.logits[:len(places)].float().cpu().numpy()
                for row, (i, j) in zip(lg, places):
                    logits[i][j] = row.copy()
        flat = [r for rs in logits for r in rs]
        if flat:
            np.stack(flat).astype("<f4").tofile(self.out / f"{msg['step']}.f32")
        for rid in msg.get("end", []):
            s = self.live.pop(rid, None)
            if s is not None:
                self.eng.close_sequence(s)


def build_engine(model_dir, dtype: str, max_tokens: int, device: str = "cuda:0"):
    import torch
    from ..models import registry
    from ..runtime.engine import Engine
    from ..runtime.state import StateConfig
    dev = torch.device(device)
    ew = registry.load_weights(model_dir, dev, None, registry.DTYPES[dtype])
    sc = StateConfig(max_slots=MAX_LIVE, max_seq_len=max_tokens, page_tokens=PAGE_TOKENS, kv_capacity_tokens=max_tokens)
    return Engine(ew, dev, sc)


def main(argv: Optional[List[str]] = None) -> int:
    a = build_parser().parse_args(argv)
    if a.max_tokens < 1:
        print("trace_run: --max-tokens must be positive", file=sys.stderr)
        return 2
    from ..models.registry import UnsupportedOption
    try:
        eng = build_engine(a.model, a.dtype, a.max_tokens, a.device)
    except UnsupportedOption as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3
    Path(a.out).mkdir(parents=True, exist_ok=True)
    run = TraceRunner(eng, a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        run.step(msg)
        print(f"done {msg['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
