"""Configurations and helpers shared by the Gebuzen tests: small models of unequal, awkward sizes with peaked attention."""
import torch

from phaseshift_b200.models.gebuzen.config import GebuzenConfig
from phaseshift_b200.models.gebuzen.weights import build_engine_weights, random_weights
from phaseshift_b200.runtime.batch import SeqRows
from phaseshift_b200.runtime.engine import Engine
from phaseshift_b200.runtime.state import StateConfig


def layer(heads, kv, dim, scale, chunk, rh, rd, rv, tau, ff):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale,
                                                   "mask": {"size": chunk}},
                                          "right": {"heads": rh, "dim": rd, "vdim": rv, "tau": tau}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, layers, loop=None, residual=0.7, logit=0.25, eps=1e-5):
    d = {"architecture": "Gebuzen", "vocab": vocab, "width": width, "layers": layers, "residual_mult": residual,
         "logit_scale": logit, "norm": {"eps": eps}}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# every layer different, a layer without a feed-forward inside the loop, odd width / vocabulary / feed-forward, 16 query heads
# on one key head, head sizes that need padding, a chunk shorter than a page
MIXED = model(301, 75, [layer(6, 2, 40, 0.3, 33, 3, 24, 20, 5.0, 101), layer(16, 1, 32, 0.2, 7, 2, 64, 64, 1.0, None),
                        layer(4, 4, 64, 0.1, 64, 1, 16, 96, 16.0, 64)], loop=(1, 3, 3))
# the shapes of the tensor-core attention kernels and of the register-resident recurrence; no loop
WIDE = model(520, 192, [layer(6, 2, 256, 0.05, 150, 2, 128, 128, 16.0, 160), layer(4, 1, 128, 0.08, 96, 3, 64, 64, 4.0, 96)])
# one layer, looped from the first to the last with one pass, a chunk of one position, a unit scale and unit multipliers
UNIT = model(64, 64, [layer(2, 2, 32, 1.0, 1, 1, 32, 32, 1.0, 64)], loop=(0, 1, 1), residual=1.0, logit=1.0)
# the last layer has no feed-forward; the loop ends before it
TAIL = model(200, 128, [layer(8, 2, 64, 0.125, 50, 2, 32, 64, 8.0, 200), layer(8, 8, 96, 0.1, 81, 4, 48, 32, 2.0, 96),
                        layer(2, 1, 160, 0.08, 1000, 2, 80, 160, 3.0, None)], loop=(0, 2, 2), residual=0.4, logit=1.5)
CASES = {"mixed": MIXED, "wide": WIDE, "unit": UNIT, "tail": TAIL}


def weights_of(raw, seed=0, peak=2.0, rank=11):
    """Random weights with q and k scaled so that single keys stand out, and sinks of the size of the scores."""
    w = random_weights(GebuzenConfig.from_dict(raw), seed, decay_rank=rank)
    for n in list(w):
        if ".left.q" in n or ".left.k" in n:
            w[n] = (w[n].float() * peak).to(torch.bfloat16)
        elif n.endswith(".sink"):
            w[n] = (w[n].float() * 2 + 1.5).to(torch.bfloat16)
    return w


def engine_of(raw, w, device="cpu", dtype=None, slots=3, max_len=400, page=16, capacity=0, graphs=True):
    ew = build_engine_weights(GebuzenConfig.from_dict(raw), lambda n: w[n], device, dtype)
    return Engine(ew, device, StateConfig(max_slots=slots, max_seq_len=max_len, page_tokens=page, kv_capacity_tokens=capacity),
                  use_graphs=graphs)


def prompt(raw, n, seed=1):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, raw["vocab"], (n,), generator=g).tolist()


def run(eng, plan, prompts):
    """plan: list of steps, a step is a list of (request, number of its next tokens).  Returns request -> logits [n, vocab]
    over all its tokens so far (cpu, float32); requests are closed when their prompt is used up."""
    live, out = {}, {}
    for step in plan:
        rows, seqs = [], []
        for r, n in step:
            s = live.get(r)
            if s is None:
                s = live[r] = eng.open_sequence()
            rows.append(SeqRows(s.slot, s.position, prompts[r][s.position:s.position + n], tuple(range(n))))
            seqs.append(s)
        _, o = eng.step(rows, seqs, sample=False, want_logits=True)
        at = 0
        for (r, n), s in zip(step, seqs):
            out.setdefault(r, []).append(o.logits[at:at + n].float().cpu().clone())
            at += n
            if s.position == len(prompts[r]):
                eng.close_sequence(live.pop(r))
    for s in live.values():
        eng.close_sequence(s)
    return {r: torch.cat(v) for r, v in out.items()}


def portions(n, sizes):
    """n cut into portions that cycle through `sizes`."""
    out, i = [], 0
    while n > 0:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n, i = n - c, i + 1
    return out


def error(got, want):
    """Worst row: rms of the logit difference (mean removed) over the standard deviation of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().std())
