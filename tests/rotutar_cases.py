"""Configurations and helpers shared by the Rotutar tests: small models of unequal, awkward sizes with peaked attention and, where
rounding must not move a token to another expert, routers whose decisions have wide margins."""
import torch

from gebuzen_cases import error, portions, prompt, run  # noqa: F401  (shared by the tests of this design)
from phaseshift_b200.models.rotutar.config import RotutarConfig
from phaseshift_b200.models.rotutar.weights import build_engine_weights, random_weights
from phaseshift_b200.runtime.engine import Engine
from phaseshift_b200.runtime.state import StateConfig


def parallel(left, right, ls=0.8, rs=0.7):
    """left: (heads, kv_heads, dim, vdim, window, scale, rotated dims, base), right: (heads, kv_heads, dim, vdim, taps)"""
    h, g, d, v, window, scale, rot, base = left
    return {"type": "parallel",
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "scale": scale, "mask": {"size": window}, "rot": {"base": base, "dims": rot}},
                      "left_scale": ls, "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)), "right_scale": rs}}


def linear(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, ff, top, groups=1, keep=1, limit=0.7):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def model(vocab, width, groups, layers, eps=1e-5, cap=20.0):
    return {"architecture": "Rotutar", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "logit_softcap": cap,
            "layers": [{**a, "mlp": b} for a, b in layers]}


# odd width, vocabulary and feed-forwards, both feed-forwards behind both mixers, layers without one, values wider and narrower than
# keys, heads that share queries and keys, windows shorter than a page, one to five taps, scales of opposite sign
MIXED = model(301, 75, 3, [(parallel((6, 2, 40, 24, 9, 0.3, 40, 900.0), (6, 3, 20, 40, 3)), moe(12, 33, 3, 4, 2)), (linear(5, 24, 40), dense(101)),
                           (linear(2, 100, 16), moe(9, 40, 4, 3, 2, 1.5)), (parallel((5, 1, 24, 48, 33, 0.4, 14, 5000.0), (2, 1, 72, 24, 5), 1.3, -0.4), None),
                           (parallel((4, 4, 36, 20, 17, 0.5, 36, 50.0), (3, 3, 33, 70, 1)), dense(64))])
# shapes of the tensor-core kernels: heads of 64 to 256 columns, states of 64 and 128, many experts
WIDE = model(520, 160, 4, [(parallel((6, 2, 128, 128, 150, 0.2, 32, 10000.0), (4, 2, 128, 128, 4)), dense(160)), (linear(2, 128, 128), moe(32, 64, 4, 4, 2)),
                           (parallel((4, 2, 256, 128, 100, 0.1, 256, 20.0), (4, 1, 64, 128, 4)), moe(15, 80, 5, 1, 1, 2.0)),
                           (linear(3, 64, 64), dense(96)), (parallel((8, 1, 64, 64, 64, 0.3, 64, 300.0), (2, 2, 128, 64, 2)), dense(64))])
# one of everything: one group, one head, a window of the position itself, one tap, one expert, unit scales
UNIT = model(64, 64, 1, [(parallel((1, 1, 32, 32, 1, 1.0, 2, 10.0), (1, 1, 32, 32, 1), 1.0, 1.0), moe(1, 32, 1)), (linear(1, 32, 32), dense(32)),
                         (linear(1, 8, 4), None)], cap=1.0)
# sizes beyond the tiled kernels: heads wider than 256, states beyond 128 and 256 channels, a long convolution, many groups of two and
# of one expert, every expert chosen
TAIL = model(200, 128, 4, [(linear(2, 272, 40), moe(40, 20, 6, 20, 4)), (parallel((2, 2, 288, 16, 90, 0.2, 100, 700.0), (2, 1, 144, 96, 9)), dense(100)),
                            (linear(1, 48, 300), moe(6, 96, 6)), (parallel((32, 2, 48, 16, 1000, 0.4, 48, 80.0), (2, 2, 40, 160, 4)), moe(7, 32, 2, 7, 3, 0.3)),
                            (linear(9, 16, 64), dense(64))])
CASES = {"mixed": MIXED, "wide": WIDE, "unit": UNIT, "tail": TAIL}

CLASSES = 8


def weights_of(raw, seed=0, peak=2.0, classes=False, rank=11):
    """Random weights with query and key norms scaled so that single keys stand out, sinks of the size of the scores, forget gates that
    keep some channels for hundreds of tokens, decays of all speeds.  ``classes``: the first dimensions of the residual hold a class
    of the token that no sublayer adds to, and routers read only those: every class has an order of the experts of its own, with gaps
    that rounding cannot close."""
    w = random_weights(RotutarConfig.from_dict(raw), seed, rank=rank)
    g = torch.Generator().manual_seed(seed + 99)
    for n in list(w):
        if n.endswith((".q.norm", ".k.norm")):
            w[n] = (w[n].float() * peak).to(torch.bfloat16)
        elif n.endswith(".sink"):
            w[n] = (w[n].float() * 3 + 1.0).to(torch.bfloat16)
        elif n.endswith(".f.b"):
            w[n] = (w[n].float() * 4 + 1.5).to(torch.bfloat16)
        elif n.endswith(".dt_bias"):
            w[n] = (w[n].float() * 1.5).to(torch.bfloat16)
        elif n.endswith((".gate", ".up")) and ".e" in n:
            w[n] = (w[n].float() * 1.5).to(torch.bfloat16)                 # (the experts' limits are reached)
    if not classes:
        return w
    C = CLASSES
    w["embed"][:, :C] = 0
    w["embed"][torch.arange(raw["vocab"]), torch.randint(0, C, (raw["vocab"],), generator=g)] = 6.0
    for n in list(w):
        if n.endswith((".o", ".down")):
            w[n][:C] = 0
        elif n.endswith("router"):
            r = torch.zeros(w[n].shape)
            groups = raw["layers"][int(n[1:].split(".")[0])]["mlp"]["router"]["groups"]["count"]
            for c in range(C):
                r[:, c] = max((_order(r.shape[0], g) for _ in range(30)), key=lambda t: _gap(t, groups))
            w[n] = r.to(torch.bfloat16)
    return w


def _order(n, g):
    """A random order as weights of a class: sums of two scores are as good as never equal."""
    return ((torch.randperm(n, generator=g) + 1) / n) ** 1.4 - 0.37


def _gap(t, groups):
    """Smallest distance between two groups' sums of their two best scores."""
    s = torch.sigmoid(6.0 * t).reshape(groups, -1)
    s = s.topk(min(2, s.shape[1]), -1).values.sum(-1).sort().values
    return float((s[1:] - s[:-1]).min()) if groups > 1 else 1.0


def engine_of(raw, w, device="cpu", dtype=None, slots=3, max_len=400, page=16, capacity=0, graphs=True):
    ew = build_engine_weights(RotutarConfig.from_dict(raw), lambda n: w[n], device, dtype)
    return Engine(ew, device, StateConfig(max_slots=slots, max_seq_len=max_len, page_tokens=page, kv_capacity_tokens=capacity),
                  use_graphs=graphs)
