"""Configurations and helpers shared by the Fudulix tests: small models of unequal, awkward sizes with peaked attention and, where
rounding must not move a token to another expert, routers whose decisions have wide margins."""
import torch

from gebuzen_cases import error, portions, prompt, run  # noqa: F401  (shared by the tests of this design)
from phaseshift_b200.models.fudulix.config import FudulixConfig
from phaseshift_b200.models.fudulix.weights import build_engine_weights, random_weights
from phaseshift_b200.runtime.engine import Engine
from phaseshift_b200.runtime.state import StateConfig


def unit(heads, kv, dim, vdim, window, scale, rot=None, base=900.0, mix=True, factor=4.0, low=1.0, high=4.0, original=100):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": mix, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot or dim, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}}}


def conv(heads, kv, dim, vdim, window, keep, taps, scale=None, rot=None, base=5000.0, mix=True, factor=8.0, original=300, fast=16.0, slow=1.0):
    return {"type": "attention_2",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "v_mix": mix, "conv": taps,
                      "mask": {"size": window, "keep_first": keep},
                      "rot": {"base": base, "dims": rot or dim, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, ff, top, groups=1, keep=1, identity=0, shared=32):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep},
                                                            "identity": identity}, "shared": {"ff": shared}}


def model(vocab, width, layers, eps=1e-5, buckets=97, mul_prev=31, mul_cur=5):
    return {"architecture": "Fudulix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": [{**a, "mlp": b} for a, b in layers]}


# odd width, vocabulary and feed-forwards, both kinds of feed-forward behind both mixers, layers without one, without value mixing
# and with other head counts of equal value size, windows shorter than a page, values wider and narrower than keys
MIXED = model(301, 75, [(conv(6, 2, 40, 24, 9, 5, 3), moe(10, 33, 3, 3, 2, 2, 50)), (unit(5, 1, 24, 48, 33, 0.5, rot=14), dense(101)),
                        (unit(4, 4, 36, 20, 17, 0.4, mix=False), moe(6, 40, 2, 4, 3, 2, 21)), (conv(9, 3, 32, 16, 40, 70, 5, rot=18), None),
                        (unit(6, 2, 70, 24, 25, 0.3), dense(64))])
# shapes of the tensor-core kernels: heads of 64 to 256 columns, query heads that share key heads, many experts
WIDE = model(520, 192, [(unit(6, 2, 128, 128, 150, 0.25, rot=32, original=60), dense(160)),
                        (conv(4, 2, 256, 128, 100, 40, 4, base=20.0), moe(30, 64, 4, 4, 2, 2, 96)),
                        (unit(4, 2, 64, 128, 64, 0.4), moe(15, 80, 5, 1, 1, 3, 64)), (conv(8, 1, 192, 256, 70, 130, 2, original=50), dense(96))])
# one of everything: one head, a window of the position itself, one tap, no kept token, one expert, one group, one bucket
UNIT = model(64, 64, [(conv(1, 1, 32, 32, 1, 0, 1), moe(1, 32, 1, shared=32)), (unit(1, 1, 32, 32, 1, 1.0, rot=2, factor=1.0), dense(32)),
                      (conv(1, 1, 2, 32, 1, 1, 1, factor=1.0), moe(1, 32, 1, 2, 1, 1, 64))], buckets=1)
# sizes beyond the tiled kernels: many query heads on one key head, heads wider than 256, a long convolution, every expert chosen,
# only identity experts left in some groups
TAIL = model(200, 128, [(conv(16, 1, 32, 32, 50, 20, 7), moe(41, 20, 6, 9, 4, 4, 64)), (unit(2, 2, 288, 16, 90, 0.2), dense(100)),
                        (unit(32, 2, 48, 16, 1000, 0.4), moe(4, 96, 6, 1, 1, 2, 33)), (conv(3, 1, 100, 260, 33, 300, 4, mix=False), moe(8, 32, 2, 5, 2, 2, 32)),
                        (conv(12, 4, 64, 8, 16, 16, 4), dense(64))])
CASES = {"mixed": MIXED, "wide": WIDE, "unit": UNIT, "tail": TAIL}

CLASSES = 8


def weights_of(raw, seed=0, peak=2.0, classes=False):
    """Random weights with query and key norms scaled so that single keys stand out and corrections that matter.  ``classes``: the
    first dimensions of the residual hold a class of the token that nothing but identity experts adds to, and routers read only
    those: every class has an order of the experts of its own, with gaps that rounding cannot close."""
    w = random_weights(FudulixConfig.from_dict(raw), seed)
    g = torch.Generator().manual_seed(seed + 99)
    for n in list(w):
        if n.endswith((".q.norm", ".k.norm")):
            w[n] = (w[n].float() * peak).to(torch.bfloat16)
        elif n.endswith("correction"):
            pick = torch.randint(0, 5, w[n].shape, generator=g)
            shift = (pick == 0) * 1.5 - (pick == 1) * 1.5 if classes else 0.1 * torch.randn(w[n].shape, generator=g)
            w[n] = (shift - 1.25).to(torch.bfloat16)
    if not classes:
        return w
    C = CLASSES
    w["embed"][:, :C] = 0
    w["embed"][torch.arange(raw["vocab"]), torch.randint(0, C, (raw["vocab"],), generator=g)] = 6.0
    w["bigram"][:, :C] = 0
    for n in list(w):
        if n.endswith((".o", ".down")):
            w[n][:C] = 0
        elif n.endswith("down.b"):
            w[n][:C] = 0
        elif n.endswith("router"):
            r = torch.zeros(w[n].shape)
            for c in range(C):
                r[:, c] = min(0.25, 3.0 / r.shape[0]) * torch.randperm(r.shape[0], generator=g)
            w[n] = r.to(torch.bfloat16)
    return w


def engine_of(raw, w, device="cpu", dtype=None, slots=3, max_len=400, page=16, capacity=0, graphs=True):
    ew = build_engine_weights(FudulixConfig.from_dict(raw), lambda n: w[n], device, dtype)
    return Engine(ew, device, StateConfig(max_slots=slots, max_seq_len=max_len, page_tokens=page, kv_capacity_tokens=capacity),
                  use_graphs=graphs)
