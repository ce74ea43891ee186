"""Configurations and helpers shared by the Luvutar tests: small models of unequal, awkward sizes with peaked attention."""
import torch

from gebuzen_cases import error, portions, prompt, run  # noqa: F401  (shared by the tests of this design)
from phaseshift_b200.models.luvutar.config import LuvutarConfig
from phaseshift_b200.models.luvutar.weights import build_engine_weights, random_weights
from phaseshift_b200.runtime.engine import Engine
from phaseshift_b200.runtime.state import StateConfig


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, ff, scale=None, base=1000.0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}, "mask": {"size": window}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads, kv, dim, vdim, ff, bias_max=70, coef=0.4, every=24, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": bias_max,
         "q_temp": {"coef": coef, "every": every}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, streams, layers, eps=1e-5):
    return {"architecture": "Luvutar", "vocab": vocab, "width": width, "streams": streams, "layers": layers, "norm": {"eps": eps}}


# odd width, vocabulary and feed-forward, layers without a feed-forward, values wider and narrower than keys, a window shorter
# than a page, keys shared by two later layers with scales, temperatures and biases of their own
MIXED = model(301, 75, 3, [attention(6, 2, 40, 24, 101, bias_max=50), latent(5, 24, 8, 40, 33, 50, 7, None),
                           attention(6, 2, 40, 24, None, 90, 0.2, 7, 0.3, kv_from=0), latent(3, 40, 22, 16, 20, 72, 41, 64, base=50.0),
                           attention(4, 4, 32, 48, 96, bias_max=33, every=100), attention(6, 2, 40, 24, 33, 20, 0.0, 5, kv_from=0)])
# shapes of the tensor-core kernels: 64-column groups, query heads that share key heads, latents in one and two value parts
WIDE = model(520, 192, 4, [latent(6, 128, 64, 128, 96, 512, 150, 160), attention(6, 2, 128, 128, 96),
                           attention(6, 2, 128, 128, 64, 100, 0.7, 16, kv_from=1), latent(20, 64, 64, 64, 64, 256, 64, 128),
                           attention(8, 1, 256, 256, 128, scale=0.05)])
# one of everything: one stream, one head, a window of the position itself, two buckets, a temperature step at every position
UNIT = model(64, 64, 1, [latent(1, 32, 2, 32, 32, 32, 1, 64, scale=1.0), attention(1, 1, 32, 32, 64, bias_max=2, coef=1.0, every=1, scale=0.05),
                         attention(1, 1, 32, 32, None, bias_max=2, every=1, scale=0.05, kv_from=1)])
# sizes beyond the tiled kernels: many streams, a wide latent, wide heads, many query heads on one key head, several row tiles
TAIL = model(200, 128, 5, [latent(2, 200, 40, 72, 48, 600, 90, 100), attention(16, 1, 32, 32, None, bias_max=200),
                           attention(2, 2, 288, 264, 96, every=50), latent(40, 16, 16, 16, 40, 64, 300, 128),
                           attention(16, 1, 32, 32, 64, kv_from=1), latent(9, 100, 130, 300, 40, 96, 33, None)])
CASES = {"mixed": MIXED, "wide": WIDE, "unit": UNIT, "tail": TAIL}


def weights_of(raw, seed=0, peak=2.0, buckets=None):
    """Random weights with queries and keys scaled so that single keys stand out, and sinks and biases of the size of the scores."""
    if buckets is None:
        buckets = min([14] + [L["mixer"]["bias_max"] for L in raw["layers"] if L["type"] == "attention"])
    w = random_weights(LuvutarConfig.from_dict(raw), seed, buckets=buckets)
    for n in list(w):
        leaf = n.rsplit(".", 1)[-1]
        if leaf in ("uq", "uk", "q", "k") and ".mix." in n:
            w[n] = (w[n].float() * peak).to(torch.bfloat16)
        elif leaf == "sink":
            w[n] = (w[n].float() * 2 + 1.5).to(torch.bfloat16)
        elif leaf == "rel":
            w[n] = (w[n].float() * 1.5).to(torch.bfloat16)
    return w


def engine_of(raw, w, device="cpu", dtype=None, slots=3, max_len=400, page=16, capacity=0, graphs=True):
    ew = build_engine_weights(LuvutarConfig.from_dict(raw), lambda n: w[n], device, dtype)
    return Engine(ew, device, StateConfig(max_slots=slots, max_seq_len=max_len, page_tokens=page, kv_capacity_tokens=capacity),
                  use_graphs=graphs)
