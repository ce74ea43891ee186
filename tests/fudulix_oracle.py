"""Plain, slow restatement of the Fudulix decoder: one function per mechanism, whole sequences, no cache, no batching.
It shares nothing with the package; every engine path of this design is compared with it.

Weights are a dict of name -> tensor (any float dtype; computed in `dtype`), the configuration is the parsed JSON.
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ embedding
def bigram_rows(ids, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; the first token has the row behind the buckets."""
    return [buckets if i == 0 else (ids[i - 1] * mul_prev + ids[i] * mul_cur) % buckets for i in range(len(ids))]


def embedding(ids, w, cfg):
    b = cfg["embedding"]["bigram"]
    x = w["embed"][torch.tensor(ids)] + w["bigram"][torch.tensor(bigram_rows(ids, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return rms_norm(x, w["embed.norm"], cfg["norm"]["eps"])


# ------------------------------------------------------------------ positions
def base_frequencies(rot):
    return [rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def stepped_frequencies(rot):
    """Long wavelengths divided by the factor, short ones kept, a blend between the two limits."""
    s, out = rot["scaling"], []
    for f in base_frequencies(rot):
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - t) * f / s["factor"] + t * f)
    return out


def ramped_frequencies(rot):
    """Blend by the pair's index, between the pairs that turn `fast` and `slow` times within the original length; and the
    factor on sine and cosine."""
    s, n = rot["scaling"], rot["dims"]
    at = lambda turns: n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), n - 1)
    out = []
    for i, f in enumerate(base_frequencies(rot)):
        r = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def turn(x, first, second, freqs, size=1.0):
    """x [n, H, D]: dimensions first[i] and second[i] turn by position * freqs[i]."""
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    c, s = (torch.cos(ang) * size).to(x.dtype)[:, None], (torch.sin(ang) * size).to(x.dtype)[:, None]
    u, v = x[..., first], x[..., second]
    y = x.clone()
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


def turn_neighbours(x, freqs):
    n = 2 * len(freqs)
    return turn(x, list(range(0, n, 2)), list(range(1, n, 2)), freqs)


def turn_halves(x, freqs, size):
    n = len(freqs)
    return turn(x, list(range(n)), list(range(n, 2 * n)), freqs, size)


# ------------------------------------------------------------------ attention
def short_conv(u, w):
    """u [n, channels], w [channels, taps]; the last tap is the token's own."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + w[:, j] * u[t - taps + 1 + j]
    return y


def window_mask(n, size):
    """allowed[i, j]: j is i itself or one of the size - 1 positions before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def kept_window_mask(n, size, keep):
    """... or one of the first `keep` positions, not later than i."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return window_mask(n, size) | ((j <= i) & (j < keep))


def softmax(scores, allowed):
    s = scores.masked_fill(~allowed, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def softmax_plus_one(scores, allowed):
    """One more term of score 0 in the denominator."""
    s = scores.masked_fill(~allowed, -math.inf)
    top = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attend(q, k, v, scale, allowed, weights):
    """q [n, H, D], k [n, G, D], v [n, G, V] -> [n, H * V]"""
    of = [i // (q.shape[1] // k.shape[1]) for i in range(q.shape[1])]
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    return torch.einsum("hij,jhv->ihv", weights(s, allowed), v[:, of]).flatten(1)


def mixed_values(v, w, p, m, shared):
    """`shared` keeps the values of the first layer that takes part (all heads of a token in a row)."""
    if not m["v_mix"]:
        return v
    if "v" not in shared:
        shared["v"] = v
        return v
    return mix_values(v, shared["v"].reshape(v.shape), w[p + "vmix"])


def attention(h, w, p, m, eps, shared):
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freqs = stepped_frequencies(m["rot"])
    q = unit_rms(turn_neighbours((h @ w[p + "q"].T).reshape(n, H, D), freqs), eps)
    k = unit_rms(turn_neighbours((h @ w[p + "k"].T).reshape(n, G, D), freqs), eps)
    v = mixed_values((h @ w[p + "v"].T).reshape(n, G, V), w, p, m, shared)
    return attend(q, k, v, m["scale"], window_mask(n, m["mask"]["size"]), softmax_plus_one) @ w[p + "o"].T


def attention_2(h, w, p, m, eps, shared):
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freqs, size = ramped_frequencies(m["rot"])
    q, k, v = (short_conv(h @ w[p + x].T, w[p + x + ".conv"]) for x in "qkv")
    q = turn_halves(rms_norm(q, w[p + "q.norm"], eps).reshape(n, H, D), freqs, size)
    k = turn_halves(rms_norm(k, w[p + "k.norm"], eps).reshape(n, G, D), freqs, size)
    v = mixed_values(v.reshape(n, G, V), w, p, m, shared)
    return attend(q, k, v, m["scale"], kept_window_mask(n, m["mask"]["size"], m["mask"]["keep_first"]), softmax) @ w[p + "o"].T


MIXERS = {"attention": attention, "attention_2": attention_2}


# ------------------------------------------------------------------ feed-forward
def dense(h, w, p):
    gate, up = h @ w[p + "gate"].T + w[p + "gate.b"], h @ w[p + "up"].T + w[p + "up.b"]
    return (gelu_tanh(gate) * up) @ w[p + "down"].T + w[p + "down.b"]


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, groups, keep, top):
    """Router logits z of one token -> [(index, weight)] of the chosen ones."""
    s = torch.softmax(z, -1)
    choice = s + correction
    size = len(z) // groups
    score = choice.reshape(groups, size).max(-1).values
    best = sorted(range(groups), key=lambda g: -float(score[g]))[:keep]
    open_ = [i for i in range(len(z)) if i // size in best]
    chosen = sorted(open_, key=lambda i: -float(choice[i]))[:top]
    total = sum(s[i] for i in chosen) + 1e-20
    return [(i, s[i] / total) for i in chosen]


def mixture(h, w, p, c):
    r, out = c["router"], []
    for row in h:
        y = torch.zeros_like(row)
        for i, weight in route(w[p + "router"] @ row, w[p + "correction"], r["groups"]["count"], r["groups"]["keep"], r["top"]):
            y = y + weight * (expert(row, w, f"{p}e{i}.") if i < r["experts"] else row)
        out.append(y + expert(row, w, p + "shared."))
    return torch.stack(out)


# ------------------------------------------------------------------ the model
def forward(cfg, weights, ids, dtype=torch.float64, after_layer=None):
    """Logits [n, vocab] of one sequence; `after_layer` collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, shared = cfg["norm"]["eps"], {}
    x = embedding(list(ids), w, cfg)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps, shared)
        c = L.get("mlp")
        if c is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            x = x + (dense(h, w, p + "mlp.") if c["kind"] == "dense" else mixture(h, w, p + "mlp.", c))
        if after_layer is not None:
            after_layer.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
