"""Plain, slow restatement of the Rotutar decoder: one function per mechanism, whole sequences, no cache, no batching.
It shares nothing with the package; every engine path of this design is compared with it.

Weights are a dict of name -> tensor (any float dtype; computed in `dtype`), the configuration is the parsed JSON.
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def group_norm(x, w, eps, groups):
    """Every one of `groups` consecutive equal parts is divided by its own root mean square."""
    parts = x.reshape(x.shape[:-1] + (groups, -1))
    return unit_rms(parts, eps).reshape(x.shape) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gated(y, h, w, b):
    """y scaled element by element by what the sublayer's input opens."""
    return y * torch.sigmoid(h @ w.T + b)


# ------------------------------------------------------------------ attention
def turn_neighbours(x, base, dims):
    """x [n, H, D]: dimensions 2i and 2i + 1 (2i < dims) turn by position * base^(-2i / dims)."""
    freq = torch.tensor([base ** (-2 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return y


def window_mask(n, size):
    """allowed[i, j]: j is i itself or one of the size - 1 positions before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def softmax_with_sink(scores, allowed, sink):
    """scores [H, n, n]; every head has one more term exp(sink) in its denominator."""
    s = scores.masked_fill(~allowed, -math.inf)
    sink = sink[:, None, None]
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale, allowed, sink):
    """q [n, H, D], k [n, G, D], v [n, G, V] -> [n, H * V]"""
    of = [i // (q.shape[1] // k.shape[1]) for i in range(q.shape[1])]
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    return torch.einsum("hij,jhv->ihv", softmax_with_sink(s, allowed, sink), v[:, of]).flatten(1)


def attention(h, w, p, m, eps):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = (rms_norm(h @ w[p + x].T, w[p + x + ".norm"], eps) for x in "qk")
    q, k = (turn_neighbours(t.reshape(n, c, m["dim"]), m["rot"]["base"], m["rot"]["dims"]) for t, c in ((q, H), (k, G)))
    v = (h @ w[p + "v"].T).reshape(n, G, m["vdim"])
    return attend(q, k, v, m["scale"], window_mask(n, m["mask"]["size"]), w[p + "sink"]) @ w[p + "o"].T


# ------------------------------------------------------------------ delta rule with a decay per channel
def short_conv(u, w):
    """u [n, channels], w [channels, taps]; the last tap is the token's own."""
    n, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + w[:, j] * u[t - taps + 1 + j]
    return y


def unit_length(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decay(h, a1, a2, A_log, dt_bias, heads):
    """[n, heads, dim], what remains of every row of the state."""
    z = softplus(h @ a1.T @ a2.T + dt_bias).reshape(h.shape[0], heads, -1)
    return torch.exp(-torch.exp(A_log)[:, None] * z)


def delta_rule(q, k, v, g, beta):
    """q, k, g [n, H, K], v [n, H, V], beta [n, H] -> [n, H, V]: decay, then write what is missing, then read."""
    S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def delta(h, w, p, m, eps):
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[p + x].T, w[p + x + ".conv"])) for x in "qkv")
    of = [i // (H // G) for i in range(H)]
    q, k = unit_length(q.reshape(n, G, D))[:, of] * D ** -0.5, unit_length(k.reshape(n, G, D))[:, of]
    g = decay(h, w[p + "a1"], w[p + "a2"], w[p + "A_log"], w[p + "dt_bias"], H)
    o = delta_rule(q, k, v.reshape(n, H, V), g, torch.sigmoid(h @ w[p + "b"].T))
    gate = torch.sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T)
    return (rms_norm(o, w[p + "norm"], eps).flatten(1) * gate) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * delta(h, w, p + "right.", m["right"], eps))


# ------------------------------------------------------------------ linear attention whose forget gate is the key
def forget_gate(z, lower):
    return lower + (1 - lower) * torch.sigmoid(z)


def forget_write(q, f, v):
    """q, f [n, H, K], v [n, H, V] -> [n, H, V]; what a channel forgets makes room for the value."""
    S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def hgrn2(h, w, p, m, eps):
    n, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(n, H, D)
    f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).reshape(n, H, D)
    o = forget_write(q, f, (h @ w[p + "v"].T).reshape(n, H, V))
    return rms_norm(o, w[p + "norm"], eps).flatten(1) @ w[p + "o"].T


MIXERS = {"parallel": parallel, "hgrn2": hgrn2}


# ------------------------------------------------------------------ feed-forward
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, limit):
    g, u = (h @ w[p + "gate"].T).clamp(max=limit), (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z, groups, keep, top):
    """Router logits z of one token -> [(index, weight)] of the chosen experts."""
    s = torch.sigmoid(z)
    size = len(z) // groups
    score = [float(s[g * size:(g + 1) * size].sort(descending=True).values[:2].sum()) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: -score[g])[:keep]
    open_ = [i for i in range(len(z)) if i // size in best]
    return [(i, s[i]) for i in sorted(open_, key=lambda i: -float(s[i]))[:top]]


def mixture(h, w, p, c):
    r, out = c["router"], []
    for row in h:
        y = torch.zeros_like(row)
        for i, weight in route(w[p + "router"] @ row, r["groups"]["count"], r["groups"]["keep"], r["top"]):
            y = y + weight * expert(row, w, f"{p}e{i}.", c["expert"]["limit"])
        out.append(y)
    return torch.stack(out)


# ------------------------------------------------------------------ the model
def forward(cfg, weights, ids, dtype=torch.float64, after_layer=None):
    """Logits [n, vocab] of one sequence; `after_layer` collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, groups, cap = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["logit_softcap"]
    x = w["embed"][torch.tensor(list(ids))]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[L["type"]](x, w, p + "mix.", L["mixer"], eps)
        x = x + group_norm(gated(y, x, w[p + "rg1"], w[p + "rg1.b"]), w[p + "norm1"], eps, groups)
        c = L.get("mlp")
        if c is not None:
            y = dense(x, w, p + "mlp.") if c["kind"] == "dense" else mixture(x, w, p + "mlp.", c)
            x = x + group_norm(gated(y, x, w[p + "rg2"], w[p + "rg2.b"]), w[p + "norm2"], eps, groups)
        if after_layer is not None:
            after_layer.append(x)
    z = group_norm(x, w["final.norm"], eps, groups) @ w["head"].T
    return cap * torch.tanh(z / cap)


def greedy(cfg, weights, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
