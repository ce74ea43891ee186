"""Plain, slow restatement of the Gebuzen decoder: one function per mechanism, whole sequences, no cache, no batching.
It shares nothing with the package; every engine path of this design is compared with it.

Weights are a dict of name -> tensor (any float dtype; computed in `dtype`), the configuration is the parsed JSON.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def chunk_mask(n, size, device="cpu"):
    """allowed[i, j]: j is not after i and lies in the same block of `size` positions, blocks counted from position 0."""
    i = torch.arange(n, device=device)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def softmax_with_sink(scores, allowed, sink):
    """scores [H, n, n]; one extra term exp(sink[h]) in every denominator, with no weight of its own."""
    s = scores.masked_fill(~allowed, -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def chunk_attention_heads(q, k, scale, size, sink):
    """q [n, H, D], k [n, G, D]; the keys are the values.  Returns [n, H, D]."""
    n, H, _ = q.shape
    G = k.shape[1]
    kk = k[:, [h // (H // G) for h in range(H)]]
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    p = softmax_with_sink(s, chunk_mask(n, size, q.device), sink)
    return torch.einsum("hij,jhd->ihd", p, kk)


def left_mixer(h, w, pre, m):
    n = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(n, H, D)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(n, G, D)
    o = chunk_attention_heads(q, k, m["scale"], m["mask"]["size"], w[pre + "sink"])
    return o.reshape(n, H * D) @ w[pre + "o"].T


def channel_decay(z, tau):
    """sigmoid(z) to the power 1 / tau."""
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_linear_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [n, H, Dk], v [n, H, Dv]; the state's rows decay per key channel, then take k v^T; read with q."""
    n, H, Dk = q.shape
    S = q.new_zeros(H, Dk, v.shape[-1]) if state is None else state.clone()
    out = []
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def right_mixer(h, w, pre, m, eps):
    n = h.shape[0]
    H, Dk, Dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).reshape(n, H, Dk) * Dk ** -0.5
    k = (h @ w[pre + "k"].T).reshape(n, H, Dk)
    v = (h @ w[pre + "v"].T).reshape(n, H, Dv)
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    o, _ = gated_linear_recurrence(q, k, v, channel_decay(z, m["tau"]).reshape(n, H, Dk))
    o = rms_norm(o, w[pre + "norm"], eps).reshape(n, H * Dv)
    g = h @ w[pre + "g"].T
    return (o * (g * torch.sigmoid(g))) @ w[pre + "o"].T


def parallel_mixer(h, w, pre, m, eps):
    a = left_mixer(h, w, pre + "left.", m["left"])
    b = right_mixer(h, w, pre + "right.", m["right"], eps)
    return 0.5 * (rms_norm(a, w[pre + "left.out"], eps) + rms_norm(b, w[pre + "right.out"], eps))


def dense_ff(h, w, pre):
    return (torch.relu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def layer(x, w, cfg, i):
    L, eps, m = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"]
    p = f"l{i}."
    x = x + m * parallel_mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
    if L.get("mlp") is not None:
        x = x + m * dense_ff(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
    return x


def layer_runs(cfg):
    """(layer, pass number or None, first of its pass) in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    runs = [(i, None, False) for i in range(a)]
    for t in range(lp["times"]):
        runs += [(i, t, i == a) for i in range(a, b)]
    return runs + [(i, None, False) for i in range(b, n)]


def forward(cfg, weights, ids, dtype=torch.float64, after_layer=None):
    """Logits [n, vocab] of one sequence; `after_layer` collects the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    x0 = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    x = x0
    for i, t, first in layer_runs(cfg):
        if first:
            if t > 0:
                x = x + x0
            x = x + w["loop.step"][t]
        x = layer(x, w, cfg, i)
        if after_layer is not None:
            after_layer.append(x.clone())
    return (rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T) * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
