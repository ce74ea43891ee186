"""Plain, slow restatement of the Luvutar decoder: one function per mechanism, whole sequences, no cache, no batching.
It shares nothing with the package; every engine path of this design is compared with it.

Weights are a dict of name -> tensor (any float dtype; computed in `dtype`), the configuration is the parsed JSON.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    """Weight as it is (the latents of the latent attention)."""
    return rms(x, eps) * w


def rms_norm_centred(x, w, eps):
    """Weight stored as its difference from one (every norm of the residual stream)."""
    return rms(x, eps) * (1 + w)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ positions
def rotate_pairs(x, pos, base):
    """x [n, H, R]: neighbouring elements (2i, 2i + 1) turn by pos * base^(-2i / R)."""
    R = x.shape[-1]
    ang = pos.to(x.dtype)[:, None] * torch.tensor([base ** (-2 * i / R) for i in range(R // 2)], dtype=x.dtype)
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def window_mask(n, size):
    """allowed[i, j]: j is i itself or one of the size - 1 positions before it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def causal_mask(n):
    return torch.ones(n, n, dtype=torch.bool).tril()


def distance_bucket(n, rows, far):
    """Bucket of distance n: one each for the first rows / 2 distances, then on a logarithmic scale that ends at `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(table, n, far):
    """[heads, n, n]: the table's entry for the distance i - j (0 where j lies after i)."""
    rows = table.shape[0]
    b = torch.tensor([distance_bucket(d, rows, far) for d in range(n)])
    d = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(min=0)
    return table[b[d]].permute(2, 0, 1)


def query_temperature(n, coef, every):
    return torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(n)], dtype=torch.float64)


# ------------------------------------------------------------------ attention
def softmax(scores, allowed):
    s = scores.masked_fill(~allowed, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def softmax_with_sink(scores, allowed, sink):
    """scores [H, n, n]; one extra term exp(sink[h]) in every denominator, with no weight of its own."""
    s = scores.masked_fill(~allowed, -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def latent_attention(h, w, p, m, eps):
    n, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = torch.arange(n)
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(n, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, None, m["kv_rank"]:], pos, m["rot"]["base"])[:, 0]
    q_rot = rotate_pairs(q[..., D:], pos, m["rot"]["base"])
    k = (c @ w[p + "uk"].T).reshape(n, H, D)
    v = (c @ w[p + "uv"].T).reshape(n, H, V)
    s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihr,jr->hij", q_rot, k_rot)) * m["scale"]
    a = softmax_with_sink(s, window_mask(n, m["mask"]["size"]), w[p + "sink"])
    o = torch.einsum("hij,jhv->ihv", a, v).reshape(n, H * V)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def keys_and_values(h, w, p, m):
    n, G = h.shape[0], m["kv_heads"]
    return (h @ w[p + "k"].T).reshape(n, G, m["dim"]), (h @ w[p + "v"].T).reshape(n, G, m["vdim"])


def biased_attention(h, w, p, m, k, v):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(n, H, m["dim"])
    t = m["q_temp"]
    q = q * query_temperature(n, t["coef"], t["every"]).to(h.dtype)[:, None, None]
    of = [i // (H // G) for i in range(H)]
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * m["scale"] + distance_bias(w[p + "rel"], n, m["bias_max"])
    o = torch.einsum("hij,jhv->ihv", softmax(s, causal_mask(n)), v[:, of])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(n, -1) @ w[p + "o"].T


# ------------------------------------------------------------------ layers
def stream_read(X, w_in):
    """X [streams, n, width] -> the sublayer's input before its norm."""
    return torch.einsum("s,snw->nw", w_in, X)


def stream_write(X, y, mix, out):
    """Every stream from the old ones (mix is [from, to]) and the sublayer's output."""
    return torch.einsum("st,snw->tnw", mix, X) + out[:, None, None] * y


def layer(X, w, cfg, i, kv):
    """`kv` keeps every attention layer's keys and values for the layers that share them."""
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    m = L["mixer"]
    h = rms_norm_centred(stream_read(X, w[p + "hc1.in"]), w[p + "norm1"], eps)
    if L["type"] == "latent_attention":
        y = latent_attention(h, w, p + "mix.", m, eps)
    else:
        src = m.get("kv_from", i)
        if src == i:
            kv[i] = keys_and_values(h, w, p + "mix.", m)
        y = biased_attention(h, w, p + "mix.", m, *kv[src])
    X = stream_write(X, y, w[p + "hc1.mix"], w[p + "hc1.out"])
    if L.get("mlp") is not None:
        h = rms_norm_centred(stream_read(X, w[p + "hc2.in"]), w[p + "norm2"], eps)
        y = gelu_tanh(h @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
        X = stream_write(X, y, w[p + "hc2.mix"], w[p + "hc2.out"])
    return X


def forward(cfg, weights, ids, dtype=torch.float64, after_layer=None):
    """Logits [n, vocab] of one sequence; `after_layer` collects the sum of the streams after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    X = x.expand(cfg["streams"], *x.shape)
    kv = {}
    for i in range(len(cfg["layers"])):
        X = layer(X, w, cfg, i, kv)
        if after_layer is not None:
            after_layer.append(X.sum(0))
    return rms_norm_centred(X.sum(0), w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T


def greedy(cfg, weights, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(torch.argmax(forward(cfg, weights, ids)[-1])))
    return ids[len(prompt):]
