"""Luvutar weights: tensor names and shapes, random initialisation, and the engine's fused layout.

Per layer the engine runs

* ``in_proj``: everything that reads the mixer's input in one launch -- latent attention [query latent | key / value latent |
  rotated key part | output gate], attention [q | k | v | head gates] (no k, v for a layer that reads another one's);
* latent attention only: ``uq``, and the per-head products ``uk_t`` / ``uv`` or their expanded form ``ukv`` (ops/specs.py);
* ``o``, then ``up`` (tanh-gelu as its epilogue) and ``down``.

Sizes are padded with zero rows and columns to what the kernels work on; zeros change no score and no sum.  Norm weights of
the residual are kept as 1 + w, the distance bias as a table by distance.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Union

import torch

from ...ops.specs import AttnSpec, LatentSpec, distance_bias_table
from ..common import pad, pad_cols, pad_heads, pad_rows, plain_linear
from ..qwen35.weights import LinearW
from .config import BiasedAttention, LatentAttention, LuvutarConfig

BIAS_BUCKETS = 32        # rows of the distance table in random-init models (a loaded model's tensors give theirs)


def tensor_shapes(cfg: LuvutarConfig, buckets: int = BIAS_BUCKETS) -> Dict[str, tuple]:
    w, s = cfg.hidden_size, cfg.streams
    out = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    for i, L in enumerate(cfg.layers):
        m, p = L.mixer, f"l{i}."
        x = p + "mix."
        out[p + "norm1"] = (w,)
        if isinstance(m, LatentAttention):
            H = m.heads
            out.update({x + "dq": (m.q_rank, w), x + "dq.norm": (m.q_rank,), x + "uq": (H * (m.dim + m.rot_dim), m.q_rank),
                        x + "dkv": (m.kv_rank + m.rot_dim, w), x + "dkv.norm": (m.kv_rank,), x + "uk": (H * m.dim, m.kv_rank),
                        x + "uv": (H * m.vdim, m.kv_rank), x + "sink": (H,), x + "g": (H * m.vdim, w), x + "o": (w, H * m.vdim)})
        else:
            out[x + "q"] = (m.heads * m.dim, w)
            if m.kv_from is None:
                out[x + "k"], out[x + "v"] = (m.kv_heads * m.dim, w), (m.kv_heads * m.vdim, w)
            out.update({x + "rel": (buckets, m.heads), x + "g": (m.heads, w), x + "o": (w, m.heads * m.vdim)})
        subs = [1]
        if L.ff is not None:
            out[p + "norm2"] = (w,)
            out[p + "mlp.up"], out[p + "mlp.down"] = (L.ff, w), (w, L.ff)
            subs.append(2)
        for q in subs:
            out[f"{p}hc{q}.in"] = out[f"{p}hc{q}.out"] = (s,)
            out[f"{p}hc{q}.mix"] = (s, s)
    return out


def random_tensor(name: str, shape: tuple, seed: int, device="cpu") -> torch.Tensor:
    """Deterministic per-tensor init, rounded to bf16: matrices N(0, fan_in^-1/2), norms around their neutral value, streams
    that are read and written unequally but keep their size."""
    g = torch.Generator(device=device)
    g.manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
    t = torch.randn(shape, device=device, generator=g)
    leaf = name.rsplit(".", 1)[-1]
    if name == "embed":
        pass
    elif leaf == "in":
        t = (1.0 + 0.5 * t) / shape[0]
    elif leaf == "out":
        t = 1.0 + 0.5 * t
    elif leaf == "mix":
        t = 0.3 * t * shape[0] ** -0.5 + 0.7 * torch.eye(shape[0], device=device)
    elif leaf == "norm" and ".mix." in name:
        t = 1.0 + 0.1 * t
    elif len(shape) == 1 and leaf != "sink":
        t = 0.1 * t
    elif leaf not in ("sink", "rel"):
        t = t * shape[1] ** -0.5
    return t.to(torch.bfloat16)


def random_weights(cfg: LuvutarConfig, seed: int = 0, device="cpu", buckets: int = BIAS_BUCKETS) -> Dict[str, torch.Tensor]:
    return {n: random_tensor(n, s, seed, device) for n, s in tensor_shapes(cfg, buckets).items()}


def random_getter(cfg: LuvutarConfig, seed: int = 0, device="cpu") -> Callable[[str], torch.Tensor]:
    shapes = tensor_shapes(cfg)
    return lambda name: random_tensor(name, shapes[name], seed, device)


@dataclass
class StreamW:
    """A sublayer's reading weights, its norm (as a plain multiplier) and its writing weights; all f32."""
    read: torch.Tensor                # [streams]
    norm: torch.Tensor                # [width]
    mix: torch.Tensor                 # [streams, streams], [from, to]
    out: torch.Tensor                 # [streams]


@dataclass
class LayerW:
    hc1: StreamW
    in_proj: LinearW
    attn: Union[LatentSpec, AttnSpec]
    appends: bool                     # the layer writes keys (and values) of its own
    uq: Optional[LinearW]
    o: LinearW
    hc2: Optional[StreamW]
    up: Optional[LinearW]
    down: Optional[LinearW]

    def linears(self) -> List[LinearW]:
        return [w for w in (self.in_proj, self.uq, self.o, self.up, self.down) if w is not None]


@dataclass
class LuvutarWeights:
    cfg: LuvutarConfig
    embed: torch.Tensor               # [vocab, width]
    layers: List[LayerW]
    read_all: torch.Tensor            # f32 [streams], ones: the final sum of the streams
    final_norm: torch.Tensor          # f32 [width]
    lm_head: LinearW
    act_dtype: torch.dtype
    tp_rank: int = 0
    tp_size: int = 1
    preset: str = "bf16"
    layout: str = "canonical"

    def linears(self) -> List[LinearW]:
        return [self.lm_head] + [w for l in self.layers for w in l.linears()]

    def decode_read_bytes(self) -> int:
        """Weight bytes one decode step streams."""
        n = sum(w.N * w.k_padded for w in self.linears())
        n += sum(l.attn.uk_t.numel() + l.attn.uv.numel() for l in self.layers if isinstance(l.attn, LatentSpec))
        return n * self.embed.element_size()

    def weight_bytes(self) -> int:
        return self.decode_read_bytes() + self.embed.numel() * self.embed.element_size()


def build_engine_weights(cfg: LuvutarConfig, get: Callable[[str], torch.Tensor], device="cpu",
                         dtype: Optional[torch.dtype] = None) -> LuvutarWeights:
    """``dtype``: what projections and activations run in, bfloat16 or float32 (default: bfloat16 on a CUDA device)."""
    dev = torch.device(device)
    dtype = dtype or (torch.bfloat16 if dev.type == "cuda" else torch.float32)
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"Luvutar runs in bfloat16 or float32, not {dtype}")
    fmt = "bf16" if dtype == torch.bfloat16 else "f32"
    W = cfg.hidden_size
    nout = pad(W, 4)                     # output rows of projections onto the residual width (paired fp32 stores need even pitches)
    kin = pad(W, 32)                     # input width of the projections that read a normed residual row

    def t(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=dtype)

    def f32(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=torch.float32).contiguous()

    def lin(w: torch.Tensor, n: int, k: int) -> LinearW:
        return plain_linear(w, n, k, fmt)

    def vec(name: str, to: int) -> torch.Tensor:
        return pad_rows(f32(name), to).contiguous()

    def stream(p: str, q: int) -> StreamW:
        hc = f"{p}hc{q}."
        return StreamW(f32(hc + "in"), 1.0 + f32(f"{p}norm{q}"), f32(hc + "mix"), f32(hc + "out"))

    def out_proj(name: str, heads: int, dim: int, to: int) -> LinearW:
        return lin(pad_heads(t(name).T.contiguous(), heads, dim, to).T, nout, heads * to)

    def latent(m: LatentAttention, x: str):
        H, D, R, V, QR, KR = m.heads, m.dim_padded, m.rot_padded, m.vdim_padded, m.q_rank_padded, m.kv_rank_padded
        dkv = t(x + "dkv")
        rows = torch.cat([pad_rows(t(x + "dq"), QR), pad_rows(dkv[:m.kv_rank], KR), pad_rows(dkv[m.kv_rank:], R),
                          pad_heads(t(x + "g"), H, m.vdim, V)], 0)
        q = t(x + "uq").reshape(H, m.dim + m.rot_dim, m.q_rank)
        uq = torch.cat([pad_heads(q[:, :m.dim].reshape(-1, m.q_rank), H, m.dim, D).reshape(H, D, -1),
                        pad_heads(q[:, m.dim:].reshape(-1, m.q_rank), H, m.rot_dim, R).reshape(H, R, -1)], 1).reshape(H * (D + R), -1)
        uk = pad_cols(pad_heads(t(x + "uk"), H, m.dim, D), KR)
        uv = pad_cols(pad_heads(t(x + "uv"), H, m.vdim, V), KR)
        inv = m.rot_base ** (-torch.arange(m.rot_dim // 2, dtype=torch.float64) * 2.0 / m.rot_dim)
        spec = LatentSpec(H, D, R, m.rot_dim, V, QR, m.q_rank, KR, m.kv_rank, m.scale, m.window, f32(x + "sink"), inv.to(dev), cfg.norm_eps,
                          vec(x + "dq.norm", QR), vec(x + "dkv.norm", KR),
                          uk.reshape(H, D, KR).transpose(1, 2).reshape(H * KR, D).contiguous(), torch.cat([uk, uv], 0).contiguous())
        return lin(rows, rows.shape[0], kin), spec, lin(uq, H * (D + R), QR), out_proj(x + "o", H, m.vdim, V)

    def attention(m: BiasedAttention, x: str):
        H, G, D = m.heads, m.kv_heads, m.dim_padded
        rows = [pad_heads(t(x + "q"), H, m.dim, D)]
        if m.kv_from is None:
            rows += [pad_heads(t(x + "k"), G, m.dim, D), pad_heads(t(x + "v"), G, m.vdim, D)]
        gate = sum(r.shape[0] for r in rows)
        rows = torch.cat(rows + [pad_rows(t(x + "g"), pad(H, 8))], 0)
        spec = AttnSpec(H, G, D, m.scale, gate_head_stride=1, gate_offset=gate, gate_per_head=True, temp_coef=m.temp_coef,
                        temp_every=m.temp_every, bias=distance_bias_table(f32(x + "rel"), m.bias_max))
        return lin(rows, rows.shape[0], kin), spec, None, out_proj(x + "o", H, m.vdim, D)

    layers = []
    for i, L in enumerate(cfg.layers):
        m, p = L.mixer, f"l{i}."
        in_proj, spec, uq, o = (latent if isinstance(m, LatentAttention) else attention)(m, p + "mix.")
        hc2 = up = down = None
        if L.ff is not None:
            fp = pad(L.ff, 32)
            hc2, up, down = stream(p, 2), lin(t(p + "mlp.up"), fp, kin), lin(t(p + "mlp.down"), nout, fp)
        layers.append(LayerW(stream(p, 1), in_proj, spec, cfg.kv_layer(i) == i, uq, o, hc2, up, down))
    return LuvutarWeights(cfg, t("embed").contiguous(), layers, torch.ones(cfg.streams, device=dev), 1.0 + f32("final.norm"),
                          lin(t("head"), pad(cfg.vocab_size, 2), kin), dtype, preset=fmt)


def load_engine_weights(model_dir, device="cpu", dtype: Optional[torch.dtype] = None) -> LuvutarWeights:
    from ...io.model_dir import ShardCollection
    col = ShardCollection(model_dir)
    return build_engine_weights(LuvutarConfig.from_dir(model_dir), col.tensor, device, dtype)
