"""Gebuzen weights: tensor names and shapes, random initialisation, and the engine's fused layout.

Per layer the engine runs four projections:

* ``in_proj``: rows [q | k] of the attention side and [q | k | v | g | a1] of the linear-attention side, one launch.
  The q and k biases ride along as one more input column: the norm kernel writes a constant 1 behind the ``width``
  real values of its output row, so every projection kernel adds them in its own accumulator.
* ``left_o``, ``right_o``: the two output projections.
* ``gate_up``: rows interleaved (gate_0, up_0, gate_1, up_1, ...), the gated activation is the projection's epilogue; ``down``.

Head sizes are padded with zero rows (of q, k, v, g, a2) and zero columns (of the output projections) to what the
attention and recurrence kernels work on, input widths to multiples of 32: zeros change no score, state or sum.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional

import torch

from ...quant.formats import QuantizedTensor
from ..common import pad, pad_cols, pad_heads, pad_rows, plain_linear
from ..qwen35.weights import LinearW
from .config import ChunkAttention, GatedLinear, GebuzenConfig

DECAY_RANK = 16          # rank of the decay projection in random-init models (a loaded model's tensors give theirs)


def tensor_shapes(cfg: GebuzenConfig, decay_rank: int = DECAY_RANK) -> Dict[str, tuple]:
    w = cfg.hidden_size
    s = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}
    if cfg.loop is not None:
        s["loop.step"] = (cfg.loop.times, w)
    for i, L in enumerate(cfg.layers):
        l, r, p = L.left, L.right, f"l{i}."
        s[p + "norm1"] = (w,)
        s[p + "mix.left.q"], s[p + "mix.left.q.b"] = (l.heads * l.dim, w), (l.heads * l.dim,)
        s[p + "mix.left.k"], s[p + "mix.left.k.b"] = (l.kv_heads * l.dim, w), (l.kv_heads * l.dim,)
        s[p + "mix.left.sink"] = (l.heads,)
        s[p + "mix.left.o"] = (w, l.heads * l.dim)
        for n, rows in (("q", r.heads * r.dim), ("k", r.heads * r.dim), ("v", r.heads * r.vdim), ("g", r.heads * r.vdim),
                        ("a1", decay_rank)):
            s[p + "mix.right." + n] = (rows, w)
        s[p + "mix.right.o"] = (w, r.heads * r.vdim)
        s[p + "mix.right.norm"] = (r.vdim,)
        s[p + "mix.right.a2"], s[p + "mix.right.a2.b"] = (r.heads * r.dim, decay_rank), (r.heads * r.dim,)
        s[p + "mix.left.out"] = s[p + "mix.right.out"] = (w,)
        if L.ff is not None:
            s[p + "norm2"] = (w,)
            s[p + "mlp.gate"] = s[p + "mlp.up"] = (L.ff, w)
            s[p + "mlp.down"] = (w, L.ff)
    return s


def random_tensor(name: str, shape: tuple, seed: int, device="cpu") -> torch.Tensor:
    """Deterministic per-tensor init, rounded to bf16: matrices N(0, fan_in^-1/2), norms around 1, sinks and decay biases
    in a range where neither the sink nor the decay is negligible."""
    g = torch.Generator(device=device)
    g.manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
    t = torch.randn(shape, device=device, generator=g)
    leaf = name.rsplit(".", 1)[-1]
    if name == "embed":
        pass
    elif name == "loop.step":
        t = t * 0.3
    elif name.endswith("a2.b"):
        t = t + 2.0
    elif leaf == "sink" or leaf == "b":
        t = t * 0.5
    elif len(shape) == 1:
        t = t * 0.1 + 1.0
    else:
        t = t * shape[1] ** -0.5
    return t.to(torch.bfloat16)


def random_weights(cfg: GebuzenConfig, seed: int = 0, device="cpu", decay_rank: int = DECAY_RANK) -> Dict[str, torch.Tensor]:
    return {n: random_tensor(n, s, seed, device) for n, s in tensor_shapes(cfg, decay_rank).items()}


def random_getter(cfg: GebuzenConfig, seed: int = 0, device="cpu") -> Callable[[str], torch.Tensor]:
    shapes = tensor_shapes(cfg)
    return lambda name: random_tensor(name, shapes[name], seed, device)


@dataclass
class ParallelLayerW:
    left: ChunkAttention
    right: GatedLinear
    norm1: torch.Tensor               # norm weights, sinks and decay biases: f32
    in_proj: LinearW
    decay_rank: int                   # columns of a2 (padded rank)
    a2: torch.Tensor                  # [heads * dim_padded, decay_rank]
    a2_bias: torch.Tensor
    sink: torch.Tensor                # [heads]
    right_norm: torch.Tensor          # [vdim_padded]
    left_o: LinearW
    right_o: LinearW
    left_out: torch.Tensor
    right_out: torch.Tensor
    norm2: Optional[torch.Tensor]
    gate_up: Optional[LinearW]
    down: Optional[LinearW]

    def linears(self) -> List[LinearW]:
        return [w for w in (self.in_proj, self.left_o, self.right_o, self.gate_up, self.down) if w is not None]


@dataclass
class GebuzenWeights:
    cfg: GebuzenConfig
    embed: torch.Tensor               # [vocab, width]
    step: Optional[torch.Tensor]      # [times, width] f32
    layers: List[ParallelLayerW]
    final_norm: torch.Tensor
    lm_head: LinearW
    act_dtype: torch.dtype
    tp_rank: int = 0
    tp_size: int = 1
    preset: str = "bf16"
    layout: str = "canonical"

    def linears(self) -> List[LinearW]:
        return [self.lm_head] + [w for l in self.layers for w in l.linears()]

    def decode_read_bytes(self) -> int:
        """Weight bytes one decode step streams (a looped layer's once per pass)."""
        per = [sum(w.N * w.k_padded for w in l.linears()) + l.a2.numel() for l in self.layers]
        esz = self.embed.element_size()
        return esz * (self.lm_head.N * self.lm_head.k_padded + sum(per[r.layer] for r in self.cfg.runs()))

    def weight_bytes(self) -> int:
        esz = self.embed.element_size()
        return esz * (self.embed.numel() + sum(w.N * w.k_padded for w in self.linears()) + sum(l.a2.numel() for l in self.layers))


def build_engine_weights(cfg: GebuzenConfig, get: Callable[[str], torch.Tensor], device="cpu",
                         dtype: Optional[torch.dtype] = None) -> GebuzenWeights:
    """``dtype``: what projections and activations run in, bfloat16 or float32 (default: bfloat16 on a CUDA device)."""
    dev = torch.device(device)
    dtype = dtype or (torch.bfloat16 if dev.type == "cuda" else torch.float32)
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"Gebuzen runs in bfloat16 or float32, not {dtype}")
    fmt = "bf16" if dtype == torch.bfloat16 else "f32"

    def t(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=dtype)

    def f32(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=torch.float32).contiguous()

    def lin(w: torch.Tensor, n: int, k: int) -> LinearW:
        return plain_linear(w, n, k, fmt)

    W = cfg.hidden_size
    nout = pad(W, 4)                     # output rows of projections onto the residual width (paired fp32 stores need even pitches)
    kin = pad(W, 32)                     # input width of projections without a bias
    kin_b = pad(W + 1, 32)               # ... and with one: column W multiplies the constant 1
    layers = []
    for i, L in enumerate(cfg.layers):
        l, r, p = L.left, L.right, f"l{i}."
        m = p + "mix."
        rank = get(m + "right.a1").shape[0]
        rp = pad(rank, 8)

        def with_bias(name: str, heads: int, dim: int, to: int) -> torch.Tensor:
            wb = torch.cat([t(name), t(name + ".b")[:, None]], 1)
            return pad_cols(pad_heads(wb, heads, dim, to), kin_b)

        def plain(name: str, heads: int, dim: int, to: int) -> torch.Tensor:
            return pad_cols(pad_heads(t(name), heads, dim, to), kin_b)

        D, dk, dv = l.dim_padded, r.dim_padded, r.vdim_padded
        rows = torch.cat([with_bias(m + "left.q", l.heads, l.dim, D), with_bias(m + "left.k", l.kv_heads, l.dim, D),
                          plain(m + "right.q", r.heads, r.dim, dk), plain(m + "right.k", r.heads, r.dim, dk),
                          plain(m + "right.v", r.heads, r.vdim, dv), plain(m + "right.g", r.heads, r.vdim, dv),
                          pad_cols(pad_rows(t(m + "right.a1"), rp), kin_b)], 0)
        in_proj = lin(rows, rows.shape[0], kin_b)
        del rows
        a2 = pad_cols(pad_heads(t(m + "right.a2"), r.heads, r.dim, dk), rp).contiguous()
        left_o = lin(pad_heads(t(m + "left.o").T.contiguous(), l.heads, l.dim, D).T, nout, l.heads * D)
        right_o = lin(pad_heads(t(m + "right.o").T.contiguous(), r.heads, r.vdim, dv).T, nout, r.heads * dv)
        gate_up = down = norm2 = None
        if L.ff is not None:
            fp = pad(L.ff, 32)
            gu = torch.stack([pad_rows(t(p + "mlp.gate"), fp), pad_rows(t(p + "mlp.up"), fp)], 1).reshape(2 * fp, W)
            gate_up, down, norm2 = lin(gu, 2 * fp, kin), lin(t(p + "mlp.down"), nout, fp), f32(p + "norm2")
            del gu
        layers.append(ParallelLayerW(l, r, f32(p + "norm1"), in_proj, rp, a2,
                                     pad_heads(f32(m + "right.a2.b"), r.heads, r.dim, dk).contiguous(), f32(m + "left.sink"),
                                     pad_rows(f32(m + "right.norm"), dv).contiguous(), left_o, right_o,
                                     f32(m + "left.out"), f32(m + "right.out"), norm2, gate_up, down))
    head = lin(t("head"), pad(cfg.vocab_size, 2), kin)
    return GebuzenWeights(cfg, t("embed").contiguous(), f32("loop.step") if cfg.loop is not None else None, layers,
                          f32("final.norm"), head, dtype, preset=fmt)


def load_engine_weights(model_dir, device="cpu", dtype: Optional[torch.dtype] = None) -> GebuzenWeights:
    from ...io.model_dir import ShardCollection
    col = ShardCollection(model_dir)
    return build_engine_weights(GebuzenConfig.from_dir(model_dir), col.tensor, device, dtype)
