"""Fudulix weights: tensor names and shapes, random initialisation, and the engine's fused layout.

Per layer the engine runs ``in_proj`` ([q | k | v heads] in one launch), ``o``, and then either ``gate_up`` (rows alternate
gate and up; the biases are the column that multiplies the constant 1 behind the normed row) and ``down``, or the router, the
experts' stacked matrices and the shared expert's ``gate_up`` and ``down``.

Sizes are padded with zero rows and columns to what the kernels work on; zeros change no score, norm or sum.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional

import torch

from ...ops.specs import AttnSpec, HeadsSpec, MoeSpec
from ..common import alternate, pad, pad_heads, pad_rows, plain_linear
from ..qwen35.weights import LinearW
from .config import ConvAttention, Dense, FudulixConfig, Mixer, Mixture


def tensor_shapes(cfg: FudulixConfig) -> Dict[str, tuple]:
    w = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, w), "bigram": (cfg.bigram.buckets + 1, w), "embed.norm": (w,), "final.norm": (w,), "head": (cfg.vocab_size, w)}

    def expert(p: str, ff: int) -> None:
        out.update({p + "gate": (ff, w), p + "up": (ff, w), p + "down": (w, ff)})
    for i, L in enumerate(cfg.layers):
        m, c, p = L.mixer, L.mlp, f"l{i}."
        x, y = p + "mix.", p + "mlp."
        sizes = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        out[p + "norm1"] = (w,)
        out.update({x + n: (s, w) for n, s in sizes.items()})
        out[x + "o"] = (w, m.heads * m.vdim)
        if isinstance(m, ConvAttention):
            out.update({f"{x}{n}.conv": (s, m.taps) for n, s in sizes.items()})
            out[x + "q.norm"], out[x + "k.norm"] = (sizes["q"],), (sizes["k"],)
        if m.v_mix:
            out[x + "vmix"] = ()
        if c is None:
            continue
        out[p + "norm2"] = (w,)
        if isinstance(c, Dense):
            expert(y, c.ff)
            out.update({y + "gate.b": (c.ff,), y + "up.b": (c.ff,), y + "down.b": (w,)})
        else:
            for e in range(c.experts):
                expert(f"{y}e{e}.", c.ff)
            n = c.experts + c.identity
            out[y + "router"], out[y + "correction"] = (n, w), (n,)
            if c.shared_ff is not None:
                expert(y + "shared.", c.shared_ff)
    return out


def random_tensor(name: str, shape: tuple, seed: int, device="cpu") -> torch.Tensor:
    """Deterministic per-tensor init, rounded to bf16: matrices N(0, fan_in^-1/2), norms around one, convolutions that mix
    their taps, corrections of the size of the scores."""
    g = torch.Generator(device=device)
    g.manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
    t = torch.randn(shape, device=device, generator=g)
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm", "norm1", "norm2"):
        t = 1.0 + 0.1 * t
    elif leaf == "vmix":
        t = 0.4 + 0.1 * t
    elif leaf == "conv":
        t = t * shape[1] ** -0.5
    elif leaf == "correction":
        t = t / shape[0]
    elif leaf == "b":
        t = 0.5 * t
    elif name not in ("embed", "bigram"):
        t = t * shape[1] ** -0.5
    return t.to(torch.bfloat16)


def random_weights(cfg: FudulixConfig, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    return {n: random_tensor(n, s, seed, device) for n, s in tensor_shapes(cfg).items()}


def random_getter(cfg: FudulixConfig, seed: int = 0, device="cpu") -> Callable[[str], torch.Tensor]:
    shapes = tensor_shapes(cfg)
    return lambda name: random_tensor(name, shapes[name], seed, device)


@dataclass
class DenseW:
    gate_up: LinearW                  # input: the normed row and a constant 1
    down: LinearW
    bias: torch.Tensor                # f32 [width], of `down`

    def linears(self) -> List[LinearW]:
        return [self.gate_up, self.down]


@dataclass
class MixtureW:
    router: LinearW
    moe: MoeSpec
    shared_gate_up: Optional[LinearW]
    shared_down: Optional[LinearW]

    def linears(self) -> List[LinearW]:
        return [w for w in (self.router, self.shared_gate_up, self.shared_down) if w is not None]


@dataclass
class LayerW:
    norm1: torch.Tensor               # f32 [width]
    in_proj: LinearW
    heads: HeadsSpec
    attn: AttnSpec
    o: LinearW
    norm2: Optional[torch.Tensor]
    mlp: object                       # DenseW, MixtureW or None

    def linears(self) -> List[LinearW]:
        return [self.in_proj, self.o] + (self.mlp.linears() if self.mlp is not None else [])


@dataclass
class FudulixWeights:
    cfg: FudulixConfig
    embed: torch.Tensor               # [vocab, width]
    bigram: torch.Tensor              # [buckets + 1, width]
    embed_norm: torch.Tensor          # f32 [width]
    layers: List[LayerW]
    final_norm: torch.Tensor          # f32 [width]
    lm_head: LinearW
    act_dtype: torch.dtype
    tp_rank: int = 0
    tp_size: int = 1
    preset: str = "bf16"
    layout: str = "canonical"

    def linears(self) -> List[LinearW]:
        return [self.lm_head] + [w for l in self.layers for w in l.linears()]

    def _mixtures(self) -> List[MoeSpec]:
        return [l.mlp.moe for l in self.layers if isinstance(l.mlp, MixtureW)]

    def decode_read_bytes(self) -> int:
        """Weight bytes a decode step of one row streams (of a mixture, the experts one row goes to at most)."""
        n = sum(w.N * w.k_padded for w in self.linears())
        n += sum((m.gate_up.numel() + m.down.numel()) // m.experts * min(m.top, m.experts) for m in self._mixtures())
        return n * self.embed.element_size()

    def weight_bytes(self) -> int:
        n = sum(w.N * w.k_padded for w in self.linears()) + self.embed.numel() + self.bigram.numel()
        return (n + sum(m.gate_up.numel() + m.down.numel() for m in self._mixtures())) * self.embed.element_size()


def build_engine_weights(cfg: FudulixConfig, get: Callable[[str], torch.Tensor], device="cpu",
                         dtype: Optional[torch.dtype] = None) -> FudulixWeights:
    """``dtype``: what projections and activations run in, bfloat16 or float32 (default: bfloat16 on a CUDA device)."""
    dev = torch.device(device)
    dtype = dtype or (torch.bfloat16 if dev.type == "cuda" else torch.float32)
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"Fudulix runs in bfloat16 or float32, not {dtype}")
    fmt = "bf16" if dtype == torch.bfloat16 else "f32"
    W = cfg.hidden_size
    nout = pad(W, 4)                     # output rows of projections onto the residual width (paired fp32 stores need even pitches)
    kin = pad(W, 32)                     # input width of the projections that read a normed residual row
    first = cfg.first_mixing()

    def t(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=dtype)

    def f32(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=torch.float32).contiguous()

    def lin(w: torch.Tensor, n: int, k: int) -> LinearW:
        return plain_linear(w, n, k, fmt)

    def mixer(i: int, m: Mixer, x: str):
        H, G, D = m.heads, m.kv_heads, m.dim_padded
        parts = (("q", H, m.dim), ("k", G, m.dim), ("v", G, m.vdim))

        def rows(suffix: str) -> torch.Tensor:
            return torch.cat([pad_heads(t(x + n + suffix), h, d, D) for n, h, d in parts], 0)

        freq, size = m.rotation()
        spec = HeadsSpec(H, G, D, m.dim, m.vdim, cfg.norm_eps, freq.to(dev), turn_size=size)
        attn = AttnSpec(H, G, D, m.scale, window=m.window)
        if isinstance(m, ConvAttention):
            spec.halves, spec.conv = True, rows(".conv").T.contiguous()
            spec.q_norm, spec.k_norm = (pad_heads(f32(x + n + ".norm"), h, d, D).contiguous() for n, h, d in parts[:2])
            attn.keep_first = m.keep_first
        else:
            spec.unit, attn.sink = True, torch.zeros(H, device=dev)
        if m.v_mix:
            spec.save = i == first
            spec.mix = None if i == first else float(get(x + "vmix").float())
        o = lin(pad_heads(t(x + "o").T.contiguous(), H, m.vdim, D).T, nout, H * D)
        return lin(rows(""), (H + 2 * G) * D, kin), spec, attn, o

    def gate_up(p: str, ff: int, ffp: int, bias: bool = False) -> torch.Tensor:
        def one(n: str) -> torch.Tensor:
            w = t(p + n)
            return pad_rows(torch.cat([w, t(f"{p}{n}.b")[:, None]], 1) if bias else w, ffp)
        return alternate(one("gate"), one("up"))

    def mixture(c: Mixture, y: str) -> MixtureW:
        n, ffp = c.experts + c.identity, pad(c.ff, 32)
        gu = torch.zeros(c.experts, 2 * ffp, kin, device=dev, dtype=dtype)
        down = torch.zeros(c.experts, nout, ffp, device=dev, dtype=dtype)
        for e in range(c.experts):
            gu[e, :, :W] = gate_up(f"{y}e{e}.", c.ff, ffp)
            down[e, :W, :c.ff] = t(f"{y}e{e}.down")
        spec = MoeSpec(c.experts, c.identity, c.top, c.groups, c.keep, ffp, nout, f32(y + "correction"), gu.flatten(0, 1), down.flatten(0, 1))
        sgu = sdown = None
        if c.shared_ff is not None:
            sp = pad(c.shared_ff, 32)
            sgu, sdown = lin(gate_up(y + "shared.", c.shared_ff, sp), 2 * sp, kin), lin(t(y + "shared.down"), nout, sp)
        return MixtureW(lin(t(y + "router"), pad(n, 4), kin), spec, sgu, sdown)

    layers = []
    for i, L in enumerate(cfg.layers):
        p, c = f"l{i}.", L.mlp
        in_proj, heads, attn, o = mixer(i, L.mixer, p + "mix.")
        norm2 = mlp = None
        if c is not None:
            norm2, y = f32(p + "norm2"), p + "mlp."
            if isinstance(c, Dense):
                fp = pad(c.ff, 32)
                mlp = DenseW(lin(gate_up(y, c.ff, fp, bias=True), 2 * fp, pad(W + 1, 32)), lin(t(y + "down"), nout, fp), f32(y + "down.b"))
            else:
                mlp = mixture(c, y)
        layers.append(LayerW(f32(p + "norm1"), in_proj, heads, attn, o, norm2, mlp))
    return FudulixWeights(cfg, t("embed").contiguous(), t("bigram").contiguous(), f32("embed.norm"), layers, f32("final.norm"),
                          lin(t("head"), pad(cfg.vocab_size, 2), kin), dtype, preset=fmt)


def load_engine_weights(model_dir, device="cpu", dtype: Optional[torch.dtype] = None) -> FudulixWeights:
    from ...io.model_dir import ShardCollection
    col = ShardCollection(model_dir)
    return build_engine_weights(FudulixConfig.from_dir(model_dir), col.tensor, device, dtype)
