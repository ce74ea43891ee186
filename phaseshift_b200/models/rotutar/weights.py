"""Rotutar weights: tensor names and shapes, random initialisation, and the engine's fused layout.

Per layer the engine runs ``in_proj`` (everything that the mixer projects from the residual and, behind it, the gate of the
mixer's result), the output projections, and then either ``gate_up`` (rows alternate gate and up), ``down`` and the gate of the
feed-forward's result, or the router with that gate in one launch and the experts' stacked matrices.

Sizes are padded with zero rows and columns to what the kernels work on; zeros change no score, state, norm or sum.
"""
from __future__ import annotations

import zlib
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Union

import torch

from ...ops.specs import AttnSpec, DeltaSpec, GlaSpec, HeadsSpec, MoeSpec, rotation_frequencies
from ..common import alternate, pad, pad_cols, pad_heads, pad_rows, plain_linear
from ..qwen35.weights import LinearW
from .config import Dense, ForgetLinear, Mixture, Parallel, RotutarConfig


def tensor_shapes(cfg: RotutarConfig, rank: Optional[int] = None) -> Dict[str, tuple]:
    """``rank`` of the low-rank projections (decay and output gate of the delta rule); a loaded model's tensors give theirs."""
    w = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, w), "final.norm": (w,), "head": (cfg.vocab_size, w)}

    def feed_forward(p: str, ff: int) -> None:
        out.update({p + "gate": (ff, w), p + "up": (ff, w), p + "down": (w, ff)})
    for i, L in enumerate(cfg.layers):
        m, c, p = L.mixer, L.mlp, f"l{i}."
        x, y = p + "mix.", p + "mlp."
        out.update({p + "norm1": (w,), p + "rg1": (w, w), p + "rg1.b": (w,)})
        if isinstance(m, Parallel):
            l, r = m.left, m.right
            sizes = {"q": l.heads * l.dim, "k": l.kv_heads * l.dim, "v": l.kv_heads * l.vdim}
            out.update({f"{x}left.{n}": (s, w) for n, s in sizes.items()})
            out.update({x + "left.q.norm": (sizes["q"],), x + "left.k.norm": (sizes["k"],), x + "left.sink": (l.heads,),
                        x + "left.o": (w, l.heads * l.vdim)})
            x += "right."
            sizes = {"q": r.kv_heads * r.dim, "k": r.kv_heads * r.dim, "v": r.heads * r.vdim}
            out.update({x + n: (s, w) for n, s in sizes.items()})
            out.update({f"{x}{n}.conv": (s, r.taps) for n, s in sizes.items()})
            n = rank or r.dim
            out.update({x + "b": (r.heads, w), x + "A_log": (r.heads,), x + "dt_bias": (r.heads * r.dim,), x + "norm": (r.vdim,),
                        x + "a1": (n, w), x + "a2": (r.heads * r.dim, n), x + "g1": (n, w), x + "g2": (r.heads * r.vdim, n),
                        x + "o": (w, r.heads * r.vdim)})
        else:
            k, v = m.heads * m.dim, m.heads * m.vdim
            out.update({x + "q": (k, w), x + "f": (k, w), x + "f.b": (k,), x + "lower": (k,), x + "v": (v, w), x + "norm": (m.vdim,),
                        x + "o": (w, v)})
        if c is None:
            continue
        out.update({p + "norm2": (w,), p + "rg2": (w, w), p + "rg2.b": (w,)})
        if isinstance(c, Dense):
            feed_forward(y, c.ff)
        else:
            for e in range(c.experts):
                feed_forward(f"{y}e{e}.", c.ff)
            out[y + "router"] = (c.experts, w)
    return out


def random_tensor(name: str, shape: tuple, seed: int, device="cpu") -> torch.Tensor:
    """Deterministic per-tensor init, rounded to bf16: matrices N(0, fan_in^-1/2), norms around one, convolutions that mix their
    taps, lower bounds in (0, 1), decays from a token or two to hundreds."""
    g = torch.Generator(device=device)
    g.manual_seed((seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
    t = torch.randn(shape, device=device, generator=g)
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm", "norm1", "norm2"):
        t = 1.0 + 0.1 * t
    elif leaf == "lower":
        t = torch.sigmoid(t)
    elif leaf == "dt_bias":
        t = t - 3.0
    elif leaf in ("A_log", "sink") or leaf == "b" and len(shape) == 1:
        t = 0.5 * t
    elif name != "embed":
        t = t * shape[1] ** -0.5
    return t.to(torch.bfloat16)


def random_weights(cfg: RotutarConfig, seed: int = 0, device="cpu", rank: Optional[int] = None) -> Dict[str, torch.Tensor]:
    return {n: random_tensor(n, s, seed, device) for n, s in tensor_shapes(cfg, rank).items()}


def random_getter(cfg: RotutarConfig, seed: int = 0, device="cpu") -> Callable[[str], torch.Tensor]:
    shapes = tensor_shapes(cfg)
    return lambda name: random_tensor(name, shapes[name], seed, device)


@dataclass
class ParallelW:
    heads: HeadsSpec
    attn: AttnSpec
    delta: DeltaSpec
    left_o: LinearW
    right_o: LinearW
    left_scale: float
    right_scale: float

    def linears(self) -> List[LinearW]:
        return [self.left_o, self.right_o]


@dataclass
class ForgetLinearW:
    gla: GlaSpec
    o: LinearW

    def linears(self) -> List[LinearW]:
        return [self.o]


@dataclass
class DenseW:
    gate_up: LinearW
    down: LinearW
    gate: LinearW                     # of the result

    def linears(self) -> List[LinearW]:
        return [self.gate_up, self.down, self.gate]


@dataclass
class MixtureW:
    router: LinearW                   # rows [experts | gate of the result]
    gate_off: int
    moe: MoeSpec

    def linears(self) -> List[LinearW]:
        return [self.router]


@dataclass
class LayerW:
    in_proj: LinearW
    gate_off: int                     # first column of the mixer result's gate
    mixer: Union[ParallelW, ForgetLinearW]
    gate1: torch.Tensor               # f32 [width]: bias of the gate, then the norm's weight
    norm1: torch.Tensor
    mlp: Union[DenseW, MixtureW, None]
    gate2: Optional[torch.Tensor]
    norm2: Optional[torch.Tensor]

    def linears(self) -> List[LinearW]:
        return [self.in_proj] + self.mixer.linears() + (self.mlp.linears() if self.mlp is not None else [])


@dataclass
class RotutarWeights:
    cfg: RotutarConfig
    embed: torch.Tensor               # [vocab, width]
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

    def _low_rank(self) -> int:
        d = [l.mixer.delta for l in self.layers if isinstance(l.mixer, ParallelW)]
        return sum(s.a2.numel() + s.g2.numel() for s in d)

    def decode_read_bytes(self) -> int:
        """Weight bytes a decode step of one row streams (of a mixture, the experts one row goes to)."""
        n = sum(w.N * w.k_padded for w in self.linears()) + self._low_rank()
        n += sum((m.gate_up.numel() + m.down.numel()) // m.experts * m.top for m in self._mixtures())
        return n * self.embed.element_size()

    def weight_bytes(self) -> int:
        n = sum(w.N * w.k_padded for w in self.linears()) + self._low_rank() + self.embed.numel()
        return (n + sum(m.gate_up.numel() + m.down.numel() for m in self._mixtures())) * self.embed.element_size()


def build_engine_weights(cfg: RotutarConfig, get: Callable[[str], torch.Tensor], device="cpu",
                         dtype: Optional[torch.dtype] = None) -> RotutarWeights:
    """``dtype``: what projections and activations run in, bfloat16 or float32 (default: bfloat16 on a CUDA device)."""
    dev = torch.device(device)
    dtype = dtype or (torch.bfloat16 if dev.type == "cuda" else torch.float32)
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"Rotutar runs in bfloat16 or float32, not {dtype}")
    fmt = "bf16" if dtype == torch.bfloat16 else "f32"
    W = cfg.hidden_size
    nout = pad(W, 4)                     # output rows of projections onto the residual width (paired fp32 stores need even pitches)
    kin = pad(W, 32)                     # input width of the projections that read the residual

    def t(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=dtype)

    def f32(name: str) -> torch.Tensor:
        return get(name).to(device=dev, dtype=torch.float32).contiguous()

    def lin(w: torch.Tensor, n: int, k: int) -> LinearW:
        return plain_linear(w, n, k, fmt)

    def out_proj(name: str, heads: int, dim: int, to: int) -> LinearW:
        return lin(pad_heads(t(name).T.contiguous(), heads, dim, to).T, nout, heads * to)

    def parallel(m: Parallel, x: str):
        """The mixer and the rows of `in_proj` that it reads."""
        l, r, y, x = m.left, m.right, x + "right.", x + "left."
        H, G, D = l.heads, l.kv_heads, l.dim_padded
        parts = (("q", H, l.dim), ("k", G, l.dim), ("v", G, l.vdim))
        rows = [pad_heads(t(x + n), h, d, D) for n, h, d in parts]
        heads = HeadsSpec(H, G, D, l.dim, l.vdim, cfg.norm_eps, rotation_frequencies(l.rot_base, l.rot_dims).to(dev))
        heads.q_norm, heads.k_norm = (pad_heads(f32(x + n + ".norm"), h, d, D).contiguous() for n, h, d in parts[:2])
        attn = AttnSpec(H, G, D, l.scale, window=l.window, sink=f32(x + "sink"))

        dk, dv = r.dim_padded, r.vdim_padded
        parts = (("q", r.kv_heads, r.dim, dk), ("k", r.kv_heads, r.dim, dk), ("v", r.heads, r.vdim, dv))
        q = (H + 2 * G) * D
        b = q + 2 * r.kv_heads * dk + r.heads * dv
        a1, g1 = t(y + "a1"), t(y + "g1")
        ra, rg = pad(a1.shape[0], 16), pad(g1.shape[0], 16)
        a = b + pad(r.heads, 16)
        rows += [pad_heads(t(y + n), h, d, to) for n, h, d, to in parts]
        rows += [pad_rows(t(y + "b"), pad(r.heads, 16)), pad_rows(a1, ra), pad_rows(g1, rg)]
        conv = torch.cat([pad_heads(t(f"{y}{n}.conv"), h, d, to) for n, h, d, to in parts], 0).T.contiguous()
        delta = DeltaSpec(r.heads, r.kv_heads, dk, dv, r.dim, r.vdim, q, b, a, a + ra, cfg.norm_eps, conv,
                          pad_cols(pad_heads(t(y + "a2"), r.heads, r.dim, dk), ra).contiguous(),
                          pad_heads(f32(y + "dt_bias"), r.heads, r.dim, dk).contiguous(), torch.exp(f32(y + "A_log")),
                          pad_cols(pad_heads(t(y + "g2"), r.heads, r.vdim, dv), rg).contiguous(),
                          pad_rows(f32(y + "norm"), dv).contiguous())
        return ParallelW(heads, attn, delta, out_proj(x + "o", H, l.vdim, D), out_proj(y + "o", r.heads, r.vdim, dv),
                         m.left_scale, m.right_scale), rows

    def forget_linear(m: ForgetLinear, x: str):
        H, dk, dv = m.heads, m.dim_padded, m.vdim_padded
        rows = [pad_heads(t(x + n), H, m.dim, dk) for n in ("q", "f")] + [pad_heads(t(x + "v"), H, m.vdim, dv)]
        lower = torch.ones(H * dk, device=dev).reshape(H, dk)                # padded channels forget and take in nothing
        lower[:, :m.dim] = f32(x + "lower").reshape(H, m.dim)
        gla = GlaSpec(H, dk, dv, m.vdim, 0, -1, 2 * H * dk, -1, H * dk, 0, 1.0, 1.0, cfg.norm_eps, None,
                      pad_heads(f32(x + "f.b"), H, m.dim, dk).contiguous(), pad_rows(f32(x + "norm"), dv).contiguous(), lower.flatten())
        return ForgetLinearW(gla, out_proj(x + "o", H, m.vdim, dv)), rows

    def gate_up(p: str, ffp: int) -> torch.Tensor:
        return alternate(pad_rows(t(p + "gate"), ffp), pad_rows(t(p + "up"), ffp))

    def mixture(c: Mixture, p: str) -> MixtureW:
        y, ffp, n = p + "mlp.", pad(c.ff, 32), pad(c.experts, 8)
        gu = torch.zeros(c.experts, 2 * ffp, kin, device=dev, dtype=dtype)
        down = torch.zeros(c.experts, nout, ffp, device=dev, dtype=dtype)
        for e in range(c.experts):
            gu[e, :, :W] = gate_up(f"{y}e{e}.", ffp)
            down[e, :W, :c.ff] = t(f"{y}e{e}.down")
        spec = MoeSpec(c.experts, 0, c.top, c.groups, c.keep, ffp, nout, None, gu.flatten(0, 1), down.flatten(0, 1), sigmoid=True, group_top=2,
                       renormalize=False, limit=c.limit)
        return MixtureW(lin(torch.cat([pad_rows(t(y + "router"), n), t(p + "rg2")], 0), n + pad(W, 8), kin), n, spec)

    layers = []
    for i, L in enumerate(cfg.layers):
        p, c = f"l{i}.", L.mlp
        mixer, rows = (parallel if isinstance(L.mixer, Parallel) else forget_linear)(L.mixer, p + "mix.")
        n = sum(r.shape[0] for r in rows)
        in_proj = lin(torch.cat(rows + [t(p + "rg1")], 0), n + pad(W, 8), kin)
        del rows
        mlp = None
        if isinstance(c, Dense):
            fp = pad(c.ff, 32)
            mlp = DenseW(lin(gate_up(p + "mlp.", fp), 2 * fp, kin), lin(t(p + "mlp.down"), nout, fp), lin(t(p + "rg2"), pad(W, 8), kin))
        elif c is not None:
            mlp = mixture(c, p)
        layers.append(LayerW(in_proj, n, mixer, f32(p + "rg1.b"), f32(p + "norm1"), mlp, None if c is None else f32(p + "rg2.b"),
                             None if c is None else f32(p + "norm2")))
    return RotutarWeights(cfg, t("embed").contiguous(), layers, f32("final.norm"), lin(t("head"), pad(cfg.vocab_size, 2), kin), dtype, preset=fmt)


def load_engine_weights(model_dir, device="cpu", dtype: Optional[torch.dtype] = None) -> RotutarWeights:
    from ...io.model_dir import ShardCollection
    col = ShardCollection(model_dir)
    return build_engine_weights(RotutarConfig.from_dir(model_dir), col.tensor, device, dtype)
