"""Rotutar decoder configuration.

A layer has one mixer -- windowed attention and a delta rule with a decay per channel side by side, or linear attention whose
forget gate is its key -- and an optional feed-forward, dense or a mixture of clamped experts in groups.  Sublayers read the
residual as it is; what they return is gated by it, normed in groups and added.

``config.json`` keys: ``architecture`` ("Rotutar"), ``vocab``, ``width``, ``norm: {eps, groups}``, ``logit_softcap``, ``layers``, a
list of ``{type, mixer, mlp | null}``.  ``type`` "parallel": ``mixer: {left: {heads, kv_heads, dim, vdim, scale, mask: {size}, rot:
{base, dims}}, left_scale, right: {heads, kv_heads, dim, vdim, conv}, right_scale}`` (``conv``: taps); ``type`` "hgrn2": ``mixer:
{heads, dim, vdim}``.  ``mlp``: ``{kind: "dense", ff}`` or ``{kind: "moe", expert: {ff, limit}, router: {experts, top, groups:
{count, keep}}}``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, Optional, Sequence, Union

from ...runtime.state import ConvSpec, KVSpec, RecurrentSpec, RunSpec
from ..common import SingleRank, eos_ids_of_dir, pad

ARCHITECTURE = "Rotutar"


@dataclass(frozen=True)
class WindowAttention:
    """Softmax attention in a window with a sink per head; queries and keys are normed over all heads and turned."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot_base: float
    rot_dims: int

    @property
    def dim_padded(self) -> int:
        """Head size of queries, keys and values in the engine's buffers and pages: the tensor-core kernels work on groups of
        64 columns (zero columns)."""
        return pad(max(self.dim, self.vdim), 64)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "mask": {"size": self.window}, "rot": {"base": self.rot_base, "dims": self.rot_dims}}


def _state_size(n: int, step: int) -> int:
    """Engine size of a delta-rule head: what the tiled kernels work on, or any multiple of `step` beyond that."""
    return pad(n, 64) if n <= 128 else pad(n, step)


@dataclass(frozen=True)
class GatedDelta:
    """Delta rule behind short convolutions, with a decay per head and key channel."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def dim_padded(self) -> int:
        return _state_size(self.dim, 16)

    @property
    def vdim_padded(self) -> int:
        return _state_size(self.vdim, 32)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.taps}


@dataclass(frozen=True)
class Parallel:
    left: WindowAttention
    left_scale: float
    right: GatedDelta
    right_scale: float

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}


@dataclass(frozen=True)
class ForgetLinear:
    """Linear attention in which what a channel forgets is how much it takes in."""
    heads: int
    dim: int
    vdim: int

    @property
    def dim_padded(self) -> int:
        return pad(self.dim, 16)

    @property
    def vdim_padded(self) -> int:
        return pad(self.vdim, 32)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}


Mixer = Union[Parallel, ForgetLinear]
TYPE_OF = {Parallel: "parallel", ForgetLinear: "hgrn2"}


@dataclass(frozen=True)
class Dense:
    ff: int

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class Mixture:
    ff: int
    limit: float
    experts: int
    top: int
    groups: int = 1
    keep: int = 1

    def to_dict(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                "router": {"experts": self.experts, "top": self.top, "groups": {"count": self.groups, "keep": self.keep}}}


@dataclass(frozen=True)
class Layer:
    mixer: Mixer
    mlp: Union[Dense, Mixture, None]


@dataclass
class RotutarConfig:
    vocab_size: int
    hidden_size: int
    layers: List[Layer]
    norm_eps: float = 1e-6
    norm_groups: int = 1
    logit_softcap: float = 30.0
    eos_token_ids: List[int] = field(default_factory=list)
    name: str = "rotutar"
    family = "rotutar"

    def __post_init__(self):
        if self.norm_groups < 1 or self.hidden_size % self.norm_groups:
            raise ValueError("the norm's groups are equal parts of the width")
        if not self.logit_softcap > 0:
            raise ValueError("the soft limit of the logits must be positive")
        for i, L in enumerate(self.layers):
            m, c = L.mixer, L.mlp
            if isinstance(m, Parallel):
                l, r = m.left, m.right
                if l.heads % l.kv_heads or r.heads % r.kv_heads:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if l.rot_dims % 2 or not 0 < l.rot_dims <= l.dim:
                    raise ValueError(f"layer {i}: rotated dimensions come in pairs and lie within the head")
                if l.window < 1:
                    raise ValueError(f"layer {i}: the window must hold the position itself")
                if r.taps < 1:
                    raise ValueError(f"layer {i}: a convolution has at least one tap")
            if isinstance(c, Mixture):
                if c.groups < 1 or c.experts % c.groups or not 1 <= c.keep <= c.groups:
                    raise ValueError(f"layer {i}: experts must form equal groups, some of which are kept")
                if not 1 <= c.top <= c.keep * (c.experts // c.groups):
                    raise ValueError(f"layer {i}: the kept groups must hold the chosen experts")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def geometry(self, tp_rank: int = 0, tp_size: int = 1) -> SingleRank:
        if tp_size != 1:
            raise ValueError("Rotutar models run on one rank")
        return SingleRank()

    def state_specs(self, geo=None) -> List[RunSpec]:
        """Pages, recurrent state and the rows that the convolutions look back to (every value head has its own copy of its
        query and key channels, so heads never share a row)."""
        out = []
        for L in self.layers:
            m = L.mixer
            if isinstance(m, ForgetLinear):
                out.append(RunSpec(None, RecurrentSpec(m.heads, m.dim_padded, m.vdim_padded)))
                continue
            l, r = m.left, m.right
            out.append(RunSpec(KVSpec(l.kv_heads, l.dim_padded), RecurrentSpec(r.heads, r.dim_padded, r.vdim_padded),
                               ConvSpec(r.heads * (2 * r.dim_padded + r.vdim_padded), r.taps - 1)))
        return out

    def to_dict(self) -> dict:
        layers = [{"type": TYPE_OF[type(L.mixer)], "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                  for L in self.layers]
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "logit_softcap": self.logit_softcap}

    def save(self, model_dir) -> None:
        Path(model_dir).mkdir(parents=True, exist_ok=True)
        (Path(model_dir) / "config.json").write_text(json.dumps(self.to_dict(), indent=1))

    @staticmethod
    def from_dict(raw: dict, eos_token_ids: Sequence[int] = ()) -> "RotutarConfig":
        layers = []
        for i, e in enumerate(raw["layers"]):
            m, c = e["mixer"], e.get("mlp")
            if e["type"] == "parallel":
                l, r = m["left"], m["right"]
                mixer: Mixer = Parallel(
                    WindowAttention(int(l["heads"]), int(l["kv_heads"]), int(l["dim"]), int(l["vdim"]), float(l["scale"]),
                                    int(l["mask"]["size"]), float(l["rot"]["base"]), int(l["rot"]["dims"])), float(m["left_scale"]),
                    GatedDelta(int(r["heads"]), int(r["kv_heads"]), int(r["dim"]), int(r["vdim"]), int(r["conv"])), float(m["right_scale"]))
            elif e["type"] == "hgrn2":
                mixer = ForgetLinear(int(m["heads"]), int(m["dim"]), int(m["vdim"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if c is None:
                mlp = None
            elif c["kind"] == "dense":
                mlp = Dense(int(c["ff"]))
            elif c["kind"] == "moe":
                r = c["router"]
                g = r.get("groups") or {"count": 1, "keep": 1}
                mlp = Mixture(int(c["expert"]["ff"]), float(c["expert"]["limit"]), int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {c['kind']!r}")
            layers.append(Layer(mixer, mlp))
        n = raw["norm"]
        return RotutarConfig(int(raw["vocab"]), int(raw["width"]), layers, float(n["eps"]), int(n["groups"]), float(raw["logit_softcap"]),
                             list(eos_token_ids))

    @staticmethod
    def from_dir(model_dir) -> "RotutarConfig":
        return RotutarConfig.from_dict(json.loads((Path(model_dir) / "config.json").read_text()), eos_ids_of_dir(model_dir))


def _alternating(preset: str, vocab: int, width: int, n_layers: int, par: Parallel, linear: ForgetLinear, dense: Dense, moe: Mixture,
                 groups: int, **over) -> RotutarConfig:
    """Attention beside the delta rule with a dense feed-forward, then linear attention with a mixture, and so on."""
    layers = [Layer(linear, moe) if i % 2 else Layer(par, dense) for i in range(n_layers)]
    kw = dict(norm_groups=groups, name=preset)
    kw.update(over)
    return RotutarConfig(vocab, width, layers, **kw)


def tiny_config(**over) -> RotutarConfig:
    return _alternating("rotutar-tiny", 512, 128, 4, Parallel(WindowAttention(4, 2, 40, 32, 0.2, 60, 10000.0, 24), 0.7, GatedDelta(4, 2, 32, 48, 4), 0.6),
                        ForgetLinear(3, 32, 64), Dense(160), Mixture(64, 2.0, 12, 3, 4, 2), 4, **over)


def rotutar_4b_config(**over) -> RotutarConfig:
    """Layer shapes of a 4B-class model (the width, heads and active feed-forward of the other families' presets)."""
    return _alternating("rotutar-4b", 151936, 2560, 32,
                        Parallel(WindowAttention(16, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 64), 0.7, GatedDelta(32, 16, 128, 128, 4), 0.7),
                        ForgetLinear(32, 128, 128), Dense(9216), Mixture(1152, 7.0, 64, 8, 4, 2), 4, **over)


def rotutar_27b_config(**over) -> RotutarConfig:
    """Layer shapes of a 27B-class model."""
    return _alternating("rotutar-27b", 151936, 5120, 64,
                        Parallel(WindowAttention(24, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 64), 0.7, GatedDelta(48, 16, 128, 128, 4), 0.7),
                        ForgetLinear(48, 128, 128), Dense(17408), Mixture(2176, 7.0, 64, 8, 4, 2), 8, **over)


PRESETS = {"rotutar-tiny": tiny_config, "rotutar-4b": rotutar_4b_config, "rotutar-27b": rotutar_27b_config}
