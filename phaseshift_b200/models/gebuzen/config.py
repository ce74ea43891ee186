"""Gebuzen decoder configuration.

A layer has one ``parallel`` mixer -- chunk-local attention (left) and gated linear attention (right) over the same
input -- and an optional dense feed-forward.  A range of layers can be looped: it runs several times with the same
weights, every pass with a cache and a state of its own.

``config.json`` keys: ``architecture`` ("Gebuzen"), ``vocab``, ``width``, ``layers`` (a list of ``{type, mixer: {left:
{heads, kv_heads, dim, vdim, scale, mask: {size}}, right: {heads, dim, vdim, tau}}, mlp: {kind, ff} | null}``), ``loop``
(``{start, stop, times}``, optional), ``norm: {eps}``, ``residual_mult``, ``logit_scale``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, NamedTuple, Optional, Sequence

from ...runtime.state import KVSpec, RecurrentSpec, RunSpec
from ..common import SingleRank, eos_ids_of_dir, pad

ARCHITECTURE = "Gebuzen"


@dataclass(frozen=True)
class ChunkAttention:
    """Softmax attention inside blocks of ``chunk`` positions with a learned sink per head; the keys are the values."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int

    @property
    def dim_padded(self) -> int:
        """Head size in the engine's buffers and pages: the attention kernels work on multiples of 32 (zero columns)."""
        return pad(self.dim, 32)


@dataclass(frozen=True)
class GatedLinear:
    """Linear attention whose state decays per key channel."""
    heads: int
    dim: int
    vdim: int
    tau: float

    @property
    def dim_padded(self) -> int:
        return pad(self.dim, 16)

    @property
    def vdim_padded(self) -> int:
        return pad(self.vdim, 32)


@dataclass(frozen=True)
class ParallelLayer:
    left: ChunkAttention
    right: GatedLinear
    ff: Optional[int]                  # None: the layer has no feed-forward


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


class LayerRun(NamedTuple):
    """One execution of a layer: ``pass_index`` is its pass of the looped range (None outside of it), ``opens_pass`` marks
    the first layer of a pass."""
    layer: int
    pass_index: Optional[int]
    opens_pass: bool


@dataclass
class GebuzenConfig:
    vocab_size: int
    hidden_size: int
    layers: List[ParallelLayer]
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    loop: Optional[Loop] = None
    eos_token_ids: List[int] = field(default_factory=list)
    name: str = "gebuzen"
    family = "gebuzen"

    def __post_init__(self):
        for i, L in enumerate(self.layers):
            if L.left.heads % L.left.kv_heads:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if L.left.chunk < 1:
                raise ValueError(f"layer {i}: the chunk size must be positive")
        if self.loop is not None and not 0 <= self.loop.start <= self.loop.stop <= len(self.layers):
            raise ValueError("the looped range lies outside the layers")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def runs(self) -> List[LayerRun]:
        """Layer executions of one forward, in order."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [LayerRun(i, None, False) for i in range(n)]
        out = [LayerRun(i, None, False) for i in range(lp.start)]
        for t in range(lp.times):
            out += [LayerRun(i, t, i == lp.start) for i in range(lp.start, lp.stop)]
        return out + [LayerRun(i, None, False) for i in range(lp.stop, n)]

    def geometry(self, tp_rank: int = 0, tp_size: int = 1) -> SingleRank:
        if tp_size != 1:
            raise ValueError("Gebuzen models run on one rank")
        return SingleRank()

    def state_specs(self, geo=None) -> List[RunSpec]:
        """Cache and state of every layer run (a looped layer has one set per pass)."""
        out = []
        for r in self.runs():
            L = self.layers[r.layer]
            out.append(RunSpec(KVSpec(L.left.kv_heads, L.left.dim_padded, shared=True),
                               RecurrentSpec(L.right.heads, L.right.dim_padded, L.right.vdim_padded)))
        return out

    def to_dict(self) -> dict:
        layers = [{"type": "parallel",
                   "mixer": {"left": {"heads": L.left.heads, "kv_heads": L.left.kv_heads, "dim": L.left.dim, "vdim": L.left.dim,
                                      "scale": L.left.scale, "mask": {"size": L.left.chunk}},
                             "right": {"heads": L.right.heads, "dim": L.right.dim, "vdim": L.right.vdim, "tau": L.right.tau}},
                   "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}} for L in self.layers]
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult, "logit_scale": self.logit_scale}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return d

    def save(self, model_dir) -> None:
        Path(model_dir).mkdir(parents=True, exist_ok=True)
        (Path(model_dir) / "config.json").write_text(json.dumps(self.to_dict(), indent=1))

    @staticmethod
    def from_dict(raw: dict, eos_token_ids: Sequence[int] = ()) -> "GebuzenConfig":
        layers = []
        for i, e in enumerate(raw["layers"]):
            if e["type"] != "parallel":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            l, r, mlp = e["mixer"]["left"], e["mixer"]["right"], e.get("mlp")
            if int(l.get("vdim", l["dim"])) != int(l["dim"]):
                raise ValueError(f"layer {i}: the keys are the values, so vdim must equal dim")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(ParallelLayer(
                ChunkAttention(int(l["heads"]), int(l["kv_heads"]), int(l["dim"]), float(l["scale"]), int(l["mask"]["size"])),
                GatedLinear(int(r["heads"]), int(r["dim"]), int(r["vdim"]), float(r["tau"])),
                None if mlp is None else int(mlp["ff"])))
        lp = raw.get("loop")
        return GebuzenConfig(int(raw["vocab"]), int(raw["width"]), layers, float(raw["norm"]["eps"]), float(raw["residual_mult"]),
                             float(raw["logit_scale"]), None if not lp else Loop(int(lp["start"]), int(lp["stop"]), int(lp["times"])),
                             list(eos_token_ids))

    @staticmethod
    def from_dir(model_dir) -> "GebuzenConfig":
        return GebuzenConfig.from_dict(json.loads((Path(model_dir) / "config.json").read_text()), eos_ids_of_dir(model_dir))


def _uniform(preset: str, vocab: int, width: int, n_layers: int, left: ChunkAttention, right: GatedLinear, ff: int, loop=None,
             **over) -> GebuzenConfig:
    kw = dict(residual_mult=0.5, name=preset)
    kw.update(over)
    return GebuzenConfig(vocab, width, [ParallelLayer(left, right, ff)] * n_layers, loop=loop, **kw)


def tiny_config(**over) -> GebuzenConfig:
    return _uniform("gebuzen-tiny", 512, 128, 3, ChunkAttention(4, 2, 32, 32 ** -0.5, 48), GatedLinear(2, 32, 64, 8.0), 192,
                    Loop(1, 3, 2), **over)


def gebuzen_4b_config(**over) -> GebuzenConfig:
    """Layer shapes of a 4B-class model (the hybrid decoder's width, heads and feed-forward)."""
    return _uniform("gebuzen-4b", 151936, 2560, 32, ChunkAttention(16, 4, 256, 256 ** -0.5, 4096), GatedLinear(32, 128, 128, 16.0), 9216,
                    **over)


def gebuzen_27b_config(**over) -> GebuzenConfig:
    """Layer shapes of a 27B-class model (the hybrid decoder's width, heads and feed-forward)."""
    return _uniform("gebuzen-27b", 151936, 5120, 64, ChunkAttention(24, 4, 256, 256 ** -0.5, 4096), GatedLinear(48, 128, 128, 16.0), 17408,
                    **over)


PRESETS = {"gebuzen-tiny": tiny_config, "gebuzen-4b": gebuzen_4b_config, "gebuzen-27b": gebuzen_27b_config}
