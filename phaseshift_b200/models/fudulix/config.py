"""Fudulix decoder configuration.

The embedding adds a row per token and one per pair of tokens.  A layer has one mixer -- rotated and normed heads in a sliding
window, or convolved, jointly normed heads in a window that also keeps the first tokens -- whose values may be blended with
those of the first layer that takes part, and an optional feed-forward: dense, or a mixture of experts in groups, some of
which are the identity, beside a shared one.

``config.json`` keys: ``architecture`` ("Fudulix"), ``vocab``, ``width``, ``norm: {eps}``, ``embedding: {bigram: {buckets,
mul_prev, mul_cur}}``, ``layers``, a list of ``{type, mixer, mlp | null}``.  ``mixer``: ``{heads, kv_heads, dim, vdim, scale,
v_mix, rot: {base, dims, scaling}}``; ``type`` "attention": ``scaling: {factor, low, high, original}``, ``mask: {size}``;
``type`` "attention_2": ``scaling: {factor, original, fast, slow}``, ``mask: {size, keep_first}`` and ``conv`` (taps).
``mlp``: ``{kind: "dense", ff}`` or ``{kind: "moe", expert: {ff}, router: {experts, top, groups: {count, keep}, identity},
shared: {ff}}``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, Optional, Sequence, Tuple, Union

import torch

from ...ops.specs import ramped_frequencies, rotation_frequencies, stepped_frequencies
from ...runtime.state import ConvSpec, KVSpec, RunSpec
from ..common import SingleRank, eos_ids_of_dir, pad

ARCHITECTURE = "Fudulix"


@dataclass(frozen=True)
class Steps:
    """Frequency scaling by wavelength (None in its place: no scaling)."""
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class Ramp:
    """Frequency scaling by pair."""
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class _Heads:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot_base: float
    rot_dims: int
    v_mix: bool

    @property
    def dim_padded(self) -> int:
        """Head size of queries, keys and values in the engine's buffers and pages: the tensor-core kernels work on groups of
        64 columns (zero columns)."""
        return pad(max(self.dim, self.vdim), 64)

    @property
    def channels(self) -> int:
        return (self.heads + 2 * self.kv_heads) * self.dim_padded

    def _dict(self, scaling, **mask) -> dict:
        rot = {"base": self.rot_base, "dims": self.rot_dims}
        if scaling is not None:
            rot["scaling"] = scaling.to_dict()
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "v_mix": self.v_mix, "mask": {"size": self.window, **mask}, "rot": rot}


@dataclass(frozen=True)
class UnitAttention(_Heads):
    """Neighbouring dimensions turn, queries and keys are divided by their root mean square per head, one is added to the
    softmax's denominator."""
    scaling: Optional[Steps] = None

    def rotation(self) -> Tuple[torch.Tensor, float]:
        f, s = rotation_frequencies(self.rot_base, self.rot_dims), self.scaling
        return (f if s is None else stepped_frequencies(f, s.factor, s.low, s.high, s.original)), 1.0

    def to_dict(self) -> dict:
        return self._dict(self.scaling)


@dataclass(frozen=True)
class ConvAttention(_Heads):
    """A short convolution over each projected channel, queries and keys normed over all heads at once, halves of a head turn,
    the first tokens stay visible."""
    scaling: Optional[Ramp] = None
    keep_first: int = 0
    taps: int = 1

    def rotation(self) -> Tuple[torch.Tensor, float]:
        f, s = rotation_frequencies(self.rot_base, self.rot_dims), self.scaling
        return (f, 1.0) if s is None else ramped_frequencies(f, self.rot_base, s.factor, s.original, s.fast, s.slow)

    def to_dict(self) -> dict:
        return {**self._dict(self.scaling, keep_first=self.keep_first), "conv": self.taps}


Mixer = Union[UnitAttention, ConvAttention]
TYPE_OF = {UnitAttention: "attention", ConvAttention: "attention_2"}


@dataclass(frozen=True)
class Dense:
    ff: int

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class Mixture:
    ff: int
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    identity: int = 0
    shared_ff: Optional[int] = None      # None: no shared expert

    def to_dict(self) -> dict:
        d = {"kind": "moe", "expert": {"ff": self.ff},
             "router": {"experts": self.experts, "top": self.top, "groups": {"count": self.groups, "keep": self.keep}, "identity": self.identity}}
        return d if self.shared_ff is None else {**d, "shared": {"ff": self.shared_ff}}


@dataclass(frozen=True)
class Layer:
    mixer: Mixer
    mlp: Union[Dense, Mixture, None]


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class FudulixConfig:
    vocab_size: int
    hidden_size: int
    bigram: Bigram
    layers: List[Layer]
    norm_eps: float = 1e-6
    eos_token_ids: List[int] = field(default_factory=list)
    name: str = "fudulix"
    family = "fudulix"
    keeps_last_token = True            # runtime/state.py: the embedding looks back one token

    def __post_init__(self):
        mixing = None
        for i, L in enumerate(self.layers):
            m, c = L.mixer, L.mlp
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if m.rot_dims % 2 or not 0 < m.rot_dims <= m.dim:
                raise ValueError(f"layer {i}: rotated dimensions come in pairs and lie within the head")
            if m.window < 1:
                raise ValueError(f"layer {i}: the window must hold the position itself")
            if isinstance(m, ConvAttention) and (m.taps < 1 or m.keep_first < 0):
                raise ValueError(f"layer {i}: a convolution has at least one tap, and no negative number of tokens is kept")
            if m.v_mix:
                mixing = m if mixing is None else mixing
                if mixing.kv_heads * mixing.vdim != m.kv_heads * m.vdim:
                    raise ValueError(f"layer {i}: its values have another size than those it mixes in")
            if isinstance(c, Mixture):
                n = c.experts + c.identity
                if c.groups < 1 or n % c.groups or not 1 <= c.keep <= c.groups:
                    raise ValueError(f"layer {i}: experts must form equal groups, some of which are kept")
                if not 1 <= c.top <= c.keep * (n // c.groups):
                    raise ValueError(f"layer {i}: the kept groups must hold the chosen experts")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def geometry(self, tp_rank: int = 0, tp_size: int = 1) -> SingleRank:
        if tp_size != 1:
            raise ValueError("Fudulix models run on one rank")
        return SingleRank()

    def state_specs(self, geo=None) -> List[RunSpec]:
        out = []
        for L in self.layers:
            m = L.mixer
            out.append(RunSpec(KVSpec(m.kv_heads, m.dim_padded), None, ConvSpec(m.channels, m.taps - 1) if isinstance(m, ConvAttention) else None))
        return out

    def first_mixing(self) -> Optional[int]:
        """The layer whose values later ones mix in."""
        return next((i for i, L in enumerate(self.layers) if L.mixer.v_mix), None)

    def to_dict(self) -> dict:
        layers = [{"type": TYPE_OF[type(L.mixer)], "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                  for L in self.layers]
        b = self.bigram
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "embedding": {"bigram": {"buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur}}, "layers": layers,
                "norm": {"eps": self.norm_eps}}

    def save(self, model_dir) -> None:
        Path(model_dir).mkdir(parents=True, exist_ok=True)
        (Path(model_dir) / "config.json").write_text(json.dumps(self.to_dict(), indent=1))

    @staticmethod
    def from_dict(raw: dict, eos_token_ids: Sequence[int] = ()) -> "FudulixConfig":
        layers = []
        for i, e in enumerate(raw["layers"]):
            m, rot = e["mixer"], e["mixer"]["rot"]
            sc = rot.get("scaling")
            heads = (int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(m["mask"]["size"]),
                     float(rot["base"]), int(rot["dims"]), bool(m.get("v_mix", False)))
            if e["type"] == "attention":
                mixer: Mixer = UnitAttention(*heads, None if sc is None else Steps(
                    float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"])))
            elif e["type"] == "attention_2":
                mixer = ConvAttention(*heads, None if sc is None else Ramp(
                    float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"])),
                    int(m["mask"].get("keep_first", 0)), int(m["conv"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            c = e.get("mlp")
            if c is None:
                mlp = None
            elif c["kind"] == "dense":
                mlp = Dense(int(c["ff"]))
            elif c["kind"] == "moe":
                r = c["router"]
                g, shared = r.get("groups") or {"count": 1, "keep": 1}, c.get("shared")
                mlp = Mixture(int(c["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]),
                              int(r.get("identity") or 0), None if shared is None else int(shared["ff"]))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {c['kind']!r}")
            layers.append(Layer(mixer, mlp))
        b = raw["embedding"]["bigram"]
        return FudulixConfig(int(raw["vocab"]), int(raw["width"]), Bigram(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])), layers,
                             float(raw["norm"]["eps"]), list(eos_token_ids))

    @staticmethod
    def from_dir(model_dir) -> "FudulixConfig":
        return FudulixConfig.from_dict(json.loads((Path(model_dir) / "config.json").read_text()), eos_ids_of_dir(model_dir))


def _alternating(preset: str, vocab: int, width: int, n_layers: int, unit: UnitAttention, conv: ConvAttention, dense: Dense, moe: Mixture,
                 **over) -> FudulixConfig:
    """Windowed attention with a dense feed-forward, then convolved attention with a mixture, and so on."""
    layers = [Layer(conv, moe) if i % 2 else Layer(unit, dense) for i in range(n_layers)]
    kw = dict(name=preset)
    kw.update(over)
    return FudulixConfig(vocab, width, Bigram(4 * vocab + 3, 8191, 31), layers, **kw)


def tiny_config(**over) -> FudulixConfig:
    return _alternating("fudulix-tiny", 512, 128, 4, UnitAttention(6, 2, 40, 32, 0.2, 60, 10000.0, 24, True, Steps(4.0, 1.0, 4.0, 64)),
                        ConvAttention(4, 2, 32, 32, 32 ** -0.5, 50, 10000.0, 32, True, Ramp(4.0, 64, 16.0, 1.0), 10, 3),
                        Dense(160), Mixture(64, 12, 3, 4, 2, 4, 96), **over)


def fudulix_4b_config(**over) -> FudulixConfig:
    """Layer shapes of a 4B-class model (the width, attention heads and active feed-forward of the other families' presets)."""
    return _alternating("fudulix-4b", 151936, 2560, 32, UnitAttention(16, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 64, True, Steps(8.0, 1.0, 4.0, 8192)),
                        ConvAttention(16, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 256, True, Ramp(8.0, 8192, 32.0, 1.0), 128, 4),
                        Dense(9216), Mixture(1024, 60, 8, 4, 2, 4, 1024), **over)


def fudulix_27b_config(**over) -> FudulixConfig:
    """Layer shapes of a 27B-class model."""
    return _alternating("fudulix-27b", 151936, 5120, 64, UnitAttention(24, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 64, True, Steps(8.0, 1.0, 4.0, 8192)),
                        ConvAttention(24, 4, 256, 256, 256 ** -0.5, 4096, 1e6, 256, True, Ramp(8.0, 8192, 32.0, 1.0), 128, 4),
                        Dense(17408), Mixture(1920, 60, 8, 4, 2, 4, 2048), **over)


PRESETS = {"fudulix-tiny": tiny_config, "fudulix-4b": fudulix_4b_config, "fudulix-27b": fudulix_27b_config}
