"""Luvutar decoder configuration.

The residual is several parallel streams that every sublayer reads, mixes and writes (hyper-connections).  A layer has one
mixer -- latent attention in a sliding window, or grouped attention with a learned bias per distance -- and an optional dense
feed-forward.  An attention layer may read the keys and values of an earlier one.

``config.json`` keys: ``architecture`` ("Luvutar"), ``vocab``, ``width``, ``streams``, ``norm: {eps}``, ``layers``, a list of
``{type, mixer, mlp: {kind, ff} | null}``.  ``type`` "latent_attention": ``mixer: {heads, dim, rot_dim, vdim, q_rank, kv_rank,
scale, rot: {base, dims}, mask: {size}}``; ``type`` "attention": ``mixer: {heads, kv_heads, dim, vdim, scale, bias_max,
q_temp: {coef, every}, kv_from (optional)}``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import List, Optional, Sequence, Union

from ...runtime.state import KVSpec, RunSpec
from ..common import SingleRank, eos_ids_of_dir, pad

ARCHITECTURE = "Luvutar"


@dataclass(frozen=True)
class LatentAttention:
    """Queries and keys / values through low-rank latents; one rotated key part shared by all heads; a window of `window`
    positions and a learned sink per head; elementwise output gate.  The cache holds the latent and the rotated part."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    window: int

    # Sizes in the engine's buffers and pages: the tensor-core kernels work on groups of 64 columns (zero columns).
    @property
    def dim_padded(self) -> int:
        return pad(self.dim, 64)

    @property
    def rot_padded(self) -> int:
        return pad(self.rot_dim, 64)

    @property
    def vdim_padded(self) -> int:
        return pad(self.vdim, 64)

    @property
    def q_rank_padded(self) -> int:
        return pad(self.q_rank, 32)

    @property
    def kv_rank_padded(self) -> int:
        return pad(self.kv_rank, 64)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dim},
                "mask": {"size": self.window}}


@dataclass(frozen=True)
class BiasedAttention:
    """Grouped causal attention without rotation: a query temperature that grows with the position, a learned bias per
    distance bucket and head, one output gate per head.  ``kv_from``: the layer whose keys and values it reads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    temp_coef: float
    temp_every: float
    kv_from: Optional[int] = None

    @property
    def dim_padded(self) -> int:
        """Head size of queries, keys and values in the engine's buffers and pages."""
        return pad(max(self.dim, self.vdim), 32)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "bias_max": self.bias_max, "q_temp": {"coef": self.temp_coef, "every": self.temp_every}}
        return d if self.kv_from is None else {**d, "kv_from": self.kv_from}


Mixer = Union[LatentAttention, BiasedAttention]
TYPE_OF = {LatentAttention: "latent_attention", BiasedAttention: "attention"}


@dataclass(frozen=True)
class Layer:
    mixer: Mixer
    ff: Optional[int]                  # None: the layer has no feed-forward


@dataclass
class LuvutarConfig:
    vocab_size: int
    hidden_size: int
    streams: int
    layers: List[Layer]
    norm_eps: float = 1e-6
    eos_token_ids: List[int] = field(default_factory=list)
    name: str = "luvutar"
    family = "luvutar"

    def __post_init__(self):
        if self.streams < 1:
            raise ValueError("there must be at least one stream")
        for i, L in enumerate(self.layers):
            m = L.mixer
            if isinstance(m, LatentAttention):
                if m.rot_dim % 2:
                    raise ValueError(f"layer {i}: rotated dimensions come in pairs")
                if m.window < 1:
                    raise ValueError(f"layer {i}: the window must hold the position itself")
                continue
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, BiasedAttention) or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own")
                if (src.heads, src.kv_heads, src.dim, src.vdim) != (m.heads, m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i}: the shared keys and values have another head geometry")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def geometry(self, tp_rank: int = 0, tp_size: int = 1) -> SingleRank:
        if tp_size != 1:
            raise ValueError("Luvutar models run on one rank")
        return SingleRank()

    def state_specs(self, geo=None) -> List[RunSpec]:
        """Cache of every layer; a layer that reads another one's keys and values has none."""
        out = []
        for L in self.layers:
            m = L.mixer
            if isinstance(m, LatentAttention):
                kv = KVSpec(1, m.kv_rank_padded + m.rot_padded, shared=True)
            else:
                kv = None if m.kv_from is not None else KVSpec(m.kv_heads, m.dim_padded)
            out.append(RunSpec(kv, None))
        return out

    def kv_layer(self, i: int) -> int:
        """Index of the layer whose pages layer `i` reads."""
        m = self.layers[i].mixer
        return i if isinstance(m, LatentAttention) or m.kv_from is None else m.kv_from

    def to_dict(self) -> dict:
        layers = [{"type": TYPE_OF[type(L.mixer)], "mixer": L.mixer.to_dict(),
                   "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}} for L in self.layers]
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                "layers": layers, "norm": {"eps": self.norm_eps}}

    def save(self, model_dir) -> None:
        Path(model_dir).mkdir(parents=True, exist_ok=True)
        (Path(model_dir) / "config.json").write_text(json.dumps(self.to_dict(), indent=1))

    @staticmethod
    def from_dict(raw: dict, eos_token_ids: Sequence[int] = ()) -> "LuvutarConfig":
        layers = []
        for i, e in enumerate(raw["layers"]):
            m, mlp = e["mixer"], e.get("mlp")
            if e["type"] == "latent_attention":
                if int(m["rot"].get("dims", m["rot_dim"])) != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: the rotated part turns as a whole, so rot.dims must equal rot_dim")
                mixer: Mixer = LatentAttention(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]),
                                               int(m["kv_rank"]), float(m["scale"]), float(m["rot"]["base"]), int(m["mask"]["size"]))
            elif e["type"] == "attention":
                src = m.get("kv_from")
                mixer = BiasedAttention(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                        float(m["bias_max"]), float(m["q_temp"]["coef"]), float(m["q_temp"]["every"]),
                                        None if src is None else int(src))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(Layer(mixer, None if mlp is None else int(mlp["ff"])))
        return LuvutarConfig(int(raw["vocab"]), int(raw["width"]), int(raw["streams"]), layers, float(raw["norm"]["eps"]), list(eos_token_ids))

    @staticmethod
    def from_dir(model_dir) -> "LuvutarConfig":
        return LuvutarConfig.from_dict(json.loads((Path(model_dir) / "config.json").read_text()), eos_ids_of_dir(model_dir))


def _pattern(preset: str, vocab: int, width: int, streams: int, n_layers: int, latent: LatentAttention, own: BiasedAttention, ff: int,
             **over) -> LuvutarConfig:
    """Groups of four layers: latent, attention, attention on the keys and values of the one before, latent."""
    layers = []
    for i in range(n_layers):
        m: Mixer = latent
        if i % 4 == 1:
            m = own
        elif i % 4 == 2:
            m = BiasedAttention(own.heads, own.kv_heads, own.dim, own.vdim, own.scale, own.bias_max, own.temp_coef, own.temp_every, i - 1)
        layers.append(Layer(m, ff))
    kw = dict(name=preset)
    kw.update(over)
    return LuvutarConfig(vocab, width, streams, layers, **kw)


def tiny_config(**over) -> LuvutarConfig:
    return _pattern("luvutar-tiny", 512, 128, 2, 4, LatentAttention(4, 32, 16, 48, 64, 80, 48 ** -0.5, 10000.0, 60),
                    BiasedAttention(6, 2, 32, 32, 32 ** -0.5, 100, 0.3, 32), 160, **over)


def luvutar_4b_config(**over) -> LuvutarConfig:
    """Layer shapes of a 4B-class model (the hybrid decoder's width, attention heads and feed-forward)."""
    return _pattern("luvutar-4b", 151936, 2560, 4, 32, LatentAttention(16, 128, 64, 128, 768, 512, 192 ** -0.5, 10000.0, 4096),
                    BiasedAttention(16, 4, 256, 256, 256 ** -0.5, 128, 0.1, 1024), 13824, **over)


def luvutar_27b_config(**over) -> LuvutarConfig:
    """Layer shapes of a 27B-class model (the hybrid decoder's width, attention heads and feed-forward)."""
    return _pattern("luvutar-27b", 151936, 5120, 4, 64, LatentAttention(40, 128, 64, 128, 1536, 512, 192 ** -0.5, 10000.0, 4096),
                    BiasedAttention(24, 4, 256, 256, 256 ** -0.5, 128, 0.1, 1024), 26112, **over)


PRESETS = {"luvutar-tiny": tiny_config, "luvutar-4b": luvutar_4b_config, "luvutar-27b": luvutar_27b_config}
