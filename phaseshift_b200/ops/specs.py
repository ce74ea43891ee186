"""Shape and constant descriptions of mechanisms that several model families share."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch


@dataclass
class AttnSpec:
    """Softmax attention over paged keys and values.

    ``chunk`` > 0: position i sees positions j <= i of its own block of `chunk` positions (blocks counted from position 0).
    ``window`` > 0: position i sees positions j with i - j < window.
    ``sink`` (f32 [heads]): one more term exp(sink[h]) in head h's denominator.
    ``temp_coef``, ``temp_every``: scores of a query at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1).
    ``bias`` (f32 [heads, distances]): added to the score of a key at distance i - j; the last entry holds for every larger one.
    ``gate`` (rows of a projection, with their layout): the output is multiplied by sigmoid(gate), element by element, or with
    ``gate_per_head`` by one number per head.  It can also be given to `attention` with every call."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int = 0
    sink: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    gate_head_stride: int = 0
    gate_offset: int = 0
    gate_per_head: bool = False
    window: int = 0
    temp_coef: float = 0.0
    temp_every: float = 1.0
    bias: Optional[torch.Tensor] = None

    def first_visible(self, pos: int) -> int:
        lo = pos // self.chunk * self.chunk if self.chunk > 0 else 0
        return max(lo, pos - self.window + 1) if self.window > 0 else lo


def distance_bias_table(table: torch.Tensor, far: float) -> torch.Tensor:
    """Bias per distance (f32 [heads, distances], the last one for everything beyond) from a learned table [buckets, heads]:
    a bucket for every distance below half their number, logarithmically wider ones up to the distance `far`."""
    rows = table.shape[0]
    half = rows // 2
    buckets, n = [], 0
    while not buckets or buckets[-1] < rows - 1:
        if n < half:
            buckets.append(n)
        elif n >= far or far <= half or half == 0:
            buckets.append(rows - 1)
        else:
            buckets.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))
        n += 1
    return table.float()[torch.tensor(buckets, device=table.device)].T.contiguous()


@dataclass
class LatentSpec:
    """Attention whose keys and values are products of one cached latent per token, plus one rotated key part shared by all
    heads.  A cached row is [latent: kv_rank | rotated part: rot]; projection rows hold [query latent | latent | rotated part |
    output gate]; query rows hold [dim | rot] per head.  Sizes are the engine's (padded with zeros), ``*_true`` the model's.

    Two ways to the same scores: with few rows the queries are taken into the latent space (``uk_t``) and the heads share the
    cached rows as keys and values; with many rows keys and values are expanded per head (``ukv``).  ``uv`` takes the latent
    outputs back to the heads."""
    heads: int
    dim: int
    rot: int
    rot_true: int
    vdim: int
    q_rank: int
    q_rank_true: int
    kv_rank: int
    kv_rank_true: int
    scale: float
    window: int
    sink: torch.Tensor          # f32 [heads]
    inv_freq: torch.Tensor      # f64 [rot_true / 2], radians per position of every pair of neighbouring elements
    eps: float
    q_norm: torch.Tensor        # f32 [q_rank]
    kv_norm: torch.Tensor       # f32 [kv_rank]
    uk_t: torch.Tensor          # [heads * kv_rank, dim]
    ukv: torch.Tensor           # [heads * dim | heads * vdim, kv_rank]

    @property
    def uv(self) -> torch.Tensor:
        return self.ukv[self.heads * self.dim:]

    @property
    def row(self) -> int:
        """Elements of a cached row."""
        return self.kv_rank + self.rot

    @property
    def c_off(self) -> int:
        return self.q_rank

    @property
    def gate_off(self) -> int:
        return self.q_rank + self.row

    def shared_keys(self) -> AttnSpec:
        """The attention in the latent space: one key / value head of `row` elements."""
        return AttnSpec(self.heads, 1, self.row, self.scale, sink=self.sink, window=self.window)


@dataclass
class GlaSpec:
    """Gated linear attention over one projection row: column offsets of q, k, v, the output gate and the low-rank decay input,
    head geometry (engine sizes, and the true value size the head norm averages over) and the decay's constants."""
    heads: int
    dk: int
    dv: int
    dv_true: int
    q_off: int
    k_off: int
    v_off: int
    g_off: int
    a_off: int
    rank: int                   # columns of the decay input
    q_scale: float
    inv_tau: float
    eps: float
    a2: torch.Tensor            # [heads * dk, rank]
    a2_bias: torch.Tensor       # f32 [heads * dk]
    norm_w: torch.Tensor        # f32 [dv]


@dataclass
class Pending:
    """What the next residual update still has to add: the normed sum of two branches (each [rows, width] with its norm
    weight) or a plain projection output, times `coef`."""
    coef: float
    branch_a: Optional[torch.Tensor] = None
    weight_a: Optional[torch.Tensor] = None
    branch_b: Optional[torch.Tensor] = None
    weight_b: Optional[torch.Tensor] = None
    plain: Optional[torch.Tensor] = None


@dataclass
class StreamWrite:
    """Pending write of a sublayer's output into parallel residual streams: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    mix: torch.Tensor           # f32 [streams, streams], [from, to]
    out: torch.Tensor           # f32 [streams]
    y: torch.Tensor             # [rows, width (+ padding columns)] f32
