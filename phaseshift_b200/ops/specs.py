"""Shape and constant descriptions of mechanisms that several model families share."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch


@dataclass
class AttnSpec:
    """Softmax attention over paged keys and values.

    ``chunk`` > 0: position i sees positions j <= i of its own block of `chunk` positions (blocks counted from position 0).
    ``window`` > 0: position i sees positions j with i - j < window, and with ``keep_first`` > 0 the first `keep_first` positions of
    its sequence as well.
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
    keep_first: int = 0

    def first_visible(self, pos: int) -> int:
        """First position of the run that ends at `pos` itself (kept first positions lie before it)."""
        lo = pos // self.chunk * self.chunk if self.chunk > 0 else 0
        return max(lo, pos - self.window + 1) if self.window > 0 else lo

    def visible(self, pos: int) -> torch.Tensor:
        lo = self.first_visible(pos)
        return torch.cat([torch.arange(min(self.keep_first, lo)), torch.arange(lo, pos + 1)])


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


def rotation_frequencies(base: float, dims: int) -> torch.Tensor:
    """f64 [dims / 2], radians per position of every rotated pair."""
    return base ** (-torch.arange(dims // 2, dtype=torch.float64) * 2.0 / dims)


def stepped_frequencies(freq: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Llama 3.1's scaling by wavelength: pairs that turn at least `high` times within the original length keep their frequency,
    those that turn at most `low` times are slowed by the factor, the ones between are blended."""
    turns = original * freq / (2.0 * math.pi)
    if high == low:
        return torch.where(turns > high, freq, freq / factor)
    keep = ((turns - low) / (high - low)).clamp(0.0, 1.0)
    return (1.0 - keep) * freq / factor + keep * freq


def ramped_frequencies(freq: torch.Tensor, base: float, factor: float, original: float, fast: float, slow: float) -> Tuple[torch.Tensor, float]:
    """YaRN's scaling by pair: a ramp from the pair that turns `fast` times within the original length (kept) to the one that
    turns `slow` times (slowed by the factor).  Returns the frequencies and the factor on sine and cosine."""
    dims = 2 * freq.numel()

    def pair_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    ramp = ((torch.arange(freq.numel(), dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


@dataclass
class HeadsSpec:
    """From a projection row [q heads | k heads | v heads] to the queries, keys and values of an attention, in this order, each
    part optional:

    ``conv`` ([taps, channels], the projection's type; the last tap is the row's own): a causal convolution over time on every
    channel; the sequence's last taps - 1 rows are state (runtime/state.py: ConvSpec).
    ``q_norm``, ``k_norm`` (f32 [heads * dim], [kv_heads * dim]): norm over all heads at once.
    ``freq`` (f64 [pairs]): the first 2 * pairs dimensions of every query and key head turn, neighbours together or (``halves``)
    dimension i with i + pairs; ``turn_size`` multiplies sine and cosine.
    ``unit``: each query and key head is divided by its root mean square.
    ``mix``: values become (1 - mix) v + mix (values that an earlier layer of the step has saved); ``save``: this layer's are
    the ones that later layers mix in."""
    heads: int
    kv_heads: int
    dim: int                    # the engine's (padded with zeros), as in AttnSpec
    dim_true: int
    vdim_true: int
    eps: float
    freq: torch.Tensor
    halves: bool = False
    turn_size: float = 1.0
    unit: bool = False
    conv: Optional[torch.Tensor] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    mix: Optional[float] = None
    save: bool = False

    @property
    def taps(self) -> int:
        return 1 if self.conv is None else self.conv.shape[0]

    @property
    def channels(self) -> int:
        return (self.heads + 2 * self.kv_heads) * self.dim


@dataclass
class MoeSpec:
    """Mixture of feed-forward experts.  A token's scores are the softmax (or the sigmoids) of its router logits over experts and,
    behind them, `identity` experts that return their input; it goes to the `top` largest of score + correction among the `keep`
    best of `groups` equal groups of neighbours (a group counts as the sum of its `group_top` best members), weighted by their
    scores, divided by the sum of these if `renormalize`.  An expert's activation is silu(gate) * up, or with a `limit` that of
    `clamped_gate`."""
    experts: int
    identity: int
    top: int
    groups: int
    keep: int
    ff: int                     # columns of an expert's activation (engine size)
    n_out: int                  # output columns (engine size)
    correction: Optional[torch.Tensor]       # f32 [experts + identity]; None: zero
    gate_up: torch.Tensor       # [experts * 2 ff, K], rows alternate gate, up
    down: torch.Tensor          # [experts * n_out, ff]
    sigmoid: bool = False
    group_top: int = 1          # 1 or 2
    renormalize: bool = True
    limit: Optional[float] = None


def clamped_gate(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u = up clamped to [-limit, limit]."""
    g = gate.clamp(max=limit)
    return g * torch.sigmoid(1.702 * g) * (up.clamp(-limit, limit) + 1.0)


@dataclass
class Routed:
    """Where the rows of a step go: expert contributions in rows sorted by expert."""
    index: torch.Tensor         # int32 [rows, top]: sorted row of the contribution, -1: none
    weight: torch.Tensor        # f32 [rows, top]
    identity: torch.Tensor      # f32 [rows]: weight of the input itself
    inputs: torch.Tensor        # [sorted rows, K]
    tiles: Optional[torch.Tensor] = None     # kernel-side list of (expert, first row, rows)
    tile_rows: int = 0
    max_tiles: int = 0


@dataclass
class ExpertSum:
    """Output of a mixture layer before its sum: sum_k weight[k] y[index[k]] + identity * h (+ shared)."""
    routed: Routed
    y: torch.Tensor             # f32 [sorted rows, width (+ padding columns)]
    h: torch.Tensor             # the layer's normed input [rows, width (+ padding columns)]
    shared: Optional[torch.Tensor] = None    # f32 [rows, width (+ padding columns)]


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
    head geometry (engine sizes, and the true value size the head norm averages over) and the decay's constants.

    With `lower` the decay is a gate of its own that also decides what is written: f = lower + (1 - lower) sigmoid(z), z a column per
    head and channel of the projection (at `a_off`) + `a2_bias`; the key is 1 - f and the query silu(q).  There is no `a2` then.
    `g_off` -1: no output gate."""
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
    a2: Optional[torch.Tensor]  # [heads * dk, rank]
    a2_bias: torch.Tensor       # f32 [heads * dk]
    norm_w: torch.Tensor        # f32 [dv]
    lower: Optional[torch.Tensor] = None     # f32 [heads * dk]


@dataclass
class DeltaSpec:
    """Delta rule with a decay per head and key channel, between a projection row and the output projection.  Projection columns:
    q and k heads (`kv_heads`; consecutive value heads share one), v heads, the input of the step size (a column per head) and the
    low-rank inputs of decay and output gate.

    q, k and v pass a causal convolution over time (`conv`, the last tap is the row's own; the sequence's last taps - 1 rows are
    state, a copy per value head: [slots, taps - 1, heads, 2 dk + dv], position p in row p % (taps - 1)) and silu; q and k are divided
    by their length, q also by sqrt(dk_true).  g = exp(-rate softplus(a2 a + dt_bias)), beta = sigmoid(b), and per head
    S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  The output is rms(o) norm_w sigmoid(g2 g)."""
    heads: int
    kv_heads: int
    dk: int                     # the engine's sizes (padded with zeros), and the model's
    dv: int
    dk_true: int
    dv_true: int
    q_off: int                  # the k and v heads lie behind the q heads
    b_off: int
    a_off: int
    g_off: int
    eps: float
    conv: torch.Tensor          # [taps, q | k | v channels], the projection's type
    a2: torch.Tensor            # [heads * dk, a rank]
    dt_bias: torch.Tensor       # f32 [heads * dk]
    rate: torch.Tensor          # f32 [heads]
    g2: torch.Tensor            # [heads * dv, g rank]
    norm_w: torch.Tensor        # f32 [dv]

    @property
    def taps(self) -> int:
        return self.conv.shape[0]

    @property
    def k_off(self) -> int:
        return self.q_off + self.kv_heads * self.dk

    @property
    def v_off(self) -> int:
        return self.k_off + self.kv_heads * self.dk


@dataclass
class GatedNorm:
    """A sublayer's result on its way into the residual: y = scale_a a + scale_b b (projection outputs, f32) or the weighted sum of a
    mixture's experts; y * sigmoid(gate + gate_bias) is normed in groups, times `norm_w`, and added."""
    gate: torch.Tensor          # [rows, width (+ padding columns)], bf16 or f32
    gate_bias: torch.Tensor     # f32 [width]
    norm_w: torch.Tensor        # f32 [width]
    a: Optional[torch.Tensor] = None
    scale_a: float = 1.0
    b: Optional[torch.Tensor] = None
    scale_b: float = 1.0
    routed: Optional[Routed] = None
    experts: Optional[torch.Tensor] = None   # f32 [sorted rows, width (+ padding columns)]


@dataclass
class Pending:
    """What the next residual update still has to add: the normed sum of two branches (each [rows, width] with its norm
    weight), a plain projection output or a mixture's sum, times `coef`; and a `bias` vector (f32 [width])."""
    coef: float
    branch_a: Optional[torch.Tensor] = None
    weight_a: Optional[torch.Tensor] = None
    branch_b: Optional[torch.Tensor] = None
    weight_b: Optional[torch.Tensor] = None
    plain: Optional[torch.Tensor] = None
    experts: Optional[ExpertSum] = None
    bias: Optional[torch.Tensor] = None


@dataclass
class StreamWrite:
    """Pending write of a sublayer's output into parallel residual streams: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    mix: torch.Tensor           # f32 [streams, streams], [from, to]
    out: torch.Tensor           # f32 [streams]
    y: torch.Tensor             # [rows, width (+ padding columns)] f32
