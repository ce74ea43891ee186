"""Shape and constant descriptions of mechanisms that several model families share."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


@dataclass
class AttnSpec:
    """Softmax attention over paged keys and values.

    ``chunk`` > 0: position i sees positions j <= i of its own block of `chunk` positions (blocks counted from position 0).
    ``sink`` (f32 [heads]): one more term exp(sink[h]) in head h's denominator.
    ``gate`` (with its row layout): the output is multiplied by sigmoid(gate)."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    chunk: int = 0
    sink: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    gate_head_stride: int = 0
    gate_offset: int = 0


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
