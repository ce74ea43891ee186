"""What every model family's runner shares."""
from __future__ import annotations

import json
from pathlib import Path
from typing import List

import torch


def pad(n: int, to: int) -> int:
    return -(-n // to) * to


class SingleRank:
    """Tensor-parallel geometry of a model that runs on one rank."""
    tp_rank, tp_size = 0, 1


def eos_ids_of_dir(model_dir) -> List[int]:
    """End-of-sequence ids of a model directory's generation_config.json (none without the file)."""
    gen = Path(model_dir) / "generation_config.json"
    eos = json.loads(gen.read_text()).get("eos_token_id", []) if gen.exists() else []
    return [eos] if isinstance(eos, int) else list(eos or [])


# ---------------------------------------------------------------- engine layouts: zero rows and columns up to what a kernel works on
def pad_heads(t: torch.Tensor, heads: int, dim: int, to: int) -> torch.Tensor:
    """[heads * dim, ...] -> [heads * to, ...], zero rows at the end of every head."""
    if dim == to:
        return t
    out = t.new_zeros((heads, to) + tuple(t.shape[1:]))
    out[:, :dim] = t.reshape((heads, dim) + tuple(t.shape[1:]))
    return out.reshape((heads * to,) + tuple(t.shape[1:]))


def pad_rows(t: torch.Tensor, to: int) -> torch.Tensor:
    return t if t.shape[0] == to else torch.cat([t, t.new_zeros((to - t.shape[0],) + tuple(t.shape[1:]))], 0)


def pad_cols(t: torch.Tensor, to: int) -> torch.Tensor:
    return t if t.shape[1] == to else torch.cat([t, t.new_zeros(t.shape[0], to - t.shape[1])], 1)


def alternate(a: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Rows a0, b0, a1, b1, ..."""
    return torch.stack([a, b], 1).flatten(0, 1)


def plain_linear(w: torch.Tensor, n: int, k: int, fmt: str):
    """Unquantised projection of `n` x `k` (zero-padded from `w`): bf16 on CUDA keeps both kernel forms, streaming tiles for
    single rows and row-major for the tensor-core GEMMs."""
    from ..quant.formats import QuantizedTensor
    from .qwen35.weights import LinearW
    w = pad_cols(pad_rows(w, n), k).contiguous()
    lw = LinearW(QuantizedTensor(fmt, (n, k), k, w))
    if w.is_cuda and fmt == "bf16":
        lw.make_tiled(True)
    return lw



class StepOutput:
    __slots__ = ("tokens", "logits", "hidden", "taps", "taps_cat", "read_back")

    def __init__(self, tokens, logits, hidden, taps, taps_cat=None):
        self.tokens, self.logits, self.hidden, self.taps = tokens, logits, hidden, taps
        self.taps_cat = taps_cat        # the tapped hidden states side by side, [rows, taps * H] (taps are views of it)
        self.read_back = None
