"""Device-resident sequence state: paged KV pools, conv/recurrent pools, block tables.

What a model keeps per sequence is described by its configuration (``cfg.state_specs(geometry)``): one `RunSpec` per layer
execution, naming the attention pages and / or the recurrent state that execution owns.  A layer may own both (attention and
a recurrence side by side), and a layer that runs several times in one forward owns one set per pass.

Layouts (chosen for Blackwell: every (page, kv-head) tile is one contiguous 8 KB / 4 KB block that a
single bulk copy can fetch; the reference interleaves heads inside a token,
include/phaseshift/models/qwen35/state/paged_kv_pool.h:59-140):

* K/V pool per attention layer: ``[num_pages, Hkv, page_tokens, D]`` in bf16 or E4M3 bytes, FP8 pools
  carry ``[num_pages, Hkv, page_tokens]`` f32 scales (one per token x head, like the reference's
  FP8_E4M3 KV mode, state/kv_cache_types.h:11-46).
  A shared spec (values are the keys) has one pool: ``v`` is ``k``.
* GDN conv history per GDN layer: ``[slots, Hv, ring, 2*Dk+Dv]`` bf16, position p in slot p % ring.
* GDN recurrent state per GDN layer: ``[slots, Hv, Dk, Dv]`` f32 (reference: gdn_state_pool.h:16-105).
* Short-convolution history of an attention layer: ``[slots, taps - 1, channels]``, position p in row p % (taps - 1).
* Last token of every sequence, for models whose embedding looks back: ``[slots]`` int32.
* Block table: ``[slots, max_blocks]`` int32, -1 = unmapped.

Sizing rules follow docs/developer/runtime.md:109-119:
``max_blocks = ceil((max_seq_len+1)/page)+1``, ``pages = ceil(capacity_tokens/page)+1``.
Page 0 is never handed out, so a zeroed block table entry cannot alias live data.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

KV_DTYPES = ("bf16", "fp8_e4m3", "nvfp4")
# names accepted on the command line for the reference's block-coded caches (src/apps/compute/main.hip:47-81): its 4-bit
# format is served by the NVFP4 pools, its 8-bit format by the FP8 pools (same E4M3 codes, one scale per row instead of
# one per 32 values)
KV_DTYPE_ALIASES = {"psq4": "nvfp4", "psq8": "fp8_e4m3"}
KV_FMT = {"bf16": 0, "fp8_e4m3": 1, "nvfp4": 2}


def kv_row_bytes(kv_dtype: str, head_dim: int) -> int:
    """Bytes of one cached row (a token of one KV head) in the pools of `kv_dtype`, without the fp32 row scale."""
    if kv_dtype == "nvfp4":
        return ((head_dim // 2 + head_dim // 16) + 15) & ~15          # codes, block scales, padded to 16 bytes
    return head_dim * (1 if kv_dtype == "fp8_e4m3" else 2)


@dataclass(frozen=True)
class KVSpec:
    """Attention pages of one layer execution: KV heads, head size, and whether the keys double as the values."""
    heads: int
    dim: int
    shared: bool = False


@dataclass(frozen=True)
class RecurrentSpec:
    """Recurrent state of one layer execution: ``[slots, heads, dk, dv]`` f32, and the channels of its short-conv history
    per head (0 = none)."""
    heads: int
    dk: int
    dv: int
    conv_channels: int = 0


@dataclass(frozen=True)
class ConvSpec:
    """Rows before the current one that a short convolution over a layer's projection looks back to."""
    channels: int
    history: int


@dataclass(frozen=True)
class RunSpec:
    kv: Optional[KVSpec]
    rec: Optional[RecurrentSpec]
    conv: Optional[ConvSpec] = None


@dataclass
class StateConfig:
    max_slots: int = 1
    max_seq_len: int = 512
    page_tokens: int = 16
    kv_capacity_tokens: int = 0          # 0 = one full context per slot
    kv_dtype: str = "bf16"
    conv_ring: int = 4                   # >= 4; 3 + max speculative rows when rollback is needed
    spec_rows: int = 0                   # > 0 allocates the alternate recurrent state + update log

    def max_blocks(self) -> int:
        return -(-(self.max_seq_len + 1) // self.page_tokens) + 1

    def num_pages(self) -> int:
        cap = self.kv_capacity_tokens or self.max_slots * (self.max_seq_len + 1)
        return -(-cap // self.page_tokens) + 1 + self.max_slots


class KVLayer:
    __slots__ = ("k", "v", "k_scale", "v_scale")

    def __init__(self, k, v, k_scale, v_scale):
        self.k, self.v, self.k_scale, self.v_scale = k, v, k_scale, v_scale


class GdnLayerState:
    """Recurrent state of one layer execution; ``conv`` is None for recurrences without a short convolution."""
    __slots__ = ("conv", "rec", "rec_alt")

    def __init__(self, conv, rec, rec_alt):
        self.conv, self.rec, self.rec_alt = conv, rec, rec_alt


class ModelState:
    """All per-sequence device state of one rank."""

    def __init__(self, cfg, sc: StateConfig, device, act_dtype=torch.bfloat16, geo=None, arenas=None):
        """``arenas`` (a core.arena.ArenaSet, CUDA only): the KV pages and the recurrent / conv state are carved from
        the named arenas "kv" and "state" (stable virtual addresses, physical memory committed for exactly what the
        configuration needs, all under the set's byte budget) instead of the framework allocator."""
        if sc.kv_dtype not in KV_DTYPES:
            raise ValueError(f"kv dtype {sc.kv_dtype!r} not in {KV_DTYPES}")
        if sc.conv_ring < 4:
            raise ValueError("conv_ring must be >= 4")
        self.cfg, self.sc, self.device = cfg, sc, device
        geo = geo or cfg.geometry(0, 1)
        self.geo = geo
        self.specs: List[RunSpec] = cfg.state_specs(geo)
        self.num_pages = sc.num_pages()
        self.max_blocks = sc.max_blocks()
        pt = sc.page_tokens
        self.kv_fp8 = sc.kv_dtype == "fp8_e4m3"
        self.kv_fmt = KV_FMT[sc.kv_dtype]            # 0 bf16, 1 FP8-E4M3 + row scale, 2 NVFP4 rows + row scale
        kv_specs = [s.kv for s in self.specs if s.kv is not None]
        rec_specs = [s.rec for s in self.specs if s.rec is not None]
        # heads of the (uniform) recurrent layers, for callers that log or replay their updates
        self.hv = rec_specs[0].heads if rec_specs else 0
        if act_dtype == torch.float32:
            kvt = torch.float32          # 32-bit engines keep full precision
            self.kv_fp8 = False
            self.kv_fmt = 0
        elif self.kv_fmt == 2:
            if any(s.dim % 32 or s.dim > 256 for s in kv_specs):
                raise ValueError("NVFP4 key/value pages need a head size that is a multiple of 32, at most 256")
            kvt = torch.uint8
        else:
            kvt = torch.uint8 if self.kv_fp8 else torch.bfloat16
        if self.kv_fmt != 0 and any(s.shared for s in kv_specs):
            raise ValueError("pages whose keys double as the values are stored in bf16 (or 32-bit) only")
        scaled = self.kv_fmt != 0                    # pools with an fp32 scale per (page, head, token)
        self.kv: List[Optional[KVLayer]] = []
        self.gdn: List[Optional[GdnLayerState]] = []
        self.conv: List[Optional[torch.Tensor]] = []
        self.arenas = arenas
        esz = lambda dt: torch.empty(0, dtype=dt).element_size()
        row_elems = lambda s: kv_row_bytes("nvfp4", s.dim) if self.kv_fmt == 2 else s.dim       # last extent of the pools
        kv_need = sum((1 if s.shared else 2) * self.num_pages * s.heads * pt * (row_elems(s) * esz(kvt) + (4 if scaled else 0)) + 1024
                      for s in kv_specs)
        conv_specs = [s.conv for s in self.specs if s.conv is not None and s.conv.history > 0]
        st_need = sum(sc.max_slots * c.history * c.channels * esz(act_dtype) + 1024 for c in conv_specs)
        st_need += sum(sc.max_slots * s.heads * (sc.conv_ring * s.conv_channels * esz(act_dtype)
                                                + s.dk * s.dv * 4 * (2 if sc.spec_rows > 0 else 1)) + 1024 for s in rec_specs)
        kv_arena = arenas.get("kv", kv_need + (2 << 20)) if arenas is not None and kv_specs else None
        st_arena = arenas.get("state", st_need + (2 << 20)) if arenas is not None and (rec_specs or conv_specs) else None

        def pool(arena, shape, dtype, fill=0):
            if arena is None:
                return torch.full(shape, fill, dtype=dtype, device=device) if fill else torch.zeros(shape, dtype=dtype, device=device)
            t = arena.alloc(shape, dtype)
            return t.fill_(fill) if fill else t.zero_()
        for spec in self.specs:
            kv = rec = None
            if spec.kv is not None:
                shape = (self.num_pages, spec.kv.heads, pt, row_elems(spec.kv))
                k = pool(kv_arena, shape, kvt)
                v = k if spec.kv.shared else pool(kv_arena, shape, kvt)
                ks = vs = None
                if scaled:
                    ks = pool(kv_arena, shape[:3], torch.float32, 1)
                    vs = pool(kv_arena, shape[:3], torch.float32, 1)
                kv = KVLayer(k, v, ks, vs)
            if spec.rec is not None:
                r = spec.rec
                conv = pool(st_arena, (sc.max_slots, r.heads, sc.conv_ring, r.conv_channels), act_dtype) if r.conv_channels else None
                main = pool(st_arena, (sc.max_slots, r.heads, r.dk, r.dv), torch.float32)
                alt = pool(st_arena, (sc.max_slots, r.heads, r.dk, r.dv), torch.float32) if sc.spec_rows > 0 else None
                rec = GdnLayerState(conv, main, alt)
            self.kv.append(kv)
            self.gdn.append(rec)
            c = spec.conv
            self.conv.append(pool(st_arena, (sc.max_slots, c.history, c.channels), act_dtype) if c is not None and c.history > 0 else None)
        self.last_token = (torch.zeros(sc.max_slots, dtype=torch.int32, device=device)
                           if getattr(cfg, "keeps_last_token", False) else None)
        self.block_table = torch.full((sc.max_slots, self.max_blocks), -1, dtype=torch.int32, device=device)
        self.status = torch.zeros(1, dtype=torch.int32, device=device)

    def kv_bytes(self) -> int:
        n = 0
        for l in self.kv:
            if l is not None:
                n += (1 if l.v is l.k else 2) * l.k.numel() * l.k.element_size()
                if l.k_scale is not None:
                    n += 2 * l.k_scale.numel() * 4
        return n

    def slot_tensors(self) -> List[torch.Tensor]:
        """Everything a sequence keeps outside its pages: tensors whose first extent is the slot."""
        out = []
        for g in self.gdn:
            if g is not None:
                out.append(g.rec)
                if g.conv is not None:
                    out.append(g.conv)
        out += [c for c in self.conv if c is not None]
        if self.last_token is not None:
            out.append(self.last_token)
        return out

    def reset_slot(self, slot: int) -> None:
        """Fresh sequence: zero recurrent state (convolution histories and the last token need no clearing: what lies before
        position 0 is defined by the kernels)."""
        for g in self.gdn:
            if g is not None:
                g.rec[slot].zero_()

    def copy_slot(self, dst: int, src: int) -> None:
        for t in self.slot_tensors():
            t[dst].copy_(t[src])
