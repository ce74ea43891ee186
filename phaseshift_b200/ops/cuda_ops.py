"""CUDA op set: thin Python wrappers over the sm_100a kernels in ``libps_kernels.so``.

Each method validates shapes/dtypes (the role of the reference's ``resolve_*_args`` functions, e.g.
src/phaseshift/models/qwen35/runtime/paged_attention_dispatch.hip:274-436), picks the kernel variant
(small-M fused GEMV vs tensor-core GEMM -- the job of the reference's linear selector,
src/.../runtime/linear_selector.cpp:202-308) and launches on the current stream.  Output buffers come
from a per-instance workspace keyed by (name, rows) so pointers are stable across steps, which is
what lets a whole step be captured in a CUDA graph.
"""
from __future__ import annotations

import ctypes
import os
from typing import Dict, Optional, Tuple

import numpy as np
import torch

from .trace import OpTrace
from ..models.qwen35.weights import AttnW, GdnW, LinearW
from ..runtime.batch import ROW_BUCKETS, StepBatch
from ..runtime.state import GdnLayerState, KVLayer, ModelState
from . import _lib
from .specs import AttnSpec, DeltaSpec, GatedNorm, GlaSpec, HeadsSpec, LatentSpec, MoeSpec, Pending, Routed, StreamWrite
from ._lib import c_float, c_int, c_ll, ptr

WFMT = {"bf16": 0, "nvfp4": 1, "mxfp8": 2}
PRO_NONE, PRO_RMSNORM, PRO_SIGMOID_GATE = 0, 1, 2
EPI_STORE, EPI_RESIDUAL, EPI_SWIGLU, EPI_REGLU, EPI_GELU, EPI_GEGLU = 0, 1, 2, 3, 4, 5
GATED = (EPI_SWIGLU, EPI_REGLU, EPI_GEGLU)
SMALL_M_MAX = 8


class AttnOptions(ctypes.Structure):
    """csrc/include/attn_options.cuh: AttnOptions."""
    _fields_ = [("chunk", ctypes.c_int), ("window", ctypes.c_int), ("temp_coef", ctypes.c_float), ("temp_every", ctypes.c_float),
                ("bias", ctypes.c_void_p), ("bias_len", ctypes.c_int), ("gate_per_head", ctypes.c_int), ("sink", ctypes.c_void_p), ("keep_first", ctypes.c_int)]

    @staticmethod
    def of(s: AttnSpec) -> "AttnOptions":
        for t in (s.bias, s.sink):
            if t is not None and (t.dtype != torch.float32 or not t.is_contiguous() or t.shape[0] != s.heads):
                raise ValueError("attention biases and sinks are contiguous f32 tensors, one row per head")
        return AttnOptions(s.chunk, s.window, s.temp_coef, s.temp_every, None if s.bias is None else s.bias.data_ptr(),
                           0 if s.bias is None else s.bias.shape[1], int(s.gate_per_head), None if s.sink is None else s.sink.data_ptr(), s.keep_first)


class CudaOps(OpTrace):
    act_dtype = torch.bfloat16
    name = "cuda"
    GDN_CHUNKED_MIN_ROWS = 16      # steps with more rows than this use the chunked GDN kernels
    ATTN_PREFILL_MIN_ROWS = 16     # ... and the tiled tensor-core attention kernel

    def __init__(self, cfg, device, attn_split_tokens: int = 64, attn_max_splits: int = 0,
                 max_seq_len: int = 4096, act_dtype: torch.dtype = torch.bfloat16):
        """``act_dtype``: bfloat16, or float32 for model families whose ops exist in 32-bit (see `linear`)."""
        if device.type != "cuda":
            raise ValueError("CudaOps needs a CUDA device")
        _lib.lib()      # fail loudly when the native library is missing
        self.cfg, self.device, self.act_dtype = cfg, device, act_dtype
        self.ws: Dict[Tuple[str, int], torch.Tensor] = {}
        self.checked = _lib.checked_build()          # PS_CHECKED=1: descriptor assertions in the kernels + workspace canaries
        self._guarded: Dict[Tuple[str, int], torch.Tensor] = {}
        half = getattr(cfg, "rotary_dim", 0) // 2                    # 0: the model rotates nothing
        inv = getattr(cfg, "rope_theta", 1.0) ** (-np.arange(half, dtype=np.float64) * 2.0 / max(1, 2 * half))
        self.inv_freq = torch.from_numpy(inv).to(device)
        # the split length is fixed per engine for steps of up to 8 rows and for Exact mode, so attention results there do not
        # depend on the batch; larger Fast-mode batches lengthen it (see paged_attention).  PS_ATTN_SPLIT_TOKENS overrides the
        # base length (a multiple of 32).
        self.split_tokens = int(os.environ.get("PS_ATTN_SPLIT_TOKENS", attn_split_tokens))
        if self.split_tokens < 32 or self.split_tokens % 32:
            raise ValueError("the attention split length must be a positive multiple of 32")
        while -(-(max_seq_len + 1) // self.split_tokens) > 512:
            self.split_tokens *= 2
        self.max_splits = attn_max_splits or -(-(max_seq_len + 1) // self.split_tokens)
        self.launches = 0
        self.use_tc_gemm = True
        self.exact_rows = False     # verify steps: keep every projection on the batch-invariant small-M kernel
        self.attn_decode_tc = os.environ.get("PS_ATTN_DECODE", "tc") != "legacy"
        self.wscratch = None
        self.status = torch.zeros(1, dtype=torch.int32, device=device)   # kernels' own bounded-wait status word
        # block-scaled tensor-core projections: stream-K partials + flags (flags must read 0 between launches)
        self.bs_ws: Optional[torch.Tensor] = None
        self.bs_flags: Optional[torch.Tensor] = None
        self.bs_grid_override = 0
        self.force_tc = os.environ.get("PS_FORCE_TC", "0") == "1"   # single-row steps on the tensor-core kernel too
        self.bs_prefetch = os.environ.get("PS_BS_PREFETCH", "1") != "0"
        self._bs_plan_cache: Dict[tuple, bool] = {}
        self.tickets = torch.zeros(ROW_BUCKETS[-1], dtype=torch.int32, device=device)      # one per sequence, zero between launches
        self.sel_counts: Dict[str, int] = {"tc_resident": 0, "tc_streamed": 0, "stream": 0, "gemm": 0}   # projection calls per kernel
        self.fallbacks: Dict[str, int] = {}

    # ------------------------------------------------------------------ workspace
    CANARY = 0xA5
    CANARY_BYTES = 256

    def buf(self, name: str, rows: int, cols: int, dtype=torch.bfloat16) -> torch.Tensor:
        key = (name, rows)
        t = self.ws.get(key)
        if t is None or t.shape[1] != cols or t.dtype != dtype:
            if self.checked:
                # checked build: every workspace sits between two guard regions that `check_canaries` inspects
                n = rows * cols * torch.empty(0, dtype=dtype).element_size()
                raw = torch.full((n + 2 * self.CANARY_BYTES,), self.CANARY, dtype=torch.uint8, device=self.device)
                t = raw[self.CANARY_BYTES:self.CANARY_BYTES + n].view(dtype).view(rows, cols)
                self._guarded[key] = raw
            else:
                t = torch.empty(rows, cols, dtype=dtype, device=self.device)
            self.ws[key] = t
        return t

    def check_canaries(self):
        """Checked build: names of the workspaces whose guard bytes were overwritten (an out-of-bounds write by some
        kernel).  Synchronises; the engine calls it after every step when the checked library is loaded."""
        bad = []
        g = self.CANARY_BYTES
        for key, raw in self._guarded.items():
            if bool((raw[:g] != self.CANARY).any()) or bool((raw[-g:] != self.CANARY).any()):
                bad.append(key[0])
        return bad

    # ------------------------------------------------------------------ ops
    SSQ_LD = 64          # partial sums of squares per row: one per 128-feature tile of the producing projection

    def ssq_buf(self, name: str, rows: int) -> torch.Tensor:
        return self.buf("ssq_" + name, rows, self.SSQ_LD, torch.float32)

    def embed(self, b: StepBatch, rows: int, table: LinearW, status, ssq_out: Optional[torch.Tensor] = None) -> torch.Tensor:
        H = table.K
        out = self.buf("x_embed", rows, H)
        ld = ssq_out.stride(0) if ssq_out is not None else 0
        if table.fmt == "bf16":
            _lib.call("ps_embedding", ptr(b.ids), ptr(table.q.codes), c_int(rows), c_int(table.N), c_int(H),
                      ptr(out), c_int(H), ptr(status), ptr(ssq_out), c_int(ld))
        elif table.fmt == "mxfp8":
            _lib.call("ps_embedding_mxfp8", ptr(b.ids), ptr(table.q.codes), ptr(table.q.scales), c_int(rows),
                      c_int(table.N), c_int(H), ptr(out), c_int(H), ptr(status), ptr(ssq_out), c_int(ld))
        else:
            raise ValueError("embedding table must be bf16 or mxfp8")
        self.launches += 1
        return out

    def linear(self, x: torch.Tensor, W: LinearW, *, name: str, norm_w: Optional[torch.Tensor] = None,
               eps: float = 0.0, residual: Optional[torch.Tensor] = None, swiglu: bool = False, reglu: bool = False, gelu: bool = False,
               geglu: bool = False, out_f32: bool = False, out: Optional[torch.Tensor] = None,
               xn_out: Optional[torch.Tensor] = None, tp_combine=None, ssq_in=None,
               ssq_out: Optional[torch.Tensor] = None, prefetch: Optional[LinearW] = None, tp_scatter=None) -> torch.Tensor:
        """``tp_combine`` (a parallel.tp.TpCombineStruct): the projection is row-parallel and the kernel sums
        the ranks' partial results over NVLink before the residual epilogue.
        ``ssq_in`` = (tensor [rows, SSQ_LD] fp32, n): n partial sums of squares per row of ``x`` left by the kernel
        that produced it, consumed by the fused RMSNorm; ``ssq_out``: receives the partial sums of the rows this
        projection stores (block-scaled tensor-core path, <= 32 rows; ignored elsewhere).
        ``prefetch``: the projection that will run next on the same rows; the tensor-core kernel warms L2 with the first
        bytes of its weights while it drains.
        ``tp_scatter`` (a parallel.tp.TpScatterStruct; tensor-core path with streamed activations only): instead of
        storing to ``out`` the kernel pushes each bf16 output row to the receive buffer of the rank that owns it.
        ``swiglu`` / ``reglu`` / ``geglu``: the weight's rows interleave (gate, up) and the output is silu / relu / tanh-gelu
        (gate) * up.
        ``gelu``: the tanh form of gelu is applied to every output.
        32-bit weights run in fp32 on the CUDA cores (activation epilogues only)."""
        M, K = x.shape
        if W.fmt == "f32":
            return self._linear_f32(x, W, name, self._epilogue(swiglu, reglu, gelu, geglu, residual), out, plain=norm_w is None and residual is None)
        assert K == W.K and x.dtype == torch.bfloat16 and x.stride(1) == 1, (x.shape, W.K, x.dtype)
        epi = self._epilogue(swiglu, reglu, gelu, geglu, residual)
        n_out = W.N // 2 if epi in GATED else W.N
        if out is None:
            out = self.buf(name, M, n_out, torch.float32 if out_f32 else torch.bfloat16)
        assert out.shape[0] == M and out.shape[1] == n_out and out.stride(1) == 1
        if W.K % 32 and W.sf_atoms is None:
            raise ValueError(f"K={W.K} must be a multiple of 32 for the streaming / bf16 tensor-core kernels")
        sel = self.select_linear(W, M)
        if sel == "tc":
            if reglu or gelu or geglu:
                raise ValueError("the block-scaled projections have no ReGLU, GeGLU or gelu epilogue")
            # block-quantised codes straight into the tensor cores (any number of rows)
            return self.linear_bs(x, W, name=name, norm_w=norm_w, eps=eps, residual=residual, swiglu=swiglu,
                                  out_f32=out_f32, out=out, xn_out=xn_out, tp_combine=tp_combine, ssq_in=ssq_in,
                                  ssq_out=ssq_out, prefetch=prefetch, tp_scatter=tp_scatter)
        if tp_scatter is not None:
            raise ValueError("tp_scatter needs the block-scaled tensor-core path")
        if tp_combine is not None and M > SMALL_M_MAX:
            raise ValueError("the fused tensor-parallel combine handles at most 8 rows")
        # bf16 tensor-core GEMM: prefill-sized steps, and batched steps (>= 2 rows) of bf16 weights whose row-major form
        # is resident (Fast mode only: Exact verification stays on the batch-invariant streaming kernel)
        batched = (M >= 2 and W.rowmajor_bf16 is not None and tp_combine is None and xn_out is None and self.use_tc_gemm
                   and not self.exact_rows)
        self.sel_counts["gemm" if (sel == "gemm" or batched) else "stream"] += 1
        if sel == "gemm" or batched:
            return self.linear_large(x, W, norm_w=norm_w, eps=eps, residual=residual, epi=epi, out_f32=out_f32, out=out)
        pro = PRO_RMSNORM if norm_w is not None else PRO_NONE
        if W.tiled is None:
            W.make_tiled()
        L = _lib.lib()
        L.ps_linear_stream_max_rows.restype = ctypes.c_int
        mmax = L.ps_linear_stream_max_rows(c_int(WFMT[W.fmt]), c_int(W.k_padded))
        if mmax < 1:
            raise ValueError(f"K={W.K} is too large for the streaming small-M linear kernel")
        for m0 in range(0, M, mmax):
            m = min(mmax, M - m0)
            rs = residual[m0:m0 + m] if residual is not None else None
            _lib.call("ps_linear_stream", c_int(WFMT[W.fmt]), ptr(x[m0:m0 + m]), c_int(m), c_int(W.N),
                      c_int(W.k_padded), c_int(x.stride(0)), ptr(W.tiled), c_float(W.tensor_scale), c_int(pro),
                      ptr(norm_w), c_float(eps), ptr(None), c_int(0), c_int(epi), ptr(rs),
                      c_int(residual.stride(0) if residual is not None else 0), ptr(out[m0:m0 + m]),
                      c_int(out.stride(0)), c_int(1 if out_f32 else 0),
                      ptr(xn_out[m0:m0 + m] if xn_out is not None else None),
                      ctypes.byref(tp_combine) if tp_combine is not None else ptr(None), ptr(self.status))
            self.launches += 1
        return out

    @staticmethod
    def _epilogue(swiglu: bool, reglu: bool, gelu: bool, geglu: bool, residual) -> int:
        if (gelu or geglu) and residual is not None:
            raise ValueError("a projection has either an activation or a residual in its epilogue")
        if swiglu or reglu or geglu:
            return EPI_SWIGLU if swiglu else EPI_REGLU if reglu else EPI_GEGLU
        return EPI_GELU if gelu else EPI_RESIDUAL if residual is not None else EPI_STORE

    def can_fuse_argmax(self, W: LinearW, M: int) -> bool:
        """True when ``linear_argmax`` can serve these rows: the streaming kernel would be chosen and holds them in one launch."""
        if M < 1 or M > SMALL_M_MAX or self.exact_rows or W.fmt == "f32" or W.K % 32 or self.select_linear(W, M) != "stream":
            return False
        if M >= 2 and W.rowmajor_bf16 is not None and self.use_tc_gemm:
            return False
        L = _lib.lib()
        L.ps_linear_stream_max_rows.restype = ctypes.c_int
        return M <= L.ps_linear_stream_max_rows(c_int(WFMT[W.fmt]), c_int(W.k_padded))

    def linear_argmax(self, x: torch.Tensor, W: LinearW, *, norm_w=None, eps: float = 1e-6) -> torch.Tensor:
        """Greedy sampling fused into the projection (lm_head of a decode step): int32 [M] indices of each row's largest
        output, ties to the lower index; the logits are never written.  One launch."""
        M = x.shape[0]
        if W.tiled is None:
            W.make_tiled()
        if getattr(self, "_amax_state", None) is None:
            self._amax_state = torch.zeros(10, dtype=torch.int64, device=self.device)       # 8 keys + control words, kept zero by the kernel
        tokens = self.buf("sampled", max(M, 1), 1, torch.int32)
        _lib.call("ps_linear_stream_argmax", c_int(WFMT[W.fmt]), ptr(x), c_int(M), c_int(W.N), c_int(W.k_padded), c_int(x.stride(0)),
                  ptr(W.tiled), c_float(W.tensor_scale), c_int(PRO_RMSNORM if norm_w is not None else PRO_NONE), ptr(norm_w),
                  c_float(eps), ptr(None), c_int(0), ptr(self._amax_state), ptr(tokens), ptr(self.status))
        self.launches += 1
        self.sel_counts["stream"] += 1
        return tokens.view(-1)[:M]

    def _linear_f32(self, x: torch.Tensor, W: LinearW, name: str, epi: int, out, plain: bool) -> torch.Tensor:
        M, K = x.shape
        if not plain or x.dtype != torch.float32 or K != W.K or x.stride(1) != 1:
            raise ValueError("32-bit projections take fp32 rows and have no fused norm or residual")
        if out is None:
            out = self.buf(name, M, W.N // 2 if epi in GATED else W.N, torch.float32)
        w = W.q.codes
        _lib.call("ps_gemm_f32", ptr(x), c_int(x.stride(0)), ptr(w), c_int(w.stride(0)), c_int(M), c_int(W.N), c_int(K),
                  c_int(epi), ptr(out), c_int(out.stride(0)))
        self.launches += 1
        self.sel_counts["f32"] = self.sel_counts.get("f32", 0) + 1
        return out

    def linear_large(self, x: torch.Tensor, W: LinearW, *, norm_w, eps, residual, epi: int, out_f32, out):
        """Prefill-sized projection: (RMSNorm kernel) -> weight expansion to a bf16 scratch matrix -> tcgen05
        GEMM with the residual / SwiGLU / dtype epilogue fused."""
        M, K = x.shape
        a = x if norm_w is None else self.rmsnorm(x, norm_w, eps, "gemm_norm_in")
        if W.tiled is None:
            W.make_tiled()
        kp = W.k_padded
        if W.rowmajor_bf16 is not None:
            wd = W.rowmajor_bf16
        else:
            need = W.N * kp
            if self.wscratch is None or self.wscratch.numel() < need:
                self.wscratch = torch.empty(need, dtype=torch.bfloat16, device=self.device)
            wd = self.wscratch[:need].view(W.N, kp)
            _lib.call("ps_dequant_tiled", c_int(WFMT[W.fmt]), ptr(W.tiled), c_int(W.N), c_int(kp),
                      c_float(W.tensor_scale), ptr(wd), c_int(kp))
            self.launches += 1
        if W.rowmajor_bf16 is not None and M <= 64 and W.N % 2 == 0:
            # batched decode: swap-AB split-K weight-streaming GEMM (gemm_smallm.cu)
            L = _lib.lib()
            L.ps_gemm_smallm_splits.restype = ctypes.c_int
            splits = L.ps_gemm_smallm_splits(c_int(W.N), c_int(kp))
            need = splits * M * W.N
            part = self.ws.get(("smallm_partial", 0))
            if part is None or part.numel() < need:
                part = torch.empty(max(need, 1 << 22), dtype=torch.float32, device=self.device)
                self.ws[("smallm_partial", 0)] = part
            _lib.call("ps_gemm_smallm", ptr(a), c_int(a.stride(0)), ptr(wd), c_int(kp), c_int(M), c_int(W.N), c_int(kp), c_int(epi),
                      ptr(residual), c_int(residual.stride(0) if residual is not None else 0), ptr(out), c_int(out.stride(0)),
                      c_int(1 if out_f32 else 0), ptr(part), ptr(self.status))
            self.launches += 2
            return out
        _lib.call("ps_gemm_bf16_tc", ptr(a), c_int(a.stride(0)), ptr(wd), c_int(kp), c_int(M), c_int(W.N), c_int(kp),
                  c_int(epi), ptr(residual), c_int(residual.stride(0) if residual is not None else 0), ptr(out),
                  c_int(out.stride(0)), c_int(1 if out_f32 else 0), ptr(self.status))
        self.launches += 1
        return out

    # ------------------------------------------------------------------ kernel selection
    def select_linear(self, W: LinearW, M: int) -> str:
        """Which projection kernel serves `M` rows of `W` -- the job of the reference's linear selector
        (src/phaseshift/models/qwen35/runtime/linear_selector.cpp:202-308), here a pure function of the weight's
        resident layouts, the row count and two switches:

        * ``"tc"``     block-scaled tcgen05 kernel (needs ``W.sf_atoms``): every multi-row step, and single-row steps
                       when only that layout is resident or ``force_tc`` is set (speculative decoding: verification
                       and plain steps must share one arithmetic);
        * ``"stream"`` CUDA-core streaming kernel over ``W.tiled`` (bf16 activations): single rows, bf16 weights up to
                       8 rows, and Exact verification of weights that have no tensor-core layout;
        * ``"gemm"``   bf16 tcgen05 GEMM after a weight expansion: more than 8 rows of weights without ``sf_atoms``."""
        if W.sf_atoms is not None:
            if M > 1 or W.tiled is None or self.force_tc:
                return "tc"
            return "stream"
        if M > SMALL_M_MAX and self.use_tc_gemm and not self.exact_rows:
            return "gemm"
        return "stream"

    # ------------------------------------------------------------------ block-scaled tensor-core projection
    # Rows up to which the activations are quantised inside the projection kernel and kept resident (every CTA repeats that
    # prologue for the K-panels it needs, which pays for a handful of rows: 27B decode batches measured 13.1 vs 14.6 ms per
    # step at 12 rows and 18.6 vs 23.6 ms at 32 rows in favour of one `ps_act_quant` launch + the streamed kernel); the
    # kernel itself supports 32.
    BS_RESIDENT_MAX_ROWS = 8

    def _bs_workspace(self):
        if self.bs_ws is None:
            L = _lib.lib()
            L.ps_gemm_bs_workspace_bytes.restype = ctypes.c_longlong
            L.ps_gemm_bs_flag_words.restype = ctypes.c_int
            with torch.cuda.device(self.device):
                nbytes, nflags = int(L.ps_gemm_bs_workspace_bytes()), int(L.ps_gemm_bs_flag_words())
            self.bs_ws = torch.empty(nbytes // 4, dtype=torch.float32, device=self.device)
            self.bs_flags = torch.zeros(nflags, dtype=torch.int32, device=self.device)
        return self.bs_ws, self.bs_flags

    def reset_after_error(self) -> None:
        """A kernel gave up on a bounded wait: stream-K flags may be left raised; clear them."""
        if self.bs_flags is not None:
            self.bs_flags.zero_()
        if getattr(self, "_amax_state", None) is not None:
            self._amax_state.zero_()              # a fused arg-max launch that did not finish leaves its keys and counter
        self.tickets.zero_()
        self.status.zero_()

    def leaves_row_stats(self, W: LinearW, M: int) -> bool:
        """Whether a residual projection of `M` rows through `W` hands the next fused RMSNorm its rows' sums of squares."""
        return M <= 32 and getattr(W, "sf_atoms", None) is not None and self.select_linear(W, M) == "tc" and self.bs_resident_ok(W, M)

    def bs_resident_ok(self, W: LinearW, M: int) -> bool:
        """Whether `M` rows of this projection fit the kernel's resident-activation path (pure host arithmetic)."""
        if M > self.BS_RESIDENT_MAX_ROWS:
            return False
        key = (W.fmt, 16 if M <= 16 else 32, W.N, W.K)
        ok = self._bs_plan_cache.get(key)
        if ok is None:
            out = (ctypes.c_int * 8)()
            L = _lib.lib()
            L.ps_gemm_bs_plan.restype = ctypes.c_int
            with torch.cuda.device(self.device):
                ok = bool(L.ps_gemm_bs_plan(c_int(WFMT[W.fmt]), c_int(M), c_int(W.N), c_int(W.K), c_int(1),
                                            c_int(self.bs_grid_override), out))
            self._bs_plan_cache[key] = ok
        return ok

    def act_quant(self, x: torch.Tensor, W: LinearW, norm_w, eps: float):
        """Quantise `x` (after the optional fused RMSNorm) to the block format of `W` for the streamed path.
        Returns (codes uint8 [M, panels * 128], scale atoms uint8, row scale fp32 [M] = 1/rms)."""
        from ..quant.act_quant import ATOMS_PER_PANEL, PANEL_K
        M, K = x.shape
        P = -(-K // PANEL_K[W.fmt])
        # one buffer per (K, format): a preset mixes formats at the same K, and a shared name would re-allocate the
        # buffer at every change of format (inside a graph capture too)
        codes = self.buf(f"bs_xq{K}_{W.fmt}", M, P * 128, torch.uint8)
        mblk = -(-M // 256) * 2
        sf = self.buf(f"bs_xsf{K}_{W.fmt}", mblk, P * ATOMS_PER_PANEL[W.fmt] * 512, torch.uint8)
        rs = self.buf("bs_xrs", M, 1, torch.float32)
        _lib.call("ps_act_quant", c_int(WFMT[W.fmt]), ptr(x), c_int(x.stride(0)), c_int(M), c_int(K), ptr(norm_w),
                  c_float(eps), c_float(W.act_scale), ptr(codes), ptr(sf), ptr(rs))
        self.launches += 1
        return codes, sf, rs

    def linear_bs(self, x: torch.Tensor, W: LinearW, *, name: str, norm_w, eps, residual, swiglu, out_f32, out,
                  xn_out=None, tp_combine=None, ssq_in=None, ssq_out=None, prefetch=None, tp_scatter=None) -> torch.Tensor:
        M, K = x.shape
        if K % 8 or x.stride(0) % 8:
            raise ValueError("block-scaled projections need K and the row pitch to be multiples of 8")
        ws, flags = self._bs_workspace()
        epi = EPI_SWIGLU if swiglu else (EPI_RESIDUAL if residual is not None else EPI_STORE)
        resident = self.bs_resident_ok(W, M)
        self.sel_counts["tc_resident" if resident else "tc_streamed"] += 1
        if M <= self.BS_RESIDENT_MAX_ROWS and not resident:
            self.fallbacks["tc_resident_to_streamed"] = self.fallbacks.get("tc_resident_to_streamed", 0) + 1
        if tp_combine is not None and M > tp_combine.max_rows:
            raise ValueError("the fused tensor-parallel combine is sized for %d rows" % tp_combine.max_rows)
        codes = W.codes
        if resident:
            xq = sf = rs = None
        else:
            if xn_out is not None:
                raise ValueError("xn_out is produced by the resident path only")
            xq, sf, rs = self.act_quant(x, W, norm_w, eps)
        ssq_t, ssq_n = ssq_in if (ssq_in is not None and resident and norm_w is not None) else (None, 0)
        if M > 32 or swiglu or (not resident and not out_f32 and tp_combine is None):
            ssq_out = None          # the streamed kernel's staged bf16 epilogue leaves no row statistics
        nxt = prefetch if (prefetch is not None and prefetch.sf_atoms is not None and self.bs_prefetch) else None
        err = _lib.lib().ps_gemm_bs
        err.restype = ctypes.c_int
        rc = err(c_int(WFMT[W.fmt]), ptr(codes), c_ll(codes.shape[1]), c_ll(codes.stride(0)), ptr(W.sf_atoms),
                 c_float(W.tensor_scale), c_int(M), c_int(W.N), c_int(K), ptr(x if resident else None),
                 c_int(x.stride(0)), ptr(norm_w if resident else None), c_float(eps), c_float(W.act_scale),
                 ptr(xn_out), ptr(ssq_t), c_int(ssq_n), c_int(ssq_t.stride(0) if ssq_t is not None else 0),
                 ptr(ssq_out), c_int(ssq_out.stride(0) if ssq_out is not None else 0), ptr(xq), ptr(sf), ptr(rs),
                 c_int(epi), ptr(residual),
                 c_int(residual.stride(0) if residual is not None else 0), ptr(out), c_int(out.stride(0)),
                 c_int(1 if out_f32 else 0), ptr(ws), ptr(flags),
                 ctypes.byref(tp_combine) if tp_combine is not None else ptr(None), ptr(self.status),
                 c_int(self.bs_grid_override), c_int(WFMT[nxt.fmt] if nxt is not None else 0),
                 ptr(nxt.codes if nxt is not None else None), c_ll(nxt.codes.shape[1] if nxt is not None else 0),
                 c_ll(nxt.codes.stride(0) if nxt is not None else 0), ptr(nxt.sf_atoms if nxt is not None else None),
                 c_int(nxt.N if nxt is not None else 0), c_int(nxt.K if nxt is not None else 0),
                 ctypes.byref(tp_scatter) if tp_scatter is not None else ptr(None), _lib.stream())
        _lib.check(rc, "ps_gemm_bs")
        self.launches += 1
        return out

    def attn_prep(self, qkv: torch.Tensor, aw: AttnW, hq: int, hkv: int, b: StepBatch, kv: KVLayer,
                  st: ModelState) -> torch.Tensor:
        cfg = self.cfg
        rows, D = qkv.shape[0], cfg.head_dim
        q = self.buf("attn_q", rows, hq * D)
        _lib.call("ps_attn_prep", ptr(qkv), c_int(qkv.stride(0)), c_int(rows), c_int(hq), c_int(hkv), c_int(D),
                  c_int(cfg.rotary_dim), ptr(aw.q_norm), ptr(aw.k_norm), c_float(cfg.rms_norm_eps),
                  ptr(self.inv_freq), ptr(b.row_slot), ptr(b.row_pos), ptr(q), ptr(kv.k), ptr(kv.v),
                  ptr(kv.k_scale), ptr(kv.v_scale), ptr(st.block_table), c_int(st.max_blocks),
                  c_int(st.sc.page_tokens), c_int(st.num_pages), c_int(st.kv_fmt), ptr(st.status))
        self.launches += 1
        return q

    def paged_attention(self, q: torch.Tensor, qkv: torch.Tensor, hq: int, hkv: int, b: StepBatch, kv: KVLayer,
                        st: ModelState, max_visible: int) -> torch.Tensor:
        """The hybrid decoder's attention: plain causal, sigmoid output gate interleaved with the queries in `qkv`."""
        D = self.cfg.head_dim
        return self.attention(q, AttnSpec(hq, hkv, D, D ** -0.5, gate=qkv, gate_head_stride=2 * D, gate_offset=D), b, kv, st, max_visible)

    def attention(self, q: torch.Tensor, spec: AttnSpec, b: StepBatch, kv: KVLayer, st: ModelState, max_visible: int,
                  gate: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Softmax attention of the step's rows over their paged keys and values (ops/specs.py: AttnSpec)."""
        rows, D, hq, hkv = q.shape[0], spec.dim, spec.heads, spec.kv_heads
        sm, opts = c_float(spec.scale), AttnOptions.of(spec)
        opt = ctypes.byref(opts)
        gate_t = spec.gate if gate is None else gate
        gate = (ptr(gate_t), c_int(gate_t.stride(0) if gate_t is not None else 0), c_int(spec.gate_head_stride), c_int(spec.gate_offset))
        if st.kv_fmt != 0 and (spec.chunk > 0 or spec.window > 0 or spec.keep_first > 0 or spec.sink is not None or spec.bias is not None or spec.temp_coef != 0.0
                               or spec.gate_per_head):
            raise ValueError("masks, sinks, score transforms and per-head gates need bf16 or 32-bit pages")
        geom = f"{hq}x{D}"                      # layers of one model may differ in head geometry: one set of buffers for each
        out = self.buf("attn_ctx" + geom, rows, hq * D, self.act_dtype)
        if self.act_dtype == torch.float32 or D % 32 or D > 256:
            return self._attn_rows(q, spec, b, kv, st, out, gate)
        # the tiled kernel pays off when some sequence brings a long run of rows (a prefill chunk); steps made of
        # many sequences with a row or two each (batched decode) keep the per-row split-KV kernel
        tiled = (not self.exact_rows and not b.graph_static
                 and any(len(sq.token_ids) > self.ATTN_PREFILL_MIN_ROWS for sq in b.seqs))
        row_pos = b.row_pos
        if tiled:
            # prefill-sized step: the long sequences' query tiles on the tensor cores (tcgen05 for head dim 256 and pages of
            # 16 / 32 / 64 tokens, FP8 pools through a bf16 scratch copy of the step's pages; mma.sync otherwise); sequences
            # with a row or two (decode rows of other requests in the same step) stay on the per-row kernel below
            T = self.ATTN_PREFILL_MIN_ROWS
            pt = st.sc.page_tokens
            any_short = T == StepBatch.SHORT_SEQ_ROWS and any(len(sq.token_ids) <= T for sq in b.seqs)
            min_rows = T if any_short else 0
            deq = (None, None, 0, None, None)
            src = (kv.k, kv.v, kv.k_scale, kv.v_scale, st.block_table, st.num_pages, b.seq_desc, 1 if st.kv_fp8 else 0)
            n_long_pages = lambda: sum(-(-(sq.pos_start + len(sq.token_ids)) // pt) for sq in b.seqs if len(sq.token_ids) > min_rows)
            if st.kv_fmt == 2:
                # NVFP4 pages: the step's pages are widened into the bf16 scratch pool, which then IS the pool of the tiled
                # kernels (with its own block table and sequence descriptors), whatever the head size
                dk, dv, n_pg, dbt, dsq = self._attn_scratch(n_long_pages(), hkv, pt, D, b.max_seqs, st.max_blocks)
                _lib.call("ps_kv_fp4_dequant", ptr(kv.k), ptr(kv.v), ptr(kv.k_scale), ptr(kv.v_scale), ptr(st.block_table),
                          c_int(st.max_blocks), c_int(st.num_pages), c_int(pt), c_int(hkv), c_int(D), ptr(b.seq_desc),
                          c_int(b.n_seqs), c_int(min_rows), ptr(dk), ptr(dv), c_int(n_pg), ptr(dbt), ptr(dsq), ptr(st.status))
                self.launches += 1
                src = (dk, dv, None, None, dbt, dk.shape[0], dsq, 0)
            elif st.kv_fp8 and D == 256 and pt in (16, 32, 64):
                deq = self._attn_scratch(n_long_pages(), hkv, pt, D, b.max_seqs, st.max_blocks)
            _lib.call("ps_attn_prefill_ex", ptr(q), ptr(src[0]), ptr(src[1]), ptr(src[2]), ptr(src[3]),
                      ptr(src[4]), c_int(st.max_blocks), c_int(pt), c_int(src[5]),
                      ptr(src[6]), c_int(b.n_seqs), c_int(rows), c_int(q.shape[0]), c_int(min_rows), c_int(hq), c_int(hkv), c_int(D),
                      sm, c_int(src[7]), *gate, ptr(deq[0]), ptr(deq[1]), c_int(deq[2]), ptr(deq[3]), ptr(deq[4]), ptr(out), ptr(st.status), opt)
            self.launches += 2 if deq[0] is not None else 1
            if not any_short:
                return out
            row_pos = b.row_pos_short
        # Split length: 64 tokens give a single row enough CTAs to fill the GPU; a batch of many rows already does, and its
        # CTAs should rather amortise their set-up over a longer run of tokens (about four CTAs per SM in total).  Exact mode
        # and small batches keep the fixed length, so a row's summation order does not depend on its neighbours there.
        split_tokens = self.split_tokens
        if rows > SMALL_M_MAX and not self.exact_rows:
            want = max(1, (4 * 148) // (rows * hkv))
            split_tokens = max(split_tokens, -(-(-(-max_visible // want)) // 32) * 32)
        pacc = self.buf("attn_part_acc" + geom, rows, hq * self.max_splits * D, torch.float32)
        pml = self.buf("attn_part_ml" + geom, rows, hq * self.max_splits * 2, torch.float32)
        # Decode / verify rows on the tensor cores: bf16 pages, head dim 256, every sequence handled here has at most 16 rows
        # (the query heads that share a KV head are packed into one MMA tile).  A row's result does not depend on the other
        # rows of its tile (every tile row has its own scores, reference maximum and accumulator lane), so Exact mode -- whose
        # verified rows must reproduce single-row decoding bit for bit -- uses it as well.  FP8 pages and other shapes keep the
        # per-row kernel.  PS_ATTN_DECODE=legacy switches it off.
        if (self.attn_decode_tc and D % 64 == 0 and st.kv_fmt == 0 and st.sc.page_tokens in (16, 32, 64) and hq // hkv <= 8
                and not (kv.k is kv.v and (spec.bias is not None or spec.temp_coef != 0.0))
                and (b.graph_static or row_pos is b.row_pos_short or all(len(sq.token_ids) <= 16 for sq in b.seqs))):
            st_tok = -(-split_tokens // 64) * 64
            n_seqs = b.max_seqs if b.graph_static else b.n_seqs
            _lib.call("ps_attn_decode_tc_ex", ptr(q), c_int(q.shape[0]), ptr(kv.k), ptr(kv.v), ptr(st.block_table),
                      c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(b.seq_desc), c_int(n_seqs),
                      c_int(16), c_int(hq), c_int(hkv), c_int(D), sm, c_int(st_tok), c_int(self.max_splits),
                      c_int(max_visible), ptr(pacc), ptr(pml), ptr(st.status), opt)
            _lib.call("ps_paged_attention_merge_ex", ptr(pacc), ptr(pml), ptr(row_pos), c_int(rows), c_int(hq), c_int(D),
                      c_int(st_tok), c_int(self.max_splits), *gate, ptr(out), opt, c_int(0))
            self.launches += 2
            return out
        if st.kv_fmt == 2:
            _lib.call("ps_paged_attention_fp4", ptr(q), ptr(kv.k), ptr(kv.v), ptr(kv.k_scale), ptr(kv.v_scale),
                      ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages),
                      ptr(b.row_slot), ptr(row_pos), c_int(rows), c_int(hq), c_int(hkv), c_int(D), sm,
                      c_int(split_tokens), c_int(self.max_splits), c_int(max_visible), ptr(pacc), ptr(pml), ptr(st.status))
            _lib.call("ps_paged_attention_merge", ptr(pacc), ptr(pml), ptr(row_pos), c_int(rows), c_int(hq), c_int(D),
                      c_int(split_tokens), c_int(self.max_splits), *gate, ptr(out))
            self.launches += 2
            return out
        _lib.call("ps_paged_attention_ex", ptr(q), ptr(kv.k), ptr(kv.v), ptr(kv.k_scale), ptr(kv.v_scale),
                  ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages),
                  ptr(b.row_slot), ptr(row_pos), c_int(rows), c_int(hq), c_int(hkv), c_int(D),
                  sm, c_int(1 if st.kv_fp8 else 0), c_int(split_tokens), c_int(self.max_splits), c_int(max_visible),
                  ptr(pacc), ptr(pml), *gate, ptr(out), ptr(st.status), opt)
        self.launches += 2
        return out

    def _attn_rows(self, q, spec: AttnSpec, b: StepBatch, kv: KVLayer, st: ModelState, out: torch.Tensor, gate) -> torch.Tensor:
        """One CTA per row and head, any head size, bf16 or 32-bit."""
        opts = AttnOptions.of(spec)
        _lib.call("ps_attn_rows", ptr(q), ptr(kv.k), ptr(kv.v), c_int(1 if self.act_dtype == torch.float32 else 0),
                  ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(b.row_slot),
                  ptr(b.row_pos), c_int(q.shape[0]), c_int(spec.heads), c_int(spec.kv_heads), c_int(spec.dim), c_float(spec.scale),
                  ctypes.byref(opts), *gate, ptr(out), ptr(st.status))
        self.launches += 1
        return out

    def _attn_scratch(self, pages: int, hkv: int, pt: int, D: int, max_seqs: int, max_blocks: int):
        """bf16 scratch pool for the tiled attention over FP8 pages: (k, v, pages, block table, sequence descriptors).  One
        allocation that grows to the largest step seen (by doubling)."""
        cap = getattr(self, "_deq_cap", 0)
        if pages > cap or getattr(self, "_deq_geom", None) != (hkv, pt, D, max_seqs, max_blocks):
            cap = max(pages, 2 * cap, 64)
            self._deq_k = torch.empty(cap, hkv, pt, D, dtype=torch.bfloat16, device=self.device)
            self._deq_v = torch.empty_like(self._deq_k)
            self._deq_bt = torch.zeros(max_seqs, max_blocks, dtype=torch.int32, device=self.device)
            self._deq_seqs = torch.zeros(max_seqs, 4, dtype=torch.int32, device=self.device)
            self._deq_cap, self._deq_geom = cap, (hkv, pt, D, max_seqs, max_blocks)
        return self._deq_k, self._deq_v, pages, self._deq_bt, self._deq_seqs

    def gdn(self, proj: torch.Tensor, gw: GdnW, hk: int, hv: int, b: StepBatch, gs: GdnLayerState,
            st: ModelState, log=None, to_alt: bool = False, xn: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``xn`` given: the kernel projects beta/decay inputs itself from the normalised rows (bf16
        ``ba_proj`` weights); otherwise they are read from the last 2*hv columns of ``proj``."""
        cfg = self.cfg
        rows = proj.shape[0]
        Dk, Dv = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        out = self.buf("gdn_o", rows, hv * Dv)
        state_out = gs.rec_alt if to_alt else gs.rec
        n_seqs = b.max_seqs if b.graph_static else b.n_seqs
        # Sequences with many rows in this step (prefill chunks) take the chunked kernels, sequences with few rows
        # (decode / verify rows of other requests in the same step) the row-sequential kernel; both can be present.
        T = self.GDN_CHUNKED_MIN_ROWS
        plain = log is None and not to_alt and not self.exact_rows and not b.graph_static
        seq_rows = [len(sq.token_ids) for sq in b.seqs] if plain else []
        any_long = any(n > T for n in seq_rows)
        any_short = (not any_long) or any(n <= T for n in seq_rows)
        if any_long:
            f32 = torch.float32
            long_rows = sum(n for n in seq_rows if n > T)
            chunks = sum((n + 63) // 64 for n in seq_rows if n > T)
            scr = self.buf("gdn_scratch", 1, chunks * hv * 64 * (3 * Dk + Dv + 64), f32)
            dc = self.buf("gdn_dc", 1, chunks * hv, f32)
            o = self.buf("gdn_of", rows, hv * Dv, f32)
            if xn is not None:
                raise ValueError("the chunked GDN path reads the b/a projections from `proj`")
            _lib.call("ps_gdn_chunked", ptr(proj), c_int(proj.stride(0)), c_int(rows), c_int(hk), c_int(hv), c_int(Dk),
                      c_int(Dv), ptr(gw.conv_w), ptr(gw.A_log), ptr(gw.dt_bias), ptr(gw.norm_w),
                      c_float(cfg.rms_norm_eps), ptr(gs.conv), c_int(st.sc.conv_ring), ptr(gs.rec), ptr(b.seq_desc),
                      c_int(n_seqs), ptr(b.row_slot), ptr(b.row_pos), c_int(T), ptr(scr), ptr(dc), ptr(o), ptr(out))
            self.launches += 4
            del long_rows
        if any_short:
            lk = ld = ldd = None
            if log is not None:
                lk, ld, ldd = log
            _lib.call("ps_gdn_rows", ptr(proj), c_int(proj.stride(0)), c_int(hk), c_int(hv), c_int(Dk), c_int(Dv),
                      ptr(gw.conv_w), ptr(gw.A_log), ptr(gw.dt_bias), ptr(gw.norm_w), c_float(cfg.rms_norm_eps),
                      ptr(gs.conv), c_int(st.sc.conv_ring), ptr(gs.rec), ptr(state_out), ptr(b.seq_desc),
                      c_int(n_seqs), ptr(out), ptr(lk), ptr(ld), ptr(ldd),
                      ptr(gw.ba_proj.q.codes if xn is not None else None), ptr(xn), c_int(gw.ba_proj.K),
                      c_int(T if any_long else 0))
            self.launches += 1
        return out

    def gdn_replay(self, gs: GdnLayerState, hv: int, seq_desc: torch.Tensor, n_seqs: int, log) -> None:
        cfg = self.cfg
        lk, ld, ldd = log
        _lib.call("ps_gdn_replay", ptr(gs.rec), c_int(hv), c_int(cfg.linear_key_head_dim),
                  c_int(cfg.linear_value_head_dim), ptr(seq_desc), c_int(n_seqs), ptr(lk), ptr(ld), ptr(ldd))
        self.launches += 1

    def gather_rows(self, x: torch.Tensor, rows_idx: torch.Tensor, n: int, name: str, status) -> torch.Tensor:
        out = self.buf(name, n, x.shape[1], x.dtype)
        rb = x.shape[1] * x.element_size()
        _lib.call("ps_gather_rows", ptr(x), c_ll(x.stride(0) * x.element_size()), ptr(rows_idx), c_int(n), ptr(out),
                  c_ll(rb), c_int(rb), c_int(x.shape[0]), ptr(status))
        self.launches += 1
        return out

    def sample(self, logits: torch.Tensor, b: StepBatch, n: int, mask=None, mask_active=None,
               status=None) -> torch.Tensor:
        out = self.buf("sampled", max(n, 1), 1, torch.int32)
        _lib.call("ps_sample", ptr(logits), c_int(logits.stride(0)), c_int(logits.shape[1]), c_int(n), ptr(b.d_samp),
                  ptr(mask), c_int(mask.shape[1] if mask is not None else 0), ptr(mask_active), ptr(out), ptr(status))
        self.launches += 1
        return out.view(-1)[:n]

    def topk(self, logits: torch.Tensor, k: int, mask: Optional[torch.Tensor] = None):
        """Exact top-k (k <= 128) per row of fp32 logits, sorted descending, ties to the lower id.
        Returns (ids int32 [rows, k], values fp32 [rows, k]); `mask` is an optional allowed-token bitmask."""
        rows, vocab = logits.shape
        ids = self.buf("topk_ids", rows, k, torch.int32)
        vals = self.buf("topk_vals", rows, k, torch.float32)
        L = _lib.lib()
        L.ps_topk_workspace_bytes.restype = ctypes.c_longlong
        need = int(L.ps_topk_workspace_bytes(c_int(vocab), c_int(rows), c_int(k)))
        ws = self.buf("topk_ws", rows * k, need // (rows * k * 8), torch.int64)
        _lib.call("ps_topk", ptr(logits), c_ll(logits.stride(0)), c_int(vocab), c_int(rows), c_int(k), ptr(mask),
                  c_int(mask.shape[1] if mask is not None else 0), ptr(ids), ptr(vals), ptr(ws), c_ll(need))
        self.launches += 2
        return ids, vals

    def rmsnorm(self, x: torch.Tensor, w: torch.Tensor, eps: float, name: str, one_plus: bool = True,
                add: Optional[torch.Tensor] = None, sum_out: Optional[torch.Tensor] = None) -> torch.Tensor:
        rows, H = x.shape
        out = self.buf(name, rows, H)
        _lib.call("ps_rmsnorm", ptr(x), c_int(x.stride(0)), ptr(add), c_int(add.stride(0) if add is not None else 0),
                  ptr(sum_out), c_int(sum_out.stride(0) if sum_out is not None else 0), ptr(w), c_float(eps),
                  c_int(rows), c_int(H), ptr(out), c_int(out.stride(0)), c_int(1 if one_plus else 0))
        self.launches += 1
        return out

    # ------------------------------------------------------------------ 32-bit residual stream
    def embed_f32(self, b: StepBatch, rows: int, table: torch.Tensor, status) -> torch.Tensor:
        out = self.buf("x_embed", rows, table.shape[1], torch.float32)
        _lib.call("ps_embed_f32", ptr(b.ids), ptr(table), c_int(1 if table.dtype == torch.float32 else 0), c_int(rows),
                  c_int(table.shape[0]), c_int(table.shape[1]), ptr(out), ptr(status))
        self.launches += 1
        return out

    def residual_norm(self, x: torch.Tensor, pend: Optional[Pending], *, add=None, step=None, norm_w=None, eps: float,
                      scale: float = 1.0, width: int = 0, one: bool = False, name: str = ""):
        """Add what is pending to the fp32 residual `x` (and `add` rows, a `step` vector), then norm the row for the next
        projection: `width` columns, zero-padded, column W = 1 when `one` (ops/specs.py: Pending).  One launch.
        Returns (residual, normed rows or None); the residual lives in one buffer of its own, `x` itself is only overwritten
        when it is that buffer."""
        rows, W = x.shape
        if pend is not None and pend.bias is not None:
            if step is not None:
                raise ValueError("a residual update adds one vector: a step or a bias")
            step = pend.bias
        changed = pend is not None or add is not None or step is not None
        xo = self.buf("x_res", rows, W, torch.float32) if changed else None
        h = self.buf(name, rows, width, self.act_dtype) if norm_w is not None else None
        if xo is None and h is None:
            return x, None
        a = b = wa = wb = y = None
        if pend is not None:
            a, b, wa, wb, y = pend.branch_a, pend.branch_b, pend.weight_a, pend.weight_b, pend.plain
        ld = lambda t: c_int(t.stride(0) if t is not None else 0)
        if pend is not None and pend.experts is not None:
            if add is not None or one or scale != 1.0:
                raise ValueError("a mixture's sum is followed by a plain norm")
            e, r = pend.experts, pend.experts.routed
            _lib.call("ps_residual_norm_experts", ptr(x), ptr(xo), c_int(rows), c_int(W), ptr(r.index), ptr(r.weight), ptr(r.identity),
                      c_int(r.index.shape[1]), ptr(e.y), ld(e.y), ptr(e.h), ld(e.h), ptr(e.shared), ld(e.shared), c_float(pend.coef), ptr(step),
                      ptr(norm_w), c_float(eps), ptr(h), c_int(1 if self.act_dtype == torch.float32 else 0), c_int(width))
            self.launches += 1
            return xo, h
        _lib.call("ps_residual_norm", ptr(x), ptr(xo), c_int(rows), c_int(W), ptr(a), ld(a), ptr(wa), ptr(b), ld(b), ptr(wb),
                  ptr(y), ld(y), c_float(pend.coef if pend is not None else 0.0), ptr(add), ptr(step), ptr(norm_w), c_float(eps),
                  c_float(scale), ptr(h), c_int(1 if self.act_dtype == torch.float32 else 0), c_int(width), c_int(1 if one else 0))
        self.launches += 1
        return (xo if changed else x), h

    # ------------------------------------------------------------------ norms behind the sublayers
    def gated_norm(self, x: torch.Tensor, pend: Optional[GatedNorm], *, eps: float, groups: int, norm_w: Optional[torch.Tensor] = None,
                   width: int = 0, name: str = ""):
        """x + the sublayer's gated and normed result (ops/specs.py: GatedNorm), and the next projection's input: the new residual
        itself, or with `norm_w` its norm in groups, zero-padded to `width` columns (0: none).  One launch.  Returns (residual, rows or
        None); the residual lives in one buffer of its own, `x` itself is only overwritten when it is that buffer."""
        rows, W = x.shape
        f32 = self.act_dtype == torch.float32
        xo = self.buf("x_res", rows, W, torch.float32) if pend is not None else None
        h = self.buf(name, rows, width, self.act_dtype) if width else None
        if xo is None and h is None:
            return x, None
        p = pend if pend is not None else GatedNorm(None, None, None)
        r = p.routed
        if p.gate is not None and f32 and p.gate.dtype != torch.float32:
            raise ValueError("32-bit engines have 32-bit gates")
        ld = lambda t: c_int(t.stride(0) if t is not None else 0)
        _lib.call("ps_gated_norm", ptr(x), ptr(xo), c_int(rows), c_int(W), c_int(groups), c_float(eps), ptr(p.a), ld(p.a), c_float(p.scale_a),
                  ptr(p.b), ld(p.b), c_float(p.scale_b), c_int(r.index.shape[1] if r is not None else 0), ptr(r.index if r is not None else None),
                  ptr(r.weight if r is not None else None), ptr(p.experts), ld(p.experts), ptr(p.gate), ld(p.gate),
                  c_int(1 if p.gate is not None and p.gate.dtype == torch.float32 else 0), ptr(p.gate_bias), ptr(p.norm_w), ptr(norm_w), ptr(h),
                  c_int(1 if f32 else 0), c_int(width))
        self.launches += 1
        return (xo if xo is not None else x), h

    def soft_limit(self, logits: torch.Tensor, cap: float) -> torch.Tensor:
        """cap * tanh(logits / cap), in place."""
        if not logits.is_contiguous() or logits.dtype != torch.float32:
            raise ValueError("soft_limit takes contiguous fp32 logits")
        _lib.call("ps_soft_limit", ptr(logits), c_ll(logits.numel()), c_float(cap))
        self.launches += 1
        return logits

    # ------------------------------------------------------------------ parallel residual streams
    def stream_norm(self, x: torch.Tensor, pend: Optional[StreamWrite], *, read: Optional[torch.Tensor] = None,
                    norm_w: Optional[torch.Tensor] = None, eps: float, width: int = 0, name: str = "", last: bool = False):
        """Write what is pending into the fp32 streams `x` [rows, streams, W], read the next sublayer's input from them and norm it
        for the next projection (`width` columns, zero-padded).  One launch.  Returns (streams, normed rows or None); the
        streams live in one buffer of their own.  ``last``: they are not needed again."""
        rows, S, W = x.shape
        xo = None
        if pend is not None and not last:
            xo = self.buf("x_streams", rows, S * W, torch.float32).view(rows, S, W)
        h = self.buf(name, rows, width, self.act_dtype) if norm_w is not None else None
        if xo is None and h is None:
            return x, None
        mix, out, y = (pend.mix, pend.out, pend.y) if pend is not None else (None, None, None)
        _lib.call("ps_stream_norm", ptr(x), c_ll(x.stride(0)), c_ll(x.stride(1)), ptr(xo), c_int(rows), c_int(W), c_int(S), ptr(mix), ptr(out),
                  ptr(y), c_int(y.stride(0) if y is not None else 0), ptr(read), ptr(norm_w), c_float(eps), ptr(h),
                  c_int(1 if self.act_dtype == torch.float32 else 0), c_int(width))
        self.launches += 1
        return (xo if xo is not None else x), h

    # ------------------------------------------------------------------ attention without rotation: query copy + key / value append
    def attn_append(self, proj: torch.Tensor, spec: AttnSpec, b: StepBatch, kv: Optional[KVLayer], st: ModelState) -> torch.Tensor:
        """``kv`` None: the layer reads another one's keys, only the queries are copied."""
        rows = proj.shape[0]
        q = self.buf(f"attn_q{spec.heads}x{spec.dim}", rows, spec.heads * spec.dim, self.act_dtype)
        k = kv.k if kv is not None else None
        v = kv.v if kv is not None and kv.v is not kv.k else None
        _lib.call("ps_attn_append", ptr(proj), c_int(proj.stride(0)), c_int(proj.element_size()), c_int(rows), c_int(spec.heads),
                  c_int(spec.kv_heads if kv is not None else 0), c_int(spec.dim), ptr(b.row_slot), ptr(b.row_pos), ptr(q), ptr(k), ptr(v),
                  ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(st.status))
        self.launches += 1
        return q

    # ------------------------------------------------------------------ embedding of a token and the pair it ends
    def embed_pairs(self, b: StepBatch, rows: int, table: torch.Tensor, pairs: torch.Tensor, mul_prev: int, mul_cur: int, norm_w, eps: float,
                    st: ModelState) -> torch.Tensor:
        """normed table[token] + pairs[(previous * mul_prev + token * mul_cur) mod buckets], fp32; the last row of `pairs` belongs
        to the first token of a sequence.  Keeps every sequence's last token."""
        W = table.shape[1]
        out = self.buf("x_embed", rows, W, torch.float32)
        _lib.call("ps_embed_pairs", ptr(b.ids), ptr(table), ptr(pairs), c_int(1 if table.dtype == torch.float32 else 0), c_int(rows),
                  c_int(table.shape[0]), c_int(pairs.shape[0] - 1), c_ll(mul_prev), c_ll(mul_cur), ptr(norm_w), c_float(eps), c_int(W),
                  ptr(b.row_slot), ptr(b.seq_desc), c_int(b.max_seqs if b.graph_static else b.n_seqs), ptr(st.last_token), ptr(out), ptr(st.status))
        self.launches += 1
        return out

    # ------------------------------------------------------------------ queries, keys and values of an attention
    def attn_heads(self, proj: torch.Tensor, s: HeadsSpec, b: StepBatch, kv: KVLayer, st: ModelState, history: Optional[torch.Tensor] = None,
                   saved: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Projection rows to queries (returned) and keys and values in their pages (ops/specs.py: HeadsSpec).  ``history``: the
        layer's convolution rows in the state; ``saved``: buffer of the values that later layers mix in.  One launch."""
        rows, dt = proj.shape[0], self.act_dtype
        if st.kv_fmt != 0:
            raise ValueError("attn_heads appends to bf16 or 32-bit pages")
        if proj.dtype != dt or (s.conv is not None and s.conv.dtype != dt):
            raise ValueError("projection rows and convolution weights have the engine's type")
        q = self.buf(f"attn_q{s.heads}x{s.dim}", rows, s.heads * s.dim, dt)
        _lib.call("ps_attn_heads", ptr(proj), c_int(proj.stride(0)), c_int(1 if dt == torch.float32 else 0), c_int(rows), c_int(s.heads),
                  c_int(s.kv_heads), c_int(s.dim), c_int(s.dim_true), c_int(s.vdim_true), c_int(s.freq.numel()), c_int(int(s.halves)),
                  c_int(int(s.unit)), c_float(s.eps), c_float(s.turn_size), ptr(s.freq), ptr(s.q_norm), ptr(s.k_norm), c_int(s.taps),
                  ptr(s.conv), ptr(history), c_float(s.mix or 0.0), ptr(saved if s.mix is not None else None), ptr(saved if s.save else None),
                  ptr(q), ptr(kv.k), ptr(kv.v), ptr(b.row_slot), ptr(b.row_pos), ptr(st.block_table), c_int(st.max_blocks),
                  c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(b.seq_desc), c_int(b.max_seqs if b.graph_static else b.n_seqs),
                  ptr(self.tickets), ptr(st.status))
        self.launches += 1
        return q

    def saved_values(self, rows: int, width: int) -> torch.Tensor:
        return self.buf(f"saved_values{width}", rows, width, self.act_dtype)

    # ------------------------------------------------------------------ mixture of experts
    def moe_route(self, logits: torch.Tensor, h: torch.Tensor, s: MoeSpec, b: StepBatch) -> Routed:
        """Router logits (fp32) to every row's experts and weights (ops/specs.py: MoeSpec), and the rows of `h` sorted by expert."""
        rows, K = h.shape
        R, i32, f32 = rows * s.top, torch.int32, torch.float32
        tile = self._moe_tile(rows, s)
        max_tiles = R // tile + min(s.experts, R)
        out = Routed(self.buf(f"moe_index{s.top}", rows, s.top, i32), self.buf(f"moe_weight{s.top}", rows, s.top, f32),
                     self.buf("moe_same", rows, 1, f32), self.buf(f"moe_x{K}", R + tile, K, self.act_dtype),
                     self.buf("moe_tiles", 1 + max_tiles, 4, i32), tile, max_tiles)
        small = rows <= 64
        pairs = None if small else self.buf(f"moe_pairs{s.top}", rows, 2 * s.top, i32)
        counts = None if small else self.buf(f"moe_counts{s.experts}", 1, s.experts, i32)
        _lib.call("ps_moe_route", ptr(logits), c_int(logits.stride(0)), ptr(s.correction), ptr(b.row_slot), c_int(rows), c_int(s.experts),
                  c_int(s.identity), c_int(s.top), c_int(s.groups), c_int(s.keep), c_int(int(s.sigmoid)), c_int(s.group_top), c_int(int(s.renormalize)),
                  ptr(out.index), ptr(out.weight), ptr(out.identity), ptr(h),
                  c_int(K * h.element_size()), ptr(out.inputs), ptr(out.tiles), c_int(tile), ptr(pairs), ptr(counts), ptr(self.status))
        self.launches += 1 if small else 3
        return out

    def _moe_tile(self, rows: int, s: MoeSpec) -> int:
        """Rows per tile of the experts' products: all that one expert can get in a small step, else about what it gets on average."""
        if self.act_dtype == torch.float32:
            return 64
        if rows <= 64:
            return 16 if rows <= 16 else 32 if rows <= 32 else 64
        each = rows * s.top / (s.experts + s.identity)
        return 64 if each <= 32 else 128

    def moe_experts(self, routed: Routed, s: MoeSpec) -> torch.Tensor:
        """Outputs of the sorted rows' experts, fp32 [sorted rows, n_out].  Two launches."""
        x, K, dt = routed.inputs, s.gate_up.shape[1], self.act_dtype
        R = x.shape[0] - routed.tile_rows
        act = self.buf(f"moe_act{s.ff}", x.shape[0], s.ff, dt)
        y = self.buf(f"moe_y{s.n_out}", R, s.n_out, torch.float32)
        limit = 0.0 if s.limit is None else s.limit

        def product(a, w, N, K, gated, out):
            if dt == torch.float32:
                _lib.call("ps_moe_gemm_f32", ptr(a), ptr(w), c_int(N), c_int(K), c_int(gated), c_float(limit), ptr(routed.tiles),
                          c_int(routed.max_tiles), ptr(out), c_int(out.stride(0)))
            else:
                _lib.call("ps_moe_gemm", ptr(a), c_int(a.shape[0]), ptr(w), c_int(s.experts), c_int(N), c_int(K), c_int(gated), c_float(limit),
                          ptr(routed.tiles), c_int(routed.tile_rows), c_int(routed.max_tiles), ptr(out), c_int(out.stride(0)), ptr(self.status))
            self.launches += 1
        product(x, s.gate_up, 2 * s.ff, K, 1 if s.limit is None else 2, act)
        product(act, s.down, s.n_out, s.ff, 0, y)
        return y

    # ------------------------------------------------------------------ latent attention
    def latent_down(self, proj: torch.Tensor, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState) -> torch.Tensor:
        """Norm both latents of the projection rows, turn the shared key part, append; returns the query latents."""
        rows = proj.shape[0]
        cq = self.buf(f"latent_cq{s.q_rank}", rows, s.q_rank, self.act_dtype)
        _lib.call("ps_latent_down", ptr(proj), c_int(proj.stride(0)), c_int(1 if self.act_dtype == torch.float32 else 0), c_int(rows),
                  c_int(s.q_rank), c_int(s.kv_rank), c_int(s.rot), c_int(s.q_rank_true), c_int(s.kv_rank_true), c_int(s.rot_true // 2),
                  ptr(s.q_norm), ptr(s.kv_norm), c_float(s.eps), ptr(s.inv_freq), ptr(cq), ptr(kv.k), ptr(b.row_slot), ptr(b.row_pos),
                  ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(st.status))
        self.launches += 1
        return cq

    def _latent_turn(self, q, head: int, off: int, out, ohead: int, ooff: int, s: LatentSpec, b: StepBatch) -> None:
        _lib.call("ps_latent_turn", ptr(q), c_int(q.stride(0)), c_int(head), c_int(off), ptr(out), c_int(out.stride(0)), c_int(ohead),
                  c_int(ooff), c_int(1 if q.dtype == torch.float32 else 0), c_int(q.shape[0]), c_int(s.heads), c_int(s.rot),
                  c_int(s.rot_true // 2), ptr(s.inv_freq), ptr(b.row_pos))
        self.launches += 1

    def _gemm_heads(self, x, x_head: int, w, heads: int, N: int, K: int, out, o_head: int, gate=None, g_head: int = 0,
                    turn: Optional[Tuple[LatentSpec, StepBatch]] = None) -> None:
        """out[:, h] = x[:, h] w[h]^T (* sigmoid(gate[:, h])); `x_head` / `o_head` / `g_head`: columns between heads.  ``turn``: the
        rotated part behind each head's `K` columns is turned by the row's position and stored behind its `N` outputs."""
        M, ldg = x.shape[0], gate.stride(0) if gate is not None else 0
        if self.act_dtype == torch.float32:
            _lib.call("ps_gemm_f32_batched", ptr(x), c_int(x.stride(0)), c_ll(x_head), ptr(w), c_int(K), c_ll(N * K), c_int(heads), c_int(M),
                      c_int(N), c_int(K), ptr(gate), c_int(ldg), c_ll(g_head), ptr(out), c_int(out.stride(0)), c_ll(o_head))
        else:
            s, b = turn if turn is not None else (None, None)
            _lib.call("ps_gemm_heads", ptr(x), c_int(x.stride(0)), c_int(x_head), ptr(w), c_int(heads), c_int(M), c_int(N), c_int(K),
                      ptr(gate), c_int(ldg), c_int(g_head), ptr(out), c_int(out.stride(0)), c_int(o_head), c_int(s.rot if s else 0),
                      c_int(s.rot_true // 2 if s else 0), ptr(s.inv_freq if s else None), ptr(b.row_pos if s else None), ptr(self.status))
        self.launches += 1
        if turn is not None and self.act_dtype == torch.float32:
            self._latent_turn(x, x_head, K, out, o_head, N, *turn)

    def latent_attention(self, q: torch.Tensor, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState, gate: torch.Tensor) -> torch.Tensor:
        """Attention of query rows [rows, heads * (dim + rot)] (not turned yet; turned in place) over the cached latents, values back
        in the heads and gated with the projection rows `gate`.  Sequences with many rows in the step attend over expanded keys
        and values, the others in the latent space."""
        rows, H, T = q.shape[0], s.heads, self.ATTN_PREFILL_MIN_ROWS
        out = self.buf(f"latent_ctx{H}x{s.vdim}", rows, H * s.vdim, self.act_dtype)
        L = _lib.lib()
        long = []
        if (self.act_dtype == torch.bfloat16 and not self.exact_rows and not b.graph_static and T == StepBatch.SHORT_SEQ_ROWS
                and L.ps_latent_prefill_ok(c_int(s.dim), c_int(s.rot), c_int(s.vdim))):
            long = [sq for sq in b.seqs if len(sq.token_ids) > T]
        if not long or any(len(sq.token_ids) <= T for sq in b.seqs):
            self._latent_absorbed(q, s, b, kv, st, gate, out, short_only=bool(long))
        if long:
            self._latent_expanded(q, s, b, kv, st, gate, out, long)
        return out

    def _latent_absorbed(self, q, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState, gate, out, short_only: bool) -> None:
        """Queries into the latent space, attention with the cached rows as the keys and values of all heads, outputs back to the
        heads with the gate.  ``short_only``: the rows of longer sequences come later and overwrite what this leaves there."""
        rows, H, L = q.shape[0], s.heads, _lib.lib()
        spec = s.shared_keys()
        qe = self.buf(f"latent_qe{H}x{s.row}", rows, H * s.row, self.act_dtype)
        self._gemm_heads(q, s.dim + s.rot, s.uk_t, H, s.kv_rank, s.dim, qe, s.row, turn=(s, b))
        pt = st.sc.page_tokens
        tc = (self.act_dtype == torch.bfloat16 and self.attn_decode_tc and bool(L.ps_latent_decode_ok(c_int(s.kv_rank), c_int(s.rot), c_int(pt)))
              and (short_only or b.graph_static or all(len(sq.token_ids) <= 16 for sq in b.seqs)))
        if tc:
            o, head = self._latent_decode(qe, s, spec, b, kv, st, b.row_pos_short if short_only else b.row_pos), s.kv_rank
        else:
            o, head = self.buf(f"latent_or{H}x{s.row}", rows, H * s.row, self.act_dtype), s.row
            self._attn_rows(qe, spec, b, kv, st, o, (ptr(None), c_int(0), c_int(0), c_int(0)))
        self._gemm_heads(o, head, s.uv, H, s.vdim, s.kv_rank, out, s.vdim, gate[:, s.gate_off:], s.vdim)

    def _latent_decode(self, qe, s: LatentSpec, spec: AttnSpec, b: StepBatch, kv: KVLayer, st: ModelState, row_pos) -> torch.Tensor:
        """Split-KV pass and merge.  The split length is a function of the step's row bucket and of the longest reach of a row
        (the window, or the engine's longest context), so buffers and captured graphs stay valid."""
        rows, H, L = qe.shape[0], s.heads, _lib.lib()
        if b.graph_static:
            n_seqs, seq_rows = b.max_seqs, b.max_rows if b.max_rows <= 16 else 1        # larger captured steps are pure decode batches
        else:
            n_seqs, seq_rows = b.n_seqs, max(n for n in (len(sq.token_ids) for sq in b.seqs) if n <= 16)
        reach = min(s.window, b.max_context) if s.window > 0 else b.max_context
        ctas = b.max_seqs * L.ps_latent_decode_ctas(c_int(H), c_int(s.kv_rank), c_int(s.rot), c_int(1))
        split = max(128, -(-reach // max(1, 296 // ctas) // 64) * 64)
        while -(-(reach + 80) // split) + 1 > 512:
            split *= 2
        ring = -(-(reach + 80) // split) + 1                 # a tile of up to 16 rows, from the tile of its first visible token on
        pacc = self.buf(f"latent_acc{H}x{s.kv_rank}x{ring}", rows, H * ring * s.kv_rank, torch.float32)
        pml = self.buf(f"latent_ml{H}x{ring}", rows, H * ring * 2, torch.float32)
        out = self.buf(f"latent_o{H}x{s.kv_rank}", rows, H * s.kv_rank)
        opts = AttnOptions.of(spec)
        _lib.call("ps_latent_decode", ptr(qe), c_int(rows), ptr(kv.k), ptr(st.block_table), c_int(st.max_blocks), c_int(st.sc.page_tokens),
                  c_int(st.num_pages), ptr(b.seq_desc), c_int(n_seqs), c_int(seq_rows), c_int(H), c_int(s.kv_rank), c_int(s.rot),
                  c_float(s.scale), c_int(split), c_int(ring), c_int(ring), ctypes.byref(opts), ptr(pacc), ptr(pml), ptr(st.status))
        _lib.call("ps_paged_attention_merge_ex", ptr(pacc), ptr(pml), ptr(row_pos), c_int(rows), c_int(H), c_int(s.kv_rank), c_int(split),
                  c_int(ring), ptr(None), c_int(0), c_int(0), c_int(0), ptr(out), ctypes.byref(opts), c_int(ring))
        self.launches += 2
        return out

    def _latent_expanded(self, q, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState, gate, out, long) -> None:
        """The tokens that the long sequences see, gathered into consecutive rows and expanded to keys and values per head."""
        T, spec = self.ATTN_PREFILL_MIN_ROWS, s.shared_keys()
        n = self.latent_rows(s, long)
        lat, rot, exp = self._latent_scratch(n, s)
        opts = AttnOptions.of(spec)
        _lib.call("ps_latent_gather", ptr(kv.k), c_int(s.kv_rank), c_int(s.rot), ptr(st.block_table), c_int(st.max_blocks),
                  c_int(st.sc.page_tokens), c_int(st.num_pages), ptr(b.seq_desc), c_int(b.n_seqs), c_int(T), ctypes.byref(opts), c_int(n),
                  ptr(lat), ptr(rot), ptr(st.status))
        N = s.ukv.shape[0]
        _lib.call("ps_gemm_bf16_tc", ptr(lat), c_int(s.kv_rank), ptr(s.ukv), c_int(s.kv_rank), c_int(n), c_int(N), c_int(s.kv_rank),
                  c_int(EPI_STORE), ptr(None), c_int(0), ptr(exp), c_int(N), c_int(0), ptr(self.status))
        self.launches += 2
        self._latent_turn(q, s.dim + s.rot, s.dim, q, s.dim + s.rot, s.dim, s, b)
        self._latent_prefill(q, s, b, st, gate, out, rot, exp, long)

    def _latent_prefill(self, q, s: LatentSpec, b: StepBatch, st: ModelState, gate, out, rot, exp, long) -> None:
        """Attention of turned queries over expanded keys and values."""
        T, g, opts = self.ATTN_PREFILL_MIN_ROWS, gate[:, s.gate_off:], AttnOptions.of(s.shared_keys())
        _lib.call("ps_latent_prefill", ptr(q), c_int(q.shape[0]), ptr(exp), ptr(rot), c_int(rot.numel() // s.rot), ptr(b.seq_desc), c_int(b.n_seqs),
                  c_int(max(len(sq.token_ids) for sq in long)), c_int(T), c_int(s.heads), c_int(s.dim), c_int(s.rot), c_int(s.vdim),
                  c_float(s.scale), ctypes.byref(opts), ptr(g), c_int(g.stride(0)), c_int(s.vdim), c_int(0), ptr(out), ptr(st.status))
        self.launches += 1

    @staticmethod
    def latent_rows(s: LatentSpec, long) -> int:
        """Gathered rows of the step's long sequences: what their rows see, in whole tiles."""
        tile, spec = int(_lib.lib().ps_latent_tile()), s.shared_keys()
        return sum(-(-(sq.pos_start + len(sq.token_ids) - spec.first_visible(sq.pos_start) // tile * tile) // tile) * tile for sq in long)

    def _latent_scratch(self, n: int, s: LatentSpec):
        """bf16 scratch of the expanded form (latents, rotated parts, keys and values); one allocation that grows to the largest step seen."""
        sizes = [n * s.kv_rank, n * s.rot, n * s.ukv.shape[0]]
        t = getattr(self, "_latent_buf", None)
        if t is None or t.numel() < sum(sizes):
            t = self._latent_buf = torch.empty(sum(sizes), dtype=torch.bfloat16, device=self.device)
        return torch.split(t[:sum(sizes)], sizes)

    # ------------------------------------------------------------------ gated linear attention
    def gla(self, proj: torch.Tensor, g: GlaSpec, b: StepBatch, gs: GdnLayerState, st: ModelState) -> torch.Tensor:
        """Sequences with many rows in the step take the chunked kernels, the others the row-sequential one."""
        rows, f32 = proj.shape[0], self.act_dtype == torch.float32
        out = self.buf(f"gla_o{g.heads}x{g.dv}", rows, g.heads * g.dv, self.act_dtype)
        n_seqs = b.max_seqs if b.graph_static else b.n_seqs
        T = self.GDN_CHUNKED_MIN_ROWS
        L = _lib.lib()
        chunk_ok = not f32 and not b.graph_static and bool(L.ps_gla_chunked_ok(c_int(g.dk), c_int(g.dv), c_int(g.rank)))
        seq_rows = [len(sq.token_ids) for sq in b.seqs] if chunk_ok else []
        long = [n for n in seq_rows if n > T]

        def call(chunked: int, limit: int, blocks: int, scratch) -> None:
            _lib.call("ps_gla", c_int(chunked), ptr(proj), c_int(proj.stride(0)), c_int(1 if f32 else 0), c_int(g.heads), c_int(g.dk),
                      c_int(g.dv), c_int(g.dv_true), c_int(g.q_off), c_int(max(g.k_off, 0)), c_int(g.v_off), c_int(g.g_off), c_int(g.a_off),
                      c_int(g.rank), c_float(g.q_scale), c_float(g.inv_tau), c_float(g.eps), ptr(g.a2), ptr(g.a2_bias), ptr(g.norm_w),
                      ptr(g.lower), ptr(gs.rec), ptr(b.seq_desc), c_int(n_seqs), c_int(limit), ptr(out), c_int(blocks), *[ptr(t) for t in scratch])
        if long:
            C = int(L.ps_gla_block_rows())
            blocks = sum(-(-n // C) for n in long)
            call(1, T, blocks, self._gla_scratch(blocks, g.heads, C, g.dk, g.dv))
            self.launches += 3
        if not long or len(long) < len(seq_rows):
            call(0, T if long else 0, 0, (None,) * 4)
            self.launches += 1
        return out

    def _gla_scratch(self, blocks: int, H: int, C: int, dk: int, dv: int):
        """fp32 scratch of the chunked linear attention (decayed queries, A v, block states, block decays); one allocation that
        grows to the largest step seen."""
        sizes = [blocks * H * C * dk, blocks * H * C * dv, blocks * H * dk * dv, blocks * H * dk]
        t = getattr(self, "_gla_buf", None)
        if t is None or t.numel() < sum(sizes):
            t = self._gla_buf = torch.empty(sum(sizes), dtype=torch.float32, device=self.device)
        return torch.split(t[:sum(sizes)], sizes)

    # ------------------------------------------------------------------ delta rule with a decay per channel
    def delta(self, proj: torch.Tensor, d: DeltaSpec, b: StepBatch, gs: GdnLayerState, st: ModelState,
              history: Optional[torch.Tensor]) -> torch.Tensor:
        """ops/specs.py: DeltaSpec.  ``history``: the layer's convolution rows in the state."""
        rows, f32 = proj.shape[0], self.act_dtype == torch.float32
        for t in (proj, d.conv, d.a2, d.g2):
            if t.dtype != self.act_dtype:
                raise ValueError("projection rows, convolution and low-rank weights have the engine's type")
        out = self.buf(f"delta_o{d.heads}x{d.dv}", rows, d.heads * d.dv, self.act_dtype)
        n_seqs = b.max_seqs if b.graph_static else b.n_seqs
        args = (c_int(d.heads), c_int(d.kv_heads), c_int(d.dk), c_int(d.dv), c_int(d.dk_true), c_int(d.dv_true), c_int(d.q_off), c_int(d.b_off),
                c_int(d.a_off), c_int(d.g_off), c_int(d.a2.shape[1]), c_int(d.g2.shape[1]), c_int(d.taps), c_float(d.eps), ptr(d.conv), ptr(d.a2),
                ptr(d.dt_bias), ptr(d.rate), ptr(d.g2), ptr(d.norm_w), ptr(history), ptr(gs.rec), ptr(b.seq_desc), c_int(n_seqs), ptr(out))
        T, L = self.GDN_CHUNKED_MIN_ROWS, _lib.lib()
        chunk_ok = (not f32 and not b.graph_static
                    and bool(L.ps_delta_chunked_ok(c_int(d.dk), c_int(d.dv), c_int(d.a2.shape[1]), c_int(d.g2.shape[1]))))
        seq_rows = [len(sq.token_ids) for sq in b.seqs] if chunk_ok else []
        long = [n for n in seq_rows if n > T]
        if long:
            C = int(L.ps_delta_block_rows())
            blocks = sum(-(-n // C) for n in long)
            _lib.call("ps_delta_chunked", ptr(proj), c_int(proj.stride(0)), *args, c_int(T), c_int(blocks),
                      *[ptr(t) for t in self._delta_scratch(blocks, rows, C, d)], ptr(self.status))
            self.launches += 3
        if not long or len(long) < len(seq_rows):
            _lib.call("ps_delta_rows", ptr(proj), c_int(proj.stride(0)), c_int(1 if f32 else 0), *args, c_int(T if long else 0))
            self.launches += 1
        return out

    def _delta_scratch(self, blocks: int, rows: int, C: int, d: DeltaSpec):
        """Scratch of the chunked delta rule (its matrices as bf16 pairs with the decays, U, outputs before the head norm); one
        allocation that grows to the largest step seen."""
        L = _lib.lib()
        L.ps_delta_mats.restype = ctypes.c_longlong
        n = blocks * d.heads
        sizes = [n * int(L.ps_delta_mats(c_int(d.dk))) // 4, n * C * d.dv, rows * d.heads * d.dv]
        t = getattr(self, "_delta_buf", None)
        if t is None or t.numel() < sum(sizes):
            t = self._delta_buf = torch.empty(sum(sizes), dtype=torch.float32, device=self.device)
        return torch.split(t[:sum(sizes)], sizes)
