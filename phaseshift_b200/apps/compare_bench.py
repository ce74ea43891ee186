"""Throughput of a model family beside the closest other one at equal size (`bench.py --compare gebuzen`: the hybrid decoder;
`--compare luvutar`: Gebuzen; `--compare fudulix`: Luvutar; `--compare rotutar`: Gebuzen, with Fudulix for the mixtures and the hybrid
decoder for the delta rule): prefill and decode of a stack of layers of real-model shapes with random bf16 weights, and the mixers'
kernels alone against their rooflines.

Every kernel row gives its time, the algorithmic bytes and FLOPs of one launch group, and the fraction of the roofline
max(bytes / measured copy bandwidth, FLOPs / measured bf16 throughput) it reaches.  Kernel timings flush L2 between samples.
"""
from __future__ import annotations

import statistics
from typing import Dict, List

import torch

from ..models import registry
from ..runtime.batch import SeqRows, StepBatch
from ..runtime.engine import Engine
from ..runtime.state import StateConfig


def luvutar_pairs(layers: int) -> List[tuple]:
    """(label, Luvutar configuration, Gebuzen configuration) of equal width, attention heads, feed-forward weights and depth."""
    from ..models.gebuzen.config import gebuzen_27b_config, gebuzen_4b_config
    from ..models.luvutar.config import BiasedAttention, LatentAttention, Layer, luvutar_27b_config, luvutar_4b_config

    def cut(cfg):
        cfg.layers = cfg.layers[:layers]
        return cfg

    def narrow(m):
        """Half the head size, twice the heads; a latent half as wide."""
        if isinstance(m, LatentAttention):
            return LatentAttention(40, 64, 32, 64, 768, 256, 96 ** -0.5, m.rot_base, m.window)
        return BiasedAttention(32, 8, 128, 128, 128 ** -0.5, m.bias_max, m.temp_coef, m.temp_every, m.kv_from)

    small = cut(luvutar_4b_config(name="luvutar-4b-d128"))
    small.layers = [Layer(narrow(L.mixer), L.ff) for L in small.layers]
    return [("4b", cut(luvutar_4b_config()), cut(gebuzen_4b_config())), ("4b, attention heads of 128, latents of 256", small, None),
            ("27b", cut(luvutar_27b_config()), cut(gebuzen_27b_config()))]


def fudulix_pairs(layers: int) -> List[tuple]:
    """(label, Fudulix configuration, Luvutar configuration) of equal width, attention heads, active feed-forward weights and depth."""
    from ..models.fudulix.config import ConvAttention, Layer, Mixture, UnitAttention, fudulix_27b_config, fudulix_4b_config
    from ..models.luvutar.config import luvutar_27b_config, luvutar_4b_config

    def cut(cfg):
        cfg.layers = cfg.layers[:layers]
        return cfg

    def narrow(L):
        """Half the head size, twice the heads; half-size experts, twice as many."""
        m, c = L.mixer, L.mlp
        common = (32, 8, 128, 128, 128 ** -0.5, m.window, m.rot_base, m.rot_dims // 2, m.v_mix, m.scaling)
        mixer = ConvAttention(*common, m.keep_first, m.taps) if isinstance(m, ConvAttention) else UnitAttention(*common)
        return Layer(mixer, Mixture(512, 124, 16, 8, 4, 4, 1024) if isinstance(c, Mixture) else c)

    small = cut(fudulix_4b_config(name="fudulix-4b-d128"))
    small.layers = [narrow(L) for L in small.layers]
    return [("4b", cut(fudulix_4b_config()), cut(luvutar_4b_config())), ("4b, attention heads of 128, experts of 512", small, None),
            ("27b", cut(fudulix_27b_config()), cut(luvutar_27b_config()))]


def rotutar_pairs(layers: int) -> List[tuple]:
    """(label, Rotutar, Gebuzen, Fudulix and hybrid configurations) of equal width, attention heads, recurrent heads, active
    feed-forward weights and depth."""
    from ..models.fudulix.config import fudulix_27b_config, fudulix_4b_config
    from ..models.gebuzen.config import gebuzen_27b_config, gebuzen_4b_config
    from ..models.qwen35.config import qwen35_27b_config, qwen35_4b_config
    from ..models.rotutar.config import ForgetLinear, GatedDelta, Layer, Mixture, Parallel, WindowAttention, rotutar_27b_config, rotutar_4b_config

    def cut(cfg):
        cfg.layers = cfg.layers[:layers]
        return cfg

    def narrow(L):
        """Half the head sizes, twice the heads; half-size experts, twice as many."""
        m, c = L.mixer, L.mlp
        if isinstance(m, Parallel):
            l, r = m.left, m.right
            m = Parallel(WindowAttention(32, 8, 128, 128, 128 ** -0.5, l.window, l.rot_base, 32), m.left_scale,
                         GatedDelta(2 * r.heads, 2 * r.kv_heads, 64, 64, r.taps), m.right_scale)
        else:
            m = ForgetLinear(2 * m.heads, 64, 64)
        return Layer(m, Mixture(c.ff // 2, c.limit, 2 * c.experts, 2 * c.top, 2 * c.groups, 2 * c.keep) if isinstance(c, Mixture) else c)

    small = cut(rotutar_4b_config(name="rotutar-4b-narrow"))
    small.layers = [narrow(L) for L in small.layers]
    return [("4b", cut(rotutar_4b_config()), cut(gebuzen_4b_config()), cut(fudulix_4b_config()), qwen35_4b_config(num_hidden_layers=layers)),
            ("4b, attention heads of 128, recurrent heads of 64, experts of 576", small, None, None, None),
            ("27b", cut(rotutar_27b_config()), cut(gebuzen_27b_config()), cut(fudulix_27b_config()), qwen35_27b_config(num_hidden_layers=layers))]


def gebuzen_pairs(layers: int) -> List[tuple]:
    """(label, Gebuzen configuration, hybrid configuration) of equal width, head and feed-forward shapes and depth."""
    from ..models.gebuzen.config import ChunkAttention, ParallelLayer, gebuzen_27b_config, gebuzen_4b_config
    from ..models.qwen35.config import qwen35_27b_config, qwen35_4b_config

    def cut(cfg):
        cfg.layers = cfg.layers[:layers]
        return cfg

    small128 = cut(gebuzen_4b_config(name="gebuzen-4b-d128"))
    small128.layers = [ParallelLayer(ChunkAttention(32, 8, 128, 128 ** -0.5, 4096), L.right, L.ff) for L in small128.layers]
    return [("4b", cut(gebuzen_4b_config()), qwen35_4b_config(num_hidden_layers=layers)),
            ("4b, attention heads of 128", small128, None),
            ("27b", cut(gebuzen_27b_config()), qwen35_27b_config(num_hidden_layers=layers))]


def _events(fn, n: int) -> float:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


class _Flushed:
    """Median device time of `fn` over samples, a buffer larger than L2 written before each."""

    def __init__(self, device):
        self.buf = torch.empty(256 << 20, dtype=torch.uint8, device=device)

    def __call__(self, fn, samples: int = 15) -> float:
        for _ in range(3):
            fn()
        ts = []
        for _ in range(samples):
            self.buf.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(); fn(); e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1))
        return statistics.median(ts) * 1e3


def model_times(eng: Engine, prompt_tokens: int, steps: int, warmup: int, batch: int) -> Dict[str, float]:
    """Prefill of one prompt, its continuation by as many tokens, and graph-replayed decode steps of 1 and `batch` rows."""
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, eng.cfg.vocab_size, (2 * prompt_tokens,), generator=g).tolist()
    out: Dict[str, float] = {}
    first, second = [], []
    for i in range(warmup + 3):
        s = eng.open_sequence()
        for store, part in ((first, ids[:prompt_tokens]), (second, ids[prompt_tokens:])):
            t = _events(lambda: eng.step([SeqRows(s.slot, s.position, part, (len(part) - 1,))], [s]), 1)
            if i >= warmup:
                store.append(t)
        eng.close_sequence(s)
    out["prefill_ms"], out["prefill_cont_ms"] = statistics.median(first), statistics.median(second)
    for rows in (1, batch):
        seqs = [eng.open_sequence() for _ in range(rows)]
        for s in seqs:
            eng.step([SeqRows(s.slot, 0, ids[:prompt_tokens], (prompt_tokens - 1,))], [s])
        for _ in range(3):
            eng.step([SeqRows(s.slot, s.position, [7 + i], (0,)) for i, s in enumerate(seqs)], seqs)      # (rows that differ in their experts)
        from ..runtime.batch import resolve_row_bucket
        key = [k for k in eng.graphs if not isinstance(k, tuple) and eng.graph_key_bucket(k) == resolve_row_bucket(rows)][0]
        graph = eng.graphs[key]
        for _ in range(warmup):
            graph.replay()
        out[f"decode{rows}_ms"] = _events(graph.replay, steps)
        out[f"launches{rows}"] = eng.launches_per_graph[key]
        for s in seqs:
            eng.close_sequence(s)
    return out


def _batch(eng: Engine, seqs) -> tuple:
    """A step batch over fresh sequences [(first position, rows)] with mapped pages; returns (batch, open sequences)."""
    opened = []
    for p, n in seqs:
        s = eng.open_sequence()
        eng._reserve(s, p + n)
        opened.append(s)
    b = StepBatch(sum(n for _, n in seqs), len(seqs), eng.device)
    b.max_context = eng.sc.max_seq_len + 1
    b.fill([SeqRows(s.slot, p, [0] * n) for s, (p, n) in zip(opened, seqs)])
    b.upload()
    return b, opened


def kernel_times(eng: Engine, timer: _Flushed, peaks: dict, rows: int, context: int, batch: int) -> Dict[str, dict]:
    """The mixers' kernels alone.  `rows` = prefill rows, `context` = tokens before them / before a decoded row."""
    hbm, tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    ops, st, r = eng.ops, eng.state, eng.runner
    gz = eng.cfg.family == "gebuzen"
    res: Dict[str, dict] = {}

    def add(name, fn, nbytes, flops):
        us = timer(fn)
        floor = max(nbytes / hbm, flops / tc) * 1e6
        res[name] = {"us": round(us, 1), "gb": round(nbytes / 1e9, 4), "gflop": round(flops / 1e9, 2), "roofline_us": round(floor, 2),
                     "roofline_frac": round(floor / us, 4)}

    def rand(n, width, dtype=torch.bfloat16):
        return torch.randn(n, width, device=eng.device, dtype=torch.float32).to(dtype)

    shapes = [("prefill", [(0, rows)]), ("prefill after context", [(context, rows)]), ("decode 1", [(context, 1)]),
              (f"decode {batch}", [(context, 1)] * batch)]
    if gz:
        L, attn, gla = eng.w0, r.attn[0], r.gla[0]
        H, G, D, width = attn.heads, attn.kv_heads, attn.dim, L.in_proj.N
        rh, dk, dv = gla.heads, gla.dk, gla.dv
        kv_bytes_tok = G * D * 2
    else:
        cfg = eng.cfg
        la, lg = cfg.layer_types.index(1), cfg.layer_types.index(0)
        m, gm = r.w.layers[la].mixer, r.w.layers[lg].mixer
        H, G, D, width = r.hq, r.hkv, cfg.head_dim, m.qkv_proj.N
        rh, dk, dv = r.hv, cfg.linear_key_head_dim, cfg.linear_value_head_dim
        kv_bytes_tok = 2 * G * D * 2
    for name, seqs in shapes:
        b, opened = _batch(eng, seqs)
        n = b.n_rows
        vis = [list(range(p, p + k)) for p, k in seqs]
        chunk = attn.chunk if gz else 0
        pairs = sum((q % chunk + 1) if chunk else q + 1 for v in vis for q in v)
        kv_tok = sum((v[-1] + 1 - (v[0] // chunk * chunk if chunk else 0)) for v in vis)
        qkv = rand(n, width)
        if gz:
            q = ops.attn_append(qkv, attn, b, st.kv[0], st)
            fa = lambda: ops.attention(q, attn, b, st.kv[0], st, b.max_visible_launch)
        else:
            q = ops.attn_prep(qkv, m, H, G, b, st.kv[la], st)
            fa = lambda: ops.paged_attention(q, qkv, H, G, b, st.kv[la], st, b.max_visible_launch)
        io = n * H * D * 2 * (2 if gz else 3)                       # queries, outputs (and the hybrid's output gate)
        add("attention, " + name, fa, io + kv_tok * kv_bytes_tok, 4.0 * pairs * H * D)
        state = len(seqs) * rh * dk * dv * 4 * 2
        if gz:
            fg = lambda: ops.gla(qkv, gla, b, st.gdn[0], st)
            io = n * rh * (2 * dk + 3 * dv) * 2
            flops = n * rh * (4.0 * dk * dv + 64.0 * (dk + dv))     # state update and read, the block-local triangle
        else:
            proj = rand(n, gm.in_proj.N + gm.ba_proj.N)
            fg = lambda: ops.gdn(proj, gm, r.hk, rh, b, st.gdn[lg], st)
            io = n * (2 * r.hk * dk + 3 * rh * dv) * 2
            flops = n * rh * (6.0 * dk * dv + 64.0 * (2 * dk + dv))
        add("recurrence, " + name, fg, io + state, flops)
        if name in ("prefill", "decode 1"):
            W = eng.cfg.hidden_size
            if gz:
                from ..ops.specs import Pending
                x, a, c = rand(n, W, torch.float32), rand(n, W, torch.float32), rand(n, W, torch.float32)
                pend = Pending(0.5, a, L.left_out, c, L.right_out)
                add("norm, " + name, lambda: ops.residual_norm(x, pend, norm_w=L.norm2, eps=1e-6, width=L.gate_up.K, name="bench_h"),
                    n * W * (4 * 4 + 2), 0.0)
            else:
                x = rand(n, W)
                add("norm, " + name, lambda: ops.rmsnorm(x, r.w.layers[0].input_norm, 1e-6, "bench_h"), n * W * 4, 0.0)
            w = L.gate_up if gz else r.w.layers[0].gate_up
            xg = rand(n, w.K)
            kw = {"reglu": True} if gz else {"swiglu": True}
            add("gate_up, " + name, lambda: ops.linear(xg, w, name="bench_act", **kw), w.N * w.k_padded * 2 + n * (w.K + w.N // 2) * 2,
                2.0 * n * w.N * w.K)
        for s in opened:
            eng.close_sequence(s)
    return res


def luvutar_kernel_times(eng: Engine, timer: _Flushed, peaks: dict, rows: int, context: int, batch: int) -> Dict[str, dict]:
    """As `kernel_times`, for the parts of both mixers and the residual streams."""
    from ..ops.specs import LatentSpec, StreamWrite
    hbm, tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    ops, st, w = eng.ops, eng.state, eng.runner.w
    res: Dict[str, dict] = {}

    def add(name, fn, nbytes, flops):
        us = timer(fn)
        floor = max(nbytes / hbm, flops / tc) * 1e6
        res[name] = {"us": round(us, 1), "gb": round(nbytes / 1e9, 4), "gflop": round(flops / 1e9, 2), "roofline_us": round(floor, 2),
                     "roofline_frac": round(floor / us, 4)}

    def rand(n, width, dtype=torch.bfloat16):
        return torch.randn(n, width, device=eng.device, dtype=torch.float32).to(dtype)

    la = next(i for i, L in enumerate(w.layers) if isinstance(L.attn, LatentSpec))
    lb = next(i for i, L in enumerate(w.layers) if not isinstance(L.attn, LatentSpec))
    A, B = w.layers[la], w.layers[lb]
    s, f = A.attn, B.attn
    S, W = eng.cfg.streams, eng.cfg.hidden_size
    shapes = [("prefill", [(0, rows)]), ("prefill after context", [(context, rows)]), ("decode 1", [(context, 1)]),
              (f"decode {batch}", [(context, 1)] * batch)]
    for name, seqs in shapes:
        b, opened = _batch(eng, seqs)
        n = b.n_rows
        vis = [(p, k) for p, k in seqs]
        full = sum(q + 1 for p, k in vis for q in range(p, p + k))
        win = sum(min(q + 1, s.window) for p, k in vis for q in range(p, p + k))
        kv_full = sum(p + k for p, k in vis)
        kv_win = sum(p + k - max(0, p - s.window + 1) for p, k in vis)
        qkv = rand(n, B.in_proj.N)
        q = ops.attn_append(qkv, f, b, st.kv[lb], st)
        add("attention, " + name, lambda: ops.attention(q, f, b, st.kv[lb], st, b.max_visible_launch, gate=qkv),
            2 * n * f.heads * f.dim * 2 + kv_full * 2 * f.kv_heads * f.dim * 2, 4.0 * full * f.heads * f.dim)
        proj = rand(n, A.in_proj.N)
        add("latents, " + name, lambda: ops.latent_down(proj, s, b, st.kv[la], st), n * (2 * s.q_rank + 2 * s.row) * 2, 0.0)
        lq = rand(n, A.uq.N)
        H = s.heads
        io = n * H * (s.dim + s.rot + 2 * s.vdim) * 2
        if name.startswith("prefill"):
            # keys and values are products of the latents of every visible token
            flops = 2.0 * win * H * (s.dim + s.rot + s.vdim) + 2.0 * kv_win * s.ukv.numel()
            add("latent attention, " + name, lambda: ops.latent_attention(lq, s, b, st.kv[la], st, proj), io + kv_win * s.row * 2, flops)
            add("latent attention core, " + name, _prefill_core(ops, lq, s, b, st, st.kv[la], proj),
                io + kv_win * (H * (s.dim + s.vdim) + s.rot) * 2, 2.0 * win * H * (s.dim + s.rot + s.vdim))
        else:
            weights = (s.uk_t.numel() + s.uv.numel()) * 2
            add("latent attention, " + name, lambda: ops.latent_attention(lq, s, b, st.kv[la], st, proj), io + kv_win * s.row * 2 + weights,
                2.0 * win * H * (s.row + s.kv_rank) + 2.0 * n * weights / 2)
            qe = rand(n, H * s.row)
            add("latent attention core, " + name, lambda: ops._latent_decode(qe, s, s.shared_keys(), b, st.kv[la], st, b.row_pos),
                n * H * (s.row + s.kv_rank) * 2 + kv_win * s.row * 2, 2.0 * win * H * (s.row + s.kv_rank))
            add("queries into the latent space, " + name,
                lambda: ops._gemm_heads(lq, s.dim + s.rot, s.uk_t, H, s.kv_rank, s.dim, qe, s.row), s.uk_t.numel() * 2 + n * H * (s.dim + s.kv_rank) * 2,
                2.0 * n * s.uk_t.numel())
        if name != "prefill after context":
            x, y = rand(n, S * W, torch.float32).view(n, S, W), rand(n, W, torch.float32)
            hc = A.hc2
            pend = StreamWrite(A.hc1.mix, A.hc1.out, y)
            add("streams + norm, " + name, lambda: ops.stream_norm(x, pend, read=hc.read, norm_w=hc.norm, eps=1e-6, width=A.up.K, name="bench_h"),
                n * W * (8 * S + 4 + 2), 0.0)
            xg = rand(n, A.up.K)
            add("up, " + name, lambda: ops.linear(xg, A.up, name="bench_act", gelu=True),
                A.up.N * A.up.k_padded * 2 + n * (A.up.K + A.up.N) * 2, 2.0 * n * A.up.N * A.up.K)
        for o in opened:
            eng.close_sequence(o)
    return res


def fudulix_kernel_times(eng: Engine, timer: _Flushed, peaks: dict, rows: int, context: int, batch: int) -> Dict[str, dict]:
    """As `kernel_times`, for both mixers and both feed-forwards.  What a mixture moves and multiplies is counted from the rows its
    random router sends to every expert."""
    from ..models.fudulix.weights import MixtureW
    from ..ops.specs import ExpertSum, Pending
    hbm, tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    ops, st, w = eng.ops, eng.state, eng.runner.w
    res: Dict[str, dict] = {}

    def add(name, fn, nbytes, flops):
        us = timer(fn)
        floor = max(nbytes / hbm, flops / tc) * 1e6
        res[name] = {"us": round(us, 1), "gb": round(nbytes / 1e9, 4), "gflop": round(flops / 1e9, 2), "roofline_us": round(floor, 2),
                     "roofline_frac": round(floor / us, 4)}

    def rand(n, width, dtype=torch.bfloat16):
        return torch.randn(n, width, device=eng.device, dtype=torch.float32).to(dtype)

    W = eng.cfg.hidden_size
    lc = next(i for i, L in enumerate(w.layers) if L.heads.conv is not None)
    lu = next(i for i, L in enumerate(w.layers) if L.heads.conv is None)
    dense = next(L.mlp for L in w.layers if not isinstance(L.mlp, MixtureW))
    mix = next(L.mlp for L in w.layers if isinstance(L.mlp, MixtureW))
    m = mix.moe
    shapes = [("prefill", [(0, rows)]), ("prefill after context", [(context, rows)]), ("decode 1", [(context, 1)]),
              (f"decode {batch}", [(context, 1)] * batch)]
    for name, seqs in shapes:
        b, opened = _batch(eng, seqs)
        n = b.n_rows
        for i, kind in ((lu, "attention"), (lc, "attention_2")):
            L, f = w.layers[i], w.layers[i].attn
            seen = [[min(q + 1, f.window + min(f.keep_first, max(0, q + 1 - f.window))) for q in range(p, p + k)] for p, k in seqs]
            pairs, kv_tok = sum(map(sum, seen)), sum(min(p + k, s[0] + k - 1) for (p, k), s in zip(seqs, seen))
            proj = rand(n, L.in_proj.N)
            saved = ops.saved_values(n, eng.runner.saved_width)
            q = ops.attn_heads(proj, L.heads, b, st.kv[i], st, st.conv[i], saved)
            if name != "prefill after context":
                io = n * 2 * L.in_proj.N * 2 + 2 * n * eng.runner.saved_width + (L.heads.conv.numel() * 2 if L.heads.conv is not None else 0)
                add(f"heads of {kind}, {name}", lambda: ops.attn_heads(proj, L.heads, b, st.kv[i], st, st.conv[i], saved), io, 0.0)
            add(f"{kind}, {name}", lambda: ops.attention(q, f, b, st.kv[i], st, b.max_visible_launch),
                2 * n * f.heads * f.dim * 2 + kv_tok * 2 * f.kv_heads * f.dim * 2, 4.0 * pairs * f.heads * f.dim)
        if name != "prefill after context":
            x, y, h = rand(n, W, torch.float32), rand(n, W, torch.float32), rand(n, mix.router.K)
            L = w.layers[lu]
            add("residual + norm, " + name, lambda: ops.residual_norm(x, Pending(1.0, plain=y), norm_w=L.norm1, eps=1e-6, width=h.shape[1], name="bench_h"),
                n * W * (3 * 4 + 2), 0.0)
            xg = rand(n, dense.gate_up.K)
            gu = dense.gate_up
            add("gate_up, " + name, lambda: ops.linear(xg, gu, name="bench_act", geglu=True), gu.N * gu.k_padded * 2 + n * (gu.K + gu.N // 2) * 2,
                2.0 * n * gu.N * gu.K)
            add("router, " + name, lambda: ops.linear(h, mix.router, name="bench_z", out_f32=True),
                mix.router.N * mix.router.K * 2 + n * (mix.router.K * 2 + mix.router.N * 4), 2.0 * n * mix.router.N * mix.router.K)
            z = ops.linear(h, mix.router, name="bench_z", out_f32=True)
            r = ops.moe_route(z, h, m, b)
            R, used = int((r.index >= 0).sum()), len(set(r.tiles[1:1 + int(r.tiles[0, 0]), 0].tolist()))
            add("routing, " + name, lambda: ops.moe_route(z, h, m, b), n * (z.shape[1] * 4 + h.shape[1] * 2 + m.top * 8) + R * h.shape[1] * 2, 0.0)
            K = m.gate_up.shape[1]
            add("experts, " + name, lambda: ops.moe_experts(r, m),
                used * 3 * m.ff * K * 2 + R * (K * 2 + 2 * m.ff * 2 + m.n_out * 4), 2.0 * R * (2 * m.ff * K + m.n_out * m.ff))
            ye = ops.moe_experts(r, m)
            pend = Pending(1.0, experts=ExpertSum(r, ye, h, y))
            add("expert sum + norm, " + name, lambda: ops.residual_norm(x, pend, norm_w=L.norm1, eps=1e-6, width=h.shape[1], name="bench_h"),
                n * W * (3 * 4 + 2) + R * m.n_out * 4 + int((r.identity > 0).sum()) * W * 2, 0.0)
        for o in opened:
            eng.close_sequence(o)
    return res


def rotutar_kernel_times(eng: Engine, timer: _Flushed, peaks: dict, rows: int, context: int, batch: int) -> Dict[str, dict]:
    """As `kernel_times`, for the mixers, both feed-forwards and the norms behind them."""
    from ..models.rotutar.weights import DenseW, MixtureW, ParallelW
    from ..ops.specs import GatedNorm
    hbm, tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    ops, st, w = eng.ops, eng.state, eng.runner.w
    res: Dict[str, dict] = {}

    def add(name, fn, nbytes, flops):
        us = timer(fn)
        floor = max(nbytes / hbm, flops / tc) * 1e6
        res[name] = {"us": round(us, 1), "gb": round(nbytes / 1e9, 4), "gflop": round(flops / 1e9, 2), "roofline_us": round(floor, 2),
                     "roofline_frac": round(floor / us, 4)}

    def rand(n, width, dtype=torch.bfloat16):
        return torch.randn(n, width, device=eng.device, dtype=torch.float32).to(dtype)

    W, groups, kin = eng.cfg.hidden_size, eng.cfg.norm_groups, w.lm_head.K
    lp = next(i for i, L in enumerate(w.layers) if isinstance(L.mixer, ParallelW))
    lf = next(i for i, L in enumerate(w.layers) if not isinstance(L.mixer, ParallelW))
    P, F = w.layers[lp], w.layers[lf]
    dense = next(L.mlp for L in w.layers if isinstance(L.mlp, DenseW))
    mix = next(L.mlp for L in w.layers if isinstance(L.mlp, MixtureW))
    a, d, f, m = P.mixer.attn, P.mixer.delta, F.mixer.gla, mix.moe
    shapes = [("prefill", [(0, rows)]), ("prefill after context", [(context, rows)]), ("decode 1", [(context, 1)]),
              (f"decode {batch}", [(context, 1)] * batch)]
    for name, seqs in shapes:
        b, opened = _batch(eng, seqs)
        n = b.n_rows
        pairs = sum(min(q + 1, a.window) for p, k in seqs for q in range(p, p + k))
        kv_tok = sum(min(p + k, a.window + k - 1) for p, k in seqs)
        proj = rand(n, P.in_proj.N)
        q = ops.attn_heads(proj, P.mixer.heads, b, st.kv[lp], st)
        add("attention, " + name, lambda: ops.attention(q, a, b, st.kv[lp], st, b.max_visible_launch),
            2 * n * a.heads * a.dim * 2 + kv_tok * 2 * a.kv_heads * a.dim * 2, 4.0 * pairs * a.heads * a.dim)
        ra, rg = d.a2.shape[1], d.g2.shape[1]
        state = len(seqs) * d.heads * d.dk * d.dv * 4 * 2
        io = n * (2 * d.kv_heads * d.dk + 2 * d.heads * d.dv + d.heads + ra + rg) * 2 + (d.a2.numel() + d.g2.numel()) * 2
        flops = n * d.heads * (6.0 * d.dk * d.dv + 64.0 * (2 * d.dk + d.dv)) + 2.0 * n * (d.a2.numel() + d.g2.numel())
        add("delta rule, " + name, lambda: ops.delta(proj, d, b, st.gdn[lp], st, st.conv[lp]), io + state, flops)
        fproj = rand(n, F.in_proj.N)
        state = len(seqs) * f.heads * f.dk * f.dv * 4 * 2
        add("forget-gate linear attention, " + name, lambda: ops.gla(fproj, f, b, st.gdn[lf], st), n * f.heads * 2 * (f.dk + f.dv) * 2 + state,
            n * f.heads * (4.0 * f.dk * f.dv + 64.0 * (f.dk + f.dv)))
        if name != "prefill after context":
            h = rand(n, kin)
            add("heads, " + name, lambda: ops.attn_heads(proj, P.mixer.heads, b, st.kv[lp], st), n * 2 * P.mixer.heads.channels * 2, 0.0)
            for what, lw, kw in (("in_proj", P.in_proj, {}), ("gate_up", dense.gate_up, {"swiglu": True}), ("gate of the result", dense.gate, {}),
                                 ("router and gate", mix.router, {"out_f32": True})):
                cols = lw.N // 2 if kw.get("swiglu") else lw.N
                add(f"{what}, {name}", lambda: ops.linear(h, lw, name="bench_" + what, **kw),
                    lw.N * lw.k_padded * 2 + n * (lw.K * 2 + cols * (4 if kw.get("out_f32") else 2)), 2.0 * n * lw.N * lw.K)
            x, ya, yb = (rand(n, W, torch.float32) for _ in range(3))
            pend = GatedNorm(proj[:, P.gate_off:], P.gate1, P.norm1, ya, 0.7, yb, 0.7)
            add("gated norm, " + name, lambda: ops.gated_norm(x, pend, eps=1e-6, groups=groups, width=kin, name="bench_h"), n * W * (4 * 4 + 2 + 2), 0.0)
            z = ops.linear(h, mix.router, name="bench_z", out_f32=True)
            r = ops.moe_route(z, h, m, b)
            R, used = int((r.index >= 0).sum()), len(set(r.tiles[1:1 + int(r.tiles[0, 0]), 0].tolist()))
            add("routing, " + name, lambda: ops.moe_route(z, h, m, b), n * (m.experts * 4 + kin * 2 + m.top * 8) + R * kin * 2, 0.0)
            K = m.gate_up.shape[1]
            add("experts, " + name, lambda: ops.moe_experts(r, m), used * 3 * m.ff * K * 2 + R * (K * 2 + 2 * m.ff * 2 + m.n_out * 4),
                2.0 * R * (2 * m.ff * K + m.n_out * m.ff))
            ye = ops.moe_experts(r, m)
            pend2 = GatedNorm(z[:, mix.gate_off:], F.gate2, F.norm2, routed=r, experts=ye)
            add("gated norm of a mixture, " + name, lambda: ops.gated_norm(x, pend2, eps=1e-6, groups=groups, width=kin, name="bench_h"),
                n * W * (2 * 4 + 4 + 2) + R * m.n_out * 4, 0.0)
        if name.startswith("decode"):
            lg = rand(n, w.lm_head.N, torch.float32)
            add("soft limit, " + name, lambda: ops.soft_limit(lg, 30.0), n * w.lm_head.N * 8, 0.0)
        for o in opened:
            eng.close_sequence(o)
    return res


def _prefill_core(ops, q, s, b, st, kv, gate):
    """The attention over keys and values that one call of `latent_attention` has gathered and expanded."""
    out = ops.latent_attention(q, s, b, kv, st, gate)
    long = list(b.seqs)
    lat, rot, exp = ops._latent_scratch(ops.latent_rows(s, long), s)
    return lambda: ops._latent_prefill(q, s, b, st, gate, out, rot, exp, long)


def run(peaks: dict, layers: int = 16, prompt_tokens: int = 2048, steps: int = 50, warmup: int = 3, batch: int = 32, sampler=None,
        which: str = "gebuzen") -> dict:
    dev = torch.device("cuda:0")
    timer = _Flushed(dev)
    out = {"layers": layers, "prompt_tokens": prompt_tokens, "batch": batch, "sizes": {}}
    pairs, names = {"gebuzen": (gebuzen_pairs, ("gebuzen", "hybrid")), "luvutar": (luvutar_pairs, ("luvutar", "gebuzen")),
                    "fudulix": (fudulix_pairs, ("fudulix", "luvutar")), "rotutar": (rotutar_pairs, ("rotutar", "gebuzen", "fudulix", "hybrid"))}[which]
    kernels = {"luvutar": luvutar_kernel_times, "fudulix": fudulix_kernel_times, "rotutar": rotutar_kernel_times}
    for label, *cfgs in pairs(layers):
        row = out["sizes"][label] = {}
        for name, cfg in zip(names, cfgs):
            if cfg is None:
                continue
            with torch.no_grad():
                ew = registry.random_weights(cfg, dev, "bf16")
                eng = Engine(ew, dev, StateConfig(max_slots=batch, max_seq_len=2 * prompt_tokens + 64, page_tokens=16))
                if name == "gebuzen":
                    eng.w0 = ew.layers[0]
                if sampler is not None:
                    sampler.begin()
                t = model_times(eng, prompt_tokens, steps, warmup, batch)
                k = kernels.get(name, kernel_times)(eng, timer, peaks, prompt_tokens, prompt_tokens, batch)
            rd = ew.decode_read_bytes()
            row[name] = {**{a: round(v, 4) for a, v in t.items()},
                         "prefill_tok_s": round(prompt_tokens / t["prefill_ms"] * 1e3), "decode1_tok_s": round(1e3 / t["decode1_ms"], 1),
                         f"decode{batch}_tok_s": round(batch * 1e3 / t[f"decode{batch}_ms"]), "weights_gb": round(rd / 1e9, 3),
                         "decode1_hbm_frac": round(rd / (t["decode1_ms"] * 1e-3) / (peaks["hbm_gbs"] * 1e9), 4), "kernels": k}
            del eng, ew
            torch.cuda.empty_cache()
    return out
