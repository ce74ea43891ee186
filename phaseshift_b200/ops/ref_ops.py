"""Reference op set in plain PyTorch (fp32, any device): the engine's correctness backend.

It implements exactly the same op contract as :class:`CudaOps` (paged KV through block tables, ring
conv history, per-slot recurrent state, batch descriptors) with straightforward tensor code, the role
the reference gives its single correctness mega-kernel
(src/phaseshift/models/qwen35/kernels/correctness/model_dispatch_correctness.hip:59): it is the
bit-reference for end-to-end token exactness on CPU and lets scheduler, batcher, prefix cache,
speculative decoding and tensor-parallel logic be tested without a GPU.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from .trace import OpTrace
import torch.nn.functional as F

from ..models.qwen35.weights import AttnW, GdnW, LinearW
from ..runtime.batch import StepBatch
from ..runtime.state import GdnLayerState, KVLayer, ModelState
from ..utils.sampling import sample_row_host
from .specs import AttnSpec, DeltaSpec, ExpertSum, GatedNorm, GlaSpec, HeadsSpec, LatentSpec, MoeSpec, Pending, Routed, StreamWrite, clamped_gate


class RefOps(OpTrace):
    act_dtype = torch.float32
    name = "ref"

    def __init__(self, cfg, device, act_quant: bool = False, **_):
        """``act_quant``: quantise the input of every block-quantised projection to the weights' block format
        (quant/act_quant.py), the arithmetic of the CUDA tensor-core layout; off = bf16/fp32 activations, the
        arithmetic of the streaming layout."""
        self.cfg, self.device = cfg, device
        self.act_quant = act_quant
        half = getattr(cfg, "rotary_dim", 0) // 2
        self.inv_freq = getattr(cfg, "rope_theta", 1.0) ** (-torch.arange(half, dtype=torch.float64) * 2.0 / max(1, 2 * half))
        self.launches = 0
        self.exact_rows = False

    def _dense(self, W: LinearW) -> torch.Tensor:
        return W.dense().to(self.device)

    def embed(self, b: StepBatch, rows: int, table: LinearW, status, ssq_out=None) -> torch.Tensor:
        return self._dense(table)[b.ids[:rows].long()]

    def linear(self, x, W: LinearW, *, name: str, norm_w=None, eps: float = 0.0, residual=None, swiglu=False,
               reglu=False, geglu=False, gelu=False, out_f32=False, out=None, ssq_in=None, ssq_out=None, prefetch=None, **_):
        x = x.float()
        if self.act_quant and W.fmt in ("nvfp4", "mxfp8"):
            # the tensor-core layout's arithmetic: quantise x (1 + w), apply the row factor 1/rms after the product
            from ..quant.act_quant import fake_quant
            inv = torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) if norm_w is not None else None
            if norm_w is not None:
                x = x * (1.0 + norm_w.float())
            y = fake_quant(x, W.fmt, W.act_scale) @ self._dense(W).T
            if inv is not None:
                y = y * inv
        else:
            if norm_w is not None:
                x = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (1.0 + norm_w.float())
            y = x @ self._dense(W).T
        if swiglu:
            y = F.silu(y[:, 0::2]) * y[:, 1::2]
        if reglu:
            y = F.relu(y[:, 0::2]) * y[:, 1::2]
        if geglu:
            y = F.gelu(y[:, 0::2], approximate="tanh") * y[:, 1::2]
        if gelu:
            y = F.gelu(y, approximate="tanh")
        if residual is not None:
            y = y + residual.float()
        if out is not None:
            out.copy_(y)
            return out
        return y

    def attn_prep(self, qkv, aw: AttnW, hq: int, hkv: int, b: StepBatch, kv: KVLayer, st: ModelState):
        cfg = self.cfg
        rows, D = qkv.shape[0], cfg.head_dim
        qg = qkv[:, :2 * hq * D].reshape(rows, hq, 2 * D)
        q = qg[..., :D]
        k = qkv[:, 2 * hq * D: 2 * hq * D + hkv * D].reshape(rows, hkv, D)
        v = qkv[:, 2 * hq * D + hkv * D:].reshape(rows, hkv, D)
        eps = cfg.rms_norm_eps
        q = q * torch.rsqrt(q.pow(2).mean(-1, keepdim=True) + eps) * (1.0 + aw.q_norm.float())
        k = k * torch.rsqrt(k.pow(2).mean(-1, keepdim=True) + eps) * (1.0 + aw.k_norm.float())
        pos = b.row_pos[:rows]
        half = cfg.rotary_dim // 2
        ang = pos.to(torch.float64)[:, None] * self.inv_freq.to(pos.device)[None, :]
        cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]

        def rope(t):
            t = t.clone()
            lo, hi = t[..., :half].double(), t[..., half:2 * half].double()
            t[..., :half] = (lo * cos - hi * sin).float()
            t[..., half:2 * half] = (hi * cos + lo * sin).float()
            return t
        q, k = rope(q), rope(k)
        pt = st.sc.page_tokens
        for r in range(rows):
            slot, p = int(b.row_slot[r]), int(pos[r])
            if slot < 0:
                continue
            page = int(st.block_table[slot, p // pt])
            if page < 0:
                raise RuntimeError("KV append into an unmapped page")
            kv.k[page, :, p % pt, :] = k[r]
            kv.v[page, :, p % pt, :] = v[r]
        return q.reshape(rows, hq * D)

    def paged_attention(self, q, qkv, hq: int, hkv: int, b: StepBatch, kv: KVLayer, st: ModelState,
                        max_visible: int):
        cfg = self.cfg
        rows, D = q.shape[0], cfg.head_dim
        G = hq // hkv
        pt = st.sc.page_tokens
        out = q.new_zeros(rows, hq, D)
        gate = qkv[:, :2 * hq * D].reshape(rows, hq, 2 * D)[..., D:]
        qh = q.reshape(rows, hq, D)
        for r in range(rows):
            slot, p = int(b.row_slot[r]), int(b.row_pos[r])
            if slot < 0:
                continue
            vis = p + 1
            nblk = -(-vis // pt)
            pages = st.block_table[slot, :nblk].long()
            K = kv.k[pages].permute(1, 0, 2, 3).reshape(hkv, nblk * pt, D)[:, :vis].float()
            V = kv.v[pages].permute(1, 0, 2, 3).reshape(hkv, nblk * pt, D)[:, :vis].float()
            K = K.repeat_interleave(G, 0)
            V = V.repeat_interleave(G, 0)
            s = torch.einsum("hd,htd->ht", qh[r].float(), K) * (D ** -0.5)
            pr = torch.softmax(s, -1)
            out[r] = torch.einsum("ht,htd->hd", pr, V)
        out = out * torch.sigmoid(gate.float())
        return out.reshape(rows, hq * D)

    def gdn(self, proj, gw: GdnW, hk: int, hv: int, b: StepBatch, gs: GdnLayerState, st: ModelState, log=None,
            to_alt: bool = False):
        cfg = self.cfg
        Dk, Dv = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        rows = proj.shape[0]
        qk = hk * Dk
        ring = st.sc.conv_ring
        rep = hv // hk
        out = proj.new_zeros(rows, hv * Dv)
        cw = gw.conv_w.float()
        A = -torch.exp(gw.A_log.float())
        z_off, b_off = 2 * qk + hv * Dv, 2 * qk + 2 * hv * Dv
        # per-head channel gather (matches the per-value-head private history layout)
        idx = []
        for h in range(hv):
            kh = h // rep
            idx.append(torch.cat([torch.arange(kh * Dk, (kh + 1) * Dk), torch.arange(qk + kh * Dk, qk + (kh + 1) * Dk),
                                  torch.arange(2 * qk + h * Dv, 2 * qk + (h + 1) * Dv)]))
        idx = torch.stack(idx).to(proj.device)          # [hv, 2Dk+Dv]
        for s in range(b.n_seqs):
            row0, n, slot, pos0 = (int(v) for v in b.seq_desc[s])
            if n <= 0:
                continue
            S = gs.rec[slot].clone()
            for i in range(n):
                row, pos = row0 + i, pos0 + i
                x = proj[row, :2 * qk + hv * Dv].float()
                xh = x[idx]                              # [hv, CH]
                wh = cw[idx]                             # [hv, CH, 4]
                y = wh[..., 3] * xh
                for j in (1, 2, 3):
                    if pos - j >= 0:
                        if i - j >= 0:
                            tap = proj[row - j, :2 * qk + hv * Dv].float()[idx]
                        else:
                            tap = gs.conv[slot, :, (pos - j) % ring, :].float()
                        y = y + wh[..., 3 - j] * tap
                gs.conv[slot, :, pos % ring, :] = xh.to(gs.conv.dtype)
                c = F.silu(y)
                q = c[:, :Dk]
                k = c[:, Dk:2 * Dk]
                v = c[:, 2 * Dk:]
                q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6) * (Dk ** -0.5)
                k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
                beta = torch.sigmoid(proj[row, b_off:b_off + hv].float())
                g = A * F.softplus(proj[row, b_off + hv:b_off + 2 * hv].float() + gw.dt_bias.float())
                d = torch.exp(g)
                S = S * d[:, None, None]
                kvm = torch.einsum("hkv,hk->hv", S, k)
                delta = (v - kvm) * beta[:, None]
                S = S + k[:, :, None] * delta[:, None, :]
                o = torch.einsum("hkv,hk->hv", S, q)
                if log is not None:
                    log[0][row] = k
                    log[1][row] = delta
                    log[2][row] = d
                o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + cfg.rms_norm_eps) * gw.norm_w.float()
                zz = proj[row, z_off:z_off + hv * Dv].float().reshape(hv, Dv)
                out[row] = (o * F.silu(zz)).reshape(-1)
            (gs.rec_alt if to_alt else gs.rec)[slot] = S
        return out

    def gdn_replay(self, gs: GdnLayerState, hv: int, seq_desc, n_seqs: int, log) -> None:
        for s in range(n_seqs):
            row0, n, slot, _ = (int(v) for v in seq_desc[s])
            S = gs.rec[slot]
            for i in range(n):
                S = S * log[2][row0 + i][:, None, None]
                S = S + log[0][row0 + i][:, :, None] * log[1][row0 + i][:, None, :]
            gs.rec[slot] = S

    def gather_rows(self, x, rows_idx, n: int, name: str, status):
        return x[rows_idx[:n].long()]

    def sample(self, logits, b: StepBatch, n: int, mask=None, mask_active=None, status=None):
        out = torch.empty(n, dtype=torch.int32)
        params = b._np_samp
        lg = logits.detach().float().cpu()
        for r in range(n):
            m = None
            if mask is not None and (mask_active is None or bool(mask_active[r])):
                m = mask[r].cpu()
            out[r] = sample_row_host(lg[r], params[r], m)
        return out.to(logits.device)

    def rmsnorm(self, x, w, eps: float, name: str, one_plus: bool = True, add=None, sum_out=None):
        x = x.float()
        if add is not None:
            x = x + add.float()
            if sum_out is not None:
                sum_out.copy_(x)
        ww = (1.0 + w.float()) if one_plus else w.float()
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * ww

    # ------------------------------------------------------------------ 32-bit residual stream
    def embed_f32(self, b: StepBatch, rows: int, table: torch.Tensor, status) -> torch.Tensor:
        return table[b.ids[:rows].long()].float()

    def residual_norm(self, x, pend: Optional[Pending], *, add=None, step=None, norm_w=None, eps: float, scale: float = 1.0,
                      width: int = 0, one: bool = False, name: str = ""):
        """x + the pending contribution (+ add + step), and the normed row padded to `width` columns (column W holds 1 when
        `one`).  Returns (new residual, normed row or None)."""
        unit = lambda t: t.float() * torch.rsqrt(t.float().pow(2).mean(-1, keepdim=True) + eps)
        if pend is not None:
            W = x.shape[1]                       # projections may carry padding columns behind the width
            if pend.experts is not None:
                y = self._expert_sum(pend.experts, W)
            elif pend.plain is not None:
                y = pend.plain[:, :W].float()
            else:
                y = unit(pend.branch_a[:, :W]) * pend.weight_a + unit(pend.branch_b[:, :W]) * pend.weight_b
            x = x + pend.coef * y
            if pend.bias is not None:
                x = x + pend.bias
        if add is not None:
            x = x + add
        if step is not None:
            x = x + step
        h = None
        if norm_w is not None:
            h = x.new_zeros(x.shape[0], width)
            h[:, :x.shape[1]] = unit(x) * norm_w * scale
            if one:
                h[:, x.shape[1]] = 1.0
        return x, h

    # ------------------------------------------------------------------ embedding of a token and the pair it ends
    def embed_pairs(self, b: StepBatch, rows: int, table, pairs, mul_prev: int, mul_cur: int, norm_w, eps: float, st: ModelState):
        """normed table[token] + pairs[(previous * mul_prev + token * mul_cur) mod buckets]; the last row of `pairs` belongs to
        the first token of a sequence.  Keeps every sequence's last token."""
        out = torch.empty(rows, table.shape[1])
        buckets = pairs.shape[0] - 1
        for s in range(b.n_seqs):
            row0, n, slot, pos0 = (int(v) for v in b.seq_desc[s])
            prev = int(st.last_token[slot])
            for r in range(row0, row0 + n):
                cur = int(b.ids[r])
                at = buckets if pos0 + r - row0 == 0 else (prev * mul_prev + cur * mul_cur) % buckets
                x = table[cur].float() + pairs[at].float()
                out[r] = x * torch.rsqrt(x.pow(2).mean() + eps) * norm_w
                prev = cur
            if n > 0:
                st.last_token[slot] = prev
        return out

    # ------------------------------------------------------------------ queries, keys and values of an attention
    def attn_heads(self, proj, s: HeadsSpec, b: StepBatch, kv: KVLayer, st: ModelState, history=None, saved=None):
        """Projection rows to queries (returned) and keys and values in their pages (ops/specs.py: HeadsSpec).  ``history``: the
        layer's convolution rows in the state; ``saved``: buffer of the values that later layers mix in."""
        rows, D, H, G = proj.shape[0], s.dim, s.heads, s.kv_heads
        x = proj[:, :s.channels].float()
        if s.conv is not None:
            x = self._short_conv(x, s, b, history)
        pos = b.row_pos[:rows].clamp(min=0)
        unit = lambda t, n: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / n + s.eps)
        q, k, v = x[:, :H * D], x[:, H * D:(H + G) * D], x[:, (H + G) * D:].reshape(rows, G, D)
        if s.q_norm is not None:
            q, k = unit(q, H * s.dim_true) * s.q_norm, unit(k, G * s.dim_true) * s.k_norm
        q, k = (self._turn_heads(t.reshape(rows, -1, D), pos, s) for t in (q, k))
        if s.unit:
            q, k = unit(q, s.dim_true), unit(k, s.dim_true)
        V = s.vdim_true
        if s.save:
            saved[:rows] = v[..., :V].reshape(rows, G * V)
        if s.mix is not None:
            v = v.clone()
            v[..., :V] = (1.0 - s.mix) * v[..., :V] + s.mix * saved[:rows].reshape(rows, G, V)
        for r in range(rows):
            at = self._page_of(b, r, st)
            if at is not None:
                kv.k[at[0], :, at[1]], kv.v[at[0], :, at[1]] = k[r], v[r]
        return q.reshape(rows, H * D)

    @staticmethod
    def _short_conv(x, s: HeadsSpec, b: StepBatch, history):
        y, back = torch.zeros_like(x), s.taps - 1
        for i in range(b.n_seqs):
            row0, n, slot, pos0 = (int(v) for v in b.seq_desc[i])
            if n <= 0:
                continue
            for r in range(n):
                for j in range(s.taps):
                    p = pos0 + r - j
                    if p >= 0:
                        u = x[row0 + r - j] if j <= r else history[slot, p % back]
                        y[row0 + r] += s.conv[back - j].float() * u
            for r in range(max(0, n - back), n):
                history[slot, (pos0 + r) % back] = x[row0 + r]
        return y

    @staticmethod
    def _turn_heads(t, pos, s: HeadsSpec):
        n = s.freq.numel()
        ang = pos.double()[:, None, None] * s.freq
        c, w = (ang.cos() * s.turn_size), (ang.sin() * s.turn_size)
        first, second = (slice(0, n), slice(n, 2 * n)) if s.halves else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
        u, v = t[..., first].double(), t[..., second].double()
        t = t.clone()
        t[..., first], t[..., second] = (u * c - v * w).float(), (v * c + u * w).float()
        return t

    def saved_values(self, rows: int, width: int):
        return torch.zeros(rows, width)

    # ------------------------------------------------------------------ mixture of experts
    def moe_route(self, logits, h, s: MoeSpec, b: StepBatch) -> Routed:
        """Router logits to every row's experts and weights (ops/specs.py: MoeSpec), and the rows of `h` sorted by expert."""
        rows, n = logits.shape[0], s.experts + s.identity
        z = logits[:, :n].float()
        score = torch.sigmoid(z) if s.sigmoid else torch.softmax(z, -1)
        choice = score if s.correction is None else score + s.correction
        best = choice.reshape(rows, s.groups, -1).topk(min(s.group_top, n // s.groups), -1).values.sum(-1).topk(s.keep, -1).indices
        open_ = torch.zeros(rows, s.groups, dtype=torch.bool).scatter_(1, best, True).repeat_interleave(n // s.groups, 1)
        ids = choice.masked_fill(~open_, -math.inf).topk(s.top, -1).indices
        weight = score.gather(1, ids)
        if s.renormalize:
            weight = weight / (weight.sum(-1, keepdim=True) + 1e-20)
        real = ids < s.experts
        order = sorted((int(ids[r, k]), r, k) for r in range(rows) for k in range(s.top) if real[r, k])
        index = torch.full((rows, s.top), -1, dtype=torch.int32)
        for at, (_, r, k) in enumerate(order):
            index[r, k] = at
        out = Routed(index, weight, (weight * ~real).sum(-1), h[[r for _, r, _ in order]])
        out.tiles = torch.tensor([e for e, _, _ in order], dtype=torch.long)
        return out

    def moe_experts(self, routed: Routed, s: MoeSpec):
        """Outputs of the sorted rows' experts, [sorted rows, n_out]."""
        K = s.gate_up.shape[1]
        out = torch.empty(routed.inputs.shape[0], s.n_out)
        for e in routed.tiles.unique().tolist():
            at = routed.tiles == e
            y = routed.inputs[at].float() @ s.gate_up.reshape(s.experts, 2 * s.ff, K)[e].float().T
            act = F.silu(y[:, 0::2]) * y[:, 1::2] if s.limit is None else clamped_gate(y[:, 0::2], y[:, 1::2], s.limit)
            out[at] = act @ s.down.reshape(s.experts, s.n_out, s.ff)[e].float().T
        return out

    @staticmethod
    def _weighted_experts(y, r: Routed, experts):
        for k in range(r.index.shape[1]):
            at = r.index[:, k].long()
            got = at >= 0
            y[got] = y[got] + r.weight[got, k][:, None] * experts[at[got], :y.shape[1]]
        return y

    def _expert_sum(self, e: ExpertSum, W: int):
        y = self._weighted_experts(e.routed.identity[:, None] * e.h[:, :W].float(), e.routed, e.y)
        return y if e.shared is None else y + e.shared[:, :W]

    # ------------------------------------------------------------------ norms behind the sublayers
    @staticmethod
    def _group_norm(x, w, eps: float, groups: int):
        p = x.reshape(x.shape[0], groups, -1)
        return (p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)).reshape(x.shape) * w

    def gated_norm(self, x, pend: Optional[GatedNorm], *, eps: float, groups: int, norm_w=None, width: int = 0, name: str = ""):
        """x + the sublayer's gated and normed result, and the next projection's input: the new residual itself, or with `norm_w` its
        norm in groups, padded to `width` columns.  Returns (new residual, rows or None)."""
        W = x.shape[1]
        if pend is not None:
            if pend.routed is not None:
                y = self._weighted_experts(torch.zeros_like(x), pend.routed, pend.experts)
            else:
                y = pend.scale_a * pend.a[:, :W].float()
                if pend.b is not None:
                    y = y + pend.scale_b * pend.b[:, :W].float()
            x = x + self._group_norm(y * torch.sigmoid(pend.gate[:, :W].float() + pend.gate_bias), pend.norm_w, eps, groups)
        if width == 0:
            return x, None
        h = x.new_zeros(x.shape[0], width)
        h[:, :W] = x if norm_w is None else self._group_norm(x, norm_w, eps, groups)
        return x, h

    def soft_limit(self, logits, cap: float):
        """cap * tanh(logits / cap), in place."""
        return logits.div_(cap).tanh_().mul_(cap)

    # ------------------------------------------------------------------ parallel residual streams
    def stream_norm(self, x, pend: Optional[StreamWrite], *, read=None, norm_w=None, eps: float, width: int = 0, name: str = "",
                    last: bool = False):
        """x [rows, streams, W]: write what is pending into all streams, then read the next sublayer's input from them and norm
        it, padded to `width` columns.  Returns (new streams, normed row or None)."""
        W = x.shape[2]
        if pend is not None:
            x = torch.einsum("st,rsw->rtw", pend.mix, x) + pend.out[:, None] * pend.y[:, None, :W].float()
        h = None
        if norm_w is not None:
            u = torch.einsum("s,rsw->rw", read, x)
            h = x.new_zeros(x.shape[0], width)
            h[:, :W] = u * torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps) * norm_w
        return x, h

    # ------------------------------------------------------------------ attention without rotation over paged keys
    def _page_of(self, b: StepBatch, r: int, st: ModelState):
        """(page, offset) of row r's position, or None for a padding row."""
        slot, p, pt = int(b.row_slot[r]), int(b.row_pos[r]), st.sc.page_tokens
        if slot < 0:
            return None
        page = int(st.block_table[slot, p // pt])
        if page < 0:
            raise RuntimeError("KV append into an unmapped page")
        return page, p % pt

    def attn_append(self, proj, spec: AttnSpec, b: StepBatch, kv: Optional[KVLayer], st: ModelState):
        """proj rows start with [q heads | k heads (| v heads)]: keys and values go to their pages, the queries are returned.
        ``kv`` None: the layer has no keys of its own."""
        rows, D, G = proj.shape[0], spec.dim, spec.kv_heads
        nq, nk = spec.heads * D, spec.kv_heads * D
        for r in range(rows if kv is not None else 0):
            at = self._page_of(b, r, st)
            if at is None:
                continue
            kv.k[at[0], :, at[1], :] = proj[r, nq:nq + nk].reshape(G, D)
            if kv.v is not kv.k:
                kv.v[at[0], :, at[1], :] = proj[r, nq + nk:nq + 2 * nk].reshape(G, D)
        return proj[:, :nq]

    def attention(self, q, spec: AttnSpec, b: StepBatch, kv: KVLayer, st: ModelState, max_visible: int, gate=None):
        rows, D, H = q.shape[0], spec.dim, spec.heads
        pt = st.sc.page_tokens
        out = q.new_zeros(rows, H, D)
        qh = q.reshape(rows, H, D)
        for r in range(rows):
            slot, p = int(b.row_slot[r]), int(b.row_pos[r])
            if slot < 0:
                continue
            tok = spec.visible(p)
            pages = st.block_table[slot, tok // pt].long()
            K = kv.k[pages, :, tok % pt].float().repeat_interleave(H // spec.kv_heads, 1)
            V = kv.v[pages, :, tok % pt].float().repeat_interleave(H // spec.kv_heads, 1)
            s = torch.einsum("hd,thd->ht", qh[r].float(), K) * spec.scale
            if spec.temp_coef != 0.0:
                s = s * (1.0 + spec.temp_coef * math.log(math.floor((p + 1) / spec.temp_every) + 1))
            if spec.bias is not None:
                s = s + spec.bias[:, (p - tok).clamp(max=spec.bias.shape[1] - 1)]
            if spec.sink is not None:
                pr = torch.softmax(torch.cat([s, spec.sink[:, None]], 1), -1)[:, :-1]
            else:
                pr = torch.softmax(s, -1)
            out[r] = torch.einsum("ht,thd->hd", pr, V)
        gate = spec.gate if gate is None else gate
        if gate is not None:
            cols = spec.gate_offset + torch.arange(H)[:, None] * spec.gate_head_stride
            out = out * torch.sigmoid(gate[:, cols if spec.gate_per_head else cols + torch.arange(D)].float())
        return out.reshape(rows, H * D)

    # ------------------------------------------------------------------ latent attention
    @staticmethod
    def _turn_pairs(t, pos, inv_freq):
        """Neighbouring elements of the first 2 * len(inv_freq) columns of t [rows, ..., R] turn by pos * inv_freq."""
        n = 2 * inv_freq.numel()
        ang = (pos.double()[:, None] * inv_freq).reshape((-1,) + (1,) * (t.dim() - 2) + (n // 2,))
        u, v = t[..., 0:n:2].double(), t[..., 1:n:2].double()
        t = t.clone()
        t[..., 0:n:2], t[..., 1:n:2] = (u * ang.cos() - v * ang.sin()).float(), (v * ang.cos() + u * ang.sin()).float()
        return t

    def latent_down(self, proj, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState):
        """proj rows are [query latent | latent | rotated key part | ...]: the latent and the turned key part go to their page,
        the normed query latent is returned."""
        unit = lambda t, true: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / true + s.eps)
        p = proj.float()
        c = unit(p[:, s.c_off:s.c_off + s.kv_rank], s.kv_rank_true) * s.kv_norm
        r = self._turn_pairs(p[:, s.c_off + s.kv_rank:s.c_off + s.row], b.row_pos[:proj.shape[0]], s.inv_freq)
        for i in range(proj.shape[0]):
            at = self._page_of(b, i, st)
            if at is not None:
                kv.k[at[0], 0, at[1]] = torch.cat([c[i], r[i]])
        return unit(p[:, :s.q_rank], s.q_rank_true) * s.q_norm

    def latent_attention(self, q, s: LatentSpec, b: StepBatch, kv: KVLayer, st: ModelState, gate):
        rows, H = q.shape[0], s.heads
        qh = q.float().reshape(rows, H, s.dim + s.rot)
        into = torch.einsum("rhd,hcd->rhc", qh[..., :s.dim], s.uk_t.float().reshape(H, s.kv_rank, s.dim))
        qe = torch.cat([into, self._turn_pairs(qh[..., s.dim:], b.row_pos[:rows], s.inv_freq)], -1)
        o = self.attention(qe.reshape(rows, -1), s.shared_keys(), b, kv, st, b.max_visible_launch).reshape(rows, H, s.row)[..., :s.kv_rank]
        o = torch.einsum("rhc,hvc->rhv", o, s.uv.float().reshape(H, s.vdim, s.kv_rank)).reshape(rows, H * s.vdim)
        return o * torch.sigmoid(gate[:, s.gate_off:s.gate_off + H * s.vdim].float())

    # ------------------------------------------------------------------ gated linear attention
    def gla(self, proj, g: GlaSpec, b: StepBatch, gs: GdnLayerState, st: ModelState):
        H, dk, dv = g.heads, g.dk, g.dv
        out = proj.new_zeros(proj.shape[0], H * dv)
        p = proj.float()
        q = p[:, g.q_off:g.q_off + H * dk].reshape(-1, H, dk)
        if g.lower is not None:
            z = p[:, g.a_off:g.a_off + H * dk] + g.a2_bias
            k = ((1.0 - g.lower) * torch.sigmoid(-z)).reshape(-1, H, dk)
            alpha, q = 1.0 - k, F.silu(q)
        else:
            z = p[:, g.a_off:g.a_off + g.rank] @ g.a2.float().T + g.a2_bias
            alpha = torch.exp(F.logsigmoid(z) * g.inv_tau).reshape(-1, H, dk)
            k = p[:, g.k_off:g.k_off + H * dk].reshape(-1, H, dk)
        q = q * g.q_scale
        v = p[:, g.v_off:g.v_off + H * dv].reshape(-1, H, dv)
        gate = F.silu(p[:, g.g_off:g.g_off + H * dv]) if g.g_off >= 0 else p.new_ones(p.shape[0], H * dv)
        for s in range(b.n_seqs):
            row0, n, slot, _ = (int(t) for t in b.seq_desc[s])
            S = gs.rec[slot]
            for row in range(row0, row0 + n):
                S = S * alpha[row][:, :, None] + k[row][:, :, None] * v[row][:, None, :]
                o = torch.einsum("hkv,hk->hv", S, q[row])
                o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / g.dv_true + g.eps) * g.norm_w
                out[row] = o.reshape(-1) * gate[row]
            if n > 0:
                gs.rec[slot] = S
        return out

    # ------------------------------------------------------------------ delta rule with a decay per channel
    def delta(self, proj, d: DeltaSpec, b: StepBatch, gs: GdnLayerState, st: ModelState, history):
        H, G, dk, dv, taps = d.heads, d.kv_heads, d.dk, d.dv, d.taps
        p, out = proj.float(), proj.new_zeros(proj.shape[0], H * dv)
        head = torch.arange(H)[:, None]
        # every value head's own channels: columns of the projection, and of the convolution
        cols = torch.cat([d.q_off + head // (H // G) * dk + torch.arange(dk), d.k_off + head // (H // G) * dk + torch.arange(dk),
                          d.v_off + head * dv + torch.arange(dv)], 1)
        w = d.conv.float()[:, cols - d.q_off]                     # [taps, heads, 2 dk + dv]
        g = torch.exp(-d.rate[:, None] * F.softplus(p[:, d.a_off:d.a_off + d.a2.shape[1]] @ d.a2.float().T + d.dt_bias).reshape(-1, H, dk))
        beta = torch.sigmoid(p[:, d.b_off:d.b_off + H])
        gate = torch.sigmoid(p[:, d.g_off:d.g_off + d.g2.shape[1]] @ d.g2.float().T)
        for s in range(b.n_seqs):
            row0, n, slot, pos0 = (int(t) for t in b.seq_desc[s])
            if n <= 0:
                continue
            S = gs.rec[slot]
            hist = None if history is None else history[slot].reshape(taps - 1, H, 2 * dk + dv)
            for r in range(n):
                x = torch.zeros(H, 2 * dk + dv)
                for j in range(min(taps, pos0 + r + 1)):
                    x = x + w[taps - 1 - j] * (p[row0 + r - j][cols] if j <= r else hist[(pos0 + r - j) % (taps - 1)].float())
                x = F.silu(x)
                unit = lambda t: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
                q, k, v = unit(x[:, :dk]) * d.dk_true ** -0.5, unit(x[:, dk:2 * dk]), x[:, 2 * dk:]
                S = S * g[row0 + r][:, :, None]
                u = beta[row0 + r][:, None] * (v - torch.einsum("hkv,hk->hv", S, k))
                S = S + k[:, :, None] * u[:, None, :]
                o = torch.einsum("hkv,hk->hv", S, q)
                o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / d.dv_true + d.eps) * d.norm_w
                out[row0 + r] = o.reshape(-1) * gate[row0 + r]
            gs.rec[slot] = S
            for r in range(max(0, n - taps + 1), n):
                hist[(pos0 + r) % (taps - 1)] = proj[row0 + r][cols]
        return out
