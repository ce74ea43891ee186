"""Gebuzen forward over an op set: one call = one scheduled step over a mixed batch of rows.

The residual stream is 32-bit.  Every residual update is fused with the norm that follows it (``ops.residual_norm``): it adds
the pending contribution -- the two normed mixer branches, or the feed-forward's output -- and, at the start of a pass of the
looped range, the embedding output and the pass's step vector, and leaves the normed row for the next projection.  A layer is
eleven launches: norm, in_proj, append, attention (split + merge), linear attention, two output projections, norm, gate_up, down.
"""
from __future__ import annotations

from typing import Optional, Sequence

from ...ops.specs import AttnSpec, GlaSpec, Pending
from ..common import StepOutput
from .weights import GebuzenWeights, ParallelLayerW


class GebuzenRunner:
    def __init__(self, weights: GebuzenWeights, state, ops, tp=None):
        if tp is not None and tp.size > 1:
            raise ValueError("Gebuzen models run on one rank")
        self.w, self.state, self.ops, self.tp = weights, state, ops, None
        self.cfg = weights.cfg
        self.runs = self.cfg.runs()
        self.imatrix_collector = self.act_collector = None
        self.attn = [self._attn_spec(L) for L in weights.layers]
        self.gla = [self._gla_spec(L) for L in weights.layers]

    def _attn_spec(self, L: ParallelLayerW) -> AttnSpec:
        l = L.left
        return AttnSpec(l.heads, l.kv_heads, l.dim_padded, l.scale, chunk=l.chunk, sink=L.sink)

    def _gla_spec(self, L: ParallelLayerW) -> GlaSpec:
        l, r = L.left, L.right
        q = (l.heads + l.kv_heads) * l.dim_padded
        k = q + r.heads * r.dim_padded
        v = k + r.heads * r.dim_padded
        g = v + r.heads * r.vdim_padded
        a = g + r.heads * r.vdim_padded
        return GlaSpec(r.heads, r.dim_padded, r.vdim_padded, r.vdim, q, k, v, g, a, L.decay_rank, r.dim ** -0.5, 1.0 / r.tau,
                       self.cfg.norm_eps, L.a2, L.a2_bias, L.right_norm)

    def forward(self, b, rows: int, n_out: int, *, tap_layers: Sequence[int] = (), gdn_log=None, gdn_to_alt: bool = False,
                mask=None, mask_active=None, sample: bool = True, greedy_only: bool = False) -> StepOutput:
        """``tap_layers``: indices of layer runs whose residual stream (after everything the run adds) is returned in ``taps``.
        ``greedy_only``: as in the hybrid decoder's runner."""
        if gdn_log is not None or gdn_to_alt:
            raise ValueError("Gebuzen's recurrent state cannot be logged or redirected (no speculative decoding)")
        cfg, ops, st, w = self.cfg, self.ops, self.state, self.w
        eps, m = cfg.norm_eps, cfg.residual_mult
        with ops.range("embed"):
            x0 = ops.embed_f32(b, rows, w.embed, st.status)
        x = x0
        pend: Optional[Pending] = None
        taps = {}
        for j, run in enumerate(self.runs):
            L = w.layers[run.layer]
            add = x0 if run.opens_pass and run.pass_index > 0 else None
            step = w.step[run.pass_index] if run.opens_pass else None
            with ops.range("norm"):
                x, h = ops.residual_norm(x, pend, add=add, step=step, norm_w=L.norm1, eps=eps, width=L.in_proj.K, one=True, name="h_mix")
            with ops.range("mixer.in_proj"):
                proj = ops.linear(h, L.in_proj, name=f"mix_proj{L.in_proj.N}")
            attn, gla = self.attn[run.layer], self.gla[run.layer]
            with ops.range("attn.append"):
                q = ops.attn_append(proj, attn, b, st.kv[j], st)
            with ops.range("attn.core"):
                ctx = ops.attention(q, attn, b, st.kv[j], st, b.max_visible_launch)
            with ops.range("gla"):
                o = ops.gla(proj, gla, b, st.gdn[j], st)
            with ops.range("attn.o_proj"):
                left = ops.linear(ctx, L.left_o, name="mix_left", out_f32=True)
            with ops.range("gla.out_proj"):
                right = ops.linear(o, L.right_o, name="mix_right", out_f32=True)
            pend = Pending(0.5 * m, left, L.left_out, right, L.right_out)
            if L.gate_up is not None:
                with ops.range("norm"):
                    x, h = ops.residual_norm(x, pend, norm_w=L.norm2, eps=eps, width=L.gate_up.K, name="h_mlp")
                with ops.range("mlp.gate_up"):
                    act = ops.linear(h, L.gate_up, name=f"mlp_act{L.gate_up.N}", reglu=True)
                with ops.range("mlp.down"):
                    pend = Pending(m, plain=ops.linear(act, L.down, name="mlp_out", out_f32=True))
            if j in tap_layers:
                x, _ = ops.residual_norm(x, pend, eps=eps)
                pend = None
                taps[j] = x.clone()
        tokens = logits = hidden = None
        if n_out > 0:
            # the logit scale rides on the final norm's output: the head is linear
            with ops.range("norm"):
                x, h = ops.residual_norm(x, pend, norm_w=w.final_norm, eps=eps, scale=cfg.logit_scale, width=w.lm_head.K, name="h_final")
            hidden = h[:n_out] if b.identity_out else ops.gather_rows(h, b.out_rows, n_out, "out_hidden", st.status)
            if (greedy_only and sample and mask is None and w.lm_head.N == cfg.vocab_size and hasattr(ops, "can_fuse_argmax")
                    and ops.can_fuse_argmax(w.lm_head, n_out)):
                with ops.range("head.lm_head"):
                    tokens = ops.linear_argmax(hidden, w.lm_head)
                return StepOutput(tokens, None, hidden, taps)
            with ops.range("head.lm_head"):
                logits = ops.linear(hidden, w.lm_head, name="logits", out_f32=True)[:, :cfg.vocab_size]
            if sample:
                with ops.range("head.sample"):
                    tokens = ops.sample(logits, b, n_out, mask=mask, mask_active=mask_active, status=st.status)
        return StepOutput(tokens, logits, hidden, taps)
