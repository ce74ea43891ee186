"""Rotutar forward over an op set: one call = one scheduled step over a mixed batch of rows.

The residual stream is 32-bit and feeds the projections as it is.  Every sublayer ends in one launch (``ops.gated_norm``): the
weighted sum of what it computed, its gate, the norm in groups, the residual update and the next projection's input.  A parallel
mixer is eight launches (in_proj, heads, attention split + merge, delta rule, two output projections, gated norm), the linear one
four; a dense feed-forward four, a mixture five.
"""
from __future__ import annotations

from typing import Optional, Sequence

from ...ops.specs import GatedNorm
from ..common import StepOutput
from .weights import DenseW, LayerW, ParallelW, RotutarWeights


class RotutarRunner:
    def __init__(self, weights: RotutarWeights, state, ops, tp=None):
        if tp is not None and tp.size > 1:
            raise ValueError("Rotutar models run on one rank")
        self.w, self.state, self.ops, self.tp = weights, state, ops, None
        self.cfg = weights.cfg
        self.imatrix_collector = self.act_collector = None

    def _mixer(self, i: int, L: LayerW, h, b) -> GatedNorm:
        ops, st, m = self.ops, self.state, L.mixer
        with ops.range("mixer.in_proj"):
            proj = ops.linear(h, L.in_proj, name=f"mix_proj{L.in_proj.N}")
        pend = GatedNorm(proj[:, L.gate_off:], L.gate1, L.norm1)
        if not isinstance(m, ParallelW):
            with ops.range("gla"):
                o = ops.gla(proj, m.gla, b, st.gdn[i], st)
            with ops.range("mixer.o_proj"):
                pend.a = ops.linear(o, m.o, name="mix_left", out_f32=True)
            return pend
        with ops.range("attn.heads"):
            q = ops.attn_heads(proj, m.heads, b, st.kv[i], st)
        with ops.range("attn.core"):
            ctx = ops.attention(q, m.attn, b, st.kv[i], st, b.max_visible_launch)
        with ops.range("delta"):
            o = ops.delta(proj, m.delta, b, st.gdn[i], st, st.conv[i])
        with ops.range("mixer.o_proj"):
            pend.a, pend.scale_a = ops.linear(ctx, m.left_o, name="mix_left", out_f32=True), m.left_scale
            pend.b, pend.scale_b = ops.linear(o, m.right_o, name="mix_right", out_f32=True), m.right_scale
        return pend

    def _feed_forward(self, L: LayerW, h, b) -> GatedNorm:
        ops, m = self.ops, L.mlp
        if isinstance(m, DenseW):
            with ops.range("mlp.gate_up"):
                act = ops.linear(h, m.gate_up, name=f"mlp_act{m.gate_up.N}", swiglu=True)
            with ops.range("mlp.down"):
                y = ops.linear(act, m.down, name="mlp_out", out_f32=True)
            with ops.range("mlp.gate"):
                gate = ops.linear(h, m.gate, name="mlp_gate")
            return GatedNorm(gate, L.gate2, L.norm2, y)
        with ops.range("moe.router"):
            z = ops.linear(h, m.router, name=f"moe_logits{m.router.N}", out_f32=True)
        with ops.range("moe.route"):
            routed = ops.moe_route(z, h, m.moe, b)
        with ops.range("moe.experts"):
            y = ops.moe_experts(routed, m.moe)
        return GatedNorm(z[:, m.gate_off:], L.gate2, L.norm2, routed=routed, experts=y)

    def forward(self, b, rows: int, n_out: int, *, tap_layers: Sequence[int] = (), gdn_log=None, gdn_to_alt: bool = False,
                mask=None, mask_active=None, sample: bool = True, greedy_only: bool = False) -> StepOutput:
        """``tap_layers``: indices of layers after which the residual is returned in ``taps``.
        ``greedy_only``: as in the hybrid decoder's runner (the soft limit of the logits keeps their order)."""
        if gdn_log is not None or gdn_to_alt:
            raise ValueError("Rotutar's recurrent state cannot be logged or redirected (no speculative decoding)")
        cfg, ops, st, w = self.cfg, self.ops, self.state, self.w
        norm = dict(eps=cfg.norm_eps, groups=cfg.norm_groups)
        kin = w.lm_head.K                      # every projection of the residual has this input width
        with ops.range("embed"):
            x = ops.embed_f32(b, rows, w.embed, st.status)
        with ops.range("norm"):
            x, h = ops.gated_norm(x, None, width=kin, name="h", **norm)
        taps = {}
        steps = [(i, L, part) for i, L in enumerate(w.layers) for part in (("mixer", "mlp") if L.mlp is not None else ("mixer",))]
        for at, (i, L, part) in enumerate(steps):
            pend = self._mixer(i, L, h, b) if part == "mixer" else self._feed_forward(L, h, b)
            last = at + 1 == len(steps)
            with ops.range("norm"):
                x, h = ops.gated_norm(x, pend, norm_w=w.final_norm if last else None, width=0 if last and n_out == 0 else kin, name="h", **norm)
            if i in tap_layers and (last or steps[at + 1][0] != i):
                taps[i] = x.clone()
        if not steps:
            x, h = ops.gated_norm(x, None, norm_w=w.final_norm, width=kin, name="h", **norm)
        tokens = logits = hidden = None
        if n_out > 0:
            hidden = h[:n_out] if b.identity_out else ops.gather_rows(h, b.out_rows, n_out, "out_hidden", st.status)
            if (greedy_only and sample and mask is None and w.lm_head.N == cfg.vocab_size and hasattr(ops, "can_fuse_argmax")
                    and ops.can_fuse_argmax(w.lm_head, n_out)):
                with ops.range("head.lm_head"):
                    tokens = ops.linear_argmax(hidden, w.lm_head)
                return StepOutput(tokens, None, hidden, taps)
            with ops.range("head.lm_head"):
                logits = ops.soft_limit(ops.linear(hidden, w.lm_head, name="logits", out_f32=True), cfg.logit_softcap)[:, :cfg.vocab_size]
            if sample:
                with ops.range("head.sample"):
                    tokens = ops.sample(logits, b, n_out, mask=mask, mask_active=mask_active, status=st.status)
        return StepOutput(tokens, logits, hidden, taps)
