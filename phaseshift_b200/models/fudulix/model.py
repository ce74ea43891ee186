"""Fudulix forward over an op set: one call = one scheduled step over a mixed batch of rows.

The residual stream is 32-bit; every update is fused with the norm that follows it (``ops.residual_norm``), the sum over a
mixture's experts included.  A mixer is six launches: norm, in_proj, heads (convolution, norms, rotation, value mixing,
append), attention (split + merge), o.  A dense feed-forward is three (norm, gate_up, down), a mixture up to seven (norm,
router, routing, the experts' two, the shared expert's two).
"""
from __future__ import annotations

from typing import Optional, Sequence

from ...ops.specs import ExpertSum, Pending
from ..common import StepOutput
from .weights import DenseW, FudulixWeights, LayerW, MixtureW


class FudulixRunner:
    def __init__(self, weights: FudulixWeights, state, ops, tp=None):
        if tp is not None and tp.size > 1:
            raise ValueError("Fudulix models run on one rank")
        self.w, self.state, self.ops, self.tp = weights, state, ops, None
        self.cfg = weights.cfg
        self.imatrix_collector = self.act_collector = None
        first = self.cfg.first_mixing()
        m = None if first is None else self.cfg.layers[first].mixer
        self.saved_width = 0 if m is None else m.kv_heads * m.vdim

    def _mixer(self, i: int, L: LayerW, h, b, saved):
        """The mixer's output before its projection back to the residual width."""
        ops, st = self.ops, self.state
        with ops.range("mixer.in_proj"):
            proj = ops.linear(h, L.in_proj, name=f"mix_proj{L.in_proj.N}")
        with ops.range("attn.heads"):
            q = ops.attn_heads(proj, L.heads, b, st.kv[i], st, st.conv[i], saved)
        with ops.range("attn.core"):
            return ops.attention(q, L.attn, b, st.kv[i], st, b.max_visible_launch)

    def _dense(self, m: DenseW, h) -> Pending:
        ops = self.ops
        with ops.range("mlp.gate_up"):
            act = ops.linear(h, m.gate_up, name=f"mlp_act{m.gate_up.N}", geglu=True)
        with ops.range("mlp.down"):
            return Pending(1.0, plain=ops.linear(act, m.down, name="mlp_out", out_f32=True), bias=m.bias)

    def _mixture(self, m: MixtureW, h, b) -> Pending:
        ops, shared = self.ops, None
        with ops.range("moe.router"):
            z = ops.linear(h, m.router, name=f"moe_logits{m.router.N}", out_f32=True)
        with ops.range("moe.route"):
            routed = ops.moe_route(z, h, m.moe, b)
        with ops.range("moe.experts"):
            y = ops.moe_experts(routed, m.moe)
        if m.shared_gate_up is not None:
            with ops.range("moe.shared"):
                act = ops.linear(h, m.shared_gate_up, name=f"mlp_act{m.shared_gate_up.N}", swiglu=True)
                shared = ops.linear(act, m.shared_down, name="mlp_out", out_f32=True)
        return Pending(1.0, experts=ExpertSum(routed, y, h, shared))

    def forward(self, b, rows: int, n_out: int, *, tap_layers: Sequence[int] = (), gdn_log=None, gdn_to_alt: bool = False,
                mask=None, mask_active=None, sample: bool = True, greedy_only: bool = False) -> StepOutput:
        """``tap_layers``: indices of layers after which the residual is returned in ``taps``.
        ``greedy_only``: as in the hybrid decoder's runner."""
        if gdn_log is not None or gdn_to_alt:
            raise ValueError("Fudulix models have no recurrent state to log or redirect (no speculative decoding)")
        cfg, ops, st, w = self.cfg, self.ops, self.state, self.w
        eps = cfg.norm_eps
        with ops.range("embed"):
            x = ops.embed_pairs(b, rows, w.embed, w.bigram, cfg.bigram.mul_prev, cfg.bigram.mul_cur, w.embed_norm, eps, st)
        saved = ops.saved_values(rows, self.saved_width) if self.saved_width else None
        pend: Optional[Pending] = None
        taps = {}
        for i, L in enumerate(w.layers):
            with ops.range("norm"):
                x, h = ops.residual_norm(x, pend, norm_w=L.norm1, eps=eps, width=L.in_proj.K, name="h_mix")
            ctx = self._mixer(i, L, h, b, saved)
            with ops.range("mixer.o_proj"):
                pend = Pending(1.0, plain=ops.linear(ctx, L.o, name="mix_out", out_f32=True))
            if L.mlp is not None:
                dense = isinstance(L.mlp, DenseW)
                width = (L.mlp.gate_up if dense else L.mlp.router).K          # (the two kinds have buffers of their own)
                with ops.range("norm"):
                    x, h = ops.residual_norm(x, pend, norm_w=L.norm2, eps=eps, width=width, one=dense, name=f"h_mlp{width}")
                pend = self._dense(L.mlp, h) if dense else self._mixture(L.mlp, h, b)
            if i in tap_layers:
                x, _ = ops.residual_norm(x, pend, eps=eps)
                pend = None
                taps[i] = x.clone()
        tokens = logits = hidden = None
        if n_out > 0:
            with ops.range("norm"):
                x, h = ops.residual_norm(x, pend, norm_w=w.final_norm, eps=eps, width=w.lm_head.K, name="h_final")
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
