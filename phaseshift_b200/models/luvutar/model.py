"""Luvutar forward over an op set: one call = one scheduled step over a mixed batch of rows.

The residual streams are 32-bit.  Writing a sublayer's output into all streams, reading the next sublayer's input from them
and its norm are one launch (``ops.stream_norm``).  An attention layer decodes in nine launches: stream norm, in_proj, append,
attention (split + merge), o, stream norm, up, down.  A latent layer decodes in twelve: stream norm, in_proj, latents (norms,
rotation, append), uq, queries into the latent space, attention (split + merge), values out of it with the output gate, o,
stream norm, up, down.
"""
from __future__ import annotations

from typing import Optional, Sequence

from ...ops.specs import LatentSpec, StreamWrite
from ..common import StepOutput
from .weights import LayerW, LuvutarWeights


class LuvutarRunner:
    def __init__(self, weights: LuvutarWeights, state, ops, tp=None):
        if tp is not None and tp.size > 1:
            raise ValueError("Luvutar models run on one rank")
        self.w, self.state, self.ops, self.tp = weights, state, ops, None
        self.cfg = weights.cfg
        self.imatrix_collector = self.act_collector = None

    def _mixer(self, i: int, L: LayerW, h, b):
        """The mixer's output before its projection back to the residual width."""
        ops, st = self.ops, self.state
        kv = st.kv[self.cfg.kv_layer(i)]
        with ops.range("mixer.in_proj"):
            proj = ops.linear(h, L.in_proj, name=f"mix_proj{L.in_proj.N}")
        if isinstance(L.attn, LatentSpec):
            with ops.range("latent.down"):
                cq = ops.latent_down(proj, L.attn, b, kv, st)
            with ops.range("latent.uq"):
                q = ops.linear(cq, L.uq, name=f"latent_q{L.uq.N}")
            with ops.range("latent.core"):
                return ops.latent_attention(q, L.attn, b, kv, st, gate=proj)
        with ops.range("attn.append"):
            q = ops.attn_append(proj, L.attn, b, kv if L.appends else None, st)
        with ops.range("attn.core"):
            return ops.attention(q, L.attn, b, kv, st, b.max_visible_launch, gate=proj)

    def forward(self, b, rows: int, n_out: int, *, tap_layers: Sequence[int] = (), gdn_log=None, gdn_to_alt: bool = False,
                mask=None, mask_active=None, sample: bool = True, greedy_only: bool = False) -> StepOutput:
        """``tap_layers``: indices of layers whose residual (the sum of the streams after the layer) is returned in ``taps``.
        ``greedy_only``: as in the hybrid decoder's runner."""
        if gdn_log is not None or gdn_to_alt:
            raise ValueError("Luvutar models have no recurrent state to log or redirect (no speculative decoding)")
        cfg, ops, st, w = self.cfg, self.ops, self.state, self.w
        eps = cfg.norm_eps
        with ops.range("embed"):
            x = ops.embed_f32(b, rows, w.embed, st.status)
        x = x[:, None].expand(-1, cfg.streams, -1)                       # every stream starts as the embedding
        pend: Optional[StreamWrite] = None
        taps = {}
        for i, L in enumerate(w.layers):
            with ops.range("norm"):
                x, h = ops.stream_norm(x, pend, read=L.hc1.read, norm_w=L.hc1.norm, eps=eps, width=L.in_proj.K, name="h_mix")
            ctx = self._mixer(i, L, h, b)
            with ops.range("mixer.o_proj"):
                pend = StreamWrite(L.hc1.mix, L.hc1.out, ops.linear(ctx, L.o, name="mix_out", out_f32=True))
            if L.hc2 is not None:
                with ops.range("norm"):
                    x, h = ops.stream_norm(x, pend, read=L.hc2.read, norm_w=L.hc2.norm, eps=eps, width=L.up.K, name="h_mlp")
                with ops.range("mlp.up"):
                    act = ops.linear(h, L.up, name=f"mlp_act{L.up.N}", gelu=True)
                with ops.range("mlp.down"):
                    pend = StreamWrite(L.hc2.mix, L.hc2.out, ops.linear(act, L.down, name="mlp_out", out_f32=True))
            if i in tap_layers:
                x, _ = ops.stream_norm(x, pend, eps=eps)
                pend = None
                taps[i] = x.sum(1)
        tokens = logits = hidden = None
        if n_out > 0:
            with ops.range("norm"):
                x, h = ops.stream_norm(x, pend, read=w.read_all, norm_w=w.final_norm, eps=eps, width=w.lm_head.K, name="h_final", last=True)
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
