"""The kernels behind Gebuzen, each alone against plain fp64 restatements: fused residual + norm, embedding, 32-bit GEMM, gated
epilogues, block-local attention with a sink (per-row, split-KV, tiled, tensor-core), gated linear attention (row and chunked)."""
import types

import pytest
import torch

import gebuzen_oracle as O
from kernel_cases import BF, F32, Paged, close, ops_of, rnd
from phaseshift_b200.models.gebuzen.weights import LinearW, QuantizedTensor
from phaseshift_b200.ops.specs import AttnSpec, GlaSpec, Pending
from phaseshift_b200.runtime.state import KVSpec, RecurrentSpec, RunSpec

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ residual + norm, embedding
@pytest.mark.parametrize("W,dtype", [(75, F32), (75, BF), (96, BF), (320 + 4, F32), (2560, BF)])
@pytest.mark.parametrize("rows", [1, 9])
def test_residual_norm(W, dtype, rows):
    ops = ops_of(dtype)
    x, add, step = rnd(rows, W, seed=1), rnd(rows, W, seed=2), rnd(W, seed=3)
    wide = (W + 3) // 4 * 4
    a, b, y = (rnd(rows, wide, seed=s, scale=3.0) for s in (4, 5, 6))       # projections with padding columns behind the width
    wa, wb, w = (rnd(W, seed=s) for s in (7, 8, 9))
    eps, width = 0.3, (W + 32) // 32 * 32                                   # an eps that would show outside the root
    branches = 0.35 * (O.rms_norm(a[:, :W].double(), wa, eps) + O.rms_norm(b[:, :W].double(), wb, eps))
    for pend, upd in ((Pending(0.35, a[:, :W], wa, b[:, :W], wb), branches), (Pending(0.7, plain=y[:, :W]), 0.7 * y[:, :W].double()), (None, 0.0)):
        for use_add, use_step, one, scale in ((False, False, True, 1.0), (True, True, False, 0.25), (False, True, True, 2.0)):
            want = x.double() + upd + (add if use_add else 0.0) + (step if use_step else 0.0)
            xo, h = ops.residual_norm(x.clone(), pend, add=add if use_add else None, step=step if use_step else None, norm_w=w, eps=eps,
                                      scale=scale, width=width, one=one, name="h")
            close(xo, want, 2e-6)
            close(h[:, :W], O.rms_norm(want, w, eps) * scale, 1e-2 if dtype == BF else 2e-6)
            assert bool((h[:, W:].float() == torch.tensor([1.0 if one else 0.0] + [0.0] * (width - W - 1), device="cuda")).all())
    xo, h = ops.residual_norm(x, Pending(0.7, plain=y[:, :W]), eps=eps)
    assert h is None and xo.data_ptr() != x.data_ptr()


@pytest.mark.parametrize("dtype", [BF, F32])
def test_embedding_rows_are_widened_and_bad_ids_reported(dtype):
    ops = ops_of(dtype)
    table = rnd(50, 75, dtype=dtype)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    b = types.SimpleNamespace(ids=torch.tensor([3, 49, 0, 7], dtype=torch.int32, device="cuda"))
    assert torch.equal(ops.embed_f32(b, 4, table, status), table[b.ids.long()].float()) and int(status) == 0
    b.ids = torch.tensor([3, 50], dtype=torch.int32, device="cuda")
    assert bool((ops.embed_f32(b, 2, table, status)[1] == 0).all()) and int(status) == 1


# ------------------------------------------------------------------ projections
@pytest.mark.parametrize("M,N,K", [(1, 64, 32), (7, 130, 96), (65, 66, 352), (200, 256, 64)])
def test_gemm_f32(M, N, K):
    ops = ops_of(F32)
    x, w = rnd(M, K, seed=1), rnd(N, K, seed=2)
    W = LinearW(QuantizedTensor("f32", (N, K), K, w))
    y = x.double() @ w.double().T
    close(ops.linear(x, W, name="y"), y, 2e-6)
    close(ops.linear(x, W, name="g", reglu=True), torch.relu(y[:, 0::2]) * y[:, 1::2], 4e-6)
    close(ops.linear(x, W, name="s", swiglu=True), torch.nn.functional.silu(y[:, 0::2]) * y[:, 1::2], 4e-6)


@pytest.mark.parametrize("M", [1, 2, 8, 33, 64, 65, 300])
def test_reglu_epilogue_of_the_bf16_projections(M):
    """One row streams, up to 64 rows run the split-K kernel, more the tiled tensor-core GEMM."""
    ops = ops_of(BF)
    N, K = 704, 288
    x, w = rnd(M, K, seed=1, dtype=BF), rnd(N, K, seed=2, scale=K ** -0.5, dtype=BF)
    W = LinearW(QuantizedTensor("bf16", (N, K), K, w)).make_tiled(True)
    y = x.double() @ w.double().T
    got = ops.linear(x, W, name="g", reglu=True)
    close(got, torch.relu(y[:, 0::2]) * y[:, 1::2], 2e-2)
    assert bool((got[y[:, 0::2] < -0.05] == 0).all())
    assert int(ops.status) == 0


# ------------------------------------------------------------------ attention
def attention_case(H, G, D, chunk, seqs, dtype, sink=True, page=16, graph=False, standout=None, scale=None, max_len=2048):
    """Runs append + attention and compares with the oracle over whole sequences.  `standout`: position whose key all queries
    score far above every other, so that seeing it or not decides the output."""
    ops = ops_of(dtype, max_len)
    pg = Paged(RunSpec(KVSpec(G, D, shared=True), None), seqs, dtype, page, graph)
    scale = scale or D ** -0.5
    sk = rnd(H, seed=9) + 1.0 if sink else None
    spec = AttnSpec(H, G, D, scale, chunk=chunk, sink=sk)
    proj = torch.zeros(pg.rows, (H + G) * D + 8, device="cuda", dtype=dtype)
    at, want = 0, []
    for i, (p, n) in enumerate(seqs):
        q, k = rnd(p + n, H, D, seed=20 + i, dtype=dtype), rnd(p + n, G, D, seed=40 + i, dtype=dtype)
        if standout is not None and standout < p + n:
            u = rnd(D, seed=3).sign()
            q = (q.float() * 0.2 + 0.7 * u).to(dtype)
            k[standout] = (u * 14.0 / (0.7 * D * scale)).to(dtype)
        pg.fill_keys(i, k[:p])
        proj[at:at + n, :H * D] = q[p:].reshape(n, -1)
        proj[at:at + n, H * D:(H + G) * D] = k[p:].reshape(n, -1)
        w = O.chunk_attention_heads(q.double(), k.double(), scale, chunk or (p + n),
                                    (sk if sink else torch.full((H,), -1e9, device="cuda")).double())
        want.append(w[p:].reshape(n, -1))
        at += n
    qb = ops.attn_append(proj, spec, pg.b, pg.st.kv[0], pg.st)
    out = ops.attention(qb, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
    assert int(pg.st.status) == 0 and int(ops.status) == 0
    at = 0
    for w in want:
        close(out[at:at + w.shape[0]], w, 2e-2 if dtype == BF else 5e-6)
        at += w.shape[0]


HEADS = [(8, 2, 128), (4, 4, 64), (4, 4, 32), (6, 2, 96), (16, 1, 64), (24, 2, 128), (4, 2, 256), (2, 1, 288), (8, 2, 160), (3, 3, 192), (20, 2, 256)]


@pytest.mark.parametrize("H,G,D", HEADS)
@pytest.mark.parametrize("chunk", [1, 7, 64, 100, 0])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_attention_of_a_mixed_batch(H, G, D, chunk, dtype):
    """A long portion that starts inside a chunk, short portions and single decoded rows together."""
    attention_case(H, G, D, chunk, [(37, 150), (130, 1), (0, 2), (63, 3), (199, 16)], dtype)


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (16, 1, 64), (8, 2, 128), (3, 3, 192), (4, 4, 64)])
@pytest.mark.parametrize("graph", [False, True])
def test_decoded_rows_alone(H, G, D, graph):
    for chunk in (50, 128, 0):
        attention_case(H, G, D, chunk, [(127, 1), (128, 1), (49, 1), (50, 1), (0, 1), (700, 1)], BF, graph=graph)


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (2, 1, 288), (24, 2, 128), (8, 2, 128), (8, 1, 64)])
@pytest.mark.parametrize("standout", [0, 15, 16, 63, 64, 99, 100, 127, 128, 199, 200, 255])
def test_a_standout_key_counts_exactly_inside_its_chunk(H, G, D, standout):
    """Rows on both sides of every border of 100-position chunks and of pages, in a prompt's portion and decoded alone."""
    attention_case(H, G, D, 100, [(90, 210), (standout, 1), (199, 1), (200, 1), (299, 1)], BF, standout=standout)
    attention_case(H, G, D, 100, [(standout, 1), (99, 1), (100, 1), (255, 4)], BF, standout=standout)
    attention_case(H, G, D, 100, [(0, 260)], F32 if D != 256 else BF, standout=standout)


@pytest.mark.parametrize("D", [64, 128, 192, 256])
@pytest.mark.parametrize("page", [16, 32, 64])
def test_page_sizes(D, page):
    attention_case(4, 2, D, 90, [(50, 200), (89, 1), (90, 1), (91, 2)], BF, page=page)


@pytest.mark.parametrize("D", [64, 256, 320])
def test_sinks_far_above_and_far_below_every_score(D):
    ops = ops_of(BF)
    for level in (-60.0, 60.0, 0.0):
        pg = Paged(RunSpec(KVSpec(2, D, shared=True), None), [(10, 80), (40, 1)], BF)
        sk = torch.full((4,), level, device="cuda")
        spec = AttnSpec(4, 2, D, 0.05, chunk=64, sink=sk)
        proj = torch.zeros(pg.rows, 6 * D, device="cuda", dtype=BF)
        ks = [rnd(90, 2, D, seed=1, dtype=BF), rnd(41, 2, D, seed=2, dtype=BF)]
        qs = [rnd(90, 4, D, seed=3, dtype=BF), rnd(41, 4, D, seed=4, dtype=BF)]
        for i, (p, n, at) in enumerate([(10, 80, 0), (40, 1, 80)]):
            pg.fill_keys(i, ks[i][:p])
            proj[at:at + n] = torch.cat([qs[i][p:].reshape(n, -1), ks[i][p:].reshape(n, -1)], 1)
        q = ops.attn_append(proj, spec, pg.b, pg.st.kv[0], pg.st)
        out = ops.attention(q, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
        for i, (p, n, at) in enumerate([(10, 80, 0), (40, 1, 80)]):
            want = O.chunk_attention_heads(qs[i].double(), ks[i].double(), 0.05, 64, sk.double())[p:].reshape(n, -1)
            if level == 60.0:
                assert float(out[at:at + n].float().abs().max()) < 1e-6 and float(want.abs().max()) < 1e-12
            else:
                close(out[at:at + n], want, 2e-2)


def test_scores_far_below_zero_keep_their_softmax():
    """All visible scores of a row around -150: the block-local mask hides the first tiles of later rows, whose reference
    maximum must then come from their own block."""
    D, H = 256, 2
    ops = ops_of(BF)
    pg = Paged(RunSpec(KVSpec(1, D, shared=True), None), [(0, 200)], BF)
    u = rnd(D, seed=3).sign()
    q = (0.5 * u + rnd(200, H, D, seed=1) * 0.02).to(BF)
    k = (-0.5 * u + rnd(200, 1, D, seed=2) * 0.3).to(BF)
    spec = AttnSpec(H, 1, D, 2.4, chunk=90)
    proj = torch.zeros(pg.rows, (H + 1) * D, device="cuda", dtype=BF)
    proj[:200] = torch.cat([q.reshape(200, -1), k.reshape(200, -1)], 1)
    qq = ops.attn_append(proj, spec, pg.b, pg.st.kv[0], pg.st)
    out = ops.attention(qq, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
    want = O.chunk_attention_heads(q.double(), k.double(), 2.4, 90, torch.full((H,), -1e9, device="cuda").double()).reshape(200, -1)
    close(out[:200], want, 2e-2)


# ------------------------------------------------------------------ gated linear attention
def gla_case(H, dk, dv, dv_true, rank, seqs, dtype, bias, tau, graph=False, steps=1):
    ops = ops_of(dtype)
    pg = Paged(RunSpec(None, RecurrentSpec(H, dk, dv)), seqs, dtype, graph=graph)
    rp = (rank + 7) // 8 * 8
    offs = [8]
    for n in (H * dk, H * dk, H * dv, H * dv):
        offs.append(offs[-1] + n)
    proj = rnd(pg.rows, offs[-1] + rp, seed=1, dtype=dtype)
    a2 = torch.zeros(H * dk, rp, device="cuda", dtype=dtype)
    a2[:, :rank] = rnd(H * dk, rank, seed=2, scale=rank ** -0.5, dtype=dtype)
    a2b = rnd(H * dk, seed=3) * 2 + bias
    nw = torch.zeros(dv, device="cuda")
    nw[:dv_true] = rnd(dv_true, seed=4) * 0.2 + 1
    if dv_true < dv:                                     # padded value columns are zero
        proj[:, offs[2]:offs[3]].view(-1, H, dv)[:, :, dv_true:] = 0
    g = GlaSpec(H, dk, dv, dv_true, *offs, rp, dk ** -0.5, 1.0 / tau, 1e-3, a2, a2b, nw)
    st0 = rnd(*pg.st.gdn[0].rec.shape, seed=6)
    if dv_true < dv:
        st0[..., dv_true:] = 0
    pg.st.gdn[0].rec.copy_(st0)
    out = ops.gla(proj, g, pg.b, pg.st.gdn[0], pg.st)
    p = proj.double().cpu()
    z = p[:, offs[4]:offs[4] + rp] @ a2.double().cpu().T + a2b.double().cpu()
    al = torch.exp(torch.nn.functional.logsigmoid(z) / tau).reshape(-1, H, dk)
    q, k = (p[:, offs[i]:offs[i + 1]].reshape(-1, H, dk) for i in (0, 1))
    v, gt = (p[:, offs[i]:offs[i + 1]].reshape(-1, H, dv) for i in (2, 3))
    at = 0
    for i, (_, n) in enumerate(seqs):
        r = slice(at, at + n)
        o, S = O.gated_linear_recurrence(q[r] * dk ** -0.5, k[r], v[r], al[r], st0[i + 1].double().cpu())
        o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / dv_true + 1e-3) * nw.double().cpu()
        want = (o * gt[r] * torch.sigmoid(gt[r])).reshape(n, -1)
        close(pg.st.gdn[0].rec[i + 1].cpu(), S, 1e-5)
        close(out[r].cpu(), want, 1.5e-2 if dtype == BF else 1e-5)
        at += n
    assert torch.equal(pg.st.gdn[0].rec[0], st0[0])        # nobody's slot stays untouched


SIZES = [(2, 128, 128, 128, 16), (3, 64, 64, 64, 11), (2, 16, 32, 20, 5), (1, 80, 160, 160, 40), (2, 48, 32, 32, 16), (1, 192, 128, 100, 64),
         (2, 256, 256, 256, 16)]


@pytest.mark.parametrize("H,dk,dv,dvt,rank", SIZES)
@pytest.mark.parametrize("bias,tau", [(2.0, 16.0), (-2.0, 1.0), (-40.0, 1.0), (20.0, 4.0)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_gla_of_a_mixed_batch(H, dk, dv, dvt, rank, bias, tau, dtype):
    """Portions longer and shorter than the chunked kernel's blocks, short ones and single rows, states from earlier steps;
    decays from none to forty e-folds per token."""
    gla_case(H, dk, dv, dvt, rank, [(5, 150), (0, 64), (9, 17), (3, 2), (70, 1), (8, 16)], dtype, bias, tau)


@pytest.mark.parametrize("graph", [False, True])
def test_gla_decoded_rows(graph):
    gla_case(2, 128, 128, 128, 16, [(5, 1), (0, 1), (9, 1)], BF, 1.0, 8.0, graph=graph)
    gla_case(2, 32, 96, 70, 3, [(5, 1), (0, 1), (9, 1)], BF, 1.0, 8.0, graph=graph)
