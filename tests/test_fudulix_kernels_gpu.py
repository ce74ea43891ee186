"""The kernels behind Fudulix, each alone against plain fp64 restatements: pair embedding, GeGLU epilogues, the heads kernel
(convolution, norms, rotation, value mixing, append), attention with kept first tokens (per-row, split-KV, tiled, tensor-core),
routing, the experts' products and the residual update that sums them."""
import types

import pytest
import torch

import fudulix_oracle as O
from kernel_cases import BF, F32, Paged, close, ops_of, rnd
from phaseshift_b200.models.common import plain_linear
from phaseshift_b200.ops.specs import AttnSpec, ExpertSum, HeadsSpec, MoeSpec, Pending
from phaseshift_b200.runtime.batch import SeqRows, StepBatch
from phaseshift_b200.runtime.state import ConvSpec, KVSpec, RunSpec

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ embedding
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("W,buckets", [(75, 1), (192, 97), (2560, 1009)])
def test_embedding_of_tokens_and_pairs(dtype, W, buckets):
    """Portions of one to many tokens over several steps: the state's last token continues a sequence; large factors do not overflow."""
    ops, V, mul = ops_of(dtype), 300, (2 ** 31 + 11, 7)
    table, pairs, w = rnd(V, W, seed=1, dtype=dtype), rnd(buckets + 1, W, seed=2, dtype=dtype), rnd(W, seed=3)
    ids = [torch.randint(0, V, (40,), generator=torch.Generator().manual_seed(i)).tolist() for i in range(3)]
    ref = {"embed": table.double().cpu(), "bigram": pairs.double().cpu(), "embed.norm": w.double().cpu()}
    cfg = {"embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), (buckets,) + mul))}, "norm": {"eps": 0.3}}
    st = types.SimpleNamespace(last_token=torch.full((5,), -1, dtype=torch.int32, device="cuda"), status=torch.zeros(1, dtype=torch.int32, device="cuda"))
    at = [0, 0, 0]
    for step in ([(0, 1), (1, 17)], [(1, 1), (0, 2), (2, 3)], [(2, 1), (0, 1), (1, 1)], [(0, 36), (2, 2)]):
        b = StepBatch(64, 3, torch.device("cuda:0"))
        b.fill([SeqRows(s + 1, at[s], ids[s][at[s]:at[s] + n]) for s, n in step])
        b.upload()
        got = ops.embed_pairs(b, 64, table, pairs, *mul, w, 0.3, st)
        r = 0
        for s, n in step:
            close(got[r:r + n].cpu(), O.embedding(ids[s], ref, cfg)[at[s]:at[s] + n], 3e-6)
            at[s], r = at[s] + n, r + n
        assert bool((got[r:] == 0).all())
    assert st.last_token.tolist() == [-1, ids[0][39], ids[1][18], ids[2][5], -1] and int(st.status) == 0


# ------------------------------------------------------------------ projections
@pytest.mark.parametrize("M", [1, 2, 8, 33, 64, 65, 300])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_geglu_epilogue(M, dtype):
    """One row streams, up to 64 rows run the split-K kernel, more the tiled tensor-core GEMM; 32-bit rows the CUDA cores."""
    ops = ops_of(dtype)
    N, K = 704, 288
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, scale=2.0 * K ** -0.5, dtype=dtype)
    y = x.double() @ w.double().T
    got = ops.linear(x, plain_linear(w, N, K, "bf16" if dtype == BF else "f32"), name="g", geglu=True)
    close(got, O.gelu_tanh(y[:, 0::2]) * y[:, 1::2], 2e-2 if dtype == BF else 4e-6)
    assert int(ops.status) == 0


# ------------------------------------------------------------------ queries, keys and values
def heads_case(H, G, dim, vdim, dtype, portions, taps=0, unit=False, halves=False, rot=None, mix=None, save=False, full_norm=False, page=16,
               graph=False):
    """Three sequences whose portions are cut differently, step by step, against whole sequences."""
    D = -(-max(dim, vdim) // 64) * 64
    C, n = (H + 2 * G) * D, [sum(p) for p in portions]
    eps, tol = 0.2, 1.5e-2 if dtype == BF else 6e-6
    freq = torch.tensor([300.0 ** (-2 * i / (rot or dim)) for i in range((rot or dim) // 2)], dtype=torch.float64)
    ops = ops_of(dtype)

    def padded(t, heads, d):
        out = torch.zeros(t.shape[:-1] + (heads, D), device=t.device, dtype=t.dtype)
        out[..., :d] = t.reshape(t.shape[:-1] + (heads, d))
        return out.flatten(-2)
    parts = ((H, dim), (G, dim), (G, vdim))
    raw = [[rnd(k, h * d, seed=10 * i + j, dtype=dtype) for j, (h, d) in enumerate(parts)] for i, k in enumerate(n)]
    cw = [rnd(h * d, taps, seed=50 + j, dtype=dtype) for j, (h, d) in enumerate(parts)] if taps else None
    nw = [1 + 0.3 * rnd(h * d, seed=60 + j) for j, (h, d) in enumerate(parts[:2])] if full_norm else None
    spec = HeadsSpec(H, G, D, dim, vdim, eps, freq.cuda(), halves, 1.3 if halves else 1.0, unit,
                     torch.cat([padded(c.T, h, d) for c, (h, d) in zip(cw, parts)], 1).contiguous() if taps else None,
                     padded(nw[0], H, dim) if nw else None, padded(nw[1], G, dim) if nw else None, mix, save)
    first = [rnd(k, G * vdim, seed=70 + i, dtype=dtype) for i, k in enumerate(n)]

    # whole sequences
    want = []
    for i in range(3):
        q, k, v = (t.double().cpu() for t in raw[i])
        if taps:
            q, k, v = (O.short_conv(t, c.double().cpu()) for t, c in zip((q, k, v), cw))
        if nw:
            q, k = O.rms_norm(q, nw[0].double().cpu(), eps), O.rms_norm(k, nw[1].double().cpu(), eps)
        q, k = q.reshape(-1, H, dim), k.reshape(-1, G, dim)
        q, k = (O.turn_halves(t, freq.tolist(), 1.3) if halves else O.turn_neighbours(t, freq.tolist()) for t in (q, k))
        if unit:
            q, k = O.unit_rms(q, eps), O.unit_rms(k, eps)
        mixed = v if mix is None else O.mix_values(v, first[i].double().cpu(), mix)
        want.append((q, k, mixed.reshape(-1, G, vdim), v))

    pg = Paged(RunSpec(KVSpec(G, D), None, ConvSpec(C, taps - 1) if taps else None), [(0, k) for k in n], dtype, page)
    hist = pg.st.conv[0]
    if hist is not None:
        hist.fill_(float("nan"))                     # what lies before a sequence's start is never read
    at = [0, 0, 0]
    for step in range(max(len(p) for p in portions)):
        live = [(i, portions[i][step]) for i in range(3) if step < len(portions[i])]
        rows = sum(c for _, c in live)
        b = StepBatch(rows + 2, 4, torch.device("cuda:0"))
        b.fill([SeqRows(i + 1, at[i], [0] * c) for i, c in live])
        b.graph_static = graph
        b.upload()
        proj = rnd(rows + 2, C + 8, seed=5, dtype=dtype)
        saved = rnd(rows + 2, G * vdim, seed=6, dtype=dtype)
        r = 0
        for i, c in live:
            proj[r:r + c, :C] = torch.cat([padded(t[at[i]:at[i] + c], h, d) for t, (h, d) in zip(raw[i], parts)], 1)
            if mix is not None:
                saved[r:r + c] = first[i][at[i]:at[i] + c]
            r += c
        got = ops.attn_heads(proj, spec, b, pg.st.kv[0], pg.st, hist, saved).reshape(rows + 2, H, D)
        r = 0
        for i, c in live:
            close(got[r:r + c, :, :dim].cpu(), want[i][0][at[i]:at[i] + c], tol)
            if save:
                close(saved[r:r + c].cpu(), want[i][3][at[i]:at[i] + c], tol)
            at[i], r = at[i] + c, r + c
        assert bool((got[:r, :, dim:] == 0).all()) and bool((got[r:] == 0).all())
    assert int(pg.st.status) == 0
    for i in range(3):
        t = torch.arange(n[i], device="cuda")
        blk = pg.st.block_table[i + 1][t // page].long()
        for pool, w in ((pg.st.kv[0].k, want[i][1]), (pg.st.kv[0].v, want[i][2])):
            g = pool[blk, :, t % page]
            close(g[..., :w.shape[-1]].cpu(), w, tol)
            assert bool((g[..., w.shape[-1]:] == 0).all())


CUTS = [[1, 1, 2, 30, 1], [40, 2], [2, 3, 1, 1, 1, 5]]
LONG = [[700, 1, 1], [1, 450], [3, 2, 1]]


@pytest.mark.parametrize("H,G,dim,vdim", [(5, 1, 40, 24), (8, 2, 128, 128), (4, 4, 20, 100), (3, 1, 300, 8)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_heads_with_unit_norms(H, G, dim, vdim, dtype):
    for cuts in (CUTS, LONG):
        heads_case(H, G, dim, vdim, dtype, cuts, unit=True)
    heads_case(H, G, dim, vdim, dtype, CUTS, unit=True, rot=dim // 2 // 2 * 2, mix=0.4, page=64)
    heads_case(H, G, dim, vdim, dtype, CUTS, unit=True, rot=2, save=True, graph=True)


@pytest.mark.parametrize("H,G,dim,vdim", [(6, 2, 40, 24), (8, 2, 128, 128), (4, 4, 18, 100), (3, 1, 300, 8)])
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_heads_with_convolutions_and_joint_norms(H, G, dim, vdim, taps, dtype):
    for cuts in (CUTS, LONG):
        heads_case(H, G, dim, vdim, dtype, cuts, taps=taps, halves=True, full_norm=True)
    heads_case(H, G, dim, vdim, dtype, CUTS, taps=taps, halves=True, full_norm=True, rot=dim // 2 // 2 * 2, mix=0.7, graph=True)
    heads_case(H, G, dim, vdim, dtype, CUTS, taps=taps, halves=True, rot=2, save=True)


# ------------------------------------------------------------------ attention with kept first tokens
def attention_case(H, G, D, seqs, dtype, window, keep, sink=False, page=16, graph=False, standout=None, max_len=2048):
    """Keys and values in scattered pages, the step's queries against the oracle over whole sequences.  `standout`: position whose
    key all queries score far above every other, so that seeing it or not decides the output."""
    ops = ops_of(dtype, max_len)
    pg = Paged(RunSpec(KVSpec(G, D), None), seqs, dtype, page, graph)
    scale = D ** -0.5
    spec = AttnSpec(H, G, D, scale, window=window, keep_first=keep, sink=torch.zeros(H, device="cuda") if sink else None)
    q_all = torch.zeros(pg.rows, H * D, device="cuda", dtype=dtype)
    at, want = 0, []
    for i, (p, n) in enumerate(seqs):
        q, k, v = (rnd(p + n, m, D, seed=s + i, dtype=dtype) for m, s in ((H, 20), (G, 40), (G, 60)))
        if standout is not None and standout < p + n:
            u = rnd(D, seed=3).sign()
            q = (q.float() * 0.2 + 0.7 * u).to(dtype)
            k[standout] = (u * 14.0 / (0.7 * D * scale)).to(dtype)
        pg.fill_keys(i, k, v)
        q_all[at:at + n] = q[p:].reshape(n, -1)
        o = O.attend(q.double().cpu(), k.double().cpu(), v.double().cpu(), scale, O.kept_window_mask(p + n, window, keep),
                     O.softmax_plus_one if sink else O.softmax)
        want.append(o[p:])
        at += n
    out = ops.attention(q_all, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
    assert int(pg.st.status) == 0 and int(ops.status) == 0
    at = 0
    for w in want:
        close(out[at:at + w.shape[0]].cpu(), w, 2e-2 if dtype == BF else 5e-6)
        at += w.shape[0]


MIX = [(37, 150), (330, 1), (0, 2), (263, 3), (399, 16)]
HEADS = [(8, 2, 128), (4, 4, 64), (4, 4, 32), (6, 2, 96), (16, 1, 64), (4, 2, 256), (2, 1, 288), (3, 3, 192), (20, 2, 256)]


@pytest.mark.parametrize("H,G,D", HEADS)
@pytest.mark.parametrize("window,keep", [(1, 1), (7, 20), (64, 64), (100, 3), (33, 200), (40, 130)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_windows_that_keep_the_first_tokens(H, G, D, window, keep, dtype):
    """A long portion, short portions and single decoded rows together; kept tokens before, inside and beyond the window's reach."""
    attention_case(H, G, D, MIX, dtype, window, keep)
    attention_case(H, G, D, MIX, dtype, window, keep, sink=True)


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (16, 1, 64), (8, 2, 128), (4, 4, 64)])
@pytest.mark.parametrize("graph", [False, True])
def test_decoded_rows_with_kept_tokens(H, G, D, graph):
    rows = [(127, 1), (128, 1), (49, 1), (50, 1), (0, 1), (1200, 1), (191, 1), (64, 1), (63, 1), (900, 1)]
    for window, keep in ((50, 20), (64, 64), (30, 300), (1, 65), (500, 1)):
        attention_case(H, G, D, rows, BF, window, keep, graph=graph)
        attention_case(H, G, D, rows[:5], BF, window, keep, graph=graph, sink=True)


@pytest.mark.parametrize("D", [64, 128, 192, 256])
@pytest.mark.parametrize("page", [16, 32, 64])
def test_page_sizes_with_kept_tokens(D, page):
    attention_case(4, 2, D, [(50, 300), (389, 1), (190, 1), (191, 2)], BF, 90, 70, page=page)


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (2, 1, 288), (8, 2, 128), (16, 1, 64)])
@pytest.mark.parametrize("standout,keep", [(0, 1), (1, 1), (15, 16), (16, 16), (63, 64), (64, 64), (64, 65), (99, 100), (100, 100), (130, 131), (131, 131), (40, 0)])
def test_a_standout_key_counts_exactly_when_it_is_kept_or_in_the_window(H, G, D, standout, keep):
    """Windows of 60: rows on both sides of the edge, the last kept token and the one behind it, far away, in a prompt's portion and
    decoded alone."""
    attention_case(H, G, D, [(50, 250), (standout, 1), (standout + 59, 1), (standout + 60, 1), (700, 1)], BF, 60, keep, standout=standout)
    attention_case(H, G, D, [(standout, 1), (standout + 58, 4), (standout + 400, 1)], BF, 60, keep, standout=standout)
    attention_case(H, G, D, [(0, 260)], F32 if D != 256 else BF, 60, keep, standout=standout)


# ------------------------------------------------------------------ mixture of experts
def moe_spec(E, identity, top, groups, keep, ff, width, K, dtype, seed=1):
    n = E + identity
    c = (-1.25 + 0.2 * rnd(n, seed=seed)).contiguous()
    return MoeSpec(E, identity, top, groups, keep, ff, width, c, rnd(E * 2 * ff, K, seed=seed + 1, scale=K ** -0.5, dtype=dtype),
                   rnd(E * width, ff, seed=seed + 2, scale=ff ** -0.5, dtype=dtype))


def step_of(rows, padding=3):
    b = StepBatch(rows + padding, 1, torch.device("cuda:0"))
    b.fill([SeqRows(0, 0, [0] * rows)])
    b.upload()
    return b


ROUTERS = [(18, 6, 2, 4, 1), (10, 2, 3, 3, 2), (1, 0, 1, 1, 1), (60, 4, 8, 4, 2), (200, 56, 10, 16, 3), (41, 4, 6, 9, 4), (8, 2, 2, 5, 2), (3, 5, 8, 1, 1)]


@pytest.mark.parametrize("rows", [1, 5, 64, 65, 300])
@pytest.mark.parametrize("shape", ROUTERS)
def test_routing(rows, shape):
    E, identity, top, groups, keep = shape
    ops, K = ops_of(BF), 96
    s = moe_spec(E, identity, top, groups, keep, 32, 16, K, BF)
    n = E + identity
    z = rnd(rows + 3, -(-n // 4) * 4, seed=4, scale=2.0)
    h = rnd(rows + 3, K, seed=5, dtype=BF)
    for _ in range(2):
        r = ops.moe_route(z, h, s, step_of(rows))
    assert int(ops.status) == 0
    index, weight, same = r.index.cpu(), r.weight.cpu(), r.identity.cpu().flatten()
    assert bool((index[rows:] == -1).all()) and bool((same[rows:] == 0).all())
    tiles = r.tiles.cpu()
    expert_at = torch.full((rows * top,), -1)
    for e, first, count, _ in tiles[1:1 + int(tiles[0, 0])].tolist():
        assert 0 < count <= r.tile_rows and bool((expert_at[first:first + count] == -1).all())
        expert_at[first:first + count] = e
    used = []
    for i in range(rows):
        want = O.route(z[i, :n].double().cpu(), s.correction.double().cpu(), groups, keep, top)
        got = {int(expert_at[p]): float(w) for p, w in zip(index[i].tolist(), weight[i]) if p >= 0}
        real = {e: float(w) for e, w in want if e < E}
        assert set(got) == set(real)
        for e in real:
            assert abs(got[e] - real[e]) < 1e-5
        assert abs(float(same[i]) - sum(float(w) for e, w in want if e >= E)) < 1e-5
        for p in index[i].tolist():
            if p >= 0:
                used.append(p)
                assert torch.equal(r.inputs[p], h[i])
    assert sorted(used) == list(range(len(used))) and bool((expert_at[len(used):] == -1).all())


def test_logits_that_are_not_finite_are_reported():
    ops = ops_of(BF)
    s = moe_spec(8, 0, 2, 1, 1, 32, 16, 32, BF)
    for rows in (2, 100):
        z = rnd(rows + 3, 8, seed=1)
        z[1] = float("nan")
        ops.moe_route(z, rnd(rows + 3, 32, dtype=BF), s, step_of(rows))
        assert int(ops.status) != 0
        ops.status.zero_()


@pytest.mark.parametrize("rows", [1, 3, 16, 17, 40, 64, 65, 200, 700])
@pytest.mark.parametrize("E,identity,top,ff,width,K", [(14, 3, 2, 96, 224, 160), (10, 2, 3, 64, 76, 96), (4, 0, 4, 160, 128, 128), (60, 4, 8, 96, 256, 320)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_experts_and_their_sum(rows, E, identity, top, ff, width, K, dtype):
    """Router, experts, shared expert, residual update and norm against the plain mixture; unequal loads, experts without rows."""
    ops, W = ops_of(dtype), width - 1 if width % 64 else width
    s = moe_spec(E, identity, top, 1, 1, ff, width, K, dtype)
    z = rnd(rows + 3, E + identity, seed=4, scale=2.0)
    z[:, 1] += 3.0                                                     # most rows go to one expert
    h = rnd(rows + 3, K, seed=5, dtype=dtype)
    h_wide = rnd(rows + 3, width, seed=6, dtype=dtype)
    shared, x, step, nw = rnd(rows + 3, width, seed=7), rnd(rows + 3, W, seed=8), rnd(W, seed=9), rnd(W, seed=10)
    r = ops.moe_route(z, h, s, step_of(rows))
    y = ops.moe_experts(r, s)
    assert int(ops.status) == 0
    gu, dn = s.gate_up.double().reshape(E, 2 * ff, K), s.down.double().reshape(E, width, ff)
    sc = torch.softmax(z.double(), -1)
    ids = (sc + s.correction.double()).topk(top, -1).indices
    wt = sc.gather(1, ids)
    wt = wt / wt.sum(-1, keepdim=True)
    want = torch.zeros(rows, width, device="cuda", dtype=torch.float64)
    hd = h.double()[:rows]
    for e in range(E + identity):
        sel = (wt[:rows] * (ids[:rows] == e)).sum(-1)
        if e < E:
            a = hd @ gu[e].T
            want += sel[:, None] * ((O.silu(a[:, 0::2]) * a[:, 1::2]) @ dn[e].T)
        else:
            want += sel[:, None] * h_wide.double()[:rows]
    tol = 2e-2 if dtype == BF else 6e-6
    for sh in (None, shared):
        for bias in (None, step):
            pend = Pending(0.7, experts=ExpertSum(r, y, h_wide, sh), bias=bias)
            xo, hn = ops.residual_norm(x.clone(), pend, norm_w=nw, eps=0.2, width=-(-W // 32) * 32, name="h")
            t = want if sh is None else want + sh.double()[:rows]
            t = x.double()[:rows] + 0.7 * t[:, :W] + (0 if bias is None else bias.double())
            close(xo[:rows], t, tol)
            close(hn[:rows, :W], O.rms_norm(t, nw.double(), 0.2), tol)
            assert bool((hn[:, W:] == 0).all())
            pad = x[rows:] + (0 if sh is None else 0.7 * sh[rows:, :W]) + (0 if bias is None else bias)
            close(xo[rows:], pad, 1e-5)                                # padding rows get no expert


def test_one_expert_takes_every_row():
    ops, s = ops_of(BF), moe_spec(4, 0, 1, 1, 1, 64, 128, 128, BF)
    z = torch.zeros(503, 4, device="cuda")
    z[:, 2] = 9.0
    h = rnd(503, 128, seed=5, dtype=BF)
    r = ops.moe_route(z, h, s, step_of(500))
    y = ops.moe_experts(r, s)
    a = h.double()[:500] @ s.gate_up.double().reshape(4, 128, 128)[2].T
    want = (O.silu(a[:, 0::2]) * a[:, 1::2]) @ s.down.double().reshape(4, 128, 64)[2].T
    close(y[r.index[:500, 0].long()], want, 2e-2)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_a_plain_update_with_a_bias(dtype):
    ops = ops_of(dtype)
    x, y, b, w = rnd(9, 75, seed=1), rnd(9, 76, seed=2), rnd(75, seed=3), rnd(75, seed=4)
    xo, h = ops.residual_norm(x.clone(), Pending(0.5, plain=y, bias=b), norm_w=w, eps=0.1, width=96, one=True, name="h")
    t = x.double() + 0.5 * y.double()[:, :75] + b.double()
    close(xo, t, 2e-6)
    close(h[:, :75], O.rms_norm(t, w.double(), 0.1), 1e-2 if dtype == BF else 5e-6)
    assert bool((h[:, 75] == 1).all()) and bool((h[:, 76:] == 0).all())
