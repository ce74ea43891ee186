"""The kernels behind Rotutar, each alone against plain fp64 restatements: gated group norms, the logits' soft limit, heads with joint
norms and rotated neighbours, windows with a learned sink, sigmoid routing in groups, limited experts, forget-gate linear attention
and the delta rule (row by row and in blocks)."""
import pytest
import torch

import rotutar_oracle as O
from kernel_cases import BF, F32, Paged, close, ops_of, rnd
from phaseshift_b200.models.common import pad_heads
from phaseshift_b200.ops.specs import AttnSpec, DeltaSpec, GatedNorm, GlaSpec, HeadsSpec, MoeSpec
from phaseshift_b200.runtime.batch import SeqRows, StepBatch
from phaseshift_b200.runtime.state import ConvSpec, KVSpec, RecurrentSpec, RunSpec

pytestmark = pytest.mark.gpu
DTYPES = [BF, F32]


def pad_to(n, to):
    return -(-n // to) * to


def step_of(rows, padding=3):
    b = StepBatch(rows + padding, 1, torch.device("cuda:0"))
    b.fill([SeqRows(0, 0, [0] * rows)])
    b.upload()
    return b


# ------------------------------------------------------------------ norms behind the sublayers
@pytest.mark.parametrize("W,groups", [(75, 3), (75, 1), (96, 8), (200, 40), (2560, 4), (3072, 96)])
@pytest.mark.parametrize("rows", [1, 9, 70])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_norm_of_projections(W, groups, rows, dtype):
    ops, wide, width, eps = ops_of(dtype), pad_to(W, 4), pad_to(W + 1, 32), 0.3       # an eps that would show outside the root
    x, a, b = rnd(rows, W, seed=1), rnd(rows, wide, seed=2, scale=2.0), rnd(rows, wide, seed=3)
    bias, nw, fw = rnd(W, seed=5), rnd(W, seed=6), rnd(W, seed=7)
    gates = [rnd(rows, pad_to(W, 8) + 16, seed=4, dtype=d)[:, 16:] for d in ({BF, F32} if dtype == BF else {F32})]
    tol = 1e-2 if dtype == BF else 4e-6
    for gate in gates:
        for p, y in ((GatedNorm(gate, bias, nw, a, 0.7, b, -1.3), 0.7 * a.double() - 1.3 * b.double()), (GatedNorm(gate, bias, nw, a), a.double())):
            y = y[:, :W] * torch.sigmoid(gate[:, :W].double() + bias.double())
            want = x.double() + O.group_norm(y, nw.double(), eps, groups)
            xo, h = ops.gated_norm(x.clone(), p, eps=eps, groups=groups, width=width, name="h")
            close(xo, want, 2e-6)
            close(h[:, :W], want, tol)
            assert bool((h[:, W:] == 0).all())
            xo, h = ops.gated_norm(x.clone(), p, eps=eps, groups=groups, norm_w=fw, width=width, name="h")
            close(xo, want, 2e-6)
            close(h[:, :W], O.group_norm(want, fw.double(), eps, groups), tol)
            xo, h = ops.gated_norm(x.clone(), p, eps=eps, groups=groups)
            close(xo, want, 2e-6)
            assert h is None
    xo, h = ops.gated_norm(x, None, eps=eps, groups=groups, width=width, name="h")
    assert xo is x and torch.equal(h[:, :W], x.to(dtype)) and bool((h[:, W:] == 0).all())


@pytest.mark.parametrize("n,cap", [(7, 3.0), (5 * 1000, 0.5), (3 * 151936, 30.0)])
def test_soft_limit(n, cap):
    ops, z = ops_of(BF), rnd(1, n, seed=1, scale=2.0 * cap)
    want = cap * torch.tanh(z.double() / cap)
    close(ops.soft_limit(z, cap), want, 1e-6)
    assert bool((z.abs() <= cap).all())


# ------------------------------------------------------------------ attention side
@pytest.mark.parametrize("H,G,dim,vdim,rot", [(6, 2, 40, 24, 40), (8, 2, 128, 128, 32), (4, 4, 20, 100, 2), (5, 1, 300, 8, 100)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_heads_with_joint_norms_and_rotated_neighbours(H, G, dim, vdim, rot, dtype):
    D, base, eps, ops = pad_to(max(dim, vdim), 64), 700.0, 0.2, ops_of(dtype)
    seqs = [(0, 40), (37, 1), (130, 2), (5, 17)]
    pg = Paged(RunSpec(KVSpec(G, D), None), seqs, dtype)
    parts = ((H, dim), (G, dim), (G, vdim))
    nw = [1 + 0.3 * rnd(h * d, seed=60 + j) for j, (h, d) in enumerate(parts[:2])]
    spec = HeadsSpec(H, G, D, dim, vdim, eps, torch.tensor([base ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64).cuda(),
                     q_norm=pad_heads(nw[0], H, dim, D), k_norm=pad_heads(nw[1], G, dim, D))
    raw = [rnd(pg.rows, h * d, seed=j, dtype=dtype) for j, (h, d) in enumerate(parts)]
    proj = torch.cat([pad_heads(t.T.contiguous(), h, d, D).T for t, (h, d) in zip(raw, parts)] + [rnd(pg.rows, 24, seed=9, dtype=dtype)], 1).contiguous()
    got = ops.attn_heads(proj, spec, pg.b, pg.st.kv[0], pg.st).reshape(pg.rows, H, D)
    at = 0
    for i, (p, n) in enumerate(seqs):
        q, k, v = (t[at:at + n].double().cpu() for t in raw)
        q, k = O.rms_norm(q, nw[0].double().cpu(), eps), O.rms_norm(k, nw[1].double().cpu(), eps)
        turned = lambda t, h: O.turn_neighbours(torch.cat([torch.zeros(p, h, dim).double(), t.reshape(n, h, dim)]), base, rot)[p:]
        tol = 1.5e-2 if dtype == BF else 6e-6
        close(got[at:at + n, :, :dim].cpu(), turned(q, H), tol)
        t = torch.arange(p, p + n, device="cuda")
        blk = pg.st.block_table[i + 1][t // 16].long()
        close(pg.st.kv[0].k[blk, :, t % 16][..., :dim].cpu(), turned(k, G), tol)
        close(pg.st.kv[0].v[blk, :, t % 16][..., :vdim].cpu(), v.reshape(n, G, vdim), tol)
        at += n
    assert int(pg.st.status) == 0


def attention_case(H, G, D, seqs, dtype, window, graph=False, standout=None, sink=None):
    """`standout`: position whose key all queries score far above every other, so that seeing it or not decides the output; `sink`:
    the same value for every head, else random ones of the scores' size."""
    ops = ops_of(dtype)
    pg = Paged(RunSpec(KVSpec(G, D), None), seqs, dtype, graph=graph)
    scale = D ** -0.5
    sinks = torch.full((H,), sink, device="cuda") if sink is not None else 2.0 * rnd(H, seed=8) + 1.0
    spec = AttnSpec(H, G, D, scale, window=window, sink=sinks)
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
        want.append(O.attend(q.double().cpu(), k.double().cpu(), v.double().cpu(), scale, O.window_mask(p + n, window), sinks.double().cpu())[p:])
        at += n
    out = ops.attention(q_all, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
    assert int(pg.st.status) == 0 and int(ops.status) == 0
    at = 0
    for w in want:
        close(out[at:at + w.shape[0]].cpu(), w, 2e-2 if dtype == BF else 5e-6)
        at += w.shape[0]


@pytest.mark.parametrize("H,G,D", [(6, 2, 64), (4, 2, 256), (2, 1, 320), (8, 2, 128), (3, 3, 192)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_windows_with_learned_sinks(H, G, D, dtype):
    for window in (1, 16, 61, 500):
        attention_case(H, G, D, [(37, 150), (330, 1), (0, 2), (0, 1), (263, 3), (399, 16)], dtype, window)
    attention_case(H, G, D, [(127, 1), (128, 1), (60, 1), (0, 1), (900, 1)], dtype, 60, graph=True)
    attention_case(H, G, D, [(10, 40), (200, 1)], dtype, 30, sink=12.0)                          # the sink takes nearly everything


@pytest.mark.parametrize("H,G,D", [(6, 2, 64), (4, 2, 256), (2, 1, 320), (8, 2, 128)])
@pytest.mark.parametrize("standout", [0, 15, 16, 63, 64, 101])
def test_a_standout_key_counts_exactly_while_it_is_in_the_window(H, G, D, standout):
    """Rows on both sides of the edge of a window of 45, in a prompt's portion and decoded alone."""
    attention_case(H, G, D, [(40, 200), (standout, 1), (standout + 44, 1), (standout + 45, 1), (700, 1)], BF, 45, standout=standout)
    attention_case(H, G, D, [(standout, 1), (standout + 43, 4)], BF, 45, standout=standout)
    attention_case(H, G, D, [(0, 200)], F32, 45, standout=standout)


# ------------------------------------------------------------------ mixture
ROUTERS = [(12, 3, 2, 1), (16, 4, 4, 2), (1, 1, 1, 1), (60, 8, 4, 2), (256, 10, 16, 3), (40, 6, 20, 4), (7, 2, 7, 3), (9, 9, 1, 1)]


def expert_at(routed, rows, top):
    at = torch.full((rows * top,), -1)
    for e, first, count, _ in routed.tiles.cpu()[1:1 + int(routed.tiles[0, 0])].tolist():
        at[first:first + count] = e
    return at


@pytest.mark.parametrize("rows", [1, 5, 64, 65, 300])
@pytest.mark.parametrize("E,top,groups,keep", ROUTERS)
def test_sigmoid_routing_by_the_two_best_of_a_group(rows, E, top, groups, keep):
    ops, K = ops_of(BF), 96
    s = MoeSpec(E, 0, top, groups, keep, 32, 16, None, rnd(E * 64, K, dtype=BF), rnd(E * 16, 32, dtype=BF), sigmoid=True, group_top=2, renormalize=False)
    z, h = rnd(rows + 3, pad_to(E, 8), seed=4, scale=2.0), rnd(rows + 3, K, seed=5, dtype=BF)
    r = ops.moe_route(z, h, s, step_of(rows))
    assert int(ops.status) == 0
    index, weight, at = r.index.cpu(), r.weight.cpu(), expert_at(r, rows, top)
    assert bool((index[rows:] == -1).all())
    for i in range(rows):
        want = {e: float(v) for e, v in O.route(z[i, :E].double().cpu(), groups, keep, top)}
        got = {int(at[p]): float(v) for p, v in zip(index[i].tolist(), weight[i])}
        assert set(got) == set(want) and all(abs(got[e] - want[e]) < 1e-6 for e in want)
        assert all(torch.equal(r.inputs[p], h[i]) for p in index[i].tolist())


@pytest.mark.parametrize("rows", [1, 3, 17, 64, 65, 300, 700])
@pytest.mark.parametrize("E,top,ff,W,groups,K,limit", [(14, 2, 96, 223, 1, 160, 0.5), (10, 3, 64, 76, 4, 96, 2.0), (40, 8, 96, 256, 8, 320, 7.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_limited_experts_and_the_gated_norm_of_their_sum(rows, E, top, ff, W, groups, K, limit, dtype):
    """Unequal loads, experts without rows, rows of padding."""
    ops, n_out = ops_of(dtype), pad_to(W, 4)
    s = MoeSpec(E, 0, top, 1, 1, ff, n_out, None, rnd(E * 2 * ff, K, seed=1, scale=2 * K ** -0.5, dtype=dtype),
                rnd(E * n_out, ff, seed=2, scale=ff ** -0.5, dtype=dtype), sigmoid=True, group_top=2, renormalize=False, limit=limit)
    z, h, x = rnd(rows + 3, pad_to(E, 8) + pad_to(W, 8), seed=4, scale=2.0), rnd(rows + 3, K, seed=5, dtype=dtype), rnd(rows + 3, W, seed=6)
    z[:, 1] += 3.0                                                     # most rows go to one expert
    gate, bias, nw = z[:, pad_to(E, 8):], rnd(W, seed=7), rnd(W, seed=8)
    r = ops.moe_route(z, h, s, step_of(rows))
    y = ops.moe_experts(r, s)
    assert int(ops.status) == 0
    gu, dn, hd = s.gate_up.double().reshape(E, 2 * ff, K), s.down.double().reshape(E, n_out, ff), h.double()[:rows]
    sc = torch.sigmoid(z[:rows, :E].double())
    wt, ids = sc.topk(top, -1)
    want = torch.zeros(rows, n_out, device="cuda", dtype=torch.float64)
    for e in range(E):
        w = {"gate": gu[e, 0::2], "up": gu[e, 1::2], "down": dn[e]}
        want += (wt * (ids == e)).sum(-1)[:, None] * O.expert(hd, w, "", limit)
    out = want[:, :W] * torch.sigmoid(gate[:rows, :W].double() + bias.double())
    want = x[:rows].double() + O.group_norm(out, nw.double(), 0.3, groups)
    xo, hn = ops.gated_norm(x.clone(), GatedNorm(gate, bias, nw, routed=r, experts=y), eps=0.3, groups=groups, width=pad_to(W, 32), name="h")
    close(xo[:rows], want, 2e-2 if dtype == BF else 6e-6)
    close(hn[:rows, :W], want, 3e-2 if dtype == BF else 6e-6)
    close(xo[rows:], x[rows:], 1e-6)                                   # padding rows get no expert


# ------------------------------------------------------------------ recurrences
CUTS = [[150, 1, 2, 30, 1, 17], [40, 2, 64], [2, 3, 1, 1, 1, 5]]
LONG = [[300, 1, 1, 70], [1, 450], [3, 64, 1, 128]]


def steps(portions, graph=False):
    """(batch, [(sequence, first position, rows, first row)]) of every step, two padding rows behind."""
    at = [0] * len(portions)
    for step in range(max(len(p) for p in portions)):
        live = [(i, p[step]) for i, p in enumerate(portions) if step < len(p)]
        b = StepBatch(sum(c for _, c in live) + 2, 4, torch.device("cuda:0"))
        b.fill([SeqRows(i + 1, at[i], [0] * c) for i, c in live])
        b.graph_static = graph
        b.upload()
        out, r = [], 0
        for i, c in live:
            out.append((i, at[i], c, r))
            at[i], r = at[i] + c, r + c
        yield b, out


def linear_case(H, dim, vdim, portions, dtype, lower, bias, graph=False):
    dk, dv, n = pad_to(dim, 16), pad_to(vdim, 32), [sum(p) for p in portions]
    ops, eps = ops_of(dtype), 1e-3
    low = {"mixed": torch.sigmoid(2 * rnd(H * dim, seed=1)), "zero": torch.zeros(H * dim, device="cuda"), "one": torch.ones(H * dim, device="cuda")}[lower]
    fb, nw = bias + rnd(H * dim, seed=2), 1 + 0.2 * rnd(vdim, seed=3)
    lower_padded = torch.ones(H, dk, device="cuda")
    lower_padded[:, :dim] = low.reshape(H, dim)
    spec = GlaSpec(H, dk, dv, vdim, 8, -1, 8 + 2 * H * dk, -1, 8 + H * dk, 0, 1.0, 1.0, eps, None, pad_heads(fb, H, dim, dk),
                   torch.nn.functional.pad(nw, (0, dv - vdim)), lower_padded.flatten())
    parts = ((dim, dk), (dim, dk), (vdim, dv))
    raw = [[rnd(k, H * d, seed=100 * i + j, scale=1.0 if j != 1 else 2.0, dtype=dtype) for j, (d, _) in enumerate(parts)] for i, k in enumerate(n)]
    want = []
    for q, z, v in ([t.double().cpu() for t in r] for r in raw):
        f = O.forget_gate(z + fb.double().cpu(), low.double().cpu())
        o = O.forget_write(O.silu(q).reshape(-1, H, dim), f.reshape(-1, H, dim), v.reshape(-1, H, vdim))
        want.append(O.rms_norm(o, nw.double().cpu(), eps))
    pg = Paged(RunSpec(None, RecurrentSpec(H, dk, dv)), [(0, k) for k in n], dtype)
    for b, live in steps(portions, graph):
        proj = rnd(b.max_rows, 8 + H * (2 * dk + dv) + 16, seed=5, dtype=dtype)
        for i, p, c, r in live:
            proj[r:r + c, 8:8 + H * (2 * dk + dv)] = torch.cat([pad_heads(t[p:p + c].T.contiguous(), H, d, to).T for t, (d, to) in zip(raw[i], parts)], 1)
        out = ops.gla(proj, spec, b, pg.st.gdn[0], pg.st).reshape(-1, H, dv)
        for i, p, c, r in live:
            close(out[r:r + c, :, :vdim].cpu(), want[i][p:p + c], 1.2e-2 if dtype == BF else 2e-5)
            assert bool((out[r:r + c, :, vdim:] == 0).all())
    assert int(pg.st.status) == 0


@pytest.mark.parametrize("H,dim,vdim", [(2, 128, 128), (3, 64, 64), (2, 24, 40), (1, 8, 4), (2, 200, 96), (1, 272, 300)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_forget_gate_linear_attention(H, dim, vdim, dtype):
    for cuts in (CUTS, LONG):
        linear_case(H, dim, vdim, cuts, dtype, "mixed", 1.0)
    linear_case(H, dim, vdim, CUTS, dtype, "zero", -6.0)               # nearly everything is forgotten at once
    linear_case(H, dim, vdim, LONG, dtype, "zero", 7.0)                # ... or kept for a thousand tokens
    linear_case(H, dim, vdim, [[1, 1, 1, 1], [1, 1], [1, 1, 1]], dtype, "mixed", 2.0, graph=True)


def test_heads_of_one_channel():
    linear_case(3, 1, 1, CUTS, F32, "mixed", 1.0)
    linear_case(2, 1, 1, LONG, F32, "zero", -6.0)


def test_a_gate_that_never_forgets_takes_nothing_in():
    linear_case(2, 64, 64, [[90, 3], [20, 20]], BF, "one", 0.0)


def delta_case(H, G, dim, vdim, rank, taps, portions, dtype, decay="mixed", graph=False):
    """`decay`: biases of the decays' inputs; "strong" leaves nothing of a token after one or two, "weak" nearly everything."""
    up = lambda n, step: pad_to(n, 64) if n <= 128 else pad_to(n, step)
    dk, dv, r16, n, eps = up(dim, 16), up(vdim, 32), pad_to(rank, 16), [sum(p) for p in portions], 1e-4
    ops = ops_of(dtype)
    R = lambda *s, seed, scale=1.0: rnd(*s, seed=seed, scale=scale, dtype=dtype)
    parts = ((G, dim, dk), (G, dim, dk), (H, vdim, dv))
    cw = [R(h * d, taps, seed=j, scale=taps ** -0.5) for j, (h, d, _) in enumerate(parts)]
    a2, g2 = R(H * dim, rank, seed=4, scale=rank ** -0.5), R(H * vdim, rank, seed=5, scale=rank ** -0.5)
    dtb = rnd(H * dim, seed=6) + {"mixed": -2.0, "strong": 1.0, "weak": -9.0}[decay]
    alog, nw = 0.5 * rnd(H, seed=7) + (2.0 if decay == "strong" else 0.0), 1 + 0.2 * rnd(vdim, seed=8)
    q_off = 24
    b_off = q_off + 2 * G * dk + H * dv
    a_off = b_off + pad_to(H, 16)
    cols = lambda t: torch.nn.functional.pad(t, (0, r16 - rank)).contiguous()
    spec = DeltaSpec(H, G, dk, dv, dim, vdim, q_off, b_off, a_off, a_off + r16, eps,
                     torch.cat([pad_heads(c, h, d, to) for c, (h, d, to) in zip(cw, parts)], 0).T.contiguous(), cols(pad_heads(a2, H, dim, dk)),
                     pad_heads(dtb, H, dim, dk).contiguous(), torch.exp(alog), cols(pad_heads(g2, H, vdim, dv)), torch.nn.functional.pad(nw, (0, dv - vdim)))
    raw = [[R(k, h * d, seed=100 * i + j) for j, (h, d, _) in enumerate(parts)] + [R(k, H, seed=100 * i + 3)]
           + [R(k, rank, seed=100 * i + j) for j in (4, 5)] for i, k in enumerate(n)]
    c64 = lambda t: t.double().cpu()
    want = []
    for x in raw:
        q, k, v = (O.silu(O.short_conv(c64(t), c64(c))) for t, c in zip(x, cw))
        of, N = [i // (H // G) for i in range(H)], q.shape[0]
        q, k = O.unit_length(q.reshape(N, G, dim))[:, of] * dim ** -0.5, O.unit_length(k.reshape(N, G, dim))[:, of]
        g = O.decay(c64(x[4]), torch.eye(rank).double(), c64(a2), c64(alog), c64(dtb), H)
        o = O.delta_rule(q, k, v.reshape(N, H, vdim), g, torch.sigmoid(c64(x[3])))
        want.append(O.rms_norm(o, c64(nw), eps) * torch.sigmoid(c64(x[5]) @ c64(g2).T).reshape(N, H, vdim))
    pg = Paged(RunSpec(None, RecurrentSpec(H, dk, dv), ConvSpec(H * (2 * dk + dv), taps - 1)), [(0, k) for k in n], dtype)
    hist = pg.st.conv[0]
    if hist is not None:
        hist.fill_(float("nan"))                     # what lies before a sequence's start is never read
    for b, live in steps(portions, graph):
        proj = R(b.max_rows, a_off + 2 * r16 + 8, seed=9)
        for i, p, c, r in live:
            x = [t[p:p + c] for t in raw[i]]
            row = [pad_heads(t.T.contiguous(), h, d, to).T for t, (h, d, to) in zip(x, parts)]
            row += [torch.nn.functional.pad(x[3], (0, pad_to(H, 16) - H)), cols(x[4]), cols(x[5])]
            proj[r:r + c, q_off:a_off + 2 * r16] = torch.cat(row, 1)
        out = ops.delta(proj, spec, b, pg.st.gdn[0], pg.st, hist).reshape(-1, H, dv)
        for i, p, c, r in live:
            close(out[r:r + c, :, :vdim].cpu(), want[i][p:p + c], 1.2e-2 if dtype == BF else 2e-5)
            assert bool((out[r:r + c, :, vdim:] == 0).all())
    assert int(pg.st.status) == 0 and int(ops.status) == 0


@pytest.mark.parametrize("H,G,dim,vdim,rank,taps", [(4, 2, 128, 128, 128, 4), (6, 3, 64, 64, 24, 4), (4, 2, 48, 100, 24, 3), (2, 1, 100, 40, 200, 2),
                                                    (3, 3, 33, 32, 8, 1), (4, 1, 64, 128, 16, 9), (2, 2, 128, 64, 150, 7), (2, 2, 144, 96, 24, 4)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule(H, G, dim, vdim, rank, taps, dtype):
    """Sequences of different lengths cut differently, blocks and single rows in one step."""
    for cuts in (CUTS, LONG):
        delta_case(H, G, dim, vdim, rank, taps, cuts, dtype)
    delta_case(H, G, dim, vdim, rank, taps, CUTS, dtype, "strong")
    delta_case(H, G, dim, vdim, rank, taps, LONG, dtype, "weak")
    delta_case(H, G, dim, vdim, rank, taps, [[1] * 9, [1, 1], [1] * 5], dtype, graph=True)


def test_delta_rule_of_more_heads_than_fit_at_once():
    """Many heads: the scan takes 64 value columns per CTA."""
    delta_case(48, 16, 128, 128, 32, 4, [[200], [1], [70]], BF)
    delta_case(80, 16, 64, 64, 32, 4, [[130], [90], [65]], BF)
