"""The kernels behind Luvutar, each alone against plain fp64 restatements: residual streams, gelu epilogues, attention with a
window, a distance bias, a query temperature and gates (per-row, split-KV, tiled, tensor-core), latents, per-head projections,
and latent attention in both of its forms."""

import pytest
import torch

import luvutar_oracle as O
from kernel_cases import BF, F32, Paged, close, ops_of, rnd
from phaseshift_b200.models.gebuzen.weights import LinearW, QuantizedTensor
from phaseshift_b200.ops.specs import AttnSpec, LatentSpec, StreamWrite, distance_bias_table
from phaseshift_b200.runtime.state import KVSpec, RunSpec

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ residual streams
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 6, 8, 17])
@pytest.mark.parametrize("W,dtype", [(75, F32), (75, BF), (96, BF), (2560, BF)])
@pytest.mark.parametrize("rows", [1, 9, 200])
def test_stream_norm(S, W, dtype, rows):
    ops = ops_of(dtype)
    x, e = rnd(rows, S, W, seed=1), rnd(rows, W, seed=2)
    y = rnd(rows, (W + 3) // 4 * 4, seed=3, scale=3.0)                      # a projection with padding columns behind the width
    mix, out, read, w = rnd(S, S, seed=4), rnd(S, seed=5), rnd(S, seed=6), rnd(W, seed=7)
    eps, width = 0.3, (W + 31) // 32 * 32                                   # an eps that would show outside the root
    tol = 1e-2 if dtype == BF else 5e-6
    for start in (x, e[:, None].expand(-1, S, -1)):
        X = start.double().transpose(0, 1)
        for pend in (None, StreamWrite(mix, out, y)):
            want = X if pend is None else O.stream_write(X, y[:, :W].double(), mix.double(), out.double())
            u = O.stream_read(want, read.double())
            for last in (False, True):
                src = start.clone() if start is x else start
                xo, h = ops.stream_norm(src, pend, read=read, norm_w=w, eps=eps, width=width, name="h", last=last)
                close(h[:, :W], O.rms_norm(u, w.double(), eps), tol)
                assert bool((h[:, W:] == 0).all())
                if not last:
                    close(xo, want.transpose(0, 1), 2e-6 * S)
                    if pend is not None:                                    # the next write is in place
                        again, _ = ops.stream_norm(xo, pend, eps=eps)
                        assert again.data_ptr() == xo.data_ptr()
                        close(again, O.stream_write(want, y[:, :W].double(), mix.double(), out.double()).transpose(0, 1), 4e-6 * S)


# ------------------------------------------------------------------ projections
@pytest.mark.parametrize("M", [1, 2, 8, 33, 64, 65, 300])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_gelu_epilogue(M, dtype):
    """One row streams, up to 64 rows run the split-K kernel, more the tiled tensor-core GEMM; 32-bit rows the CUDA cores."""
    ops = ops_of(dtype)
    N, K = 352, 288
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, scale=2.0 * K ** -0.5, dtype=dtype)
    fmt = "bf16" if dtype == BF else "f32"
    W = LinearW(QuantizedTensor(fmt, (N, K), K, w))
    if dtype == BF:
        W.make_tiled(True)
    got = ops.linear(x, W, name="g", gelu=True)
    want = O.gelu_tanh(x.double() @ w.double().T)
    close(got, want, 1e-2 if dtype == BF else 2e-6)
    assert int(ops.status) == 0


def heads_case(M, H, N, K, xh, dtype, gate):
    ops = ops_of(dtype)
    x, w = rnd(M, H * xh, seed=1, dtype=dtype), rnd(H * N, K, seed=2, scale=K ** -0.5, dtype=dtype)
    g = rnd(M, 32 + H * N, seed=3, scale=2.0, dtype=dtype)
    out = torch.full((M, H * (N + 64)), 7.0, device="cuda", dtype=dtype)
    ops._gemm_heads(x, xh, w, H, N, K, out, N + 64, g[:, 32:] if gate else None, N)
    want = torch.einsum("mhk,hnk->mhn", x.double().reshape(M, H, xh)[..., :K], w.double().reshape(H, N, K))
    if gate:
        want = want * torch.sigmoid(g[:, 32:].double().reshape(M, H, N))
    got = out.reshape(M, H, N + 64)
    close(got[..., :N], want, 1e-2 if dtype == BF else 2e-6)
    assert bool((got[..., N:] == 7).all()) and int(ops.status) == 0        # columns between the heads stay


@pytest.mark.parametrize("M", [1, 7, 16, 40, 64, 65, 200])
@pytest.mark.parametrize("H,N,K,xh", [(3, 64, 64, 128), (5, 512, 128, 192), (2, 192, 512, 512), (1, 320, 640, 704), (40, 128, 64, 128)])
def test_projections_per_head(M, H, N, K, xh):
    for gate in (False, True):
        heads_case(M, H, N, K, xh, BF, gate)


def test_projections_per_head_in_32_bit():
    heads_case(9, 3, 64, 128, 192, F32, True)
    heads_case(70, 2, 96, 64, 64, F32, False)


# ------------------------------------------------------------------ attention options
@pytest.mark.parametrize("rows,far", [(2, 2), (2, 100), (4, 3), (14, 50), (32, 128), (32, 250), (64, 1000), (8, 4096)])
def test_bias_by_distance(rows, far):
    table = rnd(rows, 3, seed=1)
    t = distance_bias_table(table, far)
    n = 3 * far + 40
    want = table[torch.tensor([O.distance_bucket(d, rows, far) for d in range(n)], device="cuda")].T
    got = t[:, torch.arange(n, device="cuda").clamp(max=t.shape[1] - 1)]
    assert torch.equal(got, want) and t.shape[1] <= max(far, rows) + 1


def oracle_heads(q, k, v, scale, window, sink, bias, far, temp):
    """q [n, H, D], k, v [n, G, D] in fp64 on the CPU -> [n, H, D]"""
    n, H, _ = q.shape
    of = [i // (H // k.shape[1]) for i in range(H)]
    if temp is not None:
        q = q * O.query_temperature(n, *temp)[:, None, None]
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    if bias is not None:
        s = s + O.distance_bias(bias, n, far)
    seen = O.window_mask(n, window) if window else O.causal_mask(n)
    a = O.softmax(s, seen) if sink is None else O.softmax_with_sink(s, seen, sink)
    return torch.einsum("hij,jhd->ihd", a, v[:, of])


def attention_case(H, G, D, seqs, dtype, window=0, far=0, temp=None, sink=False, gate="head", page=16, graph=False, standout=None, own=True,
                   buckets=14, max_len=2048, tol=None):
    """Runs append + attention and compares with the oracle over whole sequences.  `standout`: position whose key all queries
    score far above every other, so that seeing it or not (or its bias) decides the output."""
    ops = ops_of(dtype, max_len)
    pg = Paged(RunSpec(KVSpec(G, D), None), seqs, dtype, page, graph)
    scale = D ** -0.5
    rel = rnd(buckets, H, seed=8, scale=2.0) if far else None
    sk = rnd(H, seed=9) + 1.0 if sink else None
    width = (H + 2 * G) * D
    spec = AttnSpec(H, G, D, scale, window=window, sink=sk, bias=distance_bias_table(rel, far) if far else None,
                    temp_coef=temp[0] if temp else 0.0, temp_every=temp[1] if temp else 1.0, gate_offset=width,
                    gate_per_head=gate == "head", gate_head_stride=1 if gate == "head" else D)
    proj = rnd(pg.rows, width + H * D, seed=2, scale=2.0, dtype=dtype)
    at, want = 0, []
    for i, (p, n) in enumerate(seqs):
        q, k, v = (rnd(p + n, m, D, seed=s + i, dtype=dtype) for m, s in ((H, 20), (G, 40), (G, 60)))
        if standout is not None and standout < p + n:
            u = rnd(D, seed=3).sign()
            q = (q.float() * 0.2 + 0.7 * u).to(dtype)
            k[standout] = (u * 14.0 / (0.7 * D * scale)).to(dtype)
        pg.fill_keys(i, k[:p] if own else k, v[:p] if own else v)
        proj[at:at + n, :H * D] = q[p:].reshape(n, -1)
        if own:
            proj[at:at + n, H * D:width] = torch.cat([k[p:].reshape(n, -1), v[p:].reshape(n, -1)], 1)
        o = oracle_heads(q.double().cpu(), k.double().cpu(), v.double().cpu(), scale, window, None if sk is None else sk.double().cpu(),
                         None if rel is None else rel.double().cpu(), far, temp)[p:]
        g = torch.sigmoid(proj[at:at + n, width:].double().cpu())
        want.append((o * (g[:, :H, None] if gate == "head" else g.reshape(n, H, D)) if gate else o).reshape(n, -1))
        at += n
    q = ops.attn_append(proj, spec, pg.b, pg.st.kv[0] if own else None, pg.st)
    out = ops.attention(q, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch, gate=proj if gate else None)
    assert int(pg.st.status) == 0 and int(ops.status) == 0
    at = 0
    for w in want:
        close(out[at:at + w.shape[0]].cpu(), w, tol or (2e-2 if dtype == BF else 5e-6))
        at += w.shape[0]


MIX = [(37, 150), (130, 1), (0, 2), (63, 3), (199, 16)]
HEADS = [(8, 2, 128), (4, 4, 64), (4, 4, 32), (6, 2, 96), (16, 1, 64), (4, 2, 256), (2, 1, 288), (3, 3, 192), (20, 2, 256)]


@pytest.mark.parametrize("H,G,D", HEADS)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_distance_bias_temperature_and_head_gates(H, G, D, dtype):
    """A long portion, short portions and single decoded rows together; keys of its own and of another layer."""
    attention_case(H, G, D, MIX, dtype, far=60, temp=(0.4, 24))
    attention_case(H, G, D, MIX, dtype, far=60, temp=(0.4, 24), own=False)
    attention_case(H, G, D, MIX, dtype, far=2, temp=(1.0, 1), buckets=2, gate=None)
    attention_case(H, G, D, MIX, dtype, far=300, gate=None)
    attention_case(H, G, D, MIX, dtype, temp=(-0.2, 50))


@pytest.mark.parametrize("H,G,D", HEADS)
@pytest.mark.parametrize("window", [1, 7, 64, 100])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_windows_sinks_and_elementwise_gates(H, G, D, window, dtype):
    attention_case(H, G, D, MIX, dtype, window=window, sink=True, gate="element")
    attention_case(H, G, D, MIX, dtype, window=window, far=40, temp=(0.3, 10))


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (16, 1, 64), (8, 2, 128), (4, 4, 64)])
@pytest.mark.parametrize("graph", [False, True])
def test_decoded_rows_alone(H, G, D, graph):
    rows = [(127, 1), (128, 1), (49, 1), (50, 1), (0, 1), (700, 1)]
    attention_case(H, G, D, rows, BF, far=60, temp=(0.4, 24), graph=graph)
    attention_case(H, G, D, rows, BF, window=50, sink=True, far=60, gate="element", graph=graph)


@pytest.mark.parametrize("H,G,D", [(6, 2, 96), (4, 2, 256), (2, 1, 288), (8, 2, 128), (8, 1, 64)])
@pytest.mark.parametrize("standout", [0, 15, 16, 63, 64, 99, 100, 127, 128, 199, 200])
def test_a_standout_key_counts_exactly_inside_its_window(H, G, D, standout):
    """Windows of 100: rows on both sides of the edge, of pages and of tiles, in a prompt's portion and decoded alone."""
    attention_case(H, G, D, [(90, 210), (standout, 1), (standout + 99, 1), (standout + 100, 1)], BF, window=100, standout=standout, gate=None)
    attention_case(H, G, D, [(standout, 1), (standout + 98, 4), (standout + 100, 1)], BF, window=100, standout=standout)
    attention_case(H, G, D, [(0, 260)], F32 if D != 256 else BF, window=100, standout=standout)


@pytest.mark.parametrize("H,G,D", [(4, 2, 128), (2, 1, 32), (2, 1, 288)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_the_bias_of_every_distance_is_its_own(H, G, D, dtype):
    """Keys and queries that score alike: the softmax is the bias table's, so every bucket border shows in every row."""
    ops = ops_of(dtype)
    for far in (30, 150):
        seqs = [(0, 200), (199, 1), (100, 7)]
        pg = Paged(RunSpec(KVSpec(G, D), None), seqs, dtype)
        rel = rnd(16, H, seed=8, scale=3.0)
        spec = AttnSpec(H, G, D, 1.0, bias=distance_bias_table(rel, far), gate_offset=0)
        proj = torch.zeros(pg.rows, (H + 2 * G) * D, device="cuda", dtype=dtype)
        at, want = 0, []
        for i, (p, n) in enumerate(seqs):
            v = rnd(p + n, G, D, seed=60 + i, dtype=dtype)
            pg.fill_keys(i, torch.zeros_like(v)[:p], v[:p])
            proj[at:at + n, (H + G) * D:] = v[p:].reshape(n, -1)
            zero = torch.zeros(p + n, H, D, dtype=torch.float64)
            want.append(oracle_heads(zero, zero[:, :G], v.double().cpu(), 1.0, 0, None, rel.double().cpu(), far, None)[p:].reshape(n, -1))
            at += n
        q = ops.attn_append(proj, spec, pg.b, pg.st.kv[0], pg.st)
        out = ops.attention(q, spec, pg.b, pg.st.kv[0], pg.st, pg.b.max_visible_launch)
        close(out[:at].cpu(), torch.cat(want), 1e-2 if dtype == BF else 5e-6)


@pytest.mark.parametrize("page", [16, 32, 64])
def test_page_sizes(page):
    attention_case(4, 2, 128, [(50, 200), (89, 1), (90, 1), (91, 2)], BF, far=60, temp=(0.4, 24), page=page)


# ------------------------------------------------------------------ latents
def pad64(n):
    return (n + 63) // 64 * 64


def latent_spec(H, dim, rot, vdim, q_rank, kv_rank, window, dtype, seed=0, scale=None, base=100.0, peak=1.0):
    """(spec, true weights in fp64 on the CPU): engine sizes padded with zeros, as the weights of a model are."""
    D, R, V, QR, KR = pad64(dim), pad64(rot), pad64(vdim), (q_rank + 31) // 32 * 32, pad64(kv_rank)
    uk, uv = torch.zeros(H, D, KR, device="cuda", dtype=dtype), torch.zeros(H, V, KR, device="cuda", dtype=dtype)
    uk[:, :dim, :kv_rank] = rnd(H, dim, kv_rank, seed=seed + 1, scale=peak * kv_rank ** -0.5, dtype=dtype)
    uv[:, :vdim, :kv_rank] = rnd(H, vdim, kv_rank, seed=seed + 2, scale=kv_rank ** -0.5, dtype=dtype)
    qn, kn = torch.zeros(QR, device="cuda"), torch.zeros(KR, device="cuda")
    qn[:q_rank], kn[:kv_rank] = rnd(q_rank, seed=seed + 3) * 0.2 + 1, rnd(kv_rank, seed=seed + 4) * 0.2 + 1
    inv = torch.tensor([base ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device="cuda")
    s = LatentSpec(H, D, R, rot, V, QR, q_rank, KR, kv_rank, scale or (dim + rot) ** -0.5, window, rnd(H, seed=seed + 5) + 0.5, inv, 1e-3,
                   qn, kn, uk.transpose(1, 2).reshape(H * KR, D).contiguous(), torch.cat([uk.reshape(H * D, KR), uv.reshape(H * V, KR)]).contiguous())
    return s, uk[:, :dim, :kv_rank].double().cpu(), uv[:, :vdim, :kv_rank].double().cpu()


@pytest.mark.parametrize("rot,q_rank,kv_rank", [(2, 5, 7), (22, 33, 50), (64, 64, 512), (130, 768, 600)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_latents_are_normed_turned_and_appended(rot, q_rank, kv_rank, dtype):
    ops = ops_of(dtype)
    s, _, _ = latent_spec(2, 8, rot, 8, q_rank, kv_rank, 5, dtype)
    seqs = [(3, 40), (1000, 2), (0, 1)]
    pg = Paged(RunSpec(KVSpec(1, s.row, shared=True), None), seqs, dtype)
    proj = torch.zeros(pg.rows, s.gate_off + 8, device="cuda", dtype=dtype)
    for off, n, seed in ((0, q_rank, 1), (s.c_off, kv_rank, 2), (s.c_off + s.kv_rank, rot, 3)):
        proj[:, off:off + n] = rnd(pg.rows, n, seed=seed, scale=0.05, dtype=dtype)          # eps counts
    cq = ops.latent_down(proj, s, pg.b, pg.st.kv[0], pg.st)
    p = proj.double().cpu()
    tol = 1e-2 if dtype == BF else 2e-6
    close(cq[:, :q_rank].cpu(), O.rms_norm(p[:, :q_rank], s.q_norm[:q_rank].double().cpu(), s.eps), tol)
    assert bool((cq[:, q_rank:] == 0).all()) and int(pg.st.status) == 0
    at = 0
    for i, (p0, n) in enumerate(seqs):
        pos = torch.arange(p0, p0 + n)
        got = pg.st.kv[0].k[pg.st.block_table[i + 1][pos // 16].long(), 0, (pos % 16).cuda()].cpu()
        r = slice(at, at + n)
        c = O.rms_norm(p[r, s.c_off:s.c_off + kv_rank], s.kv_norm[:kv_rank].double().cpu(), s.eps)
        ang = pos.double()[:, None] * s.inv_freq.cpu()
        x = p[r, s.c_off + s.kv_rank:s.c_off + s.kv_rank + rot]
        u, v = x[:, 0::2], x[:, 1::2]
        turned = torch.stack([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin()], -1).flatten(1)
        close(got[:, :kv_rank], c, tol)
        close(got[:, s.kv_rank:s.kv_rank + rot], turned, tol)
        assert bool((got[:, kv_rank:s.kv_rank] == 0).all()) and bool((got[:, s.kv_rank + rot:] == 0).all())
        at += n


def latent_case(H, dim, rot, vdim, kv_rank, window, seqs, dtype, page=16, graph=False, standout=None, max_len=2048, peak=1.0):
    """Cache filled with the tokens before the step, the step's own rows appended by the kernel; compared with expanded keys and
    values over whole sequences.  `standout`: position whose latent all queries score far above every other."""
    ops = ops_of(dtype, max_len)
    s, uk, uv = latent_spec(H, dim, rot, vdim, 16, kv_rank, window, dtype, peak=peak)
    pg = Paged(RunSpec(KVSpec(1, s.row, shared=True), None), seqs, dtype, page, graph)
    gate = rnd(pg.rows, s.gate_off + H * s.vdim, seed=7, scale=2.0, dtype=dtype)
    q = torch.zeros(pg.rows, H, s.dim + s.rot, device="cuda", dtype=dtype)
    at, want = 0, []
    for i, (p, n) in enumerate(seqs):
        L = p + n
        rows = torch.zeros(L, 1, s.row, device="cuda", dtype=dtype)
        rows[:, 0, :kv_rank] = rnd(L, kv_rank, seed=20 + i, dtype=dtype)
        rows[:, 0, s.kv_rank:s.kv_rank + rot] = rnd(L, rot, seed=40 + i, dtype=dtype)      # already turned
        qi = rnd(n, H, dim + rot, seed=60 + i, dtype=dtype)
        if standout is not None and standout < L:
            u = rnd(kv_rank, seed=3).sign()                            # a latent whose key in every head is what its queries ask for
            rows[standout, 0, :kv_rank] = (2.0 * u).to(dtype)
            key = torch.einsum("hdc,c->hd", uk, rows[standout, 0, :kv_rank].double().cpu())
            ask = 14.0 / s.scale * key / key.pow(2).sum(-1, keepdim=True)
            qi[..., :dim] = (0.1 * qi[..., :dim].float() + ask.float().cuda()).to(dtype)
            qi[..., dim:] = (0.1 * qi[..., dim:].float()).to(dtype)
        pg.fill_keys(i, rows)
        q[at:at + n, :, :dim], q[at:at + n, :, s.dim:s.dim + rot] = qi[..., :dim], qi[..., dim:]
        c, kr = rows[:, 0, :kv_rank].double().cpu(), rows[:, 0, s.kv_rank:s.kv_rank + rot].double().cpu()
        k, v = torch.einsum("tc,hdc->thd", c, uk), torch.einsum("tc,hvc->thv", c, uv)
        pos = torch.arange(p, L)
        ang = pos.double()[:, None] * s.inv_freq.cpu()
        x = qi[..., dim:].double().cpu()
        cs, sn = ang.cos()[:, None], ang.sin()[:, None]
        qr = torch.stack([x[..., 0::2] * cs - x[..., 1::2] * sn, x[..., 1::2] * cs + x[..., 0::2] * sn], -1).flatten(-2)
        sc = (torch.einsum("ihd,jhd->hij", qi[..., :dim].double().cpu(), k) + torch.einsum("ihr,jr->hij", qr, kr)) * s.scale
        a = O.softmax_with_sink(sc, O.window_mask(L, window)[p:], s.sink.double().cpu())
        o = torch.einsum("hij,jhv->ihv", a, v)
        g = torch.sigmoid(gate[at:at + n, s.gate_off:].double().cpu()).reshape(n, H, s.vdim)[..., :vdim]
        want.append(o * g)
        at += n
    out = ops.latent_attention(q.reshape(pg.rows, -1), s, pg.b, pg.st.kv[0], pg.st, gate)
    assert int(pg.st.status) == 0 and int(ops.status) == 0
    out = out.reshape(-1, H, s.vdim).cpu()
    at = 0
    for w in want:
        close(out[at:at + w.shape[0], :, :vdim], w, 2.5e-2 if dtype == BF else 1e-5)
        assert bool((out[at:at + w.shape[0], :, vdim:] == 0).all())
        at += w.shape[0]


# one head; odd sizes; a full-size latent in two value parts; three value groups; more than one head tile's worth of rows; 128 and
# more heads; sizes beyond the expanded kernels, beyond the decode kernel, beyond both
LATENTS = [(1, 32, 2, 32, 32), (5, 24, 8, 40, 50), (16, 128, 64, 128, 512), (6, 100, 20, 200, 180), (40, 64, 64, 64, 256), (128, 16, 16, 16, 64),
           (130, 16, 16, 16, 64), (3, 200, 40, 72, 300), (2, 64, 64, 64, 600), (2, 200, 130, 300, 600)]


@pytest.mark.parametrize("H,dim,rot,vdim,kv_rank", LATENTS)
@pytest.mark.parametrize("window", [1, 7, 64, 100, 5000])
def test_latent_attention_of_a_mixed_batch(H, dim, rot, vdim, kv_rank, window):
    latent_case(H, dim, rot, vdim, kv_rank, window, MIX, BF)


@pytest.mark.parametrize("H,dim,rot,vdim,kv_rank", LATENTS[:4] + LATENTS[-1:])
@pytest.mark.parametrize("window", [1, 50, 5000])
def test_latent_attention_in_32_bit(H, dim, rot, vdim, kv_rank, window):
    latent_case(H, dim, rot, vdim, kv_rank, window, MIX, F32)


@pytest.mark.parametrize("H,dim,rot,vdim,kv_rank", LATENTS)
@pytest.mark.parametrize("graph", [False, True])
def test_decoded_rows_of_latent_attention(H, dim, rot, vdim, kv_rank, graph):
    rows = [(127, 1), (128, 1), (49, 1), (50, 1), (0, 1), (700, 1)]
    for window in (50, 128, 5000):
        latent_case(H, dim, rot, vdim, kv_rank, window, rows, BF, graph=graph)
    latent_case(H, dim, rot, vdim, kv_rank, 90, [(200, 8)], BF, graph=graph)          # a short portion replayed from a graph


def test_long_prompts_of_several_requests():
    """Expanded rows of several sequences behind one another, starts that are no tile's, windows that reach into earlier steps."""
    latent_case(4, 128, 64, 128, 512, 100, [(37, 150), (300, 17), (0, 64), (5, 3), (511, 130)], BF)
    latent_case(4, 64, 16, 64, 128, 333, [(700, 200), (0, 129), (64, 64)], BF)


def test_windows_in_long_contexts_keep_partials_in_a_ring():
    for window in (64, 65, 200, 1000):
        latent_case(4, 64, 32, 64, 128, window, [(5000, 1), (4095, 1), (4096, 1), (3000, 5)], BF, max_len=6000)
        latent_case(4, 64, 32, 64, 128, window, [(5000, 1)], BF, max_len=6000)


@pytest.mark.parametrize("H,dim,rot,vdim,kv_rank", [(5, 24, 8, 40, 50), (16, 128, 64, 128, 512), (2, 200, 130, 300, 600)])
@pytest.mark.parametrize("standout", [0, 15, 16, 63, 64, 99, 100, 127, 128, 199])
def test_a_standout_latent_counts_exactly_inside_its_window(H, dim, rot, vdim, kv_rank, standout):
    latent_case(H, dim, rot, vdim, kv_rank, 100, [(90, 210), (standout, 1), (standout + 99, 1), (standout + 100, 1)], BF, standout=standout)
    latent_case(H, dim, rot, vdim, kv_rank, 100, [(standout, 1), (standout + 98, 4), (standout + 100, 1)], BF, standout=standout)
    if standout in (0, 64, 127):
        latent_case(H, dim, rot, vdim, kv_rank, 100, [(0, 260)], F32, standout=standout)


@pytest.mark.parametrize("page", [16, 32, 64])
def test_latent_page_sizes(page):
    latent_case(5, 24, 8, 40, 50, 90, [(50, 200), (89, 1), (90, 1), (91, 2)], BF, page=page)


def test_latent_sinks_far_above_and_far_below_every_score():
    for level in (-60.0, 60.0):
        ops = ops_of(BF)
        s, _, _ = latent_spec(3, 64, 16, 64, 16, 64, 50, BF)
        s.sink = torch.full((3,), level, device="cuda")
        pg = Paged(RunSpec(KVSpec(1, s.row, shared=True), None), [(10, 80), (40, 1)], BF)
        q, gate = rnd(pg.rows, 3 * (s.dim + s.rot), seed=1, dtype=BF), torch.full((pg.rows, s.gate_off + 3 * s.vdim), 20.0, device="cuda", dtype=BF)
        for i, n in enumerate((90, 41)):
            rows = rnd(n, 1, s.row, seed=5 + i, dtype=BF)
            rows[..., :64] = rows[..., :64].abs() + 1                         # every value is positive: a lost weight would show
            pg.fill_keys(i, rows)
        s.ukv[3 * s.dim:] = s.ukv[3 * s.dim:].abs()
        out = ops.latent_attention(q, s, pg.b, pg.st.kv[0], pg.st, gate)[:81]
        if level > 0:
            assert float(out.float().abs().max()) < 1e-6
        else:
            assert float(out.float().min()) > 0.5
