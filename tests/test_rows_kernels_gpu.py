"""Row kernels of the layered decoders, each mechanism alone against the plain equations (tests/oracles/plain_fanodra.py)."""
import types

import pytest
import torch

from oracles import plain_fanodra as P
from sparkflash_b200.kv.paged import PAGE, PagedKV
from sparkflash_b200.models.mixers import log_distance_bias
from sparkflash_b200.ops import rows as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dt):
    return 2e-5 if dt == torch.float32 else 2e-2


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    return torch.zeros(4, dtype=torch.int32, device="cuda")


def _segs(lengths, src, dst, chunk=4):
    """Segment arrays as a step holds them."""
    s, row0, seg = types.SimpleNamespace(), [], []
    for k, n in enumerate(lengths):
        row0.append(len(seg)); seg += [k] * n
    c = [(k, row0[k] + r, min(chunk, n - r)) for k, n in enumerate(lengths) for r in range(0, n, chunk)]
    first = [next(i for i, x in enumerate(c) if x[0] == k) for k, _, _ in c]
    s.row_seg, s.seg_row0, s.seg_len, s.seg_src, s.seg_dst = _i32(seg), _i32(row0), _i32(lengths), _i32(src), _i32(dst)
    s.chunk_seg, s.chunk_row0, s.chunk_rows, s.chunk_first = _i32([x[0] for x in c]), _i32([x[1] for x in c]), _i32([x[2] for x in c]), _i32(first)
    s.chunks, s.summaries = len(c), int(len(c) > len(lengths))
    return s


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("d", [96, 75, 1032])
def test_seam_norms_merge_embedding_and_step_vector(dt, d):
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g)
    n, V, eps = 5, 11, 1e-4
    x, y, y2, emb = r(n, d), r(n, d).to(dt).float(), (3 * r(n, d)).to(dt).float(), r(V, d).to(dt).float()
    w = [1 + 0.3 * r(d) for _ in range(4)]
    b = [0.3 * r(d) for _ in range(2)]
    vec, tok = r(d), [3, 0, 10, 7, 3]
    merged = 0.5 * (P.rms_norm(y, w[0], eps) + P.rms_norm(y2, w[1], eps))
    want_tap = x + P.layer_norm(merged, w[2], b[0], eps)
    want_x = want_tap + emb[tok] + vec
    want_h = P.layer_norm(want_x, w[3], b[1], eps)
    c = lambda t, k=torch.float32: t.to("cuda", k)
    X, H, T = c(x), torch.zeros(n, d, dtype=dt, device="cuda"), torch.zeros(n, d, device="cuda")
    R.seam(X, n, h=H, y=c(y, dt), y2=c(y2, dt), merge_w=(c(w[0]), c(w[1])), post=(c(w[2]), c(b[0])), embed=c(emb, dt), tokens=_i32(tok),
           add_embed=True, step_vec=c(vec), tap=T, norm=(c(w[3]), c(b[1])), eps=eps, status=_status())
    assert (T.cpu() - want_tap).abs().max() < 2e-5 and (X.cpu() - want_x).abs().max() < 2e-5
    assert (H.float().cpu() - want_h).abs().max() < _tol(dt)
    # start of a step: the row is the embedding; and the last norm of selected rows
    X2, rows = torch.full((n, d), 9.0, device="cuda"), [4, 1]
    R.seam(X2, n, h=H, embed=c(emb, dt), tokens=_i32(tok), from_embed=True, norm=(c(w[3]), c(b[1])), eps=eps, status=_status())
    assert torch.equal(X2.cpu(), emb[tok])
    R.seam(X2, 2, h=H, y=c(y, dt), post=(c(w[2]), c(b[0])), norm=(c(w[3]), c(b[1])), row_map=_i32(rows), eps=eps, status=_status())
    want = P.layer_norm(emb[tok] + P.layer_norm(y, w[2], b[0], eps), w[3], b[1], eps)[rows]
    assert (H[:2].float().cpu() - want).abs().max() < _tol(dt)
    st = _status()
    R.seam(X2, n, h=H, embed=c(emb, dt), tokens=_i32([0, V, 1, 2, 3]), from_embed=True, norm=(c(w[3]), c(b[1])), eps=eps, status=st)
    assert st.tolist()[0] == 2 and st.tolist()[2] == V          # a token outside the table is reported, not read


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("taps,C", [(1, 24), (2, 40), (3, 33), (4, 512), (7, 20)])
def test_conv_portions_carry_their_inputs(dt, taps, C):
    g = torch.Generator().manual_seed(taps)
    lens = [29, 3, 17]
    xs = [torch.randn(n, C, generator=g).to(dt).float() for n in lens]
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    hist = torch.full((6, taps - 1, C), 7.0, dtype=dt, device="cuda")       # stale values: a fresh segment must not see them
    W, B = w.t().contiguous().cuda(), b.cuda()
    cuts = [[(0, 1), (1, 3), (3, 12), (12, 29)], [(0, 2), (2, 3)], [(0, 17)]]
    got, ver = [[] for _ in lens], [0, 0, 0]
    for step in range(4):
        live = [k for k in range(3) if step < len(cuts[k])]
        parts = [xs[k][slice(*cuts[k][step])] for k in live]
        seg = _segs([len(p) for p in parts], [2 * k + ver[k] if step else -1 for k in live], [2 * k + (ver[k] ^ 1) for k in live])
        x = torch.cat(parts).to("cuda", dt)
        y = torch.empty_like(x)
        for _ in range(2):          # a repeated launch gives the same result
            R.conv(x, W, B, y, hist, seg, len(x))
        for k, p in zip(live, y.float().cpu().split([len(p) for p in parts])):
            got[k].append(p); ver[k] ^= 1
    for k in range(3):
        assert (torch.cat(got[k]) - P.causal_conv(xs[k], w, b)).abs().max() < 2 * _tol(dt)
    x = xs[0].to("cuda", dt)
    y = torch.empty_like(x)
    R.conv(x, W, None, y, hist, _segs([29], [-1], [0]), 29, R.CONV_RESIDUAL)
    assert (y.float().cpu() - (xs[0] + P.causal_conv(xs[0], w))).abs().max() < 3 * _tol(dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("parts,bs,taps", [(3, 20, 2), (2, 64, 4), (1, 37, 1), (4, 128, 3)])
def test_gated_recurrence_chunks_and_single_rows(dt, parts, bs, taps):
    g = torch.Generator().manual_seed(bs)
    r = lambda *s: torch.randn(*s, generator=g)
    width, lens = parts * bs, [23, 9]
    xs, ys = [r(n, width).to(dt).float() for n in lens], [r(n, width).to(dt).float() for n in lens]
    cw, cb, lam = 0.6 * r(width, taps), 0.3 * r(width), -4 + 2 * r(width)
    ra, ri = (r(parts, bs, bs) * bs ** -0.5).to(dt).float(), (r(parts, bs, bs) * bs ** -0.5).to(dt).float()
    rb, ib = 0.5 * r(parts, bs), 0.5 * r(parts, bs)
    want = []
    for x, y in zip(xs, ys):
        u = P.causal_conv(x, cw, cb).to(dt).float()
        want.append(P.gated_recurrence(u, P.block_gate(u, ra, rb), P.block_gate(u, ri, ib), lam) * P.gelu_tanh(y))
    c = lambda t, k=torch.float32: t.to("cuda", k).contiguous()
    wg = c(torch.cat([ra, ri], 1), dt)
    decay = c(8 * P.softplus(lam.double()))
    S, hist = torch.full((4, width), 5.0, device="cuda"), torch.full((4, taps - 1, width), 5.0, dtype=dt, device="cuda")
    W, B, RB, IB = c(cw.t()), c(cb), c(rb.reshape(-1)), c(ib.reshape(-1))
    sums = torch.zeros(64 * 2 * width, device="cuda")

    def many(parts_x, parts_y, seg):
        x, y = c(torch.cat(parts_x), dt), c(torch.cat(parts_y), dt)
        n = len(x)
        u, o, gates = torch.empty_like(x), torch.empty_like(x), torch.empty(parts, n, 2 * bs, device="cuda")
        R.conv(x, W, B, u, hist, seg, n)
        for _ in range(2):          # a repeated launch gives the same result
            with R.exact_matmul():
                R.block_gates(u, wg, gates)
            R.scan(gates, RB, IB, decay, u, y, o, S, sums, seg, n, bs)
        return o.float().cpu()
    # a prompt portion of both lanes (several chunks), then single rows through the fused kernel, then a portion again
    a = [11, 2]
    got = [[p] for p in many([xs[0][:11], xs[1][:2]], [ys[0][:11], ys[1][:2]], _segs(a, [-1, -1], [0, 2])).split(a)]
    ver = 0
    for t in range(5):
        x, y = c(torch.stack([xs[0][11 + t], xs[1][2 + t]]), dt), c(torch.stack([ys[0][11 + t], ys[1][2 + t]]), dt)
        o = torch.empty_like(x)
        R.gated_step(x, y, W, B, hist, wg, RB, IB, decay, S, o, _i32([ver, 2 + ver]), _i32([ver ^ 1, 2 + (ver ^ 1)]), 2)
        for k in range(2):
            got[k].append(o[k:k + 1].float().cpu())
        ver ^= 1
    b = [7, 2]
    for k, p in enumerate(many([xs[0][16:], xs[1][7:]], [ys[0][16:], ys[1][7:]], _segs(b, [ver, 2 + ver], [ver ^ 1, 2 + (ver ^ 1)], chunk=3)).split(b)):
        got[k].append(p)
    for k in range(2):
        assert (torch.cat(got[k]) - want[k]).abs().max() < 2 * _tol(dt)


def test_recurrence_over_many_chunks_and_segments():
    """More chunks than one thread of the start-state kernel takes at once; slow and fast decays; segments of one and of many chunks."""
    g = torch.Generator().manual_seed(2)
    lens, width = [1, 700, 4, 37, 300], 40
    n = sum(lens)
    seg = _segs(lens, [-1, 3, 4, -1, 8], [0, 2, 5, 6, 9])
    u, y = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g)
    z, lam = torch.randn(2, n, width, generator=g), torch.linspace(-9, 1, width)
    S = torch.randn(10, width, generator=g)
    want, at = [], 0
    for k, m in enumerate(lens):
        r, i = torch.sigmoid(z[0, at:at + m].double()), torch.sigmoid(z[1, at:at + m].double())
        s0 = S[[-1, 3, 4, -1, 8][k]].double() if k in (1, 2, 4) else None
        want.append(P.gated_recurrence(u[at:at + m].double(), r, i, lam.double(), s0))
        at += m
    Sd, out = S.cuda(), torch.zeros(n, width, device="cuda")
    gates = torch.cat([z[0], z[1]], -1).view(1, n, 2 * width).cuda()
    zero = torch.zeros(width, device="cuda")
    R.scan(gates, zero, zero, (8 * P.softplus(lam.double())).float().cuda(), u.cuda(), y.cuda(), out, Sd, torch.zeros(2 * seg.chunks * width, device="cuda"),
           seg, n, width)
    ref = torch.cat(want)
    assert (out.cpu() - ref.float() * P.gelu_tanh(y)).abs().max() < 2e-4 * ref.abs().max()
    for k, dst in enumerate((0, 2, 5, 6, 9)):
        assert (Sd[dst].cpu() - want[k][-1].float()).abs().max() < 2e-4 * ref.abs().max()
    assert torch.equal(Sd[[1, 3, 4, 7, 8]].cpu(), S[[1, 3, 4, 7, 8]])


def _attention_case(dt, H, G, dim, vdim, lens, seed=0, scale=0.2):
    """Keys / values of several lanes in a shuffled page pool, plus queries for every position."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dt).float()
    kv = PagedKV([(G, dim, vdim)], 3 + sum(-(-n // PAGE) for n in lens), len(lens), 1024, dt, "cuda")
    case = types.SimpleNamespace(kv=kv, H=H, G=G, dim=dim, vdim=vdim, scale=scale, dt=dt)
    case.q, case.k, case.v = ([r(n, x) for n in lens] for x in (H * dim, G * dim, G * vdim))
    case.r1, case.r2 = 0.2 + torch.rand(H, generator=g), 0.1 + 2 * torch.rand(H, generator=g)
    for p in range(max(-(-n // PAGE) for n in lens)):         # pages of the lanes interleave in the pool
        for lane, n in enumerate(lens):
            kv.ensure(lane, min(n, (p + 1) * PAGE))
    return case


def _fill(case):
    kv = case.kv
    kv.upload()
    for lane, (k, v) in enumerate(zip(case.k, case.v)):
        for p, page in enumerate(kv.pages[lane]):
            kk, vv = k[p * PAGE:(p + 1) * PAGE], v[p * PAGE:(p + 1) * PAGE]
            kv.k[0][page, :, :len(kk)] = kk.view(len(kk), case.G, case.dim).transpose(0, 1).to("cuda", case.dt)
            kv.v[0][page, :, :len(vv)] = vv.view(len(vv), case.G, case.vdim).transpose(0, 1).to("cuda", case.dt)
    case.bias = log_distance_bias(case.r1, case.r2, 1024, "cuda")


def _want(case, lane):
    q, k, v, out = case.q[lane], case.k[lane], case.v[lane], []
    for h in range(case.H):
        g = h // (case.H // case.G)
        s = P.biased_scores(q[:, h * case.dim:(h + 1) * case.dim].double(), k[:, g * case.dim:(g + 1) * case.dim].double(), case.scale,
                            case.r1[h].double(), case.r2[h].double())
        out.append(torch.softmax(s, -1) @ v[:, g * case.vdim:(g + 1) * case.vdim].double())
    return torch.cat(out, -1).float()


def _run_exact(case, rows, splits):
    """rows: (lane, position) pairs."""
    q = torch.stack([case.q[a][p] for a, p in rows]).to("cuda", case.dt)
    out = torch.full((len(rows), case.H * case.vdim), 9.0, dtype=case.dt, device="cuda")
    part = torch.empty(len(rows) * case.H * splits * case.vdim, device="cuda")
    ml = torch.empty(len(rows) * case.H * splits * 2, device="cuda")
    st = _status()
    R.attn(q, case.kv.k[0], case.kv.v[0], case.kv.table, _i32([a for a, _ in rows]), _i32([p for _, p in rows]), None, len(rows), case.bias, out,
           part, ml, case.H, case.scale, splits, st)
    assert st.tolist()[0] == 0
    return out.float().cpu()


def _run_stream(case, rows, picked=None, slack=0):
    """rows: (lane, position) pairs; ``picked``: run only these of them."""
    q = torch.stack([case.q[a][p] for a, p in rows]).to("cuda", case.dt)
    out = torch.full((len(rows), case.H * case.vdim), 9.0, dtype=case.dt, device="cuda")
    n = 2 * R.STREAM_CTAS * R.attn_stream_heads(case.H, case.G, case.dim)
    part, ml, st = torch.full((n * case.vdim,), float("nan"), device="cuda"), torch.full((n * 2,), float("nan"), device="cuda"), _status()
    run = range(len(rows)) if picked is None else picked
    R.attn_stream(q, case.kv.k[0], case.kv.v[0], case.kv.table, _i32([a for a, _ in rows]), _i32([p for _, p in rows]),
                  None if picked is None else _i32(picked), len(run), case.bias, out, part, ml, case.H, case.scale,
                  slack + sum(rows[i][1] // PAGE + 1 for i in run), st)
    assert st.tolist()[0] == 0, st.tolist()
    return out.float().cpu()


def _run_tiles(case, runs):
    """runs: (lane, first position, rows) segments through the tensor-core arm."""
    lanes = [a for a, _, m in runs for _ in range(m)]
    pos = [p + i for _, p, m in runs for i in range(m)]
    q = torch.cat([case.q[a][p:p + m] for a, p, m in runs]).to("cuda", case.dt)
    tiles, row = [], 0
    for _, _, m in runs:
        for r in range(0, m, 256):
            tiles += [row + r, min(256, m - r)]
        row += m
    out = torch.full((row, case.H * case.vdim), 9.0, dtype=case.dt, device="cuda")
    st = _status()
    R.attn_tc(q, R.attn_pools(case.kv, 0, True), case.kv.table, _i32(lanes), _i32(pos), _i32(tiles), len(tiles) // 2, case.bias, out, case.H,
              case.scale, st)
    assert st.tolist()[0] == 0, st.tolist()
    return out.float().cpu()


SHAPES = [(4, 4, 64, 64), (4, 2, 40, 24), (6, 1, 16, 80), (8, 1, 128, 128), (9, 1, 24, 136), (3, 3, 10, 7), (2, 1, 96, 48)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", SHAPES)
def test_exact_attention_rows_at_page_borders_and_splits(dt, H, G, dim, vdim):
    case = _attention_case(dt, H, G, dim, vdim, [1, 64, 65, 300])
    _fill(case)
    want = [_want(case, a) for a in range(4)]
    rows = [(0, 0), (1, 0), (1, 62), (1, 63), (2, 63), (2, 64), (3, 0), (3, 63), (3, 64), (3, 127), (3, 128), (3, 191), (3, 192), (3, 299)]
    for splits in (1, 2, 3, 7):
        got = _run_exact(case, rows, splits)
        for (a, p), row in zip(rows, got):
            assert (row - want[a][p]).abs().max() < 2 * _tol(dt), (a, p, splits)


@pytest.mark.parametrize("H,G,dim,vdim", [s for s in SHAPES if s[2] % 8 == 0 and s[3] % 8 == 0 and max(s[2:]) <= 128])
def test_tensor_core_attention_runs_match_the_equations(H, G, dim, vdim):
    case = _attention_case(torch.bfloat16, H, G, dim, vdim, [700, 130, 40])
    _fill(case)
    want = [_want(case, a) for a in range(3)]
    for runs in ([(0, 0, 700)], [(1, 0, 130)], [(2, 0, 40), (0, 1, 33), (1, 97, 33)], [(0, 37, 512), (1, 64, 66)], [(0, 300, 128), (2, 5, 32)],
                 [(0, 444, 256), (1, 1, 129)]):
        got = _run_tiles(case, runs)
        for (a, p, m), o in zip(runs, got.split([m for _, _, m in runs])):
            assert (o - want[a][p:p + m]).abs().max() < 0.02, (runs, a, (o - want[a][p:p + m]).abs().max())


@pytest.mark.parametrize("H,G,dim,vdim", [(4, 4, 64, 64), (4, 2, 128, 128), (5, 1, 32, 96), (3, 1, 96, 32), (2, 1, 256, 256), (7, 1, 64, 160), (2, 2, 128, 64)])
def test_streamed_attention_of_rows_of_many_lengths(H, G, dim, vdim):
    case = _attention_case(torch.bfloat16, H, G, dim, vdim, [1, 64, 65, 1000, 300])
    _fill(case)
    want = [_want(case, a) for a in range(5)]
    many = [(a, p) for a, n in enumerate((1, 64, 65, 1000, 300)) for p in {0, n - 1, n // 2, max(0, n - 7), min(63, n - 1), min(64, n - 1)}]
    for rows in ([(3, 999)], [(0, 0)], [(0, 0), (3, 640)], [(2, 64), (1, 63), (1, 0)], many, many * 9):
        for slack in (0, 5000):                     # few CTAs, or as many as the machine takes
            got = _run_stream(case, rows, slack=slack)
            for (a, p), row in zip(rows, got):
                assert (row - want[a][p]).abs().max() < 0.03, (a, p, len(rows), slack)
    got = _run_stream(case, many, picked=[5, 1, 8])
    for i in (5, 1, 8):
        assert (got[i] - want[many[i][0]][many[i][1]]).abs().max() < 0.03
    assert (got[0] == 9).all()                      # rows that are not picked are left alone


@pytest.mark.parametrize("arm", ["exact32", "exact16", "stream", "tiles"])
def test_one_far_key_stands_out(arm):
    """One query's score against one key is far above the rest: its value must come back, wherever the key lies."""
    dt = torch.float32 if arm == "exact32" else torch.bfloat16
    _run_rows = (lambda c, rows, _: _run_stream(c, rows)) if arm == "stream" else _run_exact
    VD = 32
    for key in (0, 1, 63, 64, 65, 127, 128, 255, 256, 383, 384, 510, 511):
        case = _attention_case(dt, 2, 1, 32, VD, [512], seed=key, scale=1.0)
        q = 511 if key % 2 else max(key, 480)
        case.k[0][key] = 0
        case.k[0][key, :4] = 6.0
        case.q[0][:, :] *= 0.1
        case.q[0][q].view(2, 32)[:, :4] = 3.0                   # score 72 against the key, a few at most against any other
        _fill(case)
        got = _run_tiles(case, [(0, 400, 112)])[q - 400] if arm == "tiles" else _run_rows(case, [(0, q)], 3)[0]
        assert (got.view(2, VD) - case.v[0][key]).abs().max() < 0.02, (arm, key)
        # the row before the key does not see it
        if 0 < key < 511 and arm != "tiles":
            case.q[0][key - 1].view(2, 32)[:, :4] = 3.0
            assert (_run_rows(case, [(0, key - 1)], 2)[0].view(2, VD) - case.v[0][key]).abs().max() > 0.5
        if arm == "tiles" and key > 460:
            case.q[0][key - 1].view(2, 32)[:, :4] = 3.0
            assert (_run_tiles(case, [(0, 400, 112)])[key - 1 - 400].view(2, VD) - case.v[0][key]).abs().max() > 0.5


def test_large_scores_and_rising_maxima():
    """Scores that rise along the sequence make every tile move the running maximum (the rescale path of both arms)."""
    case = _attention_case(torch.bfloat16, 2, 2, 64, 64, [600], scale=1.0)
    ramp = torch.linspace(0.0, 60.0, 600)
    case.k[0] = (case.k[0] * 0.05).to(torch.bfloat16).float()
    case.k[0].view(600, 2, 64)[:, :, 0] = ramp[:, None].to(torch.bfloat16).float()
    case.q[0].view(600, 2, 64)[:, :, 0] = 1.0
    _fill(case)
    want = _want(case, 0)
    assert (_run_tiles(case, [(0, 0, 600)]) - want).abs().max() < 0.02
    for run in (lambda r: _run_exact(case, r, 4), lambda r: _run_stream(case, r)):
        assert (run([(0, p) for p in (63, 200, 599)]) - want[[63, 200, 599]]).abs().max() < 0.02


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 40, 24), (3, 1, 10, 7)])
def test_query_key_norm_covers_the_whole_projection(dt, H, G, dim, vdim):
    g = torch.Generator().manual_seed(1)
    n, eps = 70, 1e-3
    kv = PagedKV([(G, dim, vdim)], 4, 2, 256, dt, "cuda")
    kv.ensure(1, 130)
    kv.upload()
    HD, GD, GV = H * dim, G * dim, G * vdim
    proj = torch.randn(n, HD + GD + GV + 12, generator=g).to(dt).float()
    qw, kw = 1 + 0.3 * torch.randn(HD, generator=g), 1 + 0.3 * torch.randn(GD, generator=g)
    q, st, pos = torch.zeros(n, HD, dtype=dt, device="cuda"), _status(), list(range(60, 130))
    R.qk_append(proj.to("cuda", dt), qw.cuda(), kw.cuda(), q, kv.k[0], kv.v[0], kv.table, _i32([1] * n), _i32(pos), n, H, eps, st)
    assert st.tolist()[0] == 0
    assert (q.float().cpu() - P.rms_norm(proj[:, :HD], qw, eps)).abs().max() < 2 * _tol(dt)
    k = P.rms_norm(proj[:, HD:HD + GD], kw, eps).view(n, G, dim)
    v = proj[:, HD + GD:HD + GD + GV].view(n, G, vdim)
    for i, p in enumerate(pos):
        page = kv.pages[1][p // PAGE]
        assert (kv.k[0][page, :, p % PAGE].float().cpu() - k[i]).abs().max() < 2 * _tol(dt)
        assert torch.equal(kv.v[0][page, :, p % PAGE].float().cpu(), v[i])


@pytest.mark.parametrize("M,K", [(40, 64), (33, 24), (2048, 2048), (96, 5128), (4100, 512)])
def test_few_row_products(M, K):
    g = torch.Generator().manual_seed(M)
    for n in (1, 2, 3, 4):
        x, w, b = torch.randn(n, K, generator=g).bfloat16(), (torch.randn(M, K, generator=g) * K ** -0.5).bfloat16(), torch.randn(M, generator=g).bfloat16()
        want = x.double() @ w.double().T
        out = torch.zeros(n, M, dtype=torch.bfloat16, device="cuda")
        assert R._gemv_takes(x)
        R.linear(x.cuda(), w.cuda(), b.cuda(), out)
        assert (out.cpu().double() - want - b.double()).abs().max() < 0.04
        logits = torch.zeros(n, M, device="cuda")
        R.head(x.cuda(), w.cuda(), logits)
        assert (logits.cpu().double() - want).abs().max() < 1e-4
        if M % 2 == 0:
            act = torch.zeros(n, M // 2, dtype=torch.bfloat16, device="cuda")
            R.gated_linear(x.cuda(), w.cuda(), None, act)
            assert (act.cpu().double() - P.silu(want[:, :M // 2]) * want[:, M // 2:]).abs().max() < 0.08
