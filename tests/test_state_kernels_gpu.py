"""Matrix-state recurrences and latent attention, each kernel alone against the plain equations (tests/oracles/plain_gudutar.py)."""
import types

import pytest
import torch

from oracles import plain_gudutar as P
from sparkflash_b200.models.mixers import MatrixState, rotation_table
from sparkflash_b200.ops import rows as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    return torch.zeros(4, dtype=torch.int32, device="cuda")


def _close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-6)
    assert err < tol, float(err)


def _step(lens, starts, src, dst, tc=None):
    """The arrays of a step with these segments; ``tc``: which of them are long."""
    s, row0 = types.SimpleNamespace(), [sum(lens[:k]) for k in range(len(lens))]
    s.n, s.status = sum(lens), _status()
    s.row_pos = _i32([p0 + i for n, p0 in zip(lens, starts) for i in range(n)])
    s.row_seg = _i32([k for k, n in enumerate(lens) for _ in range(n)])
    s.seg_row0, s.seg_len, s.seg_src, s.seg_dst = _i32(row0), _i32(lens), _i32(src), _i32(dst)
    long = [k for k in range(len(lens)) if tc and tc[k]]
    short = [k for k in range(len(lens)) if k not in long]
    chunks, first = [], []
    for k in long:
        first.append(len(chunks))
        chunks += [(row0[k] + r, min(128, lens[k] - r)) for r in range(0, lens[k], 128)]
    s.nshort, s.nlong, s.nchunks = len(short), len(long), len(chunks)
    s.short_segs = _i32(short) if long else None
    s.long_seg, s.long_first = _i32(long), _i32(first + [len(chunks)])
    s.long_row0, s.long_rows = _i32([c[0] for c in chunks]), _i32([c[1] for c in chunks])
    bufs = {}

    class Scratch:
        buf = bufs

        def get(self, name, *shape):
            return bufs.setdefault(name, torch.zeros(shape, dtype=torch.bfloat16, device="cuda")).view(*shape)
    s.scratch = Scratch()
    return s


def _run_state(core, src, cols, dt, S, lens, starts, slots, tc, dtype):
    s = _step(lens, starts, *slots, tc)
    per = core.H * core.P * S.shape[3]
    for name, n, d in (("state_sums", s.nchunks * per, torch.float32), ("state_dec", s.nchunks * core.H, torch.float32),
                       ("state_rates", s.nchunks * core.H * 256, torch.float32), ("state_starts", 2 * s.nchunks * per, torch.bfloat16)):
        s.scratch.buf[name] = torch.zeros(max(1, n), dtype=d, device="cuda")
    y = torch.zeros(s.n, core.H * core.P, dtype=dtype, device="cuda")
    core.run(s, src, cols, dt, S, y)
    assert s.status.tolist()[0] == 0
    return y


# heads, groups, N, P, lengths
SIZES = [(4, 2, 32, 24, [1, 2, 33, 5]), (3, 1, 20, 7, [9, 1, 40]), (2, 2, 130, 50, [17, 3]), (5, 1, 48, 72, [128, 32, 127, 129, 1, 257]),
         (9, 1, 64, 64, [300, 2]), (2, 1, 256, 40, [130, 256]), (6, 3, 16, 8, [40])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,Pd,lens", SIZES)
def test_step_sized_decays_against_the_recurrence(H, G, N, Pd, lens, dtype):
    """Segments that start from zero and from a state; decays from almost none to almost all per token; long and short arms."""
    g = torch.Generator().manual_seed(H * N)
    n, L = sum(lens), len(lens)
    cols = (G * N, 0, 2 * G * N)                     # q, k, v somewhere in wider rows
    stride = -(-(2 * G * N + H * Pd) // 8) * 8
    src = torch.randn(n, stride, generator=g).to(dtype).cuda()
    dt = (2 * torch.randn(n, H + 3, generator=g)).to(dtype).cuda()[:, 2:]
    bias, D = torch.randn(H, generator=g) - 1, torch.randn(H, generator=g)
    A = -torch.exp(torch.linspace(-6, 2, H))
    core = MatrixState(H, G, N, Pd, A.cuda(), dtype, bias.cuda(), D.cuda())
    S = torch.zeros(2 * L, H, Pd, R.state_pad(N), device="cuda")
    S[:, :, :, :N] = torch.randn(2 * L, H, Pd, N, generator=g).cuda()
    before = S.clone()
    start = [2 * k if k % 2 else -1 for k in range(L)]
    arms = [[False] * L] + ([[x >= 32 for x in lens]] if core.tc and max(lens) >= 32 else [])
    for tc in arms:
        S.copy_(before)
        y = _run_state(core, src, cols, dt, S, lens, [0] * L, (start, [2 * k + 1 for k in range(L)]), tc, dtype)
        for k in range(L):
            rows = slice(sum(lens[:k]), sum(lens[:k]) + lens[k])
            x, d = src[rows].cpu().double(), P.softplus(dt[rows, :H].cpu().double() + bias.double())
            for h in range(H):
                i = h // (H // G)
                q, kk = x[:, cols[0] + i * N:cols[0] + (i + 1) * N], x[:, cols[1] + i * N:cols[1] + (i + 1) * N]
                v = x[:, cols[2] + h * Pd:cols[2] + (h + 1) * Pd]
                S0 = before[2 * k, h, :, :N].cpu().double().T if k % 2 else None
                o, end = P.decayed_sum(q, kk * d[:, h:h + 1], v, A[h].double() * d[:, h], S0)
                tol = 1e-5 if dtype == torch.float32 else 6e-3
                _close(y[rows, h * Pd:(h + 1) * Pd], o + D[h].double() * v, tol)
                _close(S[2 * k + 1, h, :, :N].T, end, 1e-5 if dtype == torch.float32 else 1e-4)      # inputs are exact: only the state's rounding
        assert (S[:, :, :, N:] == 0).all() and torch.equal(S[::2], before[::2])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,N,Pd,dims,lens", [(3, 32, 40, 16, [33, 1, 130]), (2, 64, 16, 64, [257]), (2, 10, 6, 4, [5, 2]), (2, 128, 136, 64, [129, 40]),
                                             (1, 16, 8, 0, [64])])
def test_constant_decays_with_turned_queries_and_keys(H, N, Pd, dims, lens, dtype):
    g = torch.Generator().manual_seed(N)
    n, L = sum(lens), len(lens)
    stride = -(-(2 * H * N + H * Pd) // 8) * 8
    src = torch.randn(n, stride, generator=g).to(dtype).cuda()
    decay = torch.linspace(0.5, 0.9995, H)
    core = MatrixState(H, H, N, Pd, decay.cuda(), dtype, rot=rotation_table(500.0, dims, 4096, "cuda") if dims else rotation_table(5.0, 2, 64, "cuda")[:, :0],
                       rot_dims=dims, k_scale=N ** -0.5)
    S = torch.zeros(2 * L, H, Pd, R.state_pad(N), device="cuda")
    for tc in [[False] * L] + ([[x >= 32 for x in lens]] if core.tc else []):
        y = _run_state(core, src, (0, H * N, 2 * H * N), None, S, lens, [0] * L, ([-1] * L, list(range(L))), tc, dtype)
        for k in range(L):
            rows = slice(sum(lens[:k]), sum(lens[:k]) + lens[k])
            x = src[rows].cpu().double()
            q = P.rotate(x[:, :H * N].reshape(-1, H, N), 500.0, dims, "half") if dims else x[:, :H * N].reshape(-1, H, N)
            kk = P.rotate(x[:, H * N:2 * H * N].reshape(-1, H, N), 500.0, dims, "half") if dims else x[:, H * N:2 * H * N].reshape(-1, H, N)
            for h in range(H):
                o, end = P.decayed_sum(q[:, h], kk[:, h] * N ** -0.5, x[:, 2 * H * N + h * Pd:2 * H * N + (h + 1) * Pd],
                                       torch.full((lens[k],), float(decay[h].double().log()), dtype=torch.float64))
                _close(y[rows, h * Pd:(h + 1) * Pd], o, 1e-5 if dtype == torch.float32 else 6e-3)
                _close(S[k, h, :, :N].T, end, 1e-5 if dtype == torch.float32 else 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_single_rows_with_their_convolution(taps, dtype):
    """Convolution, silu and recurrence of single rows in one kernel against the convolution kernel and the plain recurrence."""
    H, G, N, Pd = 4, 2, 12, 10
    C = H * Pd + 2 * G * N
    g = torch.Generator().manual_seed(taps)
    x = torch.randn(3, C + 1, generator=g).to(dtype).cuda()[:, :C]
    cw, cb = torch.randn(taps, C, generator=g).cuda(), torch.randn(C, generator=g).cuda()
    hist = torch.randn(6, taps - 1, C, generator=g).to(dtype).cuda()
    S = torch.randn(6, H, Pd, 32, generator=g).cuda()
    S[..., N:] = 0
    dt = torch.randn(3, H, generator=g).to(dtype).cuda()
    core = MatrixState(H, G, N, Pd, -torch.rand(H, generator=g).cuda(), dtype, torch.randn(H, generator=g).cuda(), torch.randn(H, generator=g).cuda())
    s = _step([1, 1, 1], [5, 0, 9], [0, -1, 4], [1, 3, 5])
    cols = (H * Pd + G * N, H * Pd, 0)
    out = []
    for fused in (True, False):
        h2, S2 = hist.clone(), S.clone()
        y = torch.zeros(3, H * Pd, dtype=dtype, device="cuda")
        if fused:
            core.run(s, x, cols, dt, S2, y, (cw, cb, h2, cols))
        else:
            u = torch.zeros(3, C, dtype=dtype, device="cuda")
            R.conv(x, cw, cb, u, h2, s, 3, R.CONV_SILU)
            want = P.silu(P.causal_conv(torch.cat([h2[0].double().cpu(), x[:1].double().cpu()]), cw.double().cpu().T, cb.double().cpu()))[-1]
            h2 = hist.clone()
            R.conv(x, cw, cb, u, h2, s, 3, R.CONV_SILU)
            if taps > 1:
                _close(u[0], want, 1e-5 if dtype == torch.float32 else 1e-2)
            core.run(s, u, cols, dt, S2, y)
        out.append((y, h2, S2))
    _close(out[0][0], out[1][0].cpu(), 1e-5 if dtype == torch.float32 else 2e-2)
    assert torch.equal(out[0][1], out[1][1])
    _close(out[0][2], out[1][2].cpu(), 1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,part", [(96, 24), (72, 72), (35, 7), (1040, 1040), (2048, 64), (4096, 1024), (520, 520)])
def test_gated_norm(width, part, dtype):
    g = torch.Generator().manual_seed(width)
    y, gate = torch.randn(5, width, generator=g).to(dtype).cuda(), torch.randn(5, width + 8, generator=g).to(dtype).cuda()[:, 8:]
    w, out, eps = 1 + torch.randn(width, generator=g).cuda(), torch.empty(5, width, dtype=dtype, device="cuda"), 1e-2
    yd, gd = y.cpu().double(), P.silu(gate.cpu().double())
    parts = lambda t: P.unit_rms(t.view(5, -1, part), eps).view(5, width)
    R.gated_norm(y, gate, w, out, part, True, eps)
    _close(out, parts(yd * gd) * w.cpu().double(), 1e-5 if dtype == torch.float32 else 1e-2)
    R.gated_norm(y, gate, None, out, part, False, eps)
    _close(out, parts(yd) * gd, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_without_a_norm_scaled_embedding_and_gelu(dtype):
    g = torch.Generator().manual_seed(3)
    for d in (40, 33):
        emb, x, h = torch.randn(7, d, generator=g).to(dtype).cuda(), torch.zeros(3, d, device="cuda"), torch.zeros(3, d, dtype=dtype, device="cuda")
        R.seam(x, 3, h=h, embed=emb, tokens=_i32([6, 0, 2]), from_embed=True, embed_scale=12.5, status=_status())
        _close(x, emb[[6, 0, 2]].cpu().double() * 12.5, 1e-6)
        assert torch.equal(h, x.to(dtype))
        y, w, b = torch.randn(3, d, generator=g).to(dtype).cuda(), torch.randn(d, generator=g).cuda(), torch.randn(d, generator=g).cuda()
        want = x.cpu().double() + P.layer_norm(y.cpu().double(), w.cpu().double(), b.cpu().double(), 1e-3)
        R.seam(x, 3, h=h, y=y, post=(w, b), eps=1e-3, status=_status())
        _close(x, want, 1e-5)
        assert torch.equal(h, x.to(dtype))
    for n, k, ff in ((2, 64, 24), (9, 40, 17), (3, 33, 8)):
        a, w = torch.randn(n, k, generator=g).to(dtype).cuda(), (torch.randn(2 * ff, k, generator=g) / k ** 0.5).to(dtype).cuda()
        out, scr = torch.empty(n, ff, dtype=dtype, device="cuda"), torch.empty(n, 2 * ff, dtype=dtype, device="cuda")
        with R.exact_matmul():
            R.gated_linear(a, w, scr, out, "gelu_tanh")
        z = a.cpu().double() @ w.cpu().double().T
        _close(out, P.gelu_tanh(z[:, :ff]) * z[:, ff:], 1e-5 if dtype == torch.float32 else 2e-2)


def test_rotation_table_is_the_rotation():
    x = torch.randn(9, 1, 12, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    cs = rotation_table(77.0, 8, 9, "cpu").double()
    want = P.rotate(x, 77.0, 8, "half")[:, 0]
    u, v = x[:, 0, :4], x[:, 0, 4:8]
    assert torch.allclose(torch.cat([u * cs[..., 0] - v * cs[..., 1], v * cs[..., 0] + u * cs[..., 1], x[:, 0, 8:]], 1), want, atol=1e-6)


# ---- latent attention ----------------------------------------------------------------------------------------------------------
def _pool(rank, rot, lens, dtype, seed=0, spread=0.5):
    """Cached vectors of lanes of these lengths in shuffled pages."""
    g = torch.Generator().manual_seed(seed)
    pages = [-(-n // 64) for n in lens]
    order = torch.randperm(sum(pages) + 2, generator=g).tolist()
    pool = (spread * torch.randn(len(order), 1, 64, rank + rot, generator=g)).to(dtype).cuda()
    table = torch.zeros(len(lens), max(pages) + 1, dtype=torch.int32)
    at = 0
    for k, p in enumerate(pages):
        table[k, :p] = torch.tensor(order[at:at + p])
        at += p
    return pool, table.cuda(), lambda k: torch.cat([pool[table[k, p].item(), 0] for p in range(pages[k])]).cpu().double()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,rot,rank", [(3, 16, 8, 24), (2, 7, 6, 13), (4, 72, 32, 48)])
def test_latent_append(H, dim, rot, rank, dtype):
    n, g = 70, torch.Generator().manual_seed(rank)
    stride = -(-(H * (dim + rot) + rank + rot) // 8) * 8
    proj, w = torch.randn(n, stride, generator=g).to(dtype).cuda(), 1 + torch.randn(rank, generator=g).cuda()
    x = proj.cpu().double()
    pool, table, read = _pool(rank, rot, [200], dtype)
    cs, first = rotation_table(50.0, rot, 256, "cuda"), 100
    R.latent_append(proj, proj[:, H * (dim + rot):], w, cs, pool, table, torch.zeros(n, dtype=torch.int32, device="cuda"), _i32(list(range(first, first + n))), n, H, dim, rot, rank, 1e-2,
                    _status())
    turned = lambda t: P.rotate(torch.cat([torch.zeros(first, *t.shape[1:], dtype=torch.float64), t]), 50.0, rot, "pairs")[first:]
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    qd = H * (dim + rot)
    q = x[:, :qd].reshape(n, H, dim + rot)
    got = proj[:, :qd].reshape(n, H, dim + rot)
    assert torch.equal(got[..., :dim].cpu().double(), q[..., :dim])
    _close(got[..., dim:], turned(q[..., dim:]), tol)
    kept = read(0)[first:first + n]
    _close(kept[:, :rank], P.unit_rms(x[:, qd:qd + rank], 1e-2) * w.cpu().double(), tol)
    _close(kept[:, rank:], turned(x[:, qd + rank:qd + rank + rot][:, None])[:, 0], tol)


def _plain_latent(q, keys, rank, pos, window, scale):
    """q [H, key] of one row, keys [positions, key]: softmax over the window, sum of the latents."""
    k = keys[max(0, pos - window + 1):pos + 1]
    e = torch.exp((q @ k.T) * scale - ((q @ k.T) * scale).max(-1, keepdim=True).values)
    return (e / e.sum(-1, keepdim=True)) @ k[:, :rank]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,rank,rot,window", [(5, 24, 8, 41), (16, 64, 32, 64), (33, 128, 16, 65), (2, 40, 8, 1), (3, 512, 64, 300), (9, 13, 6, 100)])
def test_single_rows_in_the_latent_space(H, rank, rot, window, dtype):
    """Rows at page borders and at the window's first positions; every arm of the kernel; heads merged through the output product."""
    key, lens = rank + rot, [1, 63, 64, 65, 66, 128, 129, 300, window, window + 1, window + 64]
    pool, table, read = _pool(rank, rot, lens, dtype)
    n, g = len(lens), torch.Generator().manual_seed(H)
    q = torch.randn(n, H * key, generator=g).to(dtype).cuda()
    uv = torch.randn(H, rank, 12, generator=g).to(dtype).cuda()
    pos, lane, st, scale = _i32([x - 1 for x in lens]), torch.arange(n, dtype=torch.int32, device="cuda"), _status(), key ** -0.5
    want = torch.stack([_plain_latent(q[i].view(H, key).cpu().double(), read(i), rank, lens[i] - 1, window, scale) for i in range(n)])
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    for splits in (1, 3):
        c = torch.zeros(n, H * rank, dtype=dtype, device="cuda")
        part, ml = torch.zeros(n * H * splits * rank, device="cuda"), torch.zeros(n * H * splits * 2, device="cuda")
        R.attn(q, pool, None, table, lane, pos, None, n, None, c, part, ml, H, scale, splits, st, window, rank, True)
        _close(c.view(n, H, rank), want, tol)
    out = torch.einsum("nhr,hrm->nhm", want, uv.cpu().double()).reshape(n, -1)
    o = torch.zeros(n, H * 12, dtype=dtype, device="cuda")
    R.head_proj(c, rank, uv, o, 12, n)
    _close(o, out, tol)
    if R.latent_decode_supports(dtype, rot, rank):
        parts = torch.zeros(n, 2, dtype=torch.int32, device="cuda")
        for ctas in (1, 2, 5, 11, 148):              # shares that end inside rows, at their ends, and hold several rows
            o = torch.zeros_like(o)
            part, ml = torch.full(((n + ctas) * H * rank,), float("nan"), device="cuda"), torch.full(((n + ctas) * H * 2,), float("nan"), device="cuda")
            for a in (0, 4):                         # in slices of the rows
                b = 4 if a == 0 else n
                R.latent_decode(q[a:b], pool, rank, rot, table, lane, pos, lane[a:b], b - a, H, part, ml, parts, window, ctas, sum(-(-x // 64) for x in lens), scale, st)
                R.head_proj(None, 0, uv, o, 12, b - a, lane[a:b], 2, merge=(part, ml, parts, ctas))
            _close(o, out, tol)
    assert st.tolist()[0] == 0


@pytest.mark.parametrize("dim,rot,vdim,window", [(64, 32, 56, 48), (16, 8, 24, 128), (128, 64, 128, 1), (72, 16, 80, 65), (40, 8, 64, 10000)])
def test_runs_over_multiplied_out_keys(dim, rot, vdim, window):
    """The tcgen05 arm: a run that begins at 0, runs that begin inside and past the window, more than one query tile."""
    H, rank, g = 3, 32, torch.Generator().manual_seed(dim)
    segs = [(0, 70), (37, 300), (500, 129)]                      # (first position, rows) of lanes 0, 1, 2
    key, lens, n = rank + rot, [p + m for p, m in segs], sum(m for _, m in segs)
    pool, table, read = _pool(rank, rot, lens, torch.bfloat16)
    uk, uv = (torch.randn(H, dim, rank, generator=g) / rank ** 0.5).bfloat16().cuda(), (torch.randn(H, rank, vdim, generator=g) / rank ** 0.5).bfloat16().cuda()
    stride = H * (dim + rot) + 8
    q = torch.randn(n, stride, generator=g).bfloat16().cuda()
    pages, offs, tiles, row = [], [], [], 0
    for k, (p0, m) in enumerate(segs):
        lo, hi = max(0, p0 - window + 1) // 64, (p0 + m - 1) // 64 + 1
        off = len(pages) - lo
        pages += table[k, lo:hi].tolist()
        for r in range(0, m, 256):
            tiles += [row + r, min(256, m - r)]
            offs.append(off)
        row += m
    M, st, scale = 64 * len(pages), _status(), (dim + rot) ** -0.5
    rows = torch.zeros(M, key, dtype=torch.bfloat16, device="cuda")
    R.gather_pages(pool, _i32(pages), rows, len(pages), st)
    kx, vx = torch.zeros(H, M, dim, dtype=torch.bfloat16, device="cuda"), torch.zeros(H, M, vdim, dtype=torch.bfloat16, device="cuda")
    R.expand(rows[:, :rank], uk.transpose(1, 2), kx)
    R.expand(rows[:, :rank], uv, vx)
    o = torch.zeros(n, H * vdim, dtype=torch.bfloat16, device="cuda")
    pos = _i32([p0 + i for p0, m in segs for i in range(m)])
    R.latent_attn_tc(q, stride, kx, vx, rows, rank, pos, _i32(tiles), _i32(offs), len(offs), o, H, dim, rot, vdim, window, scale, st)
    assert st.tolist()[0] == 0
    row = 0
    for k, (p0, m) in enumerate(segs):
        c = read(k)[:p0 + m]
        for h in range(H):
            kk = torch.cat([(c[:, :rank] @ uk[h].cpu().double().T).bfloat16().double(), c[:, rank:]], 1)
            vv = (c[:, :rank] @ uv[h].cpu().double()).bfloat16().double()
            qq = torch.zeros(p0 + m, dim + rot, dtype=torch.float64)
            qq[p0:] = q[row:row + m, h * (dim + rot):(h + 1) * (dim + rot)].cpu().double()
            _close(o[row:row + m, h * vdim:(h + 1) * vdim], P.window_softmax(qq, kk, vv, scale, window)[p0:], 1.5e-2)
        row += m


def test_a_key_that_stands_out_at_the_windows_edge():
    """One cached vector is the query itself, scaled up: the last position that sees it gives its latent, the next one does not."""
    H, rank, rot, window, at = 2, 64, 16, 70, 61
    pool, table, read = _pool(rank, rot, [300], torch.bfloat16, spread=0.05)
    key = rank + rot
    q1 = torch.randn(key, generator=torch.Generator().manual_seed(1)).bfloat16()
    pool[table[0, at // 64].item(), 0, at % 64] = (4 * q1).cuda()
    rows = [at, at + 1, at + window - 2, at + window - 1, at + window, at + window + 1]
    q = q1.repeat(len(rows), H).cuda()
    pos, lane, st = _i32(rows), torch.zeros(len(rows), dtype=torch.int32, device="cuda"), _status()
    ctas, parts, eye = 7, torch.zeros(len(rows), 2, dtype=torch.int32, device="cuda"), torch.eye(rank, dtype=torch.bfloat16, device="cuda").repeat(H, 1, 1)
    part, ml = torch.zeros((len(rows) + ctas) * H * rank, device="cuda"), torch.zeros((len(rows) + ctas) * H * 2, device="cuda")
    a, b = torch.zeros(len(rows), H * rank, dtype=torch.bfloat16, device="cuda"), torch.zeros(len(rows), H * rank, dtype=torch.bfloat16, device="cuda")
    R.attn(q, pool, None, table, lane, pos, None, len(rows), None, a, None, None, H, 1.0, 1, st, window, rank, True)
    R.latent_decode(q, pool, rank, rot, table, lane, pos, torch.arange(len(rows), dtype=torch.int32, device="cuda"), len(rows), H, part, ml, parts, window, ctas, 6 * 5, 1.0, st)
    R.head_proj(None, 0, eye, b, rank, len(rows), None, 0, merge=(part, ml, parts, ctas))
    for got in (a, b):
        d = (got.float().view(-1, H, rank) - 4 * q1[:rank].float().cuda()).abs().amax((1, 2))
        assert (d[:4] < 0.1).all() and (d[4:] > 1).all(), d
