"""Residual streams, attention with normed heads, latent attention with a query latent, halves and an output gate, ungated activations, and the
grouped choice of experts: each alone against the plain equations (tests/oracles/plain_dironex.py)."""
import pytest
import torch

from oracles import plain_dironex as P
from sparkflash_b200.kv.paged import PAGE, PagedKV
from sparkflash_b200.models.mixers import LatentAttention, MixtureFF, SingleFF, W, rotation_table
from sparkflash_b200.ops import rows as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    return torch.zeros(4, dtype=torch.int32, device="cuda")


def _tol(dt):
    return 3e-5 if dt == torch.float32 else 2e-2


def _dev(t, dt=torch.float32):
    return t.to("cuda", dt).contiguous()


# ---- residual streams -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n,d,S,parts", [(5, 96, 4, 3), (4, 75, 1, 1), (3, 2056, 3, 9), (400, 64, 2, 2), (310, 1160, 4, 4), (7, 130, 5, 2), (330, 4100, 8, 1), (2, 520, 7, 1)])
def test_seam_over_streams(n, d, S, parts, dt):
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g)
    rounded = lambda *s: r(*s).to(dt).double()
    embed, tok, eps, scale = rounded(11, d), torch.randint(0, 11, (n,), generator=g), 1e-4, 1.5
    into, mix, out, w = r(S) + 0.5, r(S, S) * 0.5, r(S), 1 + 0.3 * r(d)
    x, h, tap, st = torch.full((n, S, d), 9.0, device="cuda"), torch.zeros(n, d, dtype=dt, device="cuda"), torch.zeros(n, d, device="cuda"), _status()
    common = dict(h=h, norm=_dev(w), into=_dev(into), eps=eps, status=st)
    heads = lambda X: P.rms(P.collapse(X, into.double()), w.double(), eps)
    R.stream_seam(x, n, embed=_dev(embed, dt), tokens=_i32(tok.tolist()), embed_scale=scale, **common)
    X = (embed[tok] * scale).expand(S, n, d)
    close = lambda a, b, t: (a.double().cpu() - b).abs().max() < t * max(1.0, float(b.abs().max()))
    assert close(x.transpose(0, 1), X, 1e-6) and close(h, heads(X), _tol(dt))
    y, z, wt = rounded(n, d), rounded(n, parts, d), torch.rand(n, parts, generator=g)
    R.stream_seam(x, n, y=_dev(y, dt), mix=_dev(mix), out=_dev(out), tap=tap, **common)
    X = P.spread(X, mix.double(), out.double(), 1.0, y)
    assert close(x.transpose(0, 1), X, 1e-6) and close(h, heads(X), _tol(dt)) and close(tap, X.sum(0), 1e-6)
    R.stream_seam(x, n, y=_dev(z, dt), parts_w=_dev(wt), mix=_dev(mix), out=_dev(out), **common)
    X = P.spread(X, mix.double(), out.double(), 1.0, (wt.double()[..., None] * z).sum(1))
    assert close(x.transpose(0, 1), X, 2e-6) and close(h, heads(X), _tol(dt))
    # the end: chosen rows, all streams as they are, nothing stored
    pick, before = [n - 1, 0, n // 2], x.clone()
    last = torch.zeros(3, d, dtype=dt, device="cuda")
    R.stream_seam(x, 3, h=last, norm=_dev(w), y=_dev(y, dt), mix=_dev(mix), out=_dev(out), row_map=_i32(pick), keep=False, eps=eps, status=st)
    X = P.spread(X, mix.double(), out.double(), 1.0, y)
    assert close(last, P.rms(X.sum(0), w.double(), eps)[pick], _tol(dt)) and torch.equal(x, before) and st.tolist()[0] == 0
    R.stream_seam(x, n, embed=_dev(embed, dt), tokens=_i32([11] * n), **common)
    assert st.tolist()[0] == 2


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("d,S,taps", [(64, 2, 4), (75, 3, 1), (1100, 4, 3), (96, 1, 8), (2052, 2, 2)])
def test_seam_over_streams_carries_the_convolution(d, S, taps, dt):
    """Three lanes row by row: the convolution's inputs go from version to version as the plain convolution over the whole sequence has them."""
    g, lanes, T, eps = torch.Generator().manual_seed(d), 3, 11, 1e-5
    r = lambda *s: torch.randn(*s, generator=g)
    embed, tok, w, cw = r(9, d).to(dt).double(), torch.randint(0, 9, (lanes, T), generator=g), 1 + 0.3 * r(d), 0.5 * r(d, taps)
    into, hist = r(S), torch.full((2 * lanes, taps - 1, d), 7.0, dtype=dt, device="cuda")
    x, h, st, got = torch.zeros(lanes, S, d, device="cuda"), torch.zeros(lanes, d, dtype=dt, device="cuda"), _status(), []
    for t in range(T):
        src, dst = [2 * a + (t + 1) % 2 if t else -1 for a in range(lanes)], [2 * a + t % 2 for a in range(lanes)]
        R.stream_seam(x, lanes, h=h, norm=_dev(w), into=_dev(into), embed=_dev(embed, dt), tokens=_i32(tok[:, t].tolist()),
                      conv=(_dev(cw.t()), hist, _i32(src), _i32(dst)), eps=eps, status=st)
        got.append(h.double().cpu())
    for a in range(lanes):
        hs = P.rms(P.collapse(embed[tok[a]].expand(S, T, d), into.double()), w.double(), eps).to(dt).double()
        want = P.input_convolution(hs, cw.double())
        assert (torch.stack(got)[:, a] - want).abs().max() < _tol(dt) * max(1.0, float(want.abs().max()))


# ---- heads normed one by one -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 32, 16), (3, 1, 10, 7), (2, 2, 512, 40), (6, 3, 20, 12), (16, 4, 128, 128), (5, 5, 300, 8), (2, 1, 37, 64)])
def test_append_norms_every_head(H, G, dim, vdim, dt):
    g = torch.Generator().manual_seed(dim)
    lens, cols, eps = [70, 3, 129], H * dim + G * (dim + vdim), 1e-3
    kv = PagedKV([(G, dim, vdim)], 8, 3, 256, dt, "cuda")
    for lane, n in ((2, 64), (0, 70), (1, 3), (2, 129)):
        kv.ensure(lane, n)
    kv.upload()
    xs = [(torch.randn(n, cols, generator=g) * torch.rand(n, 1, generator=g)).to(dt).double() for n in lens]
    where = [(a, p) for a, n in enumerate(lens) for p in range(n)]
    qw, kw = 1 + torch.randn(dim, generator=g), 1 + torch.randn(dim, generator=g)
    proj, st = torch.nn.functional.pad(torch.cat(xs), (0, 5)).to("cuda", dt), _status()      # a wider row
    q = torch.empty(len(where), H * dim, dtype=dt, device="cuda")
    R.head_append(proj, _dev(qw), _dev(kw), q, kv.k[0], kv.v[0], kv.table, _i32([a for a, _ in where]), _i32([p for _, p in where]), len(where), H, eps, st)
    assert st.tolist()[0] == 0
    row = 0
    for a, x in enumerate(xs):
        n = len(x)
        want_q, want_k = (P.rms(x[:, i:i + m * dim].view(n, m, dim), w.double(), eps).view(n, -1) for i, m, w in ((0, H, qw), (H * dim, G, kw)))
        pool = lambda t, width: torch.cat([t[p].transpose(0, 1).reshape(PAGE, G * width) for p in kv.pages[a]])[:n].double().cpu()
        for got, want in ((q[row:row + n].double().cpu(), want_q), (pool(kv.k[0], dim), want_k), (pool(kv.v[0], vdim), x[:, (H + G) * dim:])):
            assert (got - want).abs().max() < _tol(dt) * max(1.0, float(want.abs().max()))
        row += n


# ---- ungated activations -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("p,q", [(0.3, -0.7), (-4.0, 3.0)])
def test_xielu_near_zero_and_far_out(p, q, dt):
    z = torch.cat([torch.linspace(-30, 8, 1001), torch.tensor([-0.75, -0.7501, -0.7499, -0.0625, -0.0628, -0.062, 0.0, -0.0, 1e-6, -1e-6, -1e-4, -3e-3, -100.0])]).to(dt)
    P_, Q_ = torch.tensor(p, dtype=torch.float64), torch.tensor(q, dtype=torch.float64)
    want = P.xielu(z.double(), P_, Q_)
    got = R.act_rows(_dev(z, dt), torch.empty(len(z), dtype=dt, device="cuda"), "xielu", float(P.softplus(P_)), 0.5 + float(P.softplus(Q_))).double().cpu()
    off, rest = (got - want).abs(), 2e-7 * (1 + Q_.exp()) * z.double().abs()           # rest: the difference of two large terms far below 0
    assert (off <= (2e-6 if dt == torch.float32 else 4e-3) * want.abs() + rest).all(), off.max()
    got = R.act_rows(_dev(z, dt), torch.empty(len(z), dtype=dt, device="cuda"), "relu2").double().cpu()
    assert ((got - z.double().clamp(min=0) ** 2).abs() <= 4e-3 * z.double() ** 2).all()


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n,d,ff", [(1, 64, 40), (4, 96, 264), (3, 37, 11), (70, 64, 72), (9, 520, 33)])
def test_dense_feed_forward(n, d, ff, dt):
    g = torch.Generator().manual_seed(ff)
    w = {"up": 2 * torch.randn(ff, d, generator=g) * d ** -0.5, "down": torch.randn(d, ff, generator=g) * ff ** -0.5, "act": torch.tensor([0.4, -0.9])}
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    h, s = torch.randn(n, d, generator=g).to(dt), _Step(n)
    a, b = (P.softplus(w["act"].double()) + torch.tensor([0.0, 0.5])).tolist()
    ff_ = SingleFF(W(w, "", dt, "cuda"), "xielu", a, b)
    ff_.reserve(s)
    s.reserve("y", n * d, dt)
    with R.exact_matmul():
        got = ff_.run(s, h.cuda())
    want = P.dense(h.double(), {k: v.double() for k, v in w.items()}, "")
    assert (got.double().cpu() - want).abs().max() < _tol(dt) * max(1.0, float(want.abs().max()))


class _Step:
    """A step of n rows, its engine and its scratch in one."""

    def __init__(self, n):
        self.n, self.max_rows, self.status, self.buf = n, n + 3, _status(), {}
        self.scratch = self

    def reserve(self, name, n, dt):
        if name not in self.buf or self.buf[name].numel() < n:
            self.buf[name] = torch.zeros(n, dtype=dt, device="cuda")

    def get(self, name, *shape):
        n = 1
        for k in shape:
            n *= k
        return self.buf[name][:n].view(*shape)


# ---- experts -----------------------------------------------------------------------------------------------------------------
# width, experts, choices, ff, groups, kept
MOES = [(64, 16, 2, 24, 4, 2), (96, 6, 6, 200, 1, 1), (40, 40, 3, 136, 20, 2), (37, 6, 2, 11, 3, 2), (320, 4, 1, 64, 2, 1), (520, 130, 8, 264, 10, 3), (24, 512, 4, 8, 8, 5),
        (32, 320, 2, 16, 160, 7), (64, 5, 2, 40, 5, 3), (48, 64, 8, 520, 1, 1), (64, 32, 4, 16, 8, 4),
        (32, 256, 6, 16, 8, 3), (32, 40, 3, 24, 10, 4)]


def _moe(d, E, top, ff, count, keep, n, dt, scale=1.7):
    g = torch.Generator().manual_seed(d + n)
    w = {f"e{i}.{x}": (torch.randn(*((d, ff) if x == "down" else (ff, d)), generator=g) * (ff if x == "down" else d) ** -0.5).to(torch.bfloat16)
         for i in range(E) for x in ("up", "down")}
    w["router"], w["correction"] = (2 * torch.randn(E, d, generator=g) * d ** -0.5).to(torch.bfloat16), (0.3 * torch.randn(E, generator=g) - 0.7).to(torch.bfloat16)
    spec = {"router": {"experts": E, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}, "expert": {"ff": ff}}
    choice = R.Choice(_dev(w["correction"]), count, keep, scale)
    return w, spec, MixtureFF(W({"p." + k: v for k, v in w.items()}, "p.", dt, "cuda"), spec, act="relu2", choice=choice), torch.randn(n, d, generator=g).to(dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n", [1, 3, 9, 260])
@pytest.mark.parametrize("d,E,top,ff,count,keep", MOES)
def test_mixture_of_experts(d, E, top, ff, count, keep, n, dt):
    w, spec, moe, h = _moe(d, E, top, ff, count, keep, n, dt)
    s = _Step(n)
    moe.reserve(s)
    assert moe.tc == (dt == torch.bfloat16 and d % 8 == ff % 8 == 0) and moe.slots == top
    with R.exact_matmul():
        parts, wts = moe.run(s, h.cuda())
    assert s.status.tolist()[0] == 0
    w64, near = {k: v.double() for k, v in w.items()}, []
    want_ids, want_w = P.route(h.double() @ w64["router"].T, w64["correction"], spec["router"], near)
    ids = s.get("moe_ids", n, top).cpu()
    for t in range(n):
        if near[t] < 1e-5:
            continue
        assert sorted(ids[t].tolist()) == sorted(want_ids[t])
        by = dict(zip(want_ids[t], want_w[t].tolist()))
        assert all(abs(by[e] - x) < 1e-5 for e, x in zip(ids[t].tolist(), wts[t].tolist()))
    for e in ids.unique().tolist():                # every part against its expert
        at = (ids == e).nonzero()
        want = P.expert(h[at[:, 0]].double(), w64, f"e{e}.")
        got = parts[at[:, 0].cuda(), at[:, 1].cuda()].double().cpu()
        assert (got - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max())), e


@pytest.mark.parametrize("n", [2, 50, 200])
def test_choice_scores_below_zero_and_groups_left_out(n):
    """The correction pushes every choice score below 0, the kept group's lowest; the weights do not know the correction.  By all three routes."""
    E, top = 6, 2
    w, spec, moe, h = _moe(64, E, top, 24, 3, 1, n, torch.bfloat16, 2.0)
    w["router"].zero_()
    corr = torch.tensor([-1.5, -3.0, -2.0, -2.25, -4.0, -4.0])
    moe = MixtureFF(W(w, "", torch.bfloat16, "cuda"), spec, act="relu2", choice=R.Choice(_dev(corr), 3, 1, 2.0))
    s = _Step(n)
    moe.reserve(s)
    _, wts = moe.run(s, h.cuda())
    assert (s.get("moe_ids", n, top).cpu() == torch.tensor([2, 3])).all() and (wts == 1.0).all()


# ---- latent attention ----------------------------------------------------------------------------------------------------------
class _Engine:
    """What a latent layer needs of an engine: lanes in a shuffled page pool and a step's arrays."""

    def __init__(self, mixer, lens, max_context, max_rows, max_lanes):
        self.max_context, self.max_rows, self.max_lanes = max_context, max_rows, max_lanes
        from sparkflash_b200.models.layered import LayeredEngine, Scratch
        self.scratch, self.n_pages = Scratch("cuda"), sum(-(-x // PAGE) for x in lens) + 3
        self.short_rows, self.expanded_rows = (lambda tc: LayeredEngine.short_rows(self, tc)), (lambda w: LayeredEngine.expanded_rows(self, w))
        self.splits = lambda *a: LayeredEngine.splits(self, *a)
        self._iota = torch.arange(max_rows, dtype=torch.int32, device="cuda")
        self.kv = PagedKV([mixer.kv_run], self.n_pages, len(lens), max_context, mixer.w_in.dtype, "cuda")
        for p in range(max(-(-n // PAGE) for n in lens)):
            for lane, n in enumerate(lens):
                self.kv.ensure(lane, min(n, (p + 1) * PAGE))
        self.kv.upload()
        mixer.reserve(self)


def _latent_step(e, segs, tiles):
    """Step arrays of [(lane, first position, rows)]; ``tiles``: runs of 32 rows and more go to the tensor-core arm."""
    from sparkflash_b200.models.layered import Step, _bucket
    s = Step()
    s.engine, s.scratch, s.status, s.table = e, e.scratch, _status(), e.kv.table
    s.n = sum(m for _, _, m in segs)
    s.row_lane, s.row_pos = _i32([a for a, _, m in segs for _ in range(m)]), _i32([p + i for _, p, m in segs for i in range(m)])
    short, cut, pages, offs, row = [], [], [], [], 0
    for lane, p0, m in segs:
        if tiles and m >= 32:
            off = len(pages)
            pages += e.kv.pages[lane][:(p0 + m - 1) // PAGE + 1]
            for r in range(0, m, 256):
                cut += [row + r, min(256, m - r)]
                offs.append(off)
        else:
            short += range(row, row + m)
        row += m
    s.ntiles, s.short, s.tiles, s.short_rows = len(offs), len(short), _i32(cut or [0]), _i32(short) if offs else None
    if offs and not short:
        s.short_rows = None
    s.expand = {e.max_context: (_i32(pages or [0]), len(pages), _i32(offs or [0]))}
    s.pages = _bucket(max(p + m - 1 for _, p, m in segs) // PAGE + 1)
    return s


LATENTS = [P.latent(4, 64, 32, 64, 64, 48, 0.12, 1e3, (8.0, 64, 32.0, 1.0)), P.latent(3, 7, 6, 5, 13, 9, 0.3, 50.0), P.latent(18, 40, 16, 24, 128, 72, 0.1, 2e3, (2.0, 256, 8.0, 2.0)),
           P.latent(2, 128, 64, 128, 512, 100, 0.05, 1e4, (4.0, 300, 16.0, 1.0)), P.latent(33, 16, 8, 16, 24, 12, 0.3, 300.0)]


def _latent_weights(m, d, seed):
    cfg = P.make_config(5, d, 1, 1, 1.0, 1.0, [{"type": "latent_attention", "mixer": m}])
    return {k[7:]: v for k, v in P.make_weights(cfg, seed).items() if k.startswith("l0.mix.")}


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("k", range(len(LATENTS)))
def test_latent_layer_in_portions_and_single_rows(k, dt):
    """The whole mixer, three lanes: one whole, one in portions beside it, one row by row; against the equations over the whole sequence."""
    m, d, lens = LATENTS[k]["mixer"], 72, [150, 300, 97]
    w = _latent_weights(m, d, k)
    xs = [torch.randn(n, d, generator=torch.Generator().manual_seed(n)).to(dt) for n in lens]
    want = [P.latent_attention(x.double(), {"m." + n: t.double() for n, t in w.items()}, "m.", m, 1e-4) for x in xs]
    mixer = LatentAttention(W(w, "", dt, "cuda"), m, 1e-4, 384, halves=True, gated=True)
    assert mixer.tc == mixer.dec == (dt == torch.bfloat16 and k != 1)
    e = _Engine(mixer, lens, 384, 400, 3)
    e.scratch.reserve("y", 400 * d, dt)
    e.scratch.allocate()
    at = [0, 0, 0]
    for sizes in ((150, 64, 0), (0, 1, 2), (0, 33, 90), (0, 200, 1), (0, 2, 1), (0, 0, 3)):
        segs = [(lane, at[lane], n) for lane, n in enumerate(sizes) if n]
        s = _latent_step(e, segs, mixer.tc)
        h = torch.cat([xs[a][p:p + n] for a, p, n in segs]).cuda()
        with R.exact_matmul():
            y, _ = mixer.run(s, h, {"kv": e.kv.k[0]})
        assert s.status.tolist()[0] == 0
        for (a, p, n), got in zip(segs, y.split([n for _, _, n in segs])):
            ref = want[a][p:p + n]
            assert (got.double().cpu() - ref).abs().max() < (1e-4 if dt == torch.float32 else 4e-2) * max(1.0, float(ref.abs().max())), (a, p, n)
            at[a] += n
    assert at == lens


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("direct", [False, True])
@pytest.mark.parametrize("halves", [False, True])
@pytest.mark.parametrize("H,dim,rot,rank,q_rank", [(3, 16, 8, 24, 20), (2, 7, 6, 13, 9), (4, 72, 32, 48, 64), (2, 8, 4, 8, 6)])
def test_latents_are_normed_and_parts_turned(H, dim, rot, rank, q_rank, halves, direct, dt):
    """Both layouts, queries beside the latent or out of one of their own."""
    n, g, first, eps, base = 70, torch.Generator().manual_seed(rank), 100, 1e-2, 50.0
    proj = torch.randn(n, -(-(rank + rot + q_rank) // 8) * 8, generator=g).to(dt).cuda()
    heads = torch.randn(n, H * (dim + rot), generator=g).to(dt).cuda()
    w, wq = 1 + torch.randn(rank, generator=g), 1 + torch.randn(q_rank, generator=g)
    x, q0 = proj.cpu().double(), heads.cpu().double()
    kv = PagedKV([(1, rank + rot, 0)], 6, 1, 256, dt, "cuda")
    kv.ensure(0, 200)
    kv.upload()
    cs, pos, st = rotation_table(base, rot, 256, "cuda"), _i32(list(range(first, first + n))), _status()
    cq = torch.zeros(n, q_rank, dtype=dt, device="cuda")
    latent = dict(cq=proj[:, rank + rot:], wq=_dev(wq), cq_out=cq) if not direct else {}
    R.latent_append(heads if direct else None, proj, _dev(w), cs, kv.k[0], kv.table, torch.zeros(n, dtype=torch.int32, device="cuda"), pos, n, H, dim, rot, rank, eps, st,
                    halves, **latent)
    if not direct:
        R.latent_turn(heads, cs, pos, n, H, dim, rot, halves)

    def turned(t):                                 # neighbours: the same turn after the pairs have been brought apart
        t = torch.cat([torch.zeros(first, *t.shape[1:], dtype=torch.float64), t])
        if halves:
            return P.turn(t, base, rot)[first:]
        out = P.turn(torch.cat([t[..., 0::2], t[..., 1::2]], -1), base, rot)[first:]
        return torch.stack([out[..., :rot // 2], out[..., rot // 2:]], -1).flatten(-2)
    close = lambda a, b: (a.double().cpu() - b).abs().max() < _tol(dt) * max(1.0, float(b.abs().max()))
    got, want = heads.view(n, H, dim + rot), q0.view(n, H, dim + rot)
    assert torch.equal(got[..., :dim].cpu().double(), want[..., :dim]) and close(got[..., dim:], turned(want[..., dim:]))
    kept = torch.cat([kv.k[0][p, 0] for p in kv.pages[0]])[first:first + n]
    assert close(kept[:, :rank], P.rms(x[:, :rank], w.double(), eps)) and close(kept[:, rank:], turned(x[:, None, rank:rank + rot])[:, 0]) and st.tolist()[0] == 0
    if not direct:
        assert close(cq, P.rms(x[:, rank + rot:rank + rot + q_rank], wq.double(), eps))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,rank,rot", [(2, 64, 16), (20, 128, 32), (1, 512, 64), (3, 40, 8)])
def test_one_key_stands_out_anywhere_in_a_long_context(H, rank, rot, dt):
    """One cached vector is the query itself, scaled up, at block and page borders of a context of 2,300: rows before it do not see it, all others
    return its latent."""
    key, n, edges = rank + rot, 2300, [0, 63, 64, 127, 128, 1023, 1024, 1025, 2047, 2298]
    g = torch.Generator().manual_seed(rank)
    kv = PagedKV([(1, key, 0)], 40, 1, 2304, dt, "cuda")
    kv.ensure(0, n)
    kv.upload()
    q1 = torch.randn(key, generator=g).to(dt)
    q1 = (q1.float() / q1.float().norm() * 8).to(dt)
    eye = torch.eye(rank, dtype=dt, device="cuda").repeat(H, 1, 1)
    for at in edges:
        base = 0.05 * torch.randn(n, key, generator=g)
        base[at] = 1.5 * q1.float()
        for i, page in enumerate(kv.pages[0]):
            part = base[i * PAGE:(i + 1) * PAGE]
            kv.k[0][page, 0, :len(part)] = part.to("cuda", dt)
        rows = sorted({p for p in (at - 1, at, at + 1, at + 64, at + 200, n - 1) if 0 <= p < n})
        q, pos = q1.repeat(len(rows), H).cuda(), _i32(rows)
        lane, st, out = torch.zeros(len(rows), dtype=torch.int32, device="cuda"), _status(), []
        for splits in (1, 5):
            c = torch.zeros(len(rows), H * rank, dtype=dt, device="cuda")
            part, ml = torch.zeros(len(rows) * H * splits * rank, device="cuda"), torch.zeros(len(rows) * H * splits * 2, device="cuda")
            R.attn(q, kv.k[0], None, kv.table, lane, pos, None, len(rows), None, c, part, ml, H, 1.0, splits, st, 2304, rank, True)
            out.append(c)
        if R.latent_decode_supports(dt, rot, rank):
            for ctas in (1, 3, 50, 148):
                parts = torch.zeros(len(rows), 2, dtype=torch.int32, device="cuda")
                c, places = torch.zeros(len(rows), H * rank, dtype=dt, device="cuda"), ctas + len(rows)
                part, ml = torch.full((places * H * rank,), float("nan"), device="cuda"), torch.full((places * H * 2,), float("nan"), device="cuda")
                R.latent_decode(q, kv.k[0], rank, rot, kv.table, lane, pos, torch.arange(len(rows), dtype=torch.int32, device="cuda"), len(rows), H, part, ml, parts, 2304, ctas, 36 * len(rows),
                                1.0, st)
                R.head_proj(None, 0, eye, c, rank, len(rows), None, 0, merge=(part, ml, parts, ctas))
                out.append(c)
        assert st.tolist()[0] == 0
        want = (1.5 * q1[:rank].float()).cuda()
        for c in out:
            off = (c.float().view(-1, H, rank) - want).abs().amax((1, 2))
            for p, o in zip(rows, off.tolist()):
                assert (o < 0.05) == (p >= at), (at, p, o)
