"""Windowed attention with sinks and capped scores, rotated appends with mixed values, the mixture of experts, the per-layer token input and
the scaled seam: each alone against the plain equations (tests/oracles/plain_lifulorn.py)."""
import pytest
import torch

from oracles import plain_lifulorn as P
from sparkflash_b200.kv.paged import PAGE, PagedKV
from sparkflash_b200.models.mixers import MixtureFF, W, rotation_table
from sparkflash_b200.ops import rows as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    return torch.zeros(4, dtype=torch.int32, device="cuda")


def _tol(dt):
    return 3e-5 if dt == torch.float32 else 2e-2


# ---- seam ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n,d,parts", [(5, 96, 3), (4, 75, 1), (3, 2056, 9), (400, 64, 2)])
def test_seam_scales_sums_parts_and_takes_rms_norms(dt, n, d, parts):
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(*s, generator=g)
    x, y, z, wt, eps = r(n, d), r(n, d).to(dt).float() + 2, r(n, parts, d).to(dt).float(), torch.rand(n, parts, generator=g), 1e-4
    y = y.to(dt).float()
    w = [1 + 0.3 * r(d) for _ in range(4)]
    c = lambda t, k=torch.float32: t.to("cuda", k).contiguous()
    X, H = c(x), torch.zeros(n, d, dtype=dt, device="cuda")
    common = dict(eps=eps, status=_status(), norm_kind="rms")
    R.seam(X, n, h=H, y=c(y, dt), post=(c(w[0]), None), post_kind="scale", norm=(c(w[1]), None), **common)
    want = x + y * w[0]
    assert (X.cpu() - want).abs().max() < 2e-5 and (H.float().cpu() - P.unit_rms(want, eps) * w[1]).abs().max() < 2 * _tol(dt)
    R.seam(X, n, h=H, y=c(z, dt), parts_w=c(wt), post=(c(w[2]), None), post_kind="scale", **common)
    want = want + (wt[..., None] * z).sum(1) * w[2]
    assert (X.cpu() - want).abs().max() < 5e-5 and (H.float().cpu() - want).abs().max() < 3 * _tol(dt)      # h: the residual itself
    R.seam(X, n, h=H, y=c(y, dt), post=(c(w[3]), None), post_kind="rms", norm=(c(w[1]), None), **common)
    want = want + P.unit_rms(y, eps) * w[3]
    assert (X.cpu() - want).abs().max() < 5e-5 and (H.float().cpu() - P.unit_rms(want, eps) * w[1]).abs().max() < 2 * _tol(dt)


# ---- rotation, values, cache ----------------------------------------------------------------------------------------------
SCALING = {"factor": 5.0, "original": 200, "fast": 9.0, "slow": 0.5}


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,dims", [(4, 2, 32, 16, 16), (3, 1, 10, 7, 6), (2, 2, 64, 40, 64), (6, 3, 20, 12, 8)])
def test_append_turns_queries_and_keys_and_mixes_values(dt, H, G, dim, vdim, dims):
    g = torch.Generator().manual_seed(dim)
    lens, cols = [70, 3, 129], H * dim + G * (dim + vdim)
    kv = PagedKV([(G, dim, vdim)], 8, 3, 256, dt, "cuda")
    for lane, n in ((2, 64), (0, 70), (1, 3), (2, 129)):
        kv.ensure(lane, n)
    kv.upload()
    xs = [torch.randn(n, cols, generator=g).to(dt).double() for n in lens]
    where = [(a, p) for a, n in enumerate(lens) for p in range(n)]
    first, lam = torch.zeros(len(where), G * vdim, dtype=dt, device="cuda"), torch.tensor(0.3, device="cuda")
    proj = torch.nn.functional.pad(torch.cat(xs), (0, 5)).to("cuda", dt)      # a wider row
    cs, (freqs, gain) = rotation_table(90.0, dims, 256, "cuda", SCALING), P.yarn_frequencies(90.0, dims, SCALING)
    q = torch.empty(len(where), H * dim, dtype=dt, device="cuda")
    for mixed in (False, True):
        st = _status()
        if mixed:
            first.copy_(torch.randn(len(where), G * vdim, generator=g).to(dt))
        R.rot_append(proj, cs, dims, q, kv.k[0], kv.v[0], first, lam if mixed else None, kv.table, _i32([a for a, _ in where]), _i32([p for _, p in where]),
                     len(where), H, st)
        assert st.tolist()[0] == 0
        row = 0
        for a, x in enumerate(xs):
            n = len(x)
            want_q, want_k = (P.rotate(x[:, i:i + m * dim].view(n, m, dim), freqs, gain).view(n, -1) for i, m in ((0, H), (H * dim, G)))
            want_v = x[:, (H + G) * dim:]
            if mixed:
                want_v = 0.7 * want_v + 0.3 * first[row:row + n].double().cpu()
            pool = lambda t, w: torch.cat([t[p].transpose(0, 1).reshape(PAGE, G * w) for p in kv.pages[a]])[:n].double().cpu()
            for got, want in ((q[row:row + n].double().cpu(), want_q), (pool(kv.k[0], dim), want_k), (pool(kv.v[0], vdim), want_v)):
                assert (got - want).abs().max() < 3 * _tol(dt)
            if not mixed:
                assert torch.equal(first[row:row + n].double().cpu(), want_v)
            row += n


@pytest.mark.parametrize("dt", DTYPES)
def test_token_gate_reads_its_part_of_the_table(dt):
    z, table = torch.randn(7, 12).to(dt), torch.randn(9, 40).to(dt)
    tok = [3, 8, 0, 1, 3, 5, 2]
    out = torch.empty(7, 12, dtype=dt, device="cuda")
    st = _status()
    R.token_gate(z.cuda(), table.cuda(), 24, _i32(tok), out, 7, st)
    assert (out.double().cpu() - P.gelu_tanh(z.double()) * table[tok, 24:36].double()).abs().max() < _tol(dt) and st.tolist()[0] == 0
    R.token_gate(z.cuda(), table.cuda(), 24, _i32([9] * 7), out, 7, st)
    assert st.tolist()[:1] == [2]


# ---- attention: windows, sinks, capped scores ---------------------------------------------------------------------------------
class Case:
    """Keys and values of several lanes in a shuffled page pool, and queries for every position."""

    def __init__(self, dt, H, G, dim, vdim, lens, window, cap, seed=0, scale=0.3):
        g = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=g).to(dt).float()
        self.kv = PagedKV([(G, dim, vdim)], 3 + sum(-(-n // PAGE) for n in lens), len(lens), 1024, dt, "cuda")
        self.H, self.G, self.dim, self.vdim, self.dt, self.window, self.cap, self.scale = H, G, dim, vdim, dt, window, cap, scale
        self.q, self.k, self.v = ([r(n, x) for n in lens] for x in (H * dim, G * dim, G * vdim))
        self.sink = 2 * torch.randn(H, generator=g) + 2
        for p in range(max(-(-n // PAGE) for n in lens)):
            for lane, n in enumerate(lens):
                self.kv.ensure(lane, min(n, (p + 1) * PAGE))

    def fill(self):
        self.kv.upload()
        for lane, (k, v) in enumerate(zip(self.k, self.v)):
            for p, page in enumerate(self.kv.pages[lane]):
                kk, vv = k[p * PAGE:(p + 1) * PAGE], v[p * PAGE:(p + 1) * PAGE]
                self.kv.k[0][page, :, :len(kk)] = kk.view(len(kk), self.G, self.dim).transpose(0, 1).to("cuda", self.dt)
                self.kv.v[0][page, :, :len(vv)] = vv.view(len(vv), self.G, self.vdim).transpose(0, 1).to("cuda", self.dt)
        return self

    def want(self, lane):
        q, k, v, out, rep = self.q[lane].double(), self.k[lane].double(), self.v[lane].double(), [], self.H // self.G
        for h in range(self.H):
            g = h // rep
            out.append(P.window_softmax(q[:, h * self.dim:(h + 1) * self.dim], k[:, g * self.dim:(g + 1) * self.dim], v[:, g * self.vdim:(g + 1) * self.vdim],
                                        self.scale, self.window, self.sink[h].double(), self.cap))
        return torch.cat(out, -1).float()

    def options(self):
        return dict(window=self.window, sink=self.sink.cuda(), cap=self.cap or 0.0)

    def rows(self, arm, rows, splits=1, slack=0):
        """(lane, position) pairs through the exact or the streaming arm."""
        q = torch.stack([self.q[a][p] for a, p in rows]).to("cuda", self.dt)
        out, st, n = torch.full((len(rows), self.H * self.vdim), 9.0, dtype=self.dt, device="cuda"), _status(), 1200 * 8 * max(4, len(rows) // 100)
        part, ml = torch.full((n * self.vdim,), float("nan"), device="cuda"), torch.full((n * 2,), float("nan"), device="cuda")
        args = (q, self.kv.k[0], self.kv.v[0], self.kv.table, _i32([a for a, _ in rows]), _i32([p for _, p in rows]), None, len(rows), None, out, part, ml,
                self.H, self.scale)
        if arm == "stream":
            R.attn_stream(*args, slack + sum(p // PAGE + 1 - max(0, p - self.window + 1) // PAGE for _, p in rows), st, **self.options())
        else:
            R.attn(*args, splits, st, **self.options())
        assert st.tolist()[0] == 0, st.tolist()
        return out.float().cpu()

    def tiles(self, runs):
        """(lane, first position, rows) through the tensor-core arm."""
        lanes, pos = [a for a, _, m in runs for _ in range(m)], [p + i for _, p, m in runs for i in range(m)]
        q, tiles, row = torch.cat([self.q[a][p:p + m] for a, p, m in runs]).to("cuda", self.dt), [], 0
        for _, _, m in runs:
            for r in range(0, m, 256):
                tiles += [row + r, min(256, m - r)]
            row += m
        out, st = torch.full((row, self.H * self.vdim), 9.0, dtype=self.dt, device="cuda"), _status()
        R.attn_tc(q, R.attn_pools(self.kv, 0, True), self.kv.table, _i32(lanes), _i32(pos), _i32(tiles), len(tiles) // 2, None, out, self.H, self.scale, st,
                  **self.options())
        assert st.tolist()[0] == 0, st.tolist()
        return out.float().cpu()


LENS = [1, 64, 65, 300]
ROWS = [(0, 0), (1, 0), (1, 62), (1, 63), (2, 63), (2, 64), (3, 0), (3, 39), (3, 40), (3, 63), (3, 64), (3, 127), (3, 128), (3, 191), (3, 192), (3, 299)]
WINDOWS = [(1, None), (40, 5.0), (64, None), (65, 0.7), (200, 30.0), (5000, 2.0)]


@pytest.mark.parametrize("window,cap", WINDOWS)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 24, 40), (3, 3, 10, 7), (6, 1, 64, 32)])
def test_exact_rows(H, G, dim, vdim, dt, window, cap):
    case = Case(dt, H, G, dim, vdim, LENS, window, cap).fill()
    want = [case.want(a) for a in range(4)]
    for splits in (1, 3):
        for (a, p), row in zip(ROWS, case.rows("exact", ROWS, splits)):
            assert (row - want[a][p]).abs().max() < _tol(dt), (a, p, splits)


@pytest.mark.parametrize("window,cap", WINDOWS)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 64, 32), (5, 1, 32, 96), (2, 2, 128, 128), (2, 1, 256, 32)])
def test_streamed_rows(H, G, dim, vdim, window, cap):
    case = Case(torch.bfloat16, H, G, dim, vdim, LENS, window, cap).fill()
    want = [case.want(a) for a in range(4)]
    for rows in (ROWS, ROWS * 20, [(3, 299)]):
        for slack in (0, 5000):
            for (a, p), row in zip(rows, case.rows("stream", rows, slack=slack)):
                assert (row - want[a][p]).abs().max() < 0.02, (a, p, len(rows), slack)


@pytest.mark.parametrize("window,cap", WINDOWS)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 64, 32), (2, 1, 40, 128), (3, 3, 128, 64), (2, 2, 96, 104)])
def test_runs_on_the_tensor_cores(H, G, dim, vdim, window, cap):
    case = Case(torch.bfloat16, H, G, dim, vdim, [700, 130, 40], window, cap).fill()
    want = [case.want(a) for a in range(3)]
    for runs in ([(0, 0, 700)], [(2, 0, 40), (0, 1, 33), (1, 97, 33)], [(0, 37, 512), (1, 64, 66)], [(0, 444, 256), (1, 1, 129)]):
        for (a, p, m), o in zip(runs, case.tiles(runs).split([m for _, _, m in runs])):
            assert (o - want[a][p:p + m]).abs().max() < 0.02, (runs, a)


@pytest.mark.parametrize("arm", ["exact32", "exact16", "stream", "tiles"])
@pytest.mark.parametrize("window,cap", [(37, None), (64, 60.0), (129, None)])
def test_one_key_stands_out_just_inside_and_just_outside_the_window(arm, window, cap):
    dt = torch.float32 if arm == "exact32" else torch.bfloat16
    for key in (0, 1, 63, 64, 127, 128, 200, 319):
        case = Case(dt, 2, 1, 32, 32, [512], window, cap, seed=key, scale=1.0)
        case.q[0] *= 0.1
        case.k[0][key] = 0
        case.k[0][key, :4] = 5.0
        inside, outside = key + window - 1, key + window
        for p in (inside, outside):
            case.q[0][p].view(2, 32)[:, :4] = 2.5                # score 50 (40 capped) against the key, a few at most against any other
        case.fill()
        if arm == "tiles":
            lo = max(0, inside - 40)
            got = case.tiles([(0, lo, 90)])[[inside - lo, outside - lo]]
        else:
            got = case.rows("stream" if arm == "stream" else "exact", [(0, inside), (0, outside)], 2)
        assert (got[0].view(2, 32) - case.v[0][key]).abs().max() < 0.02, (arm, key)
        assert (got[1].view(2, 32) - case.v[0][key]).abs().max() > 0.3, (arm, key)


@pytest.mark.parametrize("arm", ["exact32", "exact16", "stream", "tiles"])
def test_sinks_far_above_and_far_below_the_scores(arm):
    dt = torch.float32 if arm == "exact32" else torch.bfloat16
    for sink in (-200.0, -3.0, 9.0, 60.0, 300.0):
        case = Case(dt, 2, 2, 32, 32, [200], 150, None, seed=5)
        case.sink[:] = sink
        want = case.fill().want(0)
        got = case.tiles([(0, 0, 200)])[[0, 70, 199]] if arm == "tiles" else case.rows("stream" if arm == "stream" else "exact", [(0, 0), (0, 70), (0, 199)])
        assert (got - want[[0, 70, 199]]).abs().max() < _tol(dt), sink
        assert sink < 60 or got.abs().max() < 1e-3


# ---- mixture of experts -------------------------------------------------------------------------------------------------------
def _mixture(dt, d, E, top, ff, sff, limits, seed, n):
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, rows, cols in [(f"e{i}.{x}", *((d, ff) if x == "down" else (ff, d))) for i in range(E) for x in ("gate", "up", "down")] + \
            [(f"shared.{x}", *((d, sff) if x == "down" else (sff, d))) for x in ("gate", "up", "down") if sff]:
        w[name] = (2 * torch.randn(rows, cols, generator=g) * cols ** -0.5).to(torch.bfloat16)
    w["router"], w["shared.sg"] = (torch.randn(E, d, generator=g) * d ** -0.5).to(torch.bfloat16), (torch.randn(1, d, generator=g) * d ** -0.5).to(torch.bfloat16)
    spec = {"router": {"experts": E, "top": top}, "expert": {"ff": ff, "limit": limits[0]}}
    if sff:
        spec["shared"] = {"ff": sff, "limit": limits[1]}
    h = torch.randn(n, d, generator=g).to(dt)
    return w, spec, h


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


# width, experts, choices, ff, shared ff, limits
MOES = [(64, 16, 2, 24, 40, (1.0, 2.0)), (96, 5, 5, 200, 0, (0.5, 1.0)), (40, 40, 3, 136, 16, (3.0, 0.7)), (37, 6, 2, 11, 7, (1.0, 1.0)), (320, 3, 1, 64, 128, (9.0, 9.0)),
        (520, 130, 8, 264, 72, (0.4, 4.0)), (24, 300, 4, 8, 0, (1.0, 1.0))]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n", [1, 3, 9, 260])
@pytest.mark.parametrize("d,E,top,ff,sff,limits", MOES)
def test_mixture_of_experts(d, E, top, ff, sff, limits, n, dt):
    w, spec, h = _mixture(dt, d, E, top, ff, sff, limits, d + n, n)
    moe, s = MixtureFF(W({"p." + k: v for k, v in w.items()}, "p.", dt, "cuda"), spec, 1.702), _Step(n)
    assert moe.slots == top + (sff > 0)
    moe.reserve(s)
    assert moe.tc == (dt == torch.bfloat16 and d % 8 == ff % 8 == sff % 8 == 0)
    with R.exact_matmul():
        parts, wts = moe.run(s, h.cuda())
    assert s.status.tolist()[0] == 0
    w64 = {k: v.double() for k, v in w.items()}
    z = h.double() @ w64["router"].T
    for t in range(n):
        ids, a = P.route(z[t], top)
        assert s.get("moe_ids", n, top)[t].tolist() == ids or (z[t].sort(descending=True).values.diff().abs()[:top] < 1e-3).any()
    if n <= 9:
        got = (parts.double() * wts[..., None].double()).sum(1).cpu()
        want = P.mixture(w64, "", spec, h.double())
        assert (got - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
    else:                                          # many rows: every part against its expert
        ids = s.get("moe_ids", n, top).cpu()
        for j in range(top):
            for e in ids[:, j].unique().tolist():
                rows = ids[:, j] == e
                want = P.expert(w64, f"e{e}.", h[rows].double(), limits[0])
                assert (parts[rows.cuda(), j].double().cpu() - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
        if sff:
            want = P.expert(w64, "shared.", h.double(), limits[1])
            assert (parts[:, top].double().cpu() - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
            assert (wts[:, top].double().cpu() - P.sigmoid(h.double() @ w64["shared.sg"].T)[:, 0]).abs().max() < (1e-5 if dt == torch.float32 else 1e-5)


@pytest.mark.parametrize("n", [700, 9000])
def test_all_rows_on_one_expert_and_close_calls(n):
    """A router that sends everything to the same experts (one long list, more pairs than the plan holds at once), and equal logits (the
    lower number wins)."""
    d, E, top = 64, 9, 2
    w, spec, h = _mixture(torch.bfloat16, d, E, top, 40, 0, (2.0, 1.0), 3, n)
    w["router"].zero_()
    moe, s = MixtureFF(W({"p." + k: v for k, v in w.items()}, "p.", torch.bfloat16, "cuda"), spec, 1.702), _Step(n)
    moe.reserve(s)
    parts, wts = moe.run(s, h.cuda())
    assert (s.get("moe_ids", n, top).cpu() == torch.tensor([0, 1])).all() and (wts == 0.5).all() and s.status.tolist()[0] == 0
    w64 = {k: v.double() for k, v in w.items()}
    for j in range(2):
        want = P.expert(w64, f"e{j}.", h.double(), 2.0)
        assert (parts[:, j].double().cpu() - want).abs().max() < 2e-2 * float(want.abs().max())
