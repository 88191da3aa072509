"""The gated delta rule, each arm alone against the plain equations (tests/oracles/plain_lifulorn.py)."""
import types

import pytest
import torch

from oracles import plain_lifulorn as P
from sparkflash_b200.models.mixers import DeltaState
from sparkflash_b200.ops import rows as R

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


class _Scratch:
    def __init__(self):
        self.buf = {}

    def get(self, name, *shape):
        n = 1
        for k in shape:
            n *= k
        return self.buf[name][:n].view(*shape)


def _step(core, lens, src, dst, long):
    """The arrays of a step with these segments, of which ``long`` go to the tensor-core arm, and its scratch."""
    s, row0 = types.SimpleNamespace(), [sum(lens[:k]) for k in range(len(lens))]
    s.n, s.status = sum(lens), torch.zeros(4, dtype=torch.int32, device="cuda")
    s.row_pos = _i32([i for n in lens for i in range(n)])
    s.row_seg = _i32([k for k, n in enumerate(lens) for _ in range(n)])
    s.seg_row0, s.seg_len, s.seg_src, s.seg_dst = _i32(row0), _i32(lens), _i32(src), _i32(dst)
    short = [k for k in range(len(lens)) if k not in long]
    chunks, first = [], []
    for k in long:
        first.append(len(chunks))
        chunks += [(row0[k] + r, min(128, lens[k] - r)) for r in range(0, lens[k], 128)]
    s.nshort, s.nlong, s.nchunks = len(short), len(long), len(chunks)
    s.short_segs = _i32(short) if long else None
    s.long_seg, s.long_first = _i32(long), _i32(first + [len(chunks)])
    s.long_row0, s.long_rows = _i32([c[0] for c in chunks]), _i32([c[1] for c in chunks])
    s.scratch = _Scratch()
    s.engine = types.SimpleNamespace(max_rows=s.n + 7, state_chunks=lambda: len(chunks))
    s.engine.scratch = types.SimpleNamespace(reserve=lambda name, n, dt: s.scratch.buf.__setitem__(name, torch.zeros(max(1, n), dtype=dt, device="cuda")))
    core.reserve(s.engine)
    return s


def _close(got, want, tol):
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-6)
    assert err < tol, float(err)


# heads, groups, N, P, lengths
SIZES = [(4, 2, 32, 24, [1, 2, 33, 5]), (3, 1, 20, 7, [9, 1, 40]), (2, 2, 130, 50, [17, 3]), (5, 1, 48, 72, [128, 32, 127, 129, 1, 257]),
         (9, 1, 64, 64, [300, 2]), (2, 1, 128, 40, [130, 256]), (6, 3, 16, 8, [40]), (2, 2, 112, 128, [420])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,Pd,lens", SIZES)
def test_segments_against_the_recurrence(H, G, N, Pd, lens, dtype):
    """Segments that start from zero and from a state, short and long arms; decays from almost none to almost all per token, keys that
    repeat (so that what is written depends on what the chunk has already written)."""
    g = torch.Generator().manual_seed(H * N)
    n, L = sum(lens), len(lens)
    cols = (G * N, 0, 2 * G * N)                     # q, k, v somewhere in wider rows
    stride = -(-(2 * G * N + H * Pd) // 8) * 8
    src = torch.randn(n, stride, generator=g)
    src[:, :G * N] = src[torch.randint(0, n, (n,), generator=g) // 7, :G * N] + 0.2 * src[:, :G * N]
    src = src.to(dtype).cuda()
    side = (2 * torch.randn(n, 2 * H + 3, generator=g)).to(dtype).cuda()
    dt, beta = side[:, 2:], side[:, 2 + H:]
    bias, A = torch.randn(H, generator=g) - 1, -torch.exp(torch.linspace(-6, 2, H))
    core = DeltaState(H, G, N, Pd, A.cuda(), dtype, bias.cuda())
    assert core.tc == (dtype == torch.bfloat16 and N % 16 == 0 and N <= 128 and Pd % 8 == 0)
    S = torch.zeros(2 * L, H, Pd, R.state_pad(N), device="cuda")
    S[:, :, :, :N] = torch.randn(2 * L, H, Pd, N, generator=g).cuda()
    before = S.clone()
    start = [2 * k if k % 2 else -1 for k in range(L)]
    for long in [[]] + ([[k for k in range(L) if lens[k] >= 32]] if core.tc and max(lens) >= 32 else []):
        S.copy_(before)
        s = _step(core, lens, start, [2 * k + 1 for k in range(L)], long)
        y = torch.zeros(n, H * Pd, dtype=dtype, device="cuda")
        core.run(s, src, cols, dt, beta, S, y)
        assert s.status.tolist()[0] == 0
        for k in range(L):
            rows = slice(sum(lens[:k]), sum(lens[:k]) + lens[k])
            x, d, b = src[rows].cpu().double(), dt[rows, :H].cpu().double(), P.sigmoid(beta[rows, :H].cpu().double())
            for h in range(H):
                i = h // (H // G)
                q = P.unit(x[:, cols[0] + i * N:cols[0] + (i + 1) * N]) * N ** -0.5
                kk = P.unit(x[:, cols[1] + i * N:cols[1] + (i + 1) * N])
                decay = torch.exp(A[h].double() * P.softplus(d[:, h] + bias[h].double()))
                S0 = before[2 * k, h, :, :N].cpu().double().T if k % 2 else None
                o, end = P.delta_rule(q, kk, x[:, cols[2] + h * Pd:cols[2] + (h + 1) * Pd], decay, b[:, h], S0)
                _close(y[rows, h * Pd:(h + 1) * Pd], o, 2e-5 if dtype == torch.float32 else 6e-3)
                _close(S[2 * k + 1, h, :, :N].T, end, 2e-5 if dtype == torch.float32 else 2e-4)      # inputs are exact: only the state's rounding
        assert (S[:, :, :, N:] == 0).all() and torch.equal(S[::2], before[::2])


@pytest.mark.parametrize("n", [1, 3])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,Pd,taps", [(4, 2, 24, 40, 4), (3, 1, 7, 5, 1), (2, 1, 64, 32, 6)])
def test_single_rows_with_their_convolution(H, G, N, Pd, taps, dtype, n):
    """Few single rows: the recurrence applies the convolution itself and carries its inputs on."""
    g = torch.Generator().manual_seed(N)
    C = 2 * G * N + H * Pd
    raw, w = torch.randn(n, C, generator=g).to(dtype).cuda(), torch.randn(taps, C, generator=g).cuda()
    hist = torch.randn(2 * n, max(1, taps - 1), C, generator=g).to(dtype).cuda()[:, :taps - 1].contiguous()
    old = hist.clone()
    side, bias, A = torch.randn(n, 2 * H, generator=g).to(dtype).cuda(), torch.randn(H, generator=g), -torch.rand(H, generator=g)
    core = DeltaState(H, G, N, Pd, A.cuda(), dtype, bias.cuda())
    S = torch.zeros(2 * n, H, Pd, R.state_pad(N), device="cuda")
    S[:, :, :, :N] = torch.randn(2 * n, H, Pd, N, generator=g).cuda()
    before = S.clone()
    s = _step(core, [1] * n, [2 * k for k in range(n)], [2 * k + 1 for k in range(n)], [])
    y = torch.zeros(n, H * Pd, dtype=dtype, device="cuda")
    core.run(s, raw, (0, G * N, 2 * G * N), side[:, H:], side, S, y, (w, None, hist, (0, G * N, 2 * G * N)))
    for r in range(n):
        x = torch.cat([old[2 * r], raw[r:r + 1]]).cpu().double()
        u = P.silu((x * w.cpu().double()).sum(0)).to(dtype).double()
        if taps > 1:
            assert torch.equal(hist[2 * r + 1], torch.cat([old[2 * r], raw[r:r + 1]])[1:]) and torch.equal(hist[2 * r], old[2 * r])
        for h in range(H):
            i = h // (H // G)
            q, k = P.unit(u[None, i * N:(i + 1) * N]) * N ** -0.5, P.unit(u[None, (G + i) * N:(G + i + 1) * N])
            v = u[None, 2 * G * N + h * Pd:2 * G * N + (h + 1) * Pd]
            decay = torch.exp(A[h].double() * P.softplus(side[r, H + h].cpu().double() + bias[h].double()))[None]
            o, end = P.delta_rule(q, k, v, decay, P.sigmoid(side[r, h].cpu().double())[None], before[2 * r, h, :, :N].cpu().double().T)
            _close(y[r:r + 1, h * Pd:(h + 1) * Pd], o, 2e-5 if dtype == torch.float32 else 1e-2)
            _close(S[2 * r + 1, h, :, :N].T, end, 2e-5 if dtype == torch.float32 else 5e-3)
