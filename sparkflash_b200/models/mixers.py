"""Sublayers of the layered decoders (models/layered.py): attention with a distance bias, attention with rotated keys in a window (sinks,
capped scores, values mixed across layers), attention with normed heads in a window, the real-gated linear recurrence, two mixers side by side, matrix-state recurrences
(state-space duality, retention, the gated delta rule), latent attention, the dense feed-forward (gated or with one activation), the
mixture of experts, the per-layer token input, and the weights of residual streams.  Each takes its sizes and constants as arguments, reads its weights by
name, keeps its caches in the engine's page pool or state slots, and runs on a step's rows through the kernels of ops/rows.py.

A sublayer is built once per layer (``weights``) and bound once per run of the layer (``bind_run``): a looped layer shares its
weights between passes, every pass has its own keys, values and states.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F

from ..ops import rows as R

CONV_STEP_ROWS = 4         # up to this many single rows the matrix-state kernel applies the convolution itself (every head does B and C again)
GATED_STEP_ROWS = 16       # up to this many single rows run convolution, gates and recurrence as one kernel


class W:
    """Weight access of one layer: ``act`` in the activation type, ``f32`` for what is computed in 32-bit."""

    def __init__(self, tensors: dict[str, torch.Tensor], prefix: str, dtype: torch.dtype, device):
        self.t, self.p, self.dtype, self.device = tensors, prefix, dtype, device

    def sub(self, name: str) -> "W":
        return W(self.t, self.p + name, self.dtype, self.device)

    def act(self, *names: str, pad: int = 1) -> torch.Tensor:
        """One matrix out of several, stacked along the output dimension; zero rows up to a multiple of ``pad``."""
        t = torch.cat([self.t[self.p + n] for n in names], 0).to(self.device, self.dtype)
        if t.shape[0] % pad:
            t = torch.cat([t, t.new_zeros(pad - t.shape[0] % pad, *t.shape[1:])], 0)
        return t.contiguous()

    def f32(self, name: str) -> torch.Tensor:
        return self.t[self.p + name].to(self.device, torch.float32).contiguous()

    def taps(self, *names: str) -> torch.Tensor:
        """Convolution weights [channels, taps], stacked, as the kernels read them: [taps, channels], 32-bit."""
        return torch.cat([self.t[self.p + n] for n in names], 0).to(self.device, torch.float32).t().contiguous()


def log_distance_bias(r1: torch.Tensor, r2: torch.Tensor, length: int, device) -> torch.Tensor:
    """[heads, length]: r1 ln(1 + r2 distance), evaluated in 64-bit and rounded once."""
    d = torch.arange(length, dtype=torch.float64, device=device)
    return (r1.to(device, torch.float64)[:, None] * torch.log1p(r2.to(device, torch.float64)[:, None] * d)).to(torch.float32).contiguous()


class PagedAttention:
    """Grouped-query softmax attention over the paged cache: the rows of a step go to the arm that suits them.  ``bias`` [heads, distance]
    is taken off the scaled score, ``cap`` bounds it, a position sees the last ``window`` ones, ``sink`` [heads] joins the denominator."""

    PROJ, PROJ_BIAS = ("q", "k", "v"), ("q.b", "k.b", "v.b")
    bias: torch.Tensor | None = None
    sink: torch.Tensor | None = None
    window, cap = R.NO_WINDOW, 0.0

    def __init__(self, w: W, spec: dict):
        self.H, self.G, self.dim, self.vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        self.scale = float(spec["scale"])
        self.cols = self.H * self.dim + self.G * (self.dim + self.vdim)
        self.tc = R.attn_tc_supports(w.dtype, self.dim, self.vdim)
        self.stream = R.attn_stream_supports(w.dtype, self.dim, self.vdim)
        self.dtype = w.dtype

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.dtype
        e.scratch.reserve("attn_q", n * self.H * self.dim, dt)
        e.scratch.reserve("attn_o", n * self.H * self.vdim, dt)
        # partial outputs of split rows: rows x heads x ranges, bounded by the blocks of one launch (see LayeredEngine.splits)
        per = self.H // R.attn_blocks(self.H, self.G)
        parts = max(1, per) * 1024 + self.H * 64
        if self.stream:
            parts = max(parts, 2 * R.STREAM_CTAS * R.attn_stream_heads(self.H, self.G, self.dim))
        e.scratch.reserve("attn_part", parts * self.vdim, torch.float32)
        e.scratch.reserve("attn_ml", parts * 2, torch.float32)

    def attend(self, s, q, kv, o) -> None:
        """q [n, H dim] against this run's pools, whose rows of the step have been appended; kv from R.attn_pools."""
        k, v, opts = kv[0], kv[1], dict(window=self.window, sink=self.sink, cap=self.cap)
        rows, m = s.single_rows(self.tc)
        if s.ntiles and self.tc:
            R.attn_tc(q, kv, s.table, s.row_lane, s.row_pos, s.tiles, s.ntiles, self.bias, o, self.H, self.scale, s.status, **opts)
        if m and self.stream and m <= R.STREAM_ROWS:
            pages = min(s.pages, (self.window + R.PAGE - 2) // R.PAGE + 1)
            R.attn_stream(q, k, v, s.table, s.row_lane, s.row_pos, rows, m, self.bias, o, s.scratch.buf["attn_part"],
                          s.scratch.buf["attn_ml"], self.H, self.scale, m * pages, s.status, **opts)
        elif m:
            blocks = R.attn_blocks(self.H, self.G)
            sp = s.engine.splits(s, m, blocks, self.window)
            part = s.scratch.buf["attn_part"] if sp > 1 else None
            ml = s.scratch.buf["attn_ml"] if sp > 1 else None
            R.attn(q, k, v, s.table, s.row_lane, s.row_pos, rows, m, self.bias, o, part, ml, self.H, self.scale, sp, s.status, **opts)


class BiasedAttention(PagedAttention):
    """RMS norm over the whole query and key projections, no rotation, a distance bias taken off the scaled score.  Reads its q | k | v
    columns out of the layer's stacked projection."""

    def __init__(self, w: W, spec: dict, eps: float, max_context: int):
        super().__init__(w, spec)
        self.eps = eps
        self.q_norm, self.k_norm = w.f32("q.norm"), w.f32("k.norm")
        self.bias = log_distance_bias(w.f32("r1"), w.f32("r2"), max_context, w.device)
        self.wo, self.bo = w.act("o"), w.act("o.b")

    def run(self, s, proj, kv, out):
        """proj [n, >= cols] view whose first columns are q | k | v; kv = (k pool, v pool) of this run."""
        n = s.n
        q = s.scratch.get("attn_q", n, self.H * self.dim)
        o = s.scratch.get("attn_o", n, self.H * self.vdim)
        R.qk_append(proj, self.q_norm, self.k_norm, q, kv[0], kv[1], s.table, s.row_lane, s.row_pos, n, self.H, self.eps, s.status)
        self.attend(s, q, kv, o)
        return R.linear(o, self.wo, self.bo, out)


class GatedRecurrence:
    """Griffin-style recurrent block (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
    Language Models"): y = gelu(W_y h), u = conv(W_x h), S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with a = exp(-c r softplus(lam))
    and block-diagonal gates r, i of u; output W_o (S y).  Reads its y | x columns out of the layer's stacked projection."""

    PROJ, PROJ_BIAS = ("y", "x"), ("y.b", "x.b")

    def __init__(self, w: W, spec: dict, c: float):
        self.width, self.parts, self.n_taps = spec["width"], spec["blocks"], spec["conv"]
        self.bs, self.cols = self.width // self.parts, 2 * self.width
        self.cw, self.cb = w.taps("conv"), w.f32("conv.b")
        self.wg = torch.cat([w.t[w.p + "ra"], w.t[w.p + "ri"]], 1).to(w.device, w.dtype).contiguous()        # [parts, 2 bs, bs]
        self.rb, self.ib = w.f32("ra.b").reshape(-1), w.f32("ri.b").reshape(-1)
        self.decay = (c * F.softplus(w.t[w.p + "lam"].to(w.device, torch.float64), threshold=50.0)).to(torch.float32).contiguous()
        self.wo = w.act("o")

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.wo.dtype
        e.scratch.reserve("rec_u", n * self.width, dt)
        e.scratch.reserve("rec_o", n * self.width, dt)
        e.scratch.reserve("rec_gates", n * 2 * self.width, torch.float32)
        e.scratch.reserve("rec_sums", (-(-n // e.chunk_rows) + e.max_lanes) * 2 * self.width, torch.float32)

    def states(self, e, tag: str):
        dt = self.wo.dtype
        return (e.state.add(tag + ".conv", (self.n_taps - 1, self.width), dt), e.state.add(tag + ".scan", (self.width,), torch.float32))

    def run(self, s, proj, states, out):
        """proj [n, 2 width] view (y | x); states = (convolution inputs, scan state) of this run."""
        n, (hist, S) = s.n, states
        y, x = proj[:, :self.width], proj[:, self.width:2 * self.width]
        o = s.scratch.get("rec_o", n, self.width)
        if s.single and n <= GATED_STEP_ROWS:
            R.gated_step(x, y, self.cw, self.cb, hist, self.wg, self.rb, self.ib, self.decay, S, o, s.seg_src, s.seg_dst, n)
        else:
            u = s.scratch.get("rec_u", n, self.width)
            R.conv(x, self.cw, self.cb, u, hist, s, n)
            gates = s.scratch.get("rec_gates", self.parts, n, 2 * self.bs)
            R.block_gates(u, self.wg, gates)
            R.scan(gates, self.rb, self.ib, self.decay, u, y, o, S, s.scratch.buf["rec_sums"], s, n, self.bs)
        return R.linear(o, self.wo, None, out)


class RecurrentMixer:
    """A gated recurrence as a layer's only mixer."""

    def __init__(self, w: W, spec: dict, c: float):
        self.rec = GatedRecurrence(w, spec, c)
        self.w_in, self.b_in = w.act(*self.rec.PROJ), w.act(*self.rec.PROJ_BIAS)
        self.merge = (None, None)
        self.kv_run = None

    def reserve(self, e) -> None:
        self.rec.reserve(e)
        e.scratch.reserve("proj", e.max_rows * self.w_in.shape[0], self.w_in.dtype)

    def bind_run(self, e, tag: str, kv_index):
        return {"rec": self.rec.states(e, tag)}

    def run(self, s, h, run):
        proj = R.linear(h, self.w_in, self.b_in, s.scratch.get("proj", s.n, self.w_in.shape[0]))
        return self.rec.run(s, proj, run["rec"], s.scratch.get("y", s.n, h.shape[1])), None


class ParallelMixer:
    """Attention and a gated recurrence on the same input: one stacked projection for both, and the half sum of the two outputs'
    RMS norms, which the seam kernel applies (``merge``)."""

    def __init__(self, w: W, spec: dict, eps: float, c: float, max_context: int):
        left, right = w.sub("left."), w.sub("right.")
        self.att = BiasedAttention(left, spec["left"], eps, max_context)
        self.rec = GatedRecurrence(right, spec["right"], c)
        self.w_in = torch.cat([left.act(*self.att.PROJ), right.act(*self.rec.PROJ)], 0).contiguous()
        self.b_in = torch.cat([left.act(*self.att.PROJ_BIAS), right.act(*self.rec.PROJ_BIAS)], 0).contiguous()
        self.merge = (left.f32("out"), right.f32("out"))
        self.kv_run = (self.att.G, self.att.dim, self.att.vdim)

    def reserve(self, e) -> None:
        self.att.reserve(e)
        self.rec.reserve(e)
        e.scratch.reserve("proj", e.max_rows * self.w_in.shape[0], self.w_in.dtype)

    def bind_run(self, e, tag: str, kv_index):
        return {"kv": R.attn_pools(e.kv, kv_index, self.att.tc), "rec": self.rec.states(e, tag)}

    def run(self, s, h, run):
        proj = R.linear(h, self.w_in, self.b_in, s.scratch.get("proj", s.n, self.w_in.shape[0]))
        y = self.att.run(s, proj, run["kv"], s.scratch.get("y", s.n, h.shape[1]))
        y2 = self.rec.run(s, proj[:, self.att.cols:], run["rec"], s.scratch.get("y2", s.n, h.shape[1]))
        return y, y2


def rotation_frequencies(base: float, dims: int, scaling: dict | None = None) -> tuple[list[float], float]:
    """Radians per position of every pair, and a factor on cosine and sine.  ``scaling``: None; {factor, low, high, original}: a pair keeps its
    frequency where the original context holds more than ``high`` of its wavelengths, has it divided by ``factor`` where it holds less than
    ``low``, and a blend in between; {factor, original, fast, slow}: YaRN (Peng et al., "YaRN: Efficient Context Window Extension of Large Language
    Models"), the division comes in along a ramp over the pairs between those that turn ``fast`` and ``slow`` times in the original context."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    if "fast" in scaling:
        pair = lambda turns: dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
        first, last = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), dims - 1)
        share = [min(max((i - first) / max(last - first, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [x * (1 - r) + x / factor * r for x, r in zip(f, share)], 0.1 * math.log(factor) + 1.0
    out = []
    for x in f:
        turns = original * x / (2 * math.pi)          # wavelengths in the original context
        kept = 1.0 if turns > scaling["high"] else 0.0 if turns < scaling["low"] else (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
        out.append(kept * x + (1 - kept) * x / factor)
    return out, 1.0


def rotation_table(base: float, dims: int, length: int, device, scaling: dict | None = None) -> torch.Tensor:
    """[length, dims / 2, 2]: cosine and sine of position times frequency, evaluated in 64-bit and rounded once."""
    f, gain = rotation_frequencies(base, dims, scaling)
    a = torch.arange(length, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    return (torch.stack([a.cos(), a.sin()], -1) * gain).to(torch.float32).to(device).contiguous()


class ValueMix:
    """Values that the layers of a model share within a step: the first layer that takes part leaves its own, the others mix theirs with them."""

    def __init__(self, cols: int):
        self.cols, self.layers = cols, 0

    def reserve(self, e, dtype) -> None:
        e.scratch.reserve("v_first", e.max_rows * self.cols, dtype)


class RotaryAttention(PagedAttention):
    """Rotated queries and keys (the first ``rot`` dims of a head, rotate-half layout, scaled frequencies), a sliding window, a learned sink per
    head, optionally capped scores, and values mixed with another layer's (``mix``) ahead of the cache.  A layer's only mixer."""

    def __init__(self, w: W, spec: dict, max_context: int, mix: ValueMix | None = None):
        super().__init__(w, spec)
        rot = spec["rot"]
        self.window, self.cap = min(int(spec["mask"]["size"]), max_context), float(spec.get("softcap") or 0.0)
        self.dims, self.cs = rot["dims"], rotation_table(rot["base"], rot["dims"], max_context, w.device, rot.get("scaling"))
        self.sink = w.f32("sink")
        self.w_in, self.b_in, self.wo = w.act(*self.PROJ), w.act(*self.PROJ_BIAS), w.act("o")
        self.mix, self.lam = mix, None
        if mix is not None:
            self.lam = w.f32("vmix") if mix.layers else None        # the first such layer has nothing to mix with
            mix.layers += 1
        self.merge, self.kv_run = (None, None), (self.G, self.dim, self.vdim)

    def reserve(self, e) -> None:
        super().reserve(e)
        e.scratch.reserve("proj", e.max_rows * self.w_in.shape[0], self.dtype)
        if self.mix is not None:
            self.mix.reserve(e, self.dtype)

    def bind_run(self, e, tag: str, kv_index):
        return {"kv": R.attn_pools(e.kv, kv_index, self.tc)}

    def run(self, s, h, run):
        n, kv = s.n, run["kv"]
        proj = R.linear(h, self.w_in, self.b_in, s.scratch.get("proj", n, self.w_in.shape[0]))
        q, o = s.scratch.get("attn_q", n, self.H * self.dim), s.scratch.get("attn_o", n, self.H * self.vdim)
        first = s.scratch.get("v_first", n, self.mix.cols) if self.mix is not None else None
        R.rot_append(proj, self.cs, self.dims, q, kv[0], kv[1], first, self.lam, s.table, s.row_lane, s.row_pos, n, self.H, s.status)
        self.attend(s, q, kv, o)
        return R.linear(o, self.wo, None, s.scratch.get("y", n, h.shape[1])), None


class HeadNormAttention(PagedAttention):
    """Queries and keys RMS-normed head by head (weights that the heads share), no rotation, a sliding window.  A layer's only mixer."""

    def __init__(self, w: W, spec: dict, eps: float, max_context: int):
        super().__init__(w, spec)
        self.eps, self.window = eps, min(int(spec["mask"]["size"]), max_context)
        self.q_norm, self.k_norm = w.f32("q.norm"), w.f32("k.norm")
        self.w_in, self.wo = w.act(*self.PROJ, pad=8), w.act("o")
        self.merge, self.kv_run = (None, None), (self.G, self.dim, self.vdim)

    def reserve(self, e) -> None:
        super().reserve(e)
        e.scratch.reserve("proj", e.max_rows * self.w_in.shape[0], self.dtype)

    def bind_run(self, e, tag: str, kv_index):
        return {"kv": R.attn_pools(e.kv, kv_index, self.tc)}

    def run(self, s, h, run):
        n, kv = s.n, run["kv"]
        proj = R.linear(h, self.w_in, None, s.scratch.get("proj", n, self.w_in.shape[0]))
        q, o = s.scratch.get("attn_q", n, self.H * self.dim), s.scratch.get("attn_o", n, self.H * self.vdim)
        R.head_append(proj, self.q_norm, self.k_norm, q, kv[0], kv[1], s.table, s.row_lane, s.row_pos, n, self.H, self.eps, s.status)
        self.attend(s, q, kv, o)
        return R.linear(o, self.wo, None, s.scratch.get("y", n, h.shape[1])), None


class MatrixState:
    """S_t = a_t S_(t-1) + w_t k_t v_t^T, y_t = S_t^T q_t + D v_t: one 32-bit state [P, N] and one decay per head, q and k shared by
    groups of heads.  Decay and input weight come from a step size per token (a = exp(A dt), w = dt; ``decay`` is A), or the decay is a
    constant.  q and k may be turned by their position (``rot``) and k scaled.  Long runs of bf16 rows take the tensor-core arm."""

    def __init__(self, heads: int, groups: int, n: int, p: int, decay: torch.Tensor, dtype: torch.dtype, dt_bias=None, skip=None, rot=None,
                 rot_dims: int = 0, k_scale: float = 1.0):
        self.H, self.G, self.N, self.P = heads, groups, n, p
        self.log_decay = decay if dt_bias is not None else torch.log(decay.double()).float().contiguous()
        self.decay, self.dt_bias, self.skip, self.rot, self.rot_dims, self.k_scale = decay, dt_bias, skip, rot, rot_dims, k_scale
        self.terms = 2 if rot is not None else 1
        self.tc = R.state_tc_supports(dtype, n, p, self.terms)

    def state(self, e, tag: str) -> torch.Tensor:
        return e.state.add(tag, (self.H, self.P, R.state_pad(self.N)), torch.float32)

    def reserve(self, e) -> None:
        if self.tc:
            chunks = e.state_chunks()
            per = self.H * self.P * R.state_pad(self.N)
            e.scratch.reserve("state_sums", chunks * per, torch.float32)
            e.scratch.reserve("state_starts", 2 * chunks * per, torch.bfloat16)
            e.scratch.reserve("state_dec", chunks * self.H, torch.float32)
            e.scratch.reserve("state_rates", chunks * self.H * 256, torch.float32)
            if self.terms > 1:
                e.scratch.reserve("state_turned", e.max_rows * 4 * self.H * self.N, torch.bfloat16)

    def run(self, s, src, cols, dt, S, y, conv=None) -> None:
        """``src`` [n, stride] holds q, k, v from the columns ``cols`` on; ``conv``: they are the inputs of a convolution, see R.state_rows."""
        q, k, v = (src[:, c:] for c in cols)
        if s.nshort:
            R.state_rows(q, k, v, dt, self.dt_bias, self.decay, self.skip, self.rot, self.rot_dims, self.k_scale, s.row_pos, y, S, self.N, self.G,
                         s.short_segs, s.nshort, s, conv)
        if s.nlong:
            hn, qk, at = self.H * self.N, src, (cols[0], cols[1], 0, 0)
            if self.terms > 1:
                qk, at = s.scratch.get("state_turned", s.n, 4 * hn), (0, 2 * hn, hn, hn)
                R.state_turn(q, k, self.rot, self.rot_dims, self.k_scale, s.row_pos, qk, s.n, self.H, self.N)
            R.state_tc(qk, at, src, cols[2], dt, self.dt_bias, self.log_decay, self.skip, S, s.scratch.buf["state_sums"], s.scratch.buf["state_dec"],
                       s.scratch.buf["state_rates"], s.scratch.buf["state_starts"], y, self.N, self.G, s, self.terms, s.status)


class StateSpaceMixer:
    """Mamba-2 (Dao & Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality"):
    z | x | B | C | dt = W_in h; x, B, C through a causal convolution and silu; the matrix-state recurrence with k = B, v = x, q = C; silu(z)
    gate, RMS norm in equal parts, W_o."""

    def __init__(self, w: W, spec: dict, eps: float):
        H, P, N, G = spec["heads"], spec["vdim"], spec["state"], spec["groups"]
        self.inner, self.bc, self.taps, self.eps, self.part = H * P, G * N, spec["conv"], eps, H * P // spec["norm_groups"]
        self.channels = self.inner + 2 * self.bc
        self.w_in, self.w_out = w.act("in", pad=8), w.act("o")
        self.cw, self.cb, self.norm = w.taps("conv"), w.f32("conv.b"), w.f32("norm")
        A = -torch.exp(w.t[w.p + "A_log"].to(w.device, torch.float64)).to(torch.float32)
        self.core = MatrixState(H, G, N, P, A.contiguous(), w.dtype, w.f32("dt_bias"), w.f32("D"))
        self.merge, self.kv_run = (None, None), None

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.w_in.dtype
        e.scratch.reserve("proj", n * self.w_in.shape[0], dt)
        e.scratch.reserve("mix_u", n * self.channels, dt)
        e.scratch.reserve("mix_y", n * self.inner, dt)
        e.scratch.reserve("mix_o", n * self.inner, dt)
        self.core.reserve(e)

    def bind_run(self, e, tag: str, kv_index):
        return {"conv": e.state.add(tag + ".conv", (self.taps - 1, self.channels), self.w_in.dtype), "S": self.core.state(e, tag + ".S")}

    def run(self, s, h, run):
        n, i, bc = s.n, self.inner, self.bc
        proj = R.linear(h, self.w_in, None, s.scratch.get("proj", n, self.w_in.shape[0]))
        z, u, dt = proj[:, :i], proj[:, i:i + self.channels], proj[:, i + self.channels:]
        y = s.scratch.get("mix_y", n, i)
        conv = (self.cw, self.cb, run["conv"], (i + bc, i, 0)) if s.single and n <= CONV_STEP_ROWS else None
        if conv is None:
            raw, u = u, s.scratch.get("mix_u", n, self.channels)
            R.conv(raw, self.cw, self.cb, u, run["conv"], s, n, R.CONV_SILU)
        self.core.run(s, u, (i + bc, i, 0), dt, run["S"], y, conv)
        o = s.scratch.get("mix_o", n, i)
        R.gated_norm(y, z, self.norm, o, self.part, True, self.eps)
        return R.linear(o, self.w_out, None, s.scratch.get("y", n, h.shape[1])), None


class RetentionMixer:
    """Retention (Sun et al., "Retentive Network: A Successor to Transformer for Large Language Models"): rotated queries and keys, a
    fixed decay per head, no softmax; every head's output over its RMS, silu(W_g h) gate, W_o."""

    PROJ = ("q", "k", "v", "g")

    def __init__(self, w: W, spec: dict, eps: float, max_context: int):
        H, N, P, rot = spec["heads"], spec["dim"], spec["vdim"], spec["rot"]
        self.inner, self.qk, self.P, self.eps = H * P, H * N, P, eps
        self.w_in, self.w_out = w.act(*self.PROJ, pad=8), w.act("o")
        decay = torch.tensor(spec["decay"], dtype=torch.float64).to(w.device, torch.float32)
        self.core = MatrixState(H, H, N, P, decay, w.dtype, rot=rotation_table(rot["base"], rot["dims"], max_context, w.device), rot_dims=rot["dims"],
                                k_scale=N ** -0.5)
        self.merge, self.kv_run = (None, None), None

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.w_in.dtype
        e.scratch.reserve("proj", n * self.w_in.shape[0], dt)
        e.scratch.reserve("mix_y", n * self.inner, dt)
        e.scratch.reserve("mix_o", n * self.inner, dt)
        self.core.reserve(e)

    def bind_run(self, e, tag: str, kv_index):
        return {"S": self.core.state(e, tag + ".S")}

    def run(self, s, h, run):
        n, i, qk = s.n, self.inner, self.qk
        proj = R.linear(h, self.w_in, None, s.scratch.get("proj", n, self.w_in.shape[0]))
        y, o = s.scratch.get("mix_y", n, i), s.scratch.get("mix_o", n, i)
        self.core.run(s, proj, (0, qk, 2 * qk), None, run["S"], y)
        R.gated_norm(y, proj[:, 2 * qk + i:2 * qk + 2 * i], None, o, self.P, False, self.eps)
        return R.linear(o, self.w_out, None, s.scratch.get("y", n, h.shape[1])), None


class DeltaState(MatrixState):
    """The gated delta rule (Yang et al., "Gated Delta Networks: Improving Mamba2 with Delta Rule"): S = a_t S_(t-1), u_t = b_t (v_t - S^T k_t),
    S_t = S + k_t u_t^T, y_t = S_t^T q_t, with unit vectors q and k (q over the root of its length), a_t = exp(A softplus(.)), b_t = sigmoid(.)."""

    UNIT_EPS = 1e-6

    def __init__(self, heads: int, groups: int, n: int, p: int, decay: torch.Tensor, dtype: torch.dtype, dt_bias):
        super().__init__(heads, groups, n, p, decay, dtype, dt_bias)
        self.tc = R.delta_tc_supports(dtype, n, p)

    def reserve(self, e) -> None:
        if self.tc:
            chunks = e.state_chunks()
            e.scratch.reserve("state_rates", chunks * self.H * R.DELTA_RATES * 128, torch.float32)
            e.scratch.reserve("state_dec", chunks * self.H, torch.float32)
            e.scratch.reserve("state_starts", 2 * chunks * self.H * self.P * self.N, torch.bfloat16)
            e.scratch.reserve("delta_inv", chunks * self.H * 2 * 128 * 128, torch.bfloat16)
            e.scratch.reserve("delta_u", 2 * chunks * self.H * 128 * self.P, torch.bfloat16)

    def run(self, s, src, cols, dt, beta, S, y, conv=None) -> None:
        """``src`` [n, stride] holds q, k, v from the columns ``cols`` on; ``conv``: they are the inputs of a convolution, see R.state_rows."""
        scale = self.N ** -0.5
        if s.nshort:
            q, k, v = (src[:, c:] for c in cols)
            R.state_rows(q, k, v, dt, self.dt_bias, self.decay, None, None, 0, 1.0, s.row_pos, y, S, self.N, self.G, s.short_segs, s.nshort, s, conv,
                         beta, scale, self.UNIT_EPS)
        if s.nlong:
            buf = s.scratch.buf
            R.delta_tc(src, cols, dt, beta, self.dt_bias, self.decay, S, buf["state_rates"], buf["state_dec"], buf["delta_inv"], buf["delta_u"], buf["state_starts"], y,
                       self.N, self.G, s, scale, self.UNIT_EPS, s.status)


class DeltaMixer:
    """q | k | v through a causal convolution and silu, the gated delta rule, every head's output over its RMS times a weight that the heads
    share, silu(W_g h) gate, W_o."""

    PROJ = ("q", "k", "v", "g", "b", "a")

    def __init__(self, w: W, spec: dict, eps: float):
        H, G, N, P = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        self.H, self.P, self.qk, self.inner, self.taps, self.eps = H, P, G * N, H * P, spec["conv"], eps
        self.channels = 2 * self.qk + self.inner
        self.w_in, self.w_out = w.act(*self.PROJ, pad=8), w.act("o")
        self.cw, self.norm = w.taps("q.conv", "k.conv", "v.conv"), w.f32("norm").repeat(H).contiguous()
        A = -torch.exp(w.t[w.p + "A_log"].to(w.device, torch.float64)).to(torch.float32)
        self.core = DeltaState(H, G, N, P, A.contiguous(), w.dtype, w.f32("dt_bias"))
        self.merge, self.kv_run = (None, None), None

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.w_in.dtype
        e.scratch.reserve("proj", n * self.w_in.shape[0], dt)
        e.scratch.reserve("mix_u", n * self.channels, dt)
        e.scratch.reserve("mix_y", n * self.inner, dt)
        e.scratch.reserve("mix_o", n * self.inner, dt)
        self.core.reserve(e)

    def bind_run(self, e, tag: str, kv_index):
        return {"conv": e.state.add(tag + ".conv", (self.taps - 1, self.channels), self.w_in.dtype), "S": self.core.state(e, tag + ".S")}

    def run(self, s, h, run):
        n, c, i = s.n, self.channels, self.inner
        proj = R.linear(h, self.w_in, None, s.scratch.get("proj", n, self.w_in.shape[0]))
        u, gate, beta, dt = proj[:, :c], proj[:, c:c + i], proj[:, c + i:], proj[:, c + i + self.H:]
        y, o, cols = s.scratch.get("mix_y", n, i), s.scratch.get("mix_o", n, i), (0, self.qk, 2 * self.qk)
        conv = (self.cw, None, run["conv"], cols) if s.single and n <= CONV_STEP_ROWS else None
        if conv is None:
            raw, u = u, s.scratch.get("mix_u", n, c)
            R.conv(raw, self.cw, None, u, run["conv"], s, n, R.CONV_SILU)
        self.core.run(s, u, cols, dt, beta, run["S"], y, conv)
        R.gated_norm(y, gate, self.norm, o, self.P, False, self.eps)
        return R.linear(o, self.w_out, None, s.scratch.get("y", n, h.shape[1])), None


class LatentAttention:
    """Attention whose keys and values are products of one cached vector per token (DeepSeek-AI, "DeepSeek-V2: A Strong, Economical, and
    Efficient Mixture-of-Experts Language Model"): the RMS-normed latent c, beside one rotated key part that the heads share.  Queries are a
    product of the input, or (``q_rank``) of a normed latent of their own; the rotation may turn neighbours or halves, at scaled frequencies;
    ``gated``: the heads' outputs times sigmoid(W_g h).  A position sees the last ``mask.size`` ones, or all of them.  Single rows and short
    runs score in the latent space (W_uk on the query, W_uv on the output); long runs multiply the visible keys and values out and take the
    tensor-core attention."""

    def __init__(self, w: W, spec: dict, eps: float, max_context: int, halves: bool = False, gated: bool = False):
        self.H, self.dim, self.rot, self.vdim, self.rank = spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"], spec["kv_rank"]
        self.q_rank, self.halves, self.gated = spec.get("q_rank", 0), halves, gated
        self.scale, self.eps = float(spec["scale"]), eps
        self.window = min(int(spec["mask"]["size"]), max_context) if spec.get("mask") else max_context
        names = (["g"] if gated else []) + (["dkv", "dq"] if self.q_rank else ["q", "dkv"])
        self.w_in, self.w_out, self.norm = w.act(*names, pad=8), w.act("o"), w.f32("dkv.norm")
        # columns of the stacked projection: gate, then queries and latent, or latent and the queries' latent
        self.col_q = H_out = self.H * self.vdim if gated else 0
        self.col_c = H_out + (0 if self.q_rank else self.H * (self.dim + self.rot))
        self.col_cq = self.col_c + self.rank + self.rot
        self.uq, self.q_norm = (w.act("uq"), w.f32("dq.norm")) if self.q_rank else (None, None)
        self.uk = w.act("uk").view(self.H, self.dim, self.rank)
        self.uv = w.act("uv").view(self.H, self.vdim, self.rank).transpose(1, 2).contiguous()       # [H, rank, vdim]
        self.cs = rotation_table(spec["rot"]["base"], self.rot, max_context, w.device, spec["rot"].get("scaling"))
        self.tc = R.latent_tc_supports(w.dtype, self.dim, self.rot, self.vdim, self.rank)
        self.dec = R.latent_decode_supports(w.dtype, self.rot, self.rank)
        self.merge, self.kv_run = (None, None), (1, self.rank + self.rot, 0)

    def reserve(self, e) -> None:
        n, dt, key = e.max_rows, self.w_in.dtype, self.rank + self.rot
        e.scratch.reserve("proj", n * self.w_in.shape[0], dt)
        e.scratch.reserve("mix_o", n * self.H * self.vdim, dt)
        if self.q_rank:
            e.scratch.reserve("lat_cq", n * self.q_rank, dt)
            e.scratch.reserve("lat_heads", n * self.H * (self.dim + self.rot), dt)
        short = min(n, e.short_rows(self.tc))
        e.scratch.reserve("lat_q", short * self.H * key, dt)
        e.scratch.reserve("lat_o", short * self.H * self.rank, dt)
        if self.dec:
            self.slice = min(short, R.LATENT_ROWS)
            e.scratch.reserve("lat_parts", 2 * self.slice, torch.int32)
            parts = R.latent_places(self.slice, self.H) * self.H
        else:
            parts = max(1, self.H // R.attn_blocks(self.H, 1)) * 1024 + self.H * 64
        e.scratch.reserve("attn_part", parts * self.rank, torch.float32)
        e.scratch.reserve("attn_ml", parts * 2, torch.float32)
        if self.tc:
            m = e.expanded_rows(self.window)
            e.scratch.reserve("lat_rows", m * key, dt)
            e.scratch.reserve("lat_k", m * self.H * self.dim, dt)
            e.scratch.reserve("lat_v", m * self.H * self.vdim, dt)

    def bind_run(self, e, tag: str, kv_index):
        return {"kv": e.kv.k[kv_index]}

    def queries(self, s, h, pool):
        """Projections, norms and the cache append; (heads' queries [n, .], what head_proj still has to turn, gate or None)."""
        n, H, dim, rot = s.n, self.H, self.dim, self.rot
        proj = R.linear(h, self.w_in, None, s.scratch.get("proj", n, self.w_in.shape[0]))
        gate = proj[:, :H * self.vdim] if self.gated else None
        where, sizes = (s.table, s.row_lane, s.row_pos, n), (H, dim, rot, self.rank)
        if not self.q_rank:
            q = proj[:, self.col_q:]
            R.latent_append(q, proj[:, self.col_c:], self.norm, self.cs, pool, *where, *sizes, self.eps, s.status, self.halves)
            return q, None, gate
        cq = s.scratch.get("lat_cq", n, self.q_rank)
        R.latent_append(None, proj[:, self.col_c:], self.norm, self.cs, pool, *where, *sizes, self.eps, s.status, self.halves, proj[:, self.col_cq:], self.q_norm, cq)
        q = R.linear(cq, self.uq, None, s.scratch.get("lat_heads", n, H * (dim + rot)))
        if (s.ntiles and self.tc) or not self.halves:
            R.latent_turn(q, self.cs, s.row_pos, n, H, dim, rot, self.halves)
            return q, None, gate
        return q, (self.cs, s.row_pos), gate

    def run(self, s, h, run):
        n, H, dim, rot, key, pool = s.n, self.H, self.dim, self.rot, self.rank + self.rot, run["kv"]
        heads, turn, gate = self.queries(s, h, pool)
        o = s.scratch.get("mix_o", n, H * self.vdim)
        short_rows, m = s.single_rows(self.tc)
        if s.ntiles and self.tc:
            pages, count, offs = s.expand[self.window]
            seen = count * 64
            rows = s.scratch.get("lat_rows", seen, key)
            kx, vx = s.scratch.get("lat_k", H, seen, dim), s.scratch.get("lat_v", H, seen, self.vdim)
            R.gather_pages(pool, pages, rows, count, s.status)
            R.expand(rows[:, :self.rank], self.uk.transpose(1, 2), kx)
            R.expand(rows[:, :self.rank], self.uv, vx)
            R.latent_attn_tc(heads, heads.stride(0), kx, vx, rows, self.rank, s.row_pos, s.tiles, offs, s.ntiles, o, H, dim, rot, self.vdim, self.window,
                             self.scale, s.status, gate)
        if m:
            q, c = s.scratch.get("lat_q", m, H * key), s.scratch.get("lat_o", m, H * self.rank)
            R.head_proj(heads, dim + rot, self.uk, q, key, m, short_rows, 1, rot, turn=turn)
        if m and self.dec:
            part, ml = s.scratch.buf["attn_part"], s.scratch.buf["attn_ml"]
            parts, seen = s.scratch.get("lat_parts", self.slice, 2), min(s.pages, -(-s.engine.max_context // R.PAGE), (self.window + R.PAGE - 2) // R.PAGE + 1)
            for a in range(0, m, self.slice):
                b = min(m, a + self.slice)
                rows = None if short_rows is None and a == 0 else (short_rows if short_rows is not None else s.engine._iota)[a:b]
                ctas = R.latent_ctas(H, (b - a) * seen)
                R.latent_decode(q[a:b], pool, self.rank, rot, s.table, s.row_lane, s.row_pos, rows, b - a, H, part, ml, parts, self.window, ctas,
                                (b - a) * seen, self.scale, s.status)
                R.head_proj(None, 0, self.uv, o, self.vdim, b - a, rows, 2, merge=(part, ml, parts, ctas), gate=gate)
        elif m:
            blocks = R.attn_blocks(H, 1)
            sp = s.engine.splits(s, m, blocks, self.window)
            part, ml = (s.scratch.buf["attn_part"], s.scratch.buf["attn_ml"]) if sp > 1 else (None, None)
            R.attn(q, pool, None, s.table, s.row_lane, s.row_pos, short_rows, m, None, c, part, ml, H, self.scale, sp, s.status, self.window, self.rank, True)
            R.head_proj(c, self.rank, self.uv, o, self.vdim, m, short_rows, 2, gate=gate)
        return R.linear(o, self.w_out, None, s.scratch.get("y", n, h.shape[1])), None


class DenseFF:
    """W_down (act(W_gate h) * (W_up h)) with gate and up in one product; act: silu, or gelu_tanh."""

    def __init__(self, w: W, act: str = "silu"):
        self.act = act
        self.w_in, self.w_out = w.act("gate", "up"), w.act("down")
        self.ff = self.w_out.shape[1]

    def reserve(self, e) -> None:
        e.scratch.reserve("proj", e.max_rows * 2 * self.ff, self.w_in.dtype)
        e.scratch.reserve("ff_act", e.max_rows * self.ff, self.w_in.dtype)

    def run(self, s, h):
        act = R.gated_linear(h, self.w_in, s.scratch.get("proj", s.n, 2 * self.ff), s.scratch.get("ff_act", s.n, self.ff), self.act)
        return R.linear(act, self.w_out, None, s.scratch.get("y", s.n, h.shape[1]))


class SingleFF:
    """act(h W_up^T) W_down^T; act of one input, with up to two numbers: relu2, or xielu."""

    def __init__(self, w: W, act: str, a: float = 0.0, b: float = 0.0):
        self.act, self.a, self.b = act, a, b
        self.w_in, self.w_out = w.act("up"), w.act("down")
        self.ff = self.w_out.shape[1]

    def reserve(self, e) -> None:
        e.scratch.reserve("ff_act", e.max_rows * self.ff, self.w_in.dtype)

    def run(self, s, h):
        act = R.act_linear(h, self.w_in, s.scratch.get("ff_act", s.n, self.ff), self.act, self.a, self.b)
        return R.linear(act, self.w_out, None, s.scratch.get("y", s.n, h.shape[1]))


class MixtureFF:
    """Every row through ``top`` of ``experts`` small feed-forwards, chosen and weighted as ``choice`` says (R.Choice), and through a shared one,
    weighted by the sigmoid of a logit of its own.  An expert with the "clamp" activation: W_down (g sigmoid(alpha g) (u + 1)), g = min(W_gate h,
    limit), u = W_up h within +-limit; with one of R.SINGLE_ACT: act(h W_up^T) W_down^T.  ``run`` returns the parts [n, top + shared, width] and
    their weights; the seam adds them up."""

    def __init__(self, w: W, spec: dict, alpha: float = 0.0, act: str = "clamp", choice: R.Choice = R.SOFTMAX):
        self.E, self.top = spec["router"]["experts"], spec["router"]["top"]
        self.ff, self.limit, self.alpha, self.act, self.choice = spec["expert"]["ff"], float(spec["expert"].get("limit", 0.0)), alpha, act, choice
        first = ("gate", "up") if act == "clamp" else ("up",)
        sh = spec.get("shared")
        self.shared, self.shared_ff, self.shared_limit = int(sh is not None), sh["ff"] if sh else 0, float(sh.get("limit", 0.0)) if sh else 0.0
        self.slots = self.top + self.shared
        self.w_in = torch.stack([w.act(*(f"e{i}.{n}" for n in first)) for i in range(self.E)]).contiguous()   # [E, ff, width], gated: [E, 2 ff, width]
        self.w_out = torch.stack([w.act(f"e{i}.down") for i in range(self.E)]).contiguous()                   # [E, width, ff]
        self.router = w.act("router", *(["shared.sg"] if sh else []), pad=8)
        self.s_in, self.s_out = (w.act(*(f"shared.{n}" for n in first)), w.act("shared.down")) if sh else (None, None)

    def reserve(self, e) -> None:
        n, dt, d = e.max_rows, self.router.dtype, self.router.shape[1]
        self.tc = R.moe_tc_supports(dt, d, self.ff, self.shared_ff)
        self.tile = R.MOE_TC_TILE if self.tc else R.MOE_TILE
        e.scratch.reserve("moe_z", n * self.router.shape[0], torch.float32)
        e.scratch.reserve("moe_w", n * self.slots, torch.float32)
        for name, size in (("moe_ids", n * self.top), ("moe_order", n * self.top), ("moe_tiles", 4 * R.moe_tiles(n, self.E, self.top, self.tile)), ("moe_count", 4)):
            e.scratch.reserve(name, size, torch.int32)
        e.scratch.reserve("moe_act", n * self.top * self.ff, dt)
        e.scratch.reserve("moe_parts", n * self.slots * d, dt)
        if self.tc and n > R.MOE_GATHER_ROWS:
            e.scratch.reserve("moe_x", n * self.top * d, dt)
        if self.shared:
            e.scratch.reserve("ff_act", n * self.shared_ff, dt)
            if not self.tc:
                e.scratch.reserve("proj", n * 2 * self.shared_ff, dt)

    def run(self, s, h):
        n, d, top, slots = s.n, h.shape[1], self.top, self.slots
        z = R.head(h, self.router, s.scratch.get("moe_z", n, self.router.shape[0]), "router")
        ids, wts = s.scratch.get("moe_ids", n, top), s.scratch.get("moe_w", n, slots)
        act, parts = s.scratch.get("moe_act", n * top, self.ff), s.scratch.get("moe_parts", n, slots, d)
        s_act = s.scratch.get("ff_act", n, self.shared_ff) if self.shared else None
        first = (h, self.s_in, s_act, self.shared_ff, self.shared_limit) if self.shared else None        # the shared expert's part in both products
        second = (s_act, self.s_out, None, d, 0.0) if self.shared else None
        if R.moe_gemv_takes(h, self.ff, self.shared_ff):
            R.moe_gemv(z, ids, wts, h, self.w_in, act, first, n, self.ff, top, slots, self.act, self.alpha, self.limit, self.choice)
            R.moe_gemv(None, ids, wts, act, self.w_out, parts, second, n, d, top, slots, None)
            return parts, wts
        plan = (s.scratch.get("moe_order", n * top), s.scratch.get("moe_tiles", R.moe_tiles(n, self.E, top, self.tile), 4), s.scratch.get("moe_count", 4),
                R.moe_tiles(n, self.E, top, self.tile))
        if n > R.MOE_PLAN_ROWS:
            R.moe_route(z, ids, wts, self.E, top, self.shared, self.choice)
        R.moe_plan(z if n <= R.MOE_PLAN_ROWS else None, ids, wts, *plan[:3], self.E, top, self.shared, self.tile, self.choice)
        if self.tc:
            few, x = n <= R.MOE_GATHER_ROWS, h
            if not few:
                x = s.scratch.get("moe_x", n * top, d)
                R.moe_pick(h, plan[0], x, top)
            R.moe_gemm(x, self.w_in, act, plan, first, n, self.ff, top, slots, self.act, s.status, self.alpha, self.limit, few)
            R.moe_gemm(act, self.w_out, parts, plan, second, n, d, top, slots, None, s.status)
            return parts, wts
        R.moe_tile(h, self.w_in, act, plan, self.ff, top, slots, self.act, self.alpha, self.limit)
        R.moe_tile(act, self.w_out, parts, plan, d, top, slots, None)
        if self.shared and self.act != "clamp":
            R.act_linear(h, self.s_in, s_act, self.act, self.alpha, self.shared_limit)
            R.linear(s_act, self.s_out, None, parts[:, top])
        elif self.shared:
            R.gated_linear(h, self.s_in, s.scratch.get("proj", n, 2 * self.shared_ff), s_act, "clamp", self.alpha, self.shared_limit)
            R.linear(s_act, self.s_out, None, parts[:, top])
        return parts, wts


class TokenInput:
    """What a layer adds from a table of its own rows per token: W_proj (gelu(W_gate x) * table[token]), to be RMS-normed by the seam.  ``x``
    is the residual itself; all layers' rows lie side by side in one table."""

    def __init__(self, w: W, table: torch.Tensor, col0: int):
        self.table, self.col0 = table, col0
        self.gate, self.proj = w.act("gate"), w.act("proj")
        self.dim = self.gate.shape[0]

    def reserve(self, e) -> None:
        e.scratch.reserve("side_z", e.max_rows * self.dim, self.gate.dtype)
        e.scratch.reserve("side_g", e.max_rows * self.dim, self.gate.dtype)

    def run(self, s, h):
        n = s.n
        z, g = s.scratch.get("side_z", n, self.dim), s.scratch.get("side_g", n, self.dim)
        R.token_linear(h, self.gate, self.table, self.col0, s.tokens, z, g, s.status)
        return R.linear(g, self.proj, None, s.scratch.get("y", n, h.shape[1]))


class StreamMix:
    """How a sublayer reads the residual's streams and how its output goes back into them (R.stream_seam): ``into`` [streams], ``mix`` [from, to],
    ``out`` [streams], with the residual's factor ``m`` on the output."""

    def __init__(self, w: W, m: float):
        self.into, self.mix, self.out = w.f32("in"), w.f32("mix"), (m * w.f32("out")).contiguous()
