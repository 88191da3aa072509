"""Sublayers of the layered decoders (models/layered.py): attention with a distance bias, the real-gated linear recurrence, two
mixers side by side, and the dense gated feed-forward.  Each takes its sizes and constants as arguments, reads its weights by
name, keeps its caches in the engine's page pool or state slots, and runs on a step's rows through the kernels of ops/rows.py.

A sublayer is built once per layer (``weights``) and bound once per run of the layer (``bind_run``): a looped layer shares its
weights between passes, every pass has its own keys, values and states.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from ..ops import rows as R

GATED_STEP_ROWS = 16       # up to this many single rows run convolution, gates and recurrence as one kernel


class W:
    """Weight access of one layer: ``act`` in the activation type, ``f32`` for what is computed in 32-bit."""

    def __init__(self, tensors: dict[str, torch.Tensor], prefix: str, dtype: torch.dtype, device):
        self.t, self.p, self.dtype, self.device = tensors, prefix, dtype, device

    def sub(self, name: str) -> "W":
        return W(self.t, self.p + name, self.dtype, self.device)

    def act(self, *names: str) -> torch.Tensor:
        """One matrix out of several, stacked along the output dimension."""
        return torch.cat([self.t[self.p + n] for n in names], 0).to(self.device, self.dtype).contiguous()

    def f32(self, name: str) -> torch.Tensor:
        return self.t[self.p + name].to(self.device, torch.float32).contiguous()

    def taps(self, name: str) -> torch.Tensor:
        """Convolution weights [channels, taps] as the kernels read them: [taps, channels], 32-bit."""
        return self.t[self.p + name].to(self.device, torch.float32).t().contiguous()


def log_distance_bias(r1: torch.Tensor, r2: torch.Tensor, length: int, device) -> torch.Tensor:
    """[heads, length]: r1 ln(1 + r2 distance), evaluated in 64-bit and rounded once."""
    d = torch.arange(length, dtype=torch.float64, device=device)
    return (r1.to(device, torch.float64)[:, None] * torch.log1p(r2.to(device, torch.float64)[:, None] * d)).to(torch.float32).contiguous()


class BiasedAttention:
    """Grouped-query attention over the paged cache: RMS norm over the whole query and key projections, no rotation, a distance
    bias taken off the scaled score.  Reads its q | k | v columns out of the layer's stacked projection."""

    def __init__(self, w: W, spec: dict, eps: float, max_context: int):
        self.H, self.G, self.dim, self.vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        self.scale, self.eps = float(spec["scale"]), eps
        self.cols = self.H * self.dim + self.G * (self.dim + self.vdim)
        self.q_norm, self.k_norm = w.f32("q.norm"), w.f32("k.norm")
        self.bias = log_distance_bias(w.f32("r1"), w.f32("r2"), max_context, w.device)
        self.wo, self.bo = w.act("o"), w.act("o.b")
        self.tc = R.attn_tc_supports(self.wo.dtype, self.dim, self.vdim)
        self.stream = R.attn_stream_supports(self.wo.dtype, self.dim, self.vdim)

    PROJ, PROJ_BIAS = ("q", "k", "v"), ("q.b", "k.b", "v.b")

    def reserve(self, e) -> None:
        n, dt = e.max_rows, self.wo.dtype
        e.scratch.reserve("attn_q", n * self.H * self.dim, dt)
        e.scratch.reserve("attn_o", n * self.H * self.vdim, dt)
        # partial outputs of split rows: rows x heads x ranges, bounded by the blocks of one launch (see LayeredEngine.splits)
        per = self.H // R.attn_blocks(self.H, self.G)
        parts = max(1, per) * 1024 + self.H * 64
        if self.stream:
            parts = max(parts, 2 * R.STREAM_CTAS * R.attn_stream_heads(self.H, self.G, self.dim))
        e.scratch.reserve("attn_part", parts * self.vdim, torch.float32)
        e.scratch.reserve("attn_ml", parts * 2, torch.float32)

    def run(self, s, proj, kv, out):
        """proj [n, >= cols] view whose first columns are q | k | v; kv = (k pool, v pool) of this run."""
        n, k, v = s.n, kv[0], kv[1]
        q = s.scratch.get("attn_q", n, self.H * self.dim)
        o = s.scratch.get("attn_o", n, self.H * self.vdim)
        R.qk_append(proj, self.q_norm, self.k_norm, q, k, v, s.table, s.row_lane, s.row_pos, n, self.H, self.eps, s.status)
        if s.ntiles:
            R.attn_tc(q, kv, s.table, s.row_lane, s.row_pos, s.tiles, s.ntiles, self.bias, o, self.H, self.scale, s.status)
        if s.short and self.stream and s.short <= R.STREAM_ROWS:
            R.attn_stream(q, k, v, s.table, s.row_lane, s.row_pos, s.short_rows, s.short, self.bias, o, s.scratch.buf["attn_part"],
                          s.scratch.buf["attn_ml"], self.H, self.scale, s.short * s.pages, s.status)
        elif s.short:
            blocks = R.attn_blocks(self.H, self.G)
            sp = s.engine.splits(s, s.short, blocks)
            part = s.scratch.buf["attn_part"] if sp > 1 else None
            ml = s.scratch.buf["attn_ml"] if sp > 1 else None
            R.attn(q, k, v, s.table, s.row_lane, s.row_pos, s.short_rows, s.short, self.bias, o, part, ml, self.H, self.scale, sp, s.status)
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
            R.conv(x, self.cw, self.cb, u, hist, s, n, residual=False)
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


class DenseFF:
    """W_down (silu(W_gate h) * (W_up h)) with gate and up in one product."""

    def __init__(self, w: W):
        self.w_in, self.w_out = w.act("gate", "up"), w.act("down")
        self.ff = self.w_out.shape[1]

    def reserve(self, e) -> None:
        e.scratch.reserve("proj", e.max_rows * 2 * self.ff, self.w_in.dtype)
        e.scratch.reserve("ff_act", e.max_rows * self.ff, self.w_in.dtype)

    def run(self, s, h):
        act = R.gated_linear(h, self.w_in, s.scratch.get("proj", s.n, 2 * self.ff), s.scratch.get("ff_act", s.n, self.ff))
        return R.linear(act, self.w_out, None, s.scratch.get("y", s.n, h.shape[1]))
