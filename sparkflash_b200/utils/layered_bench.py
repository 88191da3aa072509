"""Throughput of a layered decoder (models/fanodra.py) at sizes that resemble a real model's layers, per-kernel roofline fractions,
and the same for the closest model of the package, the hybrid decoder of models/qwen.py (linear attention three layers in four,
softmax attention in the fourth).  ``python bench.py --design fanodra`` prints it as one JSON line.

Everything is timed on the device with CUDA events after warm-up; inputs are larger than L2, or L2 is flushed in between.
"""
from __future__ import annotations

import statistics

import torch

from ..models.fanodra import Fanodra, FanodraConfig, random_tensors
from ..models.layered import LayeredEngine
from . import roofline

# width, layers, heads, kv heads, dim, recurrence width beside attention, recurrence width alone, parts, ff, vocabulary, loop
SIZES = {
    "w1024": (1024, 8, 8, 8, 128, 1024, 1024, 8, 3072, 32768, (0, 8, 2)),
    "w2048": (2048, 12, 16, 8, 128, 2048, 2048, 16, 6144, 65536, (2, 10, 2)),
    "w4096": (4096, 8, 32, 8, 128, 4096, 4096, 16, 12288, 65536, None),
}


def config(name: str) -> FanodraConfig:
    w, n, H, G, dim, rp, ra, parts, ff, vocab, loop = SIZES[name]
    mlp = {"kind": "dense", "ff": ff}
    par = {"type": "parallel", "mlp": mlp, "mixer": {"left": {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": dim ** -0.5},
                                                     "right": {"width": rp, "blocks": parts, "conv": 4}}}
    rec = {"type": "rglru", "mlp": mlp, "mixer": {"width": ra, "blocks": parts, "conv": 4}}
    return FanodraConfig.from_dict({"architecture": "Fanodra", "name": f"fanodra-{name}", "vocab": vocab, "width": w, "norm": {"eps": 1e-6},
                                    "canon": {"taps": 4}, "layers": [par if i % 4 == 0 else rec for i in range(n)],
                                    "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None})


def engine(name: str, lanes: int, context: int, rows: int) -> LayeredEngine:
    cfg = config(name)
    return LayeredEngine(Fanodra(cfg, random_tensors(cfg, 0, "cuda"), max_context=context), max_lanes=lanes, max_context=context, max_rows=rows)


def timed(fn, reps: int, warm: int = 3, flush=None) -> float:
    """Median milliseconds of ``fn`` between events."""
    ts = []
    for i in range(warm + reps):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warm:
            ts.append(a.elapsed_time(b))
    return statistics.median(ts)


def throughput(name: str, prompt: int = 8192, chunk: int = 4096, streams=(1, 16, 64), steps: int = 32) -> dict:
    """Prefill tok/s of one prompt in portions, decode tok/s at several stream counts against ``prompt`` cached tokens (and end to
    end through ``step``, which copies inputs from pinned memory and reads the tokens back)."""
    import time
    lanes, out = max(streams), {}
    g = torch.Generator().manual_seed(0)
    eng = engine(name, lanes, prompt + 256, chunk)
    ids = torch.randint(0, eng.model.vocab, (prompt,), generator=g).tolist()
    cuts = [(p, min(p + chunk, prompt)) for p in range(0, prompt, chunk)]

    def prefill(lane):
        for a, b in cuts:
            eng.step(ids[a:b], [lane] * (b - a), list(range(a, b)), head="last" if b == prompt else False, sync=False)
    ms = timed(lambda: prefill(0), 5)
    out["prefill"] = {"tok_s": prompt / ms * 1e3, "ms": ms, "prompt": prompt, "chunk": chunk}
    for lane in range(1, lanes):
        prefill(lane)
    torch.cuda.synchronize()
    for n in streams:
        tok, lane, pos = [5] * n, list(range(n)), prompt

        def one(sync):
            nonlocal pos
            r = eng.step(tok, lane, [pos] * n, sync=sync)
            pos += 1
            return r
        for _ in range(3):
            one(True)
        key = max(eng.graphs, key=lambda k: (k[0] == n, k[1]))
        graph = eng.graphs[key]
        ms = timed(graph.replay, steps)
        t0 = time.perf_counter()
        for _ in range(steps):
            one(True)
        wall = (time.perf_counter() - t0) / steps * 1e3
        for k in range(n):                      # back to the prompt's end for the next stream count
            eng.state.lanes[k].rows = prompt
        out[f"decode_{n}"] = {"tok_s": n / ms * 1e3, "ms": ms, "e2e_tok_s": n / wall * 1e3, "context": prompt, "own_launches": eng.launches[key]}
    eng.check_status()
    out["gb"] = {k: round(v / 1e9, 2) for k, v in eng.nbytes().items()}
    eng.close()
    return out


def work(cfg: FanodraConfig, n: int, ctx: int, head_rows: int, decode: bool) -> dict[str, roofline.ClassWork]:
    """Bytes that must move and FLOPs that must be done by a step of n rows that ends at ``ctx`` cached positions (prefill: one
    segment; decode: one row in each of n lanes), per launch name."""
    d, W = cfg.width, roofline.ClassWork
    out = {k: W() for k in ("rows_seam", "rows_conv", "rows_scan", "rows_gated_step", "rows_qk_append", "rows_attn", "rows_attn_tc", "rows_act_mul",
                            "linear", "block_gates", "head")}

    def linear(k, m):
        out["linear"].flops += 2.0 * n * k * m
        out["linear"].bytes += 2.0 * (k * m + n * (k + m))
    for i, _ in cfg.runs():
        L = cfg.layers[i]
        rec = L.mixer["right"] if L.type == "parallel" else L.mixer
        w, bs = rec["width"], rec["width"] // rec["blocks"]
        linear(d, 2 * w)
        linear(w, d)
        if L.type == "parallel":
            m = L.mixer["left"]
            H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            cols = H * dim + G * (dim + vdim)
            linear(d, cols)
            linear(H * vdim, d)
            out["rows_qk_append"].bytes += 2.0 * n * cols * 2
            if decode:
                out["rows_attn"].bytes += 2.0 * n * ctx * G * (dim + vdim)
            else:
                keys = n * (ctx - n) + n * (n + 1) / 2
                out["rows_attn_tc"].flops += 2.0 * H * keys * (dim + vdim)
                out["rows_attn_tc"].bytes += 2.0 * (n * H * (dim + vdim) + ctx * G * (dim + vdim))
        out["rows_seam"].bytes += n * d * (8 + 2 + 2 + (2 if L.type == "parallel" else 0))
        if not decode:
            out["rows_conv"].bytes += 4.0 * n * (d + w)
            out["rows_scan"].bytes += n * w * (8.0 + 6.0)
            out["block_gates"].flops += 4.0 * n * w * bs
            out["block_gates"].bytes += n * w * 10.0 + 4.0 * w * bs
        else:
            out["rows_gated_step"].bytes += 4.0 * w * bs + n * w * 20.0
        if L.ff is not None:
            linear(d, 2 * L.ff)
            linear(L.ff, d)
            out["rows_act_mul"].bytes += n * L.ff * 6.0
            out["rows_seam"].bytes += n * d * 12.0
    out["head"].flops += 2.0 * head_rows * cfg.vocab * d
    out["head"].bytes += 2.0 * cfg.vocab * d
    return out


def _fractions(timings: list[list[tuple[str, float]]], wk: dict[str, roofline.ClassWork]) -> list[dict]:
    """Median over repetitions of every launch name's total, beside its roofline time."""
    by: dict[str, list[float]] = {}
    for rep in timings:
        one: dict[str, float] = {}
        for nm, us in rep:
            one[nm] = one.get(nm, 0.0) + us
        for nm, us in one.items():
            by.setdefault(nm, []).append(us)
    pk, out = roofline.peaks(), []
    for nm, ts in sorted(by.items(), key=lambda kv: -statistics.median(kv[1])):
        us, k = statistics.median(ts), wk.get(nm)
        row = {"kernel": nm, "us": round(us, 1)}
        if k is not None and (k.bytes or k.flops):
            mem, cmp = k.bytes / pk["hbm_gbs"] * 1e-3, k.flops / pk["bf16_tflops_sustained"] * 1e-6
            row.update(roofline_us=round(max(mem, cmp), 1), bound="memory" if mem >= cmp else "compute", fraction=round(max(mem, cmp) / us, 3))
        out.append(row)
    return out


def kernel_table(name: str, rows: int = 4096, ctx: int = 8192, reps: int = 5) -> list[dict]:
    """Roofline fractions per kernel of one prompt portion (the last ``rows`` of ``ctx`` positions)."""
    eng = engine(name, 1, ctx + 64, rows)
    ids = torch.randint(0, eng.model.vocab, (ctx,), generator=torch.Generator().manual_seed(0)).tolist()
    for a in range(0, ctx - rows, rows):
        eng.step(ids[a:a + rows], [0] * rows, list(range(a, a + rows)), head=False)
    call, ts = (ids[ctx - rows:], [0] * rows, list(range(ctx - rows, ctx))), []
    for _ in range(reps + 1):
        eng.state.lanes[0].rows = ctx - rows
        ts.append(roofline.timed_step(eng, *call, lead_cycles=60_000_000, head="last"))
    eng.check_status()
    cfg = eng.cfg
    eng.close()
    return _fractions(ts[1:], work(cfg, rows, ctx, 1, False))


def decode_table(name: str, n: int = 16, ctx: int = 8192, reps: int = 5) -> list[dict]:
    """The same of a decode step of n rows against ``ctx`` cached tokens each."""
    eng = engine(name, n, ctx + 64, 4096)
    eng.use_graphs = False
    ids = torch.randint(0, eng.model.vocab, (ctx,), generator=torch.Generator().manual_seed(0)).tolist()
    for lane in range(n):
        for a in range(0, ctx, 4096):
            b = min(ctx, a + 4096)
            eng.step(ids[a:b], [lane] * (b - a), list(range(a, b)), head=False)
    ts = [roofline.timed_step(eng, [5] * n, list(range(n)), [ctx + i] * n, lead_cycles=30_000_000) for i in range(reps + 1)]
    eng.check_status()
    cfg = eng.cfg
    eng.close()
    wk = work(cfg, n, ctx, n, True)
    if n <= 4:           # the streaming products take the projections and the head, gate and up fused with their activation
        wk["rows_gemv"] = roofline.ClassWork(wk["linear"].bytes + wk["head"].bytes, wk["linear"].flops + wk["head"].flops)
    wk["rows_attn_stream"] = wk["rows_attn"]
    return _fractions(ts[1:], wk)


# ---- the closest model of the package: models/qwen.py ------------------------------------------------------------------
def closest(name: str, rows: int = 256, lanes: int = 4, steps: int = 3) -> dict:
    """models/qwen.py at the same width, depth, head sizes and active feed-forward width (one expert plus the shared one): tok/s of
    its rows step, and its recurrence and convolution kernels alone on ``kernel_rows`` rows beside their rooflines."""
    from ..models import linear_attn as LA
    from ..models import qwen as Q
    w, n, H, G, dim, _, _, _, ff, vocab, _ = SIZES[name]
    c = Q.HybridConfig(vocab=vocab, d=w, layers=n, heads=H, head_dim=dim, lin_heads=H, dk=dim, dv=dim, experts=1, top_k=1, inter=ff // 2)
    torch.manual_seed(0)
    weights = {k: torch.randn_like(v, device="cuda") * v.shape[-1] ** -0.5 for k, v in _meta_weights(c).items()}
    eng = Q.HybridEngine(c, weights, lanes=lanes, max_context=rows + 64)
    ids = list(range(rows))
    out = {}
    ms = timed(lambda: eng.step(ids, [0] * rows, ids), 1, warm=1)
    out["prefill"] = {"tok_s": rows / ms * 1e3, "rows": rows}
    for m in (1, lanes):
        ms = timed(lambda: eng.step([5] * m, list(range(m)), [rows] * m), steps, warm=1)
        out[f"decode_{m}"] = {"tok_s": m / ms * 1e3, "context": rows}
    del eng, weights
    kr, pk = 4096, roofline.peaks()
    r = lambda *s: torch.randn(*s, device="cuda")
    st, cv = LA.DeltaState(1, H, dim, dim), LA.ConvState(1, H * 3 * dim, 4)
    q, k, v, a, b = r(kr, H, dim), torch.nn.functional.normalize(r(kr, H, dim), dim=-1), r(kr, H, dim), torch.rand(kr, H, device="cuda"), torch.rand(kr, H, device="cuda")
    x, cw = r(kr, H * 3 * dim).bfloat16(), r(H * 3 * dim, 4)
    for nm, fn, nbytes in (("delta_rule", lambda: st.step(q, k, v, a, b, [0] * kr), kr * H * dim * 16.0), ("short_conv", lambda: cv.step(x, cw, [0] * kr), x.numel() * 4.0)):
        us, roof = timed(fn, 3, warm=1) * 1e3, nbytes / pk["hbm_gbs"] * 1e-3
        out[nm] = {"rows": kr, "us": round(us, 1), "roofline_us": round(roof, 1), "fraction": round(roof / us, 4)}
    qq, kc = r(H, dim), r(8192, H, dim)

    def row_attention():       # what the hybrid's step does per row and full-attention layer
        s = torch.einsum("hd,shd->hs", qq, kc) * dim ** -0.5
        return torch.einsum("hs,shd->hd", torch.softmax(s, -1), kc)
    flush = torch.empty(64 << 20, device="cuda")
    us, roof = timed(row_attention, 5, flush=flush) * 1e3, 2 * kc.numel() * 4 / pk["hbm_gbs"] * 1e-3
    out["row_attention"] = {"context": 8192, "us": round(us, 1), "roofline_us": round(roof, 1), "fraction": round(roof / us, 4)}
    h, wt = r(kr, w), r(ff, w)
    us, roof = timed(lambda: h @ wt.t(), 5) * 1e3, 2.0 * kr * w * ff / pk["bf16_tflops_sustained"] * 1e-6
    out["projection_32bit"] = {"rows": kr, "us": round(us, 1), "roofline_us": round(roof, 1), "fraction": round(roof / us, 4)}
    return out


def _meta_weights(c):
    """Shapes of a hybrid model's weights without filling them on the host."""
    from ..models import qwen as Q
    real = torch.randn
    try:
        torch.randn = lambda *s, generator=None, **kw: torch.empty(*s, device="meta")
        with torch.device("meta"):
            return Q.init_weights(c)
    finally:
        torch.randn = real


def run(sizes: list[str], steps: int, compare: bool = True) -> dict:
    out = {}
    for name in sizes:
        out[name] = {"throughput": throughput(name, steps=steps), "prefill_kernels": kernel_table(name), "decode16_kernels": decode_table(name, 16),
                     "decode1_kernels": decode_table(name, 1)}
        if compare:
            out[name]["closest_model"] = closest(name)
        torch.cuda.empty_cache()
    return out
