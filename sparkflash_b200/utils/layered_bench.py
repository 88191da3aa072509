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
    out = {k: W() for k in ("rows_seam", "rows_conv", "rows_scan", "rows_gated_step", "rows_qk_append", "rows_attn", "rows_attn_tc", "rows_silu_mul",
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
            out["rows_silu_mul"].bytes += n * L.ff * 6.0
            out["rows_seam"].bytes += n * d * 12.0
    out["head"].flops += 2.0 * head_rows * cfg.vocab * d
    out["head"].bytes += 2.0 * cfg.vocab * d
    return out


def kernel_table(name: str, rows: int = 4096, ctx: int = 8192) -> list[dict]:
    """Roofline fractions per kernel of one prompt portion (the last ``rows`` of ``ctx`` positions), event after every launch."""
    eng = engine(name, 1, ctx + 64, rows)
    ids = torch.randint(0, eng.model.vocab, (ctx,), generator=torch.Generator().manual_seed(0)).tolist()
    for a in range(0, ctx - rows, rows):
        eng.step(ids[a:a + rows], [0] * rows, list(range(a, a + rows)), head=False)
    call = (ids[ctx - rows:], [0] * rows, list(range(ctx - rows, ctx)))
    best: dict[str, list[float]] = {}
    for _ in range(5):
        eng.state.lanes[0].rows = ctx - rows
        by: dict[str, list[float]] = {}
        for nm, us in roofline.timed_step(eng, *call, head="last"):
            by.setdefault(nm, []).append(us)
        for nm, ts in by.items():
            best.setdefault(nm, []).append(sum(ts))
    eng.check_status()
    wk, pk, table = work(eng.cfg, rows, ctx, 1, False), roofline.peaks(), []
    for nm, ts in sorted(best.items(), key=lambda kv: -min(kv[1])):
        us, k = min(ts), wk.get(nm, roofline.ClassWork())
        mem, cmp = k.bytes / pk["hbm_gbs"] * 1e-3, k.flops / pk["bf16_tflops_sustained"] * 1e-6
        table.append({"kernel": nm, "us": round(us, 1), "roofline_us": round(max(mem, cmp), 1), "bound": "memory" if mem >= cmp else "compute",
                      "fraction": round(max(mem, cmp) / us, 3)})
    eng.close()
    return table
