"""Throughput of a layered decoder (models/fanodra.py, models/gudutar.py, models/lifulorn.py, models/dironex.py) at sizes that resemble a real model's layers,
per-kernel roofline fractions, and the same for the closest model of the package: for Fanodra the hybrid decoder of models/qwen.py (linear
attention three layers in four, softmax attention in the fourth), for Gudutar the Fanodra of the same width, head size, feed-forward
width and number of layer runs, for Lifulorn the Gudutar of the same width, number of layers, head size and active feed-forward width, for
Dironex the Lifulorn (windowed attention, experts) and the Gudutar (latent attention) of the same sizes.  ``python bench.py --design NAME`` prints it as one JSON line.

Everything is timed on the device with CUDA events after warm-up; inputs are larger than L2, or L2 is flushed in between.
"""
from __future__ import annotations

import statistics

import torch

from ..models import dironex, fanodra, gudutar, lifulorn
from ..models.dironex import DironexConfig
from ..models.fanodra import FanodraConfig
from ..models.gudutar import GudutarConfig
from ..models.lifulorn import LifulornConfig
from ..models.layered import LayeredEngine
from . import roofline

# width, layers, heads, kv heads, dim, recurrence width beside attention, recurrence width alone, parts, ff, vocabulary, loop
SIZES = {
    "w1024": (1024, 8, 8, 8, 128, 1024, 1024, 8, 3072, 32768, (0, 8, 2)),
    "w2048": (2048, 12, 16, 8, 128, 2048, 2048, 16, 6144, 65536, (2, 10, 2)),
    "w4096": (4096, 8, 32, 8, 128, 4096, 4096, 16, 12288, 65536, None),
}


def fanodra_config(name: str) -> FanodraConfig:
    w, n, H, G, dim, rp, ra, parts, ff, vocab, loop = SIZES[name]
    mlp = {"kind": "dense", "ff": ff}
    par = {"type": "parallel", "mlp": mlp, "mixer": {"left": {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": dim ** -0.5},
                                                     "right": {"width": rp, "blocks": parts, "conv": 4}}}
    rec = {"type": "rglru", "mlp": mlp, "mixer": {"width": ra, "blocks": parts, "conv": 4}}
    return FanodraConfig.from_dict({"architecture": "Fanodra", "name": f"fanodra-{name}", "vocab": vocab, "width": w, "norm": {"eps": 1e-6},
                                    "canon": {"taps": 4}, "layers": [par if i % 4 == 0 else rec for i in range(n)],
                                    "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None})


WINDOW, RANK, ROT = 1024, 512, 64        # latent attention
ORDER = ("mamba2", "retention", "latent_attention", "mamba2")


def gudutar_config(name: str) -> GudutarConfig:
    """As many layers as the Fanodra of that size has layer runs; recurrences of twice / once the width, heads of 64 x 128 and 128 x 128."""
    w, n, H, _, dim, _, _, _, ff, vocab, loop = SIZES[name]
    runs = n + (loop[1] - loop[0]) * (loop[2] - 1) if loop else n
    rot = lambda dims: {"base": 10000.0, "dims": dims}
    mixers = {"mamba2": {"heads": 2 * w // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1},
              "retention": {"heads": w // dim, "dim": dim, "vdim": dim, "rot": rot(dim), "decay": [1 - 2.0 ** (-5 - 7 * i / (w // dim)) for i in range(w // dim)]},
              "latent_attention": {"heads": H, "dim": dim, "rot_dim": ROT, "vdim": dim, "kv_rank": RANK, "scale": (dim + ROT) ** -0.5,
                                   "mask": {"size": WINDOW}, "rot": rot(ROT)}}
    return GudutarConfig.from_dict({"architecture": "Gudutar", "name": f"gudutar-{name}", "vocab": vocab, "width": w, "norm": {"eps": 1e-6},
                                    "embedding": {"scale": 1.0}, "layers": [{"type": t, "mixer": mixers[t], "mlp": {"kind": "dense", "ff": ff}}
                                                                            for t in (ORDER[i % 4] for i in range(runs))]})


EXPERTS, TOP, SIDE = 32, 4, 128
RULES = ("delta", "attention", "delta", "attention_2")


def lifulorn_config(name: str) -> LifulornConfig:
    """As many layers as the Gudutar of that size; the delta rule with a head of 128 x 128 per 128 of the width, attention with the Gudutar's heads
    and window.  Every row uses TOP of EXPERTS experts and the shared one, together as wide as the other design's feed-forward."""
    w, _, H, G, dim, _, _, _, ff, vocab, _ = SIZES[name]
    each = ff // (TOP + 2)
    mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": each, "limit": 7.0}, "shared": {"ff": ff - TOP * each, "limit": 7.0}}
    att = {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": WINDOW}, "v_mix": True}
    wave = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 4096}
    yarn = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    mixers = {"delta": {"heads": w // dim, "kv_heads": w // dim, "dim": dim, "vdim": dim, "conv": 4},
              "attention": {**att, "rot": {"base": 500000.0, "dims": dim, "scaling": wave}},
              "attention_2": {**att, "softcap": 50.0, "rot": {"base": 500000.0, "dims": dim, "scaling": yarn}}}
    return LifulornConfig.from_dict({"architecture": "Lifulorn", "name": f"lifulorn-{name}", "vocab": vocab, "width": w, "norm": {"eps": 1e-6},
                                     "residual_mult": 0.5, "token_side": {"dim": SIDE},
                                     "layers": [{"type": t, "mixer": mixers[t], "mlp": mlp} for t in (RULES[i % 4] for i in range(len(gudutar_config(name).layers)))]})


STREAMS, GROUPS, KEEP = 4, 8, 4
SUBLAYERS = (("attention", "moe"), ("latent_attention", "dense"), ("attention", "dense"), ("latent_attention", "moe"))


def dironex_config(name: str) -> DironexConfig:
    """The Fanodra's layers and loop; attention with the other designs' heads and window, latent attention with their heads, latent and rotated part,
    over the whole context.  A feed-forward has two matrices instead of three and is half as wide again, so that a row uses as many weights."""
    w, n, H, G, dim, _, _, _, ff, vocab, loop = SIZES[name]
    wide = ff * 3 // 2
    mlp = {"dense": {"kind": "dense", "ff": wide},
           "moe": {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "groups": {"count": GROUPS, "keep": KEEP}, "scale": 1.0}, "expert": {"ff": wide // TOP}}}
    yarn = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    mixers = {"attention": {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": WINDOW}},
              "latent_attention": {"heads": H, "dim": dim, "rot_dim": ROT, "vdim": dim, "kv_rank": RANK, "q_rank": min(w // 2, 1536), "scale": (dim + ROT) ** -0.5,
                                   "rot": {"base": 500000.0, "dims": ROT, "scaling": yarn}}}
    return DironexConfig.from_dict({"architecture": "Dironex", "name": f"dironex-{name}", "vocab": vocab, "width": w, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
                                    "residual_mult": 0.5, "streams": STREAMS, "canon": {"taps": 4}, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None,
                                    "layers": [{"type": t, "mixer": mixers[t], "mlp": mlp[f]} for t, f in (SUBLAYERS[i % 4] for i in range(n))]})


CONFIGS = {"fanodra": (fanodra_config, fanodra.Fanodra, fanodra.random_tensors), "gudutar": (gudutar_config, gudutar.Gudutar, gudutar.random_tensors),
           "lifulorn": (lifulorn_config, lifulorn.Lifulorn, lifulorn.random_tensors), "dironex": (dironex_config, dironex.Dironex, dironex.random_tensors)}


def engine(design: str, name: str, lanes: int, context: int, rows: int) -> LayeredEngine:
    make, cls, weights = CONFIGS[design]
    cfg = make(name)
    return LayeredEngine(cls(cfg, weights(cfg, 0, "cuda"), max_context=context), max_lanes=lanes, max_context=context, max_rows=rows)


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


def _own(ids: list[int], lane: int) -> list[int]:
    """A lane's prompt: the same tokens from another place on, so that lanes do not choose the same experts."""
    k = 97 * lane % len(ids)
    return ids[k:] + ids[:k]


def throughput(design: str, name: str, prompt: int = 8192, chunk: int = 4096, streams=(1, 16, 64), steps: int = 32) -> dict:
    """Prefill tok/s of one prompt in portions, decode tok/s at several stream counts against ``prompt`` cached tokens (and end to
    end through ``step``, which copies inputs from pinned memory and reads the tokens back)."""
    import time
    lanes, out = max(streams), {}
    g = torch.Generator().manual_seed(0)
    eng = engine(design, name, lanes, prompt + 256, chunk)
    ids = torch.randint(0, eng.model.vocab, (prompt,), generator=g).tolist()
    cuts = [(p, min(p + chunk, prompt)) for p in range(0, prompt, chunk)]

    def prefill(lane):
        own = _own(ids, lane)
        for a, b in cuts:
            eng.step(own[a:b], [lane] * (b - a), list(range(a, b)), head="last" if b == prompt else False, sync=False)
    ms = timed(lambda: prefill(0), 5)
    out["prefill"] = {"tok_s": prompt / ms * 1e3, "ms": ms, "prompt": prompt, "chunk": chunk}
    for lane in range(1, lanes):
        prefill(lane)
    torch.cuda.synchronize()
    for n in streams:
        tok, lane, pos = [(5 + 37 * k) % eng.model.vocab for k in range(n)], list(range(n)), prompt

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


def gudutar_work(cfg: GudutarConfig, n: int, ctx: int, head_rows: int, decode: bool) -> dict[str, roofline.ClassWork]:
    """The same accounting for Gudutar.  Recurrences: inputs and outputs once, the state of every segment in and out, and for prompts the
    products of chunks of 128 rows, those with a 32-bit operand counted once per pair of bf16 terms (the products the chunked form needs
    at that precision); attention: the window's keys (prompts: multiplied out, in ``linear``)."""
    d, W = cfg.width, roofline.ClassWork
    out = {k: W() for k in ("rows_seam", "rows_conv", "rows_state", "rows_state_tc", "rows_state_turn", "rows_gated_norm", "rows_latent_append", "rows_head_proj",
                            "rows_latent_decode", "rows_attn_tc", "rows_gather_pages", "rows_act_mul", "linear", "head")}
    out["rows_attn"] = out["rows_latent_decode"]

    def linear(k, m, rows=n):
        out["linear"].flops += 2.0 * rows * k * m
        out["linear"].bytes += 2.0 * (k * m + rows * (k + m))

    def state(H, G, N, P, cols, turned):
        segs = n if decode else 1
        if decode:
            out["rows_state"].bytes += segs * H * N * P * 8.0 + 2.0 * n * (cols + H * P)
        else:
            out["rows_state_tc"].bytes += segs * H * N * P * 8.0 + 2.0 * n * (cols + H * P)
            # q k^T of a group (visible half), weights times v, q S, k^T v; turned q and k have two terms: three products, less lo x lo
            s, i = (3, 3) if turned else (1, 2)
            out["rows_state_tc"].flops += n * (G * s * 128.0 * N + H * (2 * 128.0 * P + 2.0 * i * N * P + 2.0 * i * N * P))
            out["rows_state_turn"].bytes += 2.0 * n * 6 * H * N if turned else 0.0
    out["rows_seam"].bytes += n * d * 8.0
    for L in cfg.layers:
        m, H = L.mixer, L.mixer["heads"]
        inner = H * m["vdim"]
        linear(inner, d)
        if L.type == "mamba2":
            bc = 2 * m["groups"] * m["state"]
            linear(d, 2 * inner + bc + H)
            state(H, m["groups"], m["state"], m["vdim"], inner + bc + H, False)
            out["rows_conv"].bytes += 0.0 if decode else 4.0 * n * (inner + bc)
            out["rows_gated_norm"].bytes += 6.0 * n * inner
        elif L.type == "retention":
            linear(d, 2 * H * m["dim"] + 2 * inner)
            state(H, H, m["dim"], m["vdim"], 2 * H * m["dim"] + inner, True)
            out["rows_gated_norm"].bytes += 6.0 * n * inner
        else:
            r, key, win = m["kv_rank"], m["kv_rank"] + m["rot_dim"], min(m["mask"]["size"], ctx)
            qd = m["dim"] + m["rot_dim"]
            linear(d, H * qd + key)
            out["rows_latent_append"].bytes += 2.0 * n * (2 * H * m["rot_dim"] + 2 * key)
            if decode:
                out["rows_head_proj"].bytes += 2.0 * H * r * (m["dim"] + m["vdim"]) + 2.0 * n * H * (m["dim"] + m["vdim"] + r + key)
                out["rows_latent_decode"].bytes += 2.0 * n * (win * key + H * (key + r))
                out["rows_latent_decode"].flops += 2.0 * n * H * win * (key + r)
            else:
                keys = n + min(ctx - n, win - 1)
                out["rows_gather_pages"].bytes += 4.0 * keys * key
                linear(r, H * (m["dim"] + m["vdim"]), keys)
                seen = n * win if ctx - n >= win else n * (ctx - n) + n * (n + 1) / 2
                out["rows_attn_tc"].flops += 2.0 * H * seen * (qd + m["vdim"])
                out["rows_attn_tc"].bytes += 2.0 * (n * H * (qd + m["vdim"]) + keys * H * (m["dim"] + m["vdim"]))
        out["rows_seam"].bytes += n * d * 12.0
        if L.ff is not None:
            linear(d, 2 * L.ff)
            linear(L.ff, d)
            out["rows_act_mul"].bytes += n * L.ff * 6.0
            out["rows_seam"].bytes += n * d * 12.0
    out["head"].flops += 2.0 * head_rows * cfg.vocab * d
    out["head"].bytes += 2.0 * cfg.vocab * d
    return out


def lifulorn_work(cfg: LifulornConfig, n: int, ctx: int, head_rows: int, decode: bool) -> dict[str, roofline.ClassWork]:
    """The same accounting for Lifulorn.  Delta rule: as the other recurrences, the chunked products (with the inverse of every chunk's triangle) once
    per pair of bf16 terms; experts: the weights of those that the rows can touch, and their products."""
    d, W, side = cfg.width, roofline.ClassWork, cfg.side_dim
    out = {k: W() for k in ("rows_seam", "rows_conv", "rows_state", "rows_delta_tc", "rows_gated_norm", "rows_rot_append", "rows_attn_stream", "rows_attn_tc",
                            "rows_token_gate", "rows_moe_gemm", "rows_moe_gemv", "rows_moe_route", "rows_moe_plan", "rows_moe_pick", "linear", "router", "head")}
    few = n <= 4

    def linear(k, m, name="linear"):
        out[name].flops += 2.0 * n * k * m
        out[name].bytes += 2.0 * (k * m + n * (k + m))
    out["rows_seam"].bytes += n * d * 8.0
    for L in cfg.layers:
        m, H, G = L.mixer, L.mixer["heads"], L.mixer["kv_heads"]
        dim, vdim = m["dim"], m["vdim"]
        inner = H * vdim
        linear(inner, d)
        if L.type == "delta":
            cols = 2 * G * dim + inner
            linear(d, cols + inner + 2 * H)
            segs, nbytes = n if decode else 1, 2.0 * n * (cols + 2 * H + inner)
            if decode:
                out["rows_state"].bytes += segs * H * dim * vdim * 8.0 + nbytes
            else:
                # visible halves of k k^T and q k^T, the inverse (a third of a full product, 32-bit: as three), then per value dim: K S and Q S, inverse X
                # and weights U (visible halves, three products), K^T U; two products where one operand has two terms
                out["rows_delta_tc"].bytes += segs * H * dim * vdim * 8.0 + nbytes
                out["rows_delta_tc"].flops += n * (G * 2 * 128.0 * dim + H * (3 * 2 * 128.0 * 128 / 6 + vdim * (3 * 4.0 * dim + 2 * 3 * 128.0)))
                out["rows_conv"].bytes += 4.0 * n * cols
            if decode and n > 4:
                out["rows_conv"].bytes += 4.0 * n * cols
            out["rows_gated_norm"].bytes += 6.0 * n * inner
        else:
            cols, win = H * dim + G * (dim + vdim), min(m["mask"]["size"], ctx)
            linear(d, cols)
            out["rows_rot_append"].bytes += 4.0 * n * cols
            if decode:
                out["rows_attn_stream"].bytes += 2.0 * n * (win * G * (dim + vdim) + H * (dim + vdim))
            else:
                seen, keys = n * win if ctx - n >= win else n * (ctx - n) + n * (n + 1) / 2, n + min(ctx - n, win - 1)
                out["rows_attn_tc"].flops += 2.0 * H * seen * (dim + vdim)
                out["rows_attn_tc"].bytes += 2.0 * (n * H * (dim + vdim) + keys * G * (dim + vdim))
        out["rows_seam"].bytes += n * d * 12.0
        if L.mlp is not None:
            E, top, ff, sff = L.mlp["router"]["experts"], L.mlp["router"]["top"], L.mlp["expert"]["ff"], L.mlp["shared"]["ff"]
            used = E * (1 - (1 - top / E) ** n)              # experts that n rows touch, on average
            linear(d, E + 1, "router")
            out["rows_moe_route"].bytes += n * (4.0 * E + 8.0 * top)
            out["rows_moe_plan"].bytes += n * top * 16.0
            if few:
                out["rows_moe_gemv"].bytes += 2.0 * 3 * d * (n * top * ff + sff)
            else:
                out["rows_moe_gemm"].bytes += 2.0 * (3 * d * (used * ff + sff) + n * (d + top * (2 * ff + d) + 2 * sff + d))
                out["rows_moe_pick"].bytes += 0.0 if decode else 2.0 * n * d * (1 + top)
                out["rows_moe_gemm"].flops += 2.0 * n * 3 * d * (top * ff + sff)
            out["rows_seam"].bytes += n * d * (10.0 + 2.0 * (top + 1))
        linear(d, side)
        linear(side, d)
        out["rows_token_gate"].bytes += n * side * 6.0
        out["rows_seam"].bytes += n * d * 12.0
    out["head"].flops += 2.0 * head_rows * cfg.vocab * d
    out["head"].bytes += 2.0 * cfg.vocab * d
    return out


def dironex_work(cfg: DironexConfig, n: int, ctx: int, head_rows: int, decode: bool) -> dict[str, roofline.ClassWork]:
    """The same accounting for Dironex.  Seam: every stream in and out once per sublayer."""
    d, W, few = cfg.width, roofline.ClassWork, n <= 4
    out = {k: W() for k in ("rows_streams", "rows_conv", "rows_head_append", "rows_attn_stream", "rows_attn_tc", "rows_latent_append", "rows_latent_turn",
                            "rows_head_proj", "rows_latent_decode", "rows_gather_pages", "rows_act", "rows_moe_gemm", "rows_moe_gemv", "rows_moe_route", "rows_moe_plan",
                            "rows_moe_pick", "linear", "router", "head")}

    def linear(k, m, rows=n, name="linear"):
        out[name].flops += 2.0 * rows * k * m
        out[name].bytes += 2.0 * (k * m + rows * (k + m))

    def seam(parts=1):
        out["rows_streams"].bytes += n * d * (8.0 * cfg.streams + 2.0 * parts + 2.0)
        out["rows_conv"].bytes += 0.0 if decode else 4.0 * n * d
    out["rows_streams"].bytes += n * d * (4.0 * cfg.streams + 4.0) + head_rows * d * (4.0 * cfg.streams + 4.0)
    out["rows_conv"].bytes += 0.0 if decode else 4.0 * n * d
    for at, i in enumerate(cfg.runs()):
        L = cfg.layers[i]
        m, H, dim, vdim = L.mixer, L.mixer["heads"], L.mixer["dim"], L.mixer["vdim"]
        inner = H * vdim
        linear(inner, d)
        if L.type == "attention":
            G = m["kv_heads"]
            cols, win = H * dim + G * (dim + vdim), min(m["mask"]["size"], ctx)
            linear(d, cols)
            out["rows_head_append"].bytes += 4.0 * n * cols
            if decode:
                out["rows_attn_stream"].bytes += 2.0 * n * (win * G * (dim + vdim) + H * (dim + vdim))
            else:
                seen, keys = n * win if ctx - n >= win else n * (ctx - n) + n * (n + 1) / 2, n + min(ctx - n, win - 1)
                out["rows_attn_tc"].flops += 2.0 * H * seen * (dim + vdim)
                out["rows_attn_tc"].bytes += 2.0 * (n * H * (dim + vdim) + keys * G * (dim + vdim))
        else:
            r, rot, qr = m["kv_rank"], m["rot_dim"], m["q_rank"]
            key, qd = r + rot, dim + rot
            linear(d, inner + key + qr)
            linear(qr, H * qd)
            out["rows_latent_append"].bytes += 4.0 * n * (key + qr)
            if decode:
                out["rows_head_proj"].bytes += 2.0 * H * r * (dim + vdim) + 2.0 * n * H * (dim + 2 * vdim + r + key)
                out["rows_latent_decode"].bytes += 2.0 * n * (ctx * key + H * (key + r))
                out["rows_latent_decode"].flops += 2.0 * n * H * ctx * (key + r)
            else:
                out["rows_latent_turn"].bytes += 4.0 * n * H * rot
                out["rows_gather_pages"].bytes += 4.0 * ctx * key
                linear(r, H * (dim + vdim), ctx)
                seen = n * (ctx - n) + n * (n + 1) / 2
                out["rows_attn_tc"].flops += 2.0 * H * seen * (qd + vdim)
                out["rows_attn_tc"].bytes += 2.0 * (n * H * (qd + 2 * vdim) + ctx * H * (dim + vdim))
        if L.mlp is not None and L.mlp["kind"] == "dense":
            ff = L.mlp["ff"]
            seam()
            linear(d, ff)
            linear(ff, d)
            out["rows_act"].bytes += 0.0 if few else 4.0 * n * ff
        elif L.mlp is not None:
            E, top, ff = L.mlp["router"]["experts"], L.mlp["router"]["top"], L.mlp["expert"]["ff"]
            used = E * (1 - (1 - top / E) ** n)              # experts that n rows touch, on average
            seam()
            linear(d, E, name="router")
            out["rows_moe_route"].bytes += n * (4.0 * E + 8.0 * top)
            out["rows_moe_plan"].bytes += n * top * 16.0
            if few:
                out["rows_moe_gemv"].bytes += 2.0 * 2 * d * n * top * ff
            else:
                out["rows_moe_gemm"].bytes += 2.0 * (2 * d * used * ff + n * (d + top * (2 * ff + d)))
                out["rows_moe_pick"].bytes += 0.0 if decode else 2.0 * n * d * (1 + top)
                out["rows_moe_gemm"].flops += 2.0 * n * 2 * d * top * ff
        if at + 1 < len(cfg.runs()):
            seam(L.mlp["router"]["top"] if L.mlp is not None and L.mlp["kind"] == "moe" else 1)
    out["head"].flops += 2.0 * head_rows * cfg.vocab * d
    out["head"].bytes += 2.0 * cfg.vocab * d
    return out


def fanodra_work(cfg: FanodraConfig, n: int, ctx: int, head_rows: int, decode: bool) -> dict[str, roofline.ClassWork]:
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


WORK = {"fanodra": fanodra_work, "gudutar": gudutar_work, "lifulorn": lifulorn_work, "dironex": dironex_work}
CLOSEST = {"gudutar": ("fanodra",), "lifulorn": ("gudutar",), "dironex": ("lifulorn", "gudutar")}


def kernel_table(design: str, name: str, rows: int = 4096, ctx: int = 8192, reps: int = 5) -> list[dict]:
    """Roofline fractions per kernel of one prompt portion (the last ``rows`` of ``ctx`` positions)."""
    eng = engine(design, name, 1, ctx + 64, rows)
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
    return _fractions(ts[1:], WORK[design](cfg, rows, ctx, 1, False))


def decode_table(design: str, name: str, n: int = 16, ctx: int = 8192, reps: int = 5) -> list[dict]:
    """The same of a decode step of n rows against ``ctx`` cached tokens each."""
    eng = engine(design, name, n, ctx + 64, 4096)
    eng.use_graphs = False
    ids = torch.randint(0, eng.model.vocab, (ctx,), generator=torch.Generator().manual_seed(0)).tolist()
    for lane in range(n):
        for a in range(0, ctx, 4096):
            b = min(ctx, a + 4096)
            eng.step(_own(ids, lane)[a:b], [lane] * (b - a), list(range(a, b)), head=False)
    ts = [roofline.timed_step(eng, [(5 + 37 * k) % eng.model.vocab for k in range(n)], list(range(n)), [ctx + i] * n, lead_cycles=30_000_000) for i in range(reps + 1)]
    eng.check_status()
    cfg = eng.cfg
    eng.close()
    wk = WORK[design](cfg, n, ctx, n, True)
    if n <= 4:           # the streaming products take the projections and the head, gate and up fused with their activation
        wk["rows_gemv"] = roofline.ClassWork(*(sum(getattr(wk[k], f) for k in ("linear", "head", "router") if k in wk) for f in ("bytes", "flops")))
    if design == "fanodra":
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


def measure(design: str, name: str, steps: int) -> dict:
    out = {"throughput": throughput(design, name, steps=steps), "prefill_kernels": kernel_table(design, name),
           "decode16_kernels": decode_table(design, name, 16), "decode1_kernels": decode_table(design, name, 1)}
    torch.cuda.empty_cache()
    return out


def run(design: str, sizes: list[str], steps: int, compare: bool = True) -> dict:
    out = {}
    for name in sizes:
        out[name] = measure(design, name, steps)
        if compare:
            if design == "fanodra":
                out[name]["closest_model"] = closest(name)
            else:
                for key, other in zip(("closest_model", "second_closest_model"), CLOSEST[design]):
                    out[name][key] = {"design": other, **measure(other, name, steps)}
        torch.cuda.empty_cache()
    return out
