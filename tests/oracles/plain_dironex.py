"""Plain, slow implementation of the Dironex design, one function per mechanism, on the CPU.

Nothing here is shared with the product path: weights are a dict of tensors under their file names, the configuration is the
parsed ``config.json`` dict, and every function spells its equation out over a whole sequence (no cache, no chunks, no batching).
``dtype`` chooses the arithmetic (float64 for a sharp oracle)."""
from __future__ import annotations

import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


# ---- residual streams ---------------------------------------------------------------------------------------------------
def collapse(X, into):
    """X [streams, T, d]: what a sublayer reads of the streams."""
    return sum(into[s] * X[s] for s in range(X.shape[0]))


def spread(X, mix, out, m, y):
    """New streams from all the old ones (mix[from, to]) and a sublayer's output."""
    S = X.shape[0]
    return torch.stack([sum(mix[s, t] * X[s] for s in range(S)) + m * out[t] * y for t in range(S)])


def input_convolution(h, w):
    """Every row plus its channels' weighted sum over itself (last column of w) and the rows before it; rows that do not exist count as zero."""
    T, taps, out = h.shape[0], w.shape[1], h.clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] = out[back:] + w[:, j] * h[:T - back]
    return out


# ---- rotation -----------------------------------------------------------------------------------------------------------
def frequencies(base, dims, sc=None):
    """Radians per position of every pair, and the factor on cosine and sine."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return f, 1.0

    def where(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1


def turn(x, base, dims, sc=None):
    """x [T, heads, >= dims]: dimension i turns with dimension i + dims / 2."""
    f, gain = frequencies(base, dims, sc)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    c, s = (gain * a.cos()).to(x.dtype)[:, None], (gain * a.sin()).to(x.dtype)[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ---- attention ----------------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, window=None):
    """q [T, H, .], k and v [T, H, .]: softmax over the visible keys."""
    T = q.shape[0]
    dist = torch.arange(T)[:, None] - torch.arange(T)
    seen = (dist >= 0) & (dist < (window if window is not None else T))
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~seen, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hij,jhd->ihd", e / e.sum(-1, keepdim=True), v)


def window_attention(h, w, p, m, eps):
    """Grouped-query attention in a window; queries and keys normed head by head; no rotation."""
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].t()).view(T, H, dim), w[p + "q.norm"], eps)
    k = rms((h @ w[p + "k"].t()).view(T, G, dim), w[p + "k.norm"], eps).repeat_interleave(H // G, 1)
    v = (h @ w[p + "v"].t()).view(T, G, vdim).repeat_interleave(H // G, 1)
    return attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, H * vdim) @ w[p + "o"].t()


def latent_attention(h, w, p, m, eps):
    """Keys and values out of a normed latent, queries out of another one, one rotated key part for all heads, gated output."""
    T, H, dim, rd, vdim, rank, rot = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["rot"]
    q = (rms(h @ w[p + "dq"].t(), w[p + "dq.norm"], eps) @ w[p + "uq"].t()).view(T, H, dim + rd)
    down = h @ w[p + "dkv"].t()
    c, shared = rms(down[:, :rank], w[p + "dkv.norm"], eps), down[:, None, rank:]
    turned = lambda x: turn(x, rot["base"], rot["dims"], rot.get("scaling"))
    q = torch.cat([q[..., :dim], turned(q[..., dim:])], -1)
    k = torch.cat([(c @ w[p + "uk"].t()).view(T, H, dim), turned(shared).expand(T, H, rd)], -1)
    v = (c @ w[p + "uv"].t()).view(T, H, vdim)
    o = attend(q, k, v, m["scale"]).reshape(T, H * vdim)
    return (o * sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def xielu(z, p, q):
    return torch.where(z > 0, softplus(p) * z * z + z / 2, (0.5 + softplus(q)) * (torch.exp(z) - 1 - z) + z / 2)


def dense(h, w, p):
    return xielu(h @ w[p + "up"].t(), *w[p + "act"]) @ w[p + "down"].t()


def route(z, correction, r, margins=None):
    """Chosen experts and weights of every row of logits; ``margins`` collects how far each row is from another choice."""
    s, E = sigmoid(z), z.shape[1]
    choice = s + correction
    g = r.get("groups") or {"count": 1, "keep": 1}
    per = E // g["count"]
    ids, wts = [], []
    for t in range(z.shape[0]):
        row = choice[t].tolist()
        score = [sum(sorted(row[a * per:(a + 1) * per], reverse=True)[:2]) for a in range(g["count"])]
        groups = sorted(range(g["count"]), key=lambda a: (-score[a], a))
        open_ = [e for a in groups[:g["keep"]] for e in range(a * per, (a + 1) * per)]
        ranked = sorted(open_, key=lambda e: (-row[e], e))
        best = ranked[:r["top"]]
        v = s[t, best]
        ids.append(best)
        wts.append(v / (v.sum() + 1e-20) * r["scale"])
        if margins is not None:
            gap = [score[groups[g["keep"] - 1]] - score[groups[g["keep"]]]] if g["keep"] < g["count"] else []
            gap += [row[best[-1]] - row[ranked[r["top"]]]] if r["top"] < len(ranked) else []
            margins.append(min(gap, default=float("inf")))
    return ids, wts


def expert(h, w, p):
    u = (h @ w[p + "up"].t()).clamp(min=0)
    return (u * u) @ w[p + "down"].t()


def mixture(h, w, p, r, margins=None):
    ids, wts = route(h @ w[p + "router"].t(), w[p + "correction"], r, margins)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        at = [(t, k) for t in range(h.shape[0]) for k in range(r["top"]) if ids[t][k] == e]
        if at:
            rows = [t for t, _ in at]
            out[rows] += torch.stack([wts[t][k] for t, k in at])[:, None] * expert(h[rows], w, f"{p}e{e}.")
    return out


# ---- model --------------------------------------------------------------------------------------------------------------
def order(cfg):
    """Layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, tensors, tokens, taps=None, dtype=torch.float64, margins=None):
    """Logits [T, vocab] of one sequence; ``taps`` collects the sum of the streams after every layer run, ``margins`` every mixture's [T] distances
    from another choice of experts."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    X = (w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]).expand(cfg["streams"], -1, -1)
    for i in order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        for q in (1, 2):
            if q == 2 and L.get("mlp") is None:
                continue
            h = rms(collapse(X, w[f"{p}hc{q}.in"]), w[f"{p}norm{q}"], eps)
            h = input_convolution(h, w[f"{p}canon{q}"])
            if q == 1:
                y = (window_attention if L["type"] == "attention" else latent_attention)(h, w, p + "mix.", L["mixer"], eps)
            else:
                near = []
                y = dense(h, w, p + "mlp.") if L["mlp"]["kind"] == "dense" else mixture(h, w, p + "mlp.", L["mlp"]["router"], near)
                if margins is not None and near:
                    margins.append(torch.tensor(near))
            X = spread(X, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"], m, y)
        if taps is not None:
            taps.append(X.sum(0))
    return rms(X.sum(0), w["final.norm"], eps) @ w["head"].t()


# ---- models for tests ---------------------------------------------------------------------------------------------------
def windowed(heads, kv_heads, dim, vdim, window, scale, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, q_rank, scale, base, scaling=None, mlp=None):
    turned = {"base": base, "dims": rot}
    if scaling:
        turned["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                                                              "scale": scale, "rot": turned}}


def ff(width):
    return {"kind": "dense", "ff": width}


def moe(experts, top, width, count, keep, scale):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}, "expert": {"ff": width}}


def make_config(vocab, width, streams, taps, mult, embed, layers, loop=None, eps=1e-5):
    out = {"architecture": "Dironex", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps}, "residual_mult": mult,
           "embedding": {"scale": embed}, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def make_weights(cfg, seed=0, spread=False):
    """Random bf16 tensors; norm weights, mixes, corrections and activations' numbers differ from 1 and 0, so that leaving one out shows.
    ``spread``: corrections so far apart that no rounding turns a choice of experts over."""
    g = torch.Generator().manual_seed(seed)
    w, d, S = {}, cfg["width"], cfg["streams"]

    def put(name, *shape, s=None, mean=0.0):
        w[name] = (mean + torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if s is None else s)).to(torch.bfloat16)
    put("embed", cfg["vocab"], d, s=1.0)
    put("head", cfg["vocab"], d)
    put("final.norm", d, s=0.3, mean=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q, H, dim, vdim = p + "mix.", m["heads"], m["dim"], m["vdim"]
        for k in (1, 2) if L.get("mlp") else (1,):
            put(f"{p}norm{k}", d, s=0.3, mean=1.0)
            put(f"{p}canon{k}", d, cfg["canon"]["taps"], s=0.4)
            put(f"{p}hc{k}.in", S, s=0.3, mean=1 / S)
            put(f"{p}hc{k}.out", S, s=0.4, mean=0.8)
            put(f"{p}hc{k}.mix", S, S, s=0.25)
            w[f"{p}hc{k}.mix"] = (w[f"{p}hc{k}.mix"].float() + 0.8 * torch.eye(S)).to(torch.bfloat16)
        put(q + "o", d, H * vdim)
        if L["type"] == "attention":
            G = m["kv_heads"]
            put(q + "q", H * dim, d); put(q + "k", G * dim, d); put(q + "v", G * vdim, d)
            put(q + "q.norm", dim, s=0.4, mean=1.2); put(q + "k.norm", dim, s=0.4, mean=1.2)
        else:
            r, qr, rot = m["kv_rank"], m["q_rank"], m["rot_dim"]
            put(q + "dq", qr, d); put(q + "dq.norm", qr, s=0.4, mean=1.2); put(q + "uq", H * (dim + rot), qr)
            put(q + "dkv", r + rot, d); put(q + "dkv.norm", r, s=0.4, mean=1.2)
            put(q + "uk", H * dim, r); put(q + "uv", H * vdim, r); put(q + "g", H * vdim, d)
        f = L.get("mlp")
        if f and f["kind"] == "dense":
            put(p + "mlp.up", f["ff"], d); put(p + "mlp.down", d, f["ff"]); put(p + "mlp.act", 2, s=1.0)
        elif f:
            E, e_ff = f["router"]["experts"], f["expert"]["ff"]
            put(p + "mlp.router", E, d, s=2 * d ** -0.5); put(p + "mlp.correction", E, s=20.0 if spread else 0.3, mean=-0.3)
            for e in range(E):
                put(f"{p}mlp.e{e}.up", e_ff, d); put(f"{p}mlp.e{e}.down", d, e_ff)
    return w
