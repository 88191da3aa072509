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
    """h_t + sum_j w[:, j] h_(t - taps + 1 + j), zeros before the start."""
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


def route(z, correction, r):
    """Chosen experts and weights of every row of logits."""
    s, E = sigmoid(z), z.shape[1]
    choice = s + correction
    g = r.get("groups") or {"count": 1, "keep": 1}
    per = E // g["count"]
    ids, wts = [], []
    for t in range(z.shape[0]):
        row = choice[t].tolist()
        score = [sum(sorted(row[a * per:(a + 1) * per], reverse=True)[:2]) for a in range(g["count"])]
        kept = sorted(range(g["count"]), key=lambda a: -score[a])[:g["keep"]]
        open_ = [e for a in kept for e in range(a * per, (a + 1) * per)]
        best = sorted(open_, key=lambda e: (-row[e], e))[:r["top"]]
        v = s[t, best]
        ids.append(best)
        wts.append(v / (v.sum() + 1e-20) * r["scale"])
    return ids, wts


def mixture(h, w, p, r):
    ids, wts = route(h @ w[p + "router"].t(), w[p + "correction"], r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, v in zip(ids[t], wts[t]):
            u = (w[f"{p}e{e}.up"] @ h[t]).clamp(min=0)
            out[t] += v * (w[f"{p}e{e}.down"] @ (u * u))
    return out


# ---- model --------------------------------------------------------------------------------------------------------------
def order(cfg):
    """Layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, tensors, tokens, taps=None, dtype=torch.float64):
    """Logits [T, vocab] of one sequence; ``taps`` collects the sum of the streams after every layer run."""
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
                y = dense(h, w, p + "mlp.") if L["mlp"]["kind"] == "dense" else mixture(h, w, p + "mlp.", L["mlp"]["router"])
            X = spread(X, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"], m, y)
        if taps is not None:
            taps.append(X.sum(0))
    return rms(X.sum(0), w["final.norm"], eps) @ w["head"].t()
