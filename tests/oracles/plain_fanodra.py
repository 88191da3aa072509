"""Plain, slow implementation of the Fanodra design, one function per mechanism, on the CPU.

Nothing here is shared with the product path: weights are a dict of tensors under their file names, the configuration is the
parsed ``config.json`` dict, and every function spells its equation out over a whole sequence (no cache, no state carried,
no batching).  ``dtype`` chooses the arithmetic (float64 for a sharp oracle, float32 for speed)."""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * w + b over the last axis."""
    mu = x.mean(-1, keepdim=True)
    dev = x - mu
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def causal_conv(x, w, bias=None):
    """x [T, C], w [C, taps], last column = the current token: y_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before token 0."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y if bias is None else y + bias


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def linear(x, w, b=None):
    y = x @ w.T
    return y if b is None else y + b


def block_gate(u, w, b):
    """sigmoid(w[k] u_k + b[k]) on each of the equal parts u_k of u; w [parts, n, n], b [parts, n]."""
    parts, n = w.shape[0], w.shape[1]
    out = torch.empty_like(u)
    for k in range(parts):
        z = u[:, k * n:(k + 1) * n] @ w[k].T + b[k]
        out[:, k * n:(k + 1) * n] = 1 / (1 + torch.exp(-z))
    return out


def gated_recurrence(u, r, i, lam, S0=None):
    """log a = -8 r softplus(lam);  S_t = a S_(t-1) + sqrt(1 - a^2) i u.  Returns S at every t."""
    S = torch.zeros_like(u[0]) if S0 is None else S0
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(-8 * r[t] * softplus(lam))
        S = a * S + torch.sqrt(1 - a * a) * i[t] * u[t]
        out[t] = S
    return out


def recurrent_block(w, p, h):
    y = gelu_tanh(linear(h, w[p + "y"], w[p + "y.b"]))
    u = causal_conv(linear(h, w[p + "x"], w[p + "x.b"]), w[p + "conv"], w[p + "conv.b"])
    r = block_gate(u, w[p + "ra"], w[p + "ra.b"])
    i = block_gate(u, w[p + "ri"], w[p + "ri.b"])
    return linear(gated_recurrence(u, r, i, w[p + "lam"]) * y, w[p + "o"])


def biased_scores(q, k, scale, r1, r2):
    """q, k [T, dim] of one head: (q . k) scale - r1 ln(1 + r2 (i - j)) for j <= i, -inf elsewhere."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(s.dtype)
    s = s - r1 * torch.log(1 + r2 * dist.clamp(min=0))
    return s.masked_fill(dist < 0, float("-inf"))


def attention(w, p, m, h, eps):
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(linear(h, w[p + "q"], w[p + "q.b"]), w[p + "q.norm"], eps)
    k = rms_norm(linear(h, w[p + "k"], w[p + "k.b"]), w[p + "k.norm"], eps)
    v = linear(h, w[p + "v"], w[p + "v.b"])
    out = []
    for x in range(H):
        g = x // (H // G)
        s = biased_scores(q[:, x * dim:(x + 1) * dim], k[:, g * dim:(g + 1) * dim], m["scale"], w[p + "r1"][x], w[p + "r2"][x])
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((e / e.sum(-1, keepdim=True)) @ v[:, g * vdim:(g + 1) * vdim])
    return linear(torch.cat(out, -1), w[p + "o"], w[p + "o.b"])


def parallel_mixer(w, p, m, h, eps):
    left = rms_norm(attention(w, p + "left.", m["left"], h, eps), w[p + "left.out"], eps)
    right = rms_norm(recurrent_block(w, p + "right.", h), w[p + "right.out"], eps)
    return 0.5 * (left + right)


def dense_ff(w, p, h):
    return linear(silu(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


def layer(w, cfg, i, x):
    eps, L, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    n = lambda t, name: layer_norm(t, w[p + name], w[p + name + ".b"], eps)
    h = n(x, "norm1")
    h = h + causal_conv(h, w[p + "canon1"])
    y = recurrent_block(w, p + "mix.", h) if L["type"] == "rglru" else parallel_mixer(w, p + "mix.", L["mixer"], h, eps)
    x = x + n(y, "norm1b")
    if L["mlp"] is not None:
        x = x + n(dense_ff(w, p + "mlp.", n(x, "norm2")), "norm2b")
    return x


def forward(w, cfg, tokens, dtype=torch.float64, taps=None):
    """Logits [T, vocab]; ``taps``: optional list that collects the residual after every layer run."""
    w = {k: v.to(dtype) for k, v in w.items()}
    emb = w["embed"][torch.tensor(tokens)]
    x = emb.clone()
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    order = list(range(0, loop["start"]))
    runs = [(i, None) for i in order]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    runs += [(i, None) for i in range(loop["stop"], len(cfg["layers"]))]
    for i, begins in runs:
        if begins is not None:
            if begins > 0:
                x = x + emb
            x = x + w["loop.step"][begins]
        x = layer(w, cfg, i, x)
        if taps is not None:
            taps.append(x.clone())
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"])
    return x @ w["embed"].T


# ---- small random models ---------------------------------------------------------------------------------------------
def recurrent(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def attending(heads, kv_heads, dim, vdim, scale):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}


def make_config(vocab, width, taps, layers, loop=None, eps=1e-5):
    """layers: ("rglru", recurrent(...), ff or None) or ("parallel", attending(...), recurrent(...), ff or None)."""
    out = []
    for L in layers:
        mixer = L[1] if L[0] == "rglru" else {"left": L[1], "right": L[2]}
        out.append({"type": L[0], "mixer": mixer, "mlp": {"kind": "dense", "ff": L[-1]} if L[-1] else None})
    return {"architecture": "Fanodra", "vocab": vocab, "width": width, "canon": {"taps": taps}, "norm": {"eps": eps}, "layers": out,
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


def make_weights(cfg, seed=0):
    """Random bf16 tensors; every norm weight, bias, tap and gate differs from 1 and 0, so that leaving one out shows."""
    g = torch.Generator().manual_seed(seed)
    w, d = {}, cfg["width"]

    def put(name, *shape, s=None, mean=0.0):
        w[name] = (mean + torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if s is None else s)).to(torch.bfloat16)

    def norm(name):
        put(name, d, s=0.3, mean=1.0)
        put(name + ".b", d, s=0.3)

    def rec(p, m):
        n, b = m["width"], m["blocks"]
        for k in ("y", "x"):
            put(p + k, n, d); put(p + k + ".b", n, s=0.3)
        put(p + "conv", n, m["conv"], s=0.6); put(p + "conv.b", n, s=0.3)
        for k in ("ra", "ri"):
            put(p + k, b, n // b, n // b); put(p + k + ".b", b, n // b, s=0.5)
        put(p + "lam", n, s=2.0, mean=-4.0)          # decays from a few tokens to thousands
        put(p + "o", d, n)
    put("embed", cfg["vocab"], d, s=0.2)          # small, so that greedy decoding does not just repeat its input
    norm("final.norm")
    if cfg.get("loop"):
        put("loop.step", cfg["loop"]["times"], d, s=0.5)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L["mlp"] else ()):
            norm(p + n)
        put(p + "canon1", d, cfg["canon"]["taps"], s=0.4)
        if L["type"] == "rglru":
            rec(p + "mix.", L["mixer"])
        else:
            m, q = L["mixer"]["left"], p + "mix.left."
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                put(q + n, rows, d); put(q + n + ".b", rows, s=0.3)
            put(q + "q.norm", m["heads"] * m["dim"], s=0.3, mean=1.5); put(q + "k.norm", m["kv_heads"] * m["dim"], s=0.3, mean=1.5)
            w[q + "r1"] = (0.1 + torch.rand(m["heads"], generator=g)).to(torch.bfloat16)
            w[q + "r2"] = (0.05 + 2 * torch.rand(m["heads"], generator=g)).to(torch.bfloat16)
            put(q + "o", d, m["heads"] * m["vdim"]); put(q + "o.b", d, s=0.3)
            put(q + "out", d, s=0.3, mean=1.0)
            rec(p + "mix.right.", L["mixer"]["right"])
            put(p + "mix.right.out", d, s=0.3, mean=1.0)
        if L["mlp"]:
            put(p + "mlp.gate", L["mlp"]["ff"], d); put(p + "mlp.up", L["mlp"]["ff"], d); put(p + "mlp.down", d, L["mlp"]["ff"])
    return w
