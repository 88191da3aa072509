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
