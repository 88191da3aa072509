"""Plain, slow implementation of the Gudutar design, one function per mechanism, on the CPU.

Nothing here is shared with the product path: weights are a dict of tensors under their file names, the configuration is the
parsed ``config.json`` dict, and every function spells its equation out over a whole sequence (no cache, no chunks, no batching).
``dtype`` chooses the arithmetic (float64 for a sharp oracle)."""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdim=True)
    dev = x - mu
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def causal_conv(x, w, bias):
    """x [T, C], w [C, taps], last column = the current token; zeros before token 0."""
    T, taps = x.shape[0], w.shape[1]
    y = bias.expand_as(x).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y


def rotate(x, base, dims, layout):
    """x [T, heads, dim] at positions 0..T-1: the first ``dims`` dimensions turned pair by pair, the rest untouched."""
    x, half = x.clone(), dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = t * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            p, q = (i, i + half) if layout == "half" else (2 * i, 2 * i + 1)
            u, v = x[t, :, p].clone(), x[t, :, q].clone()
            x[t, :, p], x[t, :, q] = u * c - v * s, v * c + u * s
    return x


def decayed_sum(q, k, v, log_decay, S=None):
    """One head: S_t = exp(log_decay_t) S_(t-1) + k_t v_t^T, out_t = S_t^T q_t.  q, k [T, N], v [T, P], log_decay [T].
    Returns (out [T, P], final S [N, P])."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if S is None else S
    out = torch.empty(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t]) * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def mamba2(w, p, m, h, eps):
    H, P, N, G, T = m["heads"], m["vdim"], m["state"], m["groups"], h.shape[0]
    inner = H * P
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    x, B, C = torch.split(silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])), [inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[p + "dt_bias"])
    y = torch.empty(T, inner, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        xa = x[:, a * P:(a + 1) * P]
        o, _ = decayed_sum(C[:, g * N:(g + 1) * N], B[:, g * N:(g + 1) * N] * dt[:, a:a + 1], xa, -torch.exp(w[p + "A_log"][a]) * dt[:, a])
        y[:, a * P:(a + 1) * P] = o + w[p + "D"][a] * xa
    y = y * silu(z)
    part = inner // m["norm_groups"]
    for a in range(m["norm_groups"]):
        y[:, a * part:(a + 1) * part] = unit_rms(y[:, a * part:(a + 1) * part], eps)
    return (y * w[p + "norm"]) @ w[p + "o"].T


def retention(w, p, m, h, eps):
    H, N, P, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = rotate((h @ w[p + "q"].T).view(T, H, N), m["rot"]["base"], m["rot"]["dims"], "half")
    k = rotate((h @ w[p + "k"].T).view(T, H, N), m["rot"]["base"], m["rot"]["dims"], "half") * N ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, P)
    out = torch.empty(T, H, P, dtype=h.dtype)
    for a in range(H):
        la = torch.full((T,), math.log(m["decay"][a]), dtype=h.dtype)
        out[:, a] = unit_rms(decayed_sum(q[:, a], k[:, a], v[:, a], la)[0], eps)
    return (out.reshape(T, H * P) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def window_softmax(q, k, v, scale, window):
    """One head: q, k [T, d], v [T, P]; position i sees i - window + 1 .. i."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = s.masked_fill((back < 0) | (back >= window), float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return (e / e.sum(-1, keepdim=True)) @ v


def latent_attention(w, p, m, h, eps):
    H, dim, rd, vd, r, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    rot = m["rot"]
    q = (h @ w[p + "q"].T).view(T, H, dim + rd)
    q_rot = rotate(q[:, :, dim:], rot["base"], rot["dims"], "pairs")
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :r], eps) * w[p + "dkv.norm"]
    k_rot = rotate(down[:, None, r:], rot["base"], rot["dims"], "pairs")[:, 0]
    k, v = (c @ w[p + "uk"].T).view(T, H, dim), (c @ w[p + "uv"].T).view(T, H, vd)
    out = [window_softmax(torch.cat([q[:, a, :dim], q_rot[:, a]], 1), torch.cat([k[:, a], k_rot], 1), v[:, a], m["scale"], m["mask"]["size"])
           for a in range(H)]
    return torch.cat(out, 1) @ w[p + "o"].T


def dense_ff(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"mamba2": mamba2, "retention": retention, "latent_attention": latent_attention}


def layer(w, cfg, i, x):
    L, eps = cfg["layers"][i], cfg["norm"]["eps"]
    j = i
    while "weights_of" in cfg["layers"][j]:
        j = cfg["layers"][j]["weights_of"]
    p = f"l{j}."
    x = x + layer_norm(MIXERS[L["type"]](w, p + "mix.", L["mixer"], x, eps), w[p + "norm1"], w[p + "norm1.b"], eps)
    if L.get("mlp"):
        x = x + layer_norm(dense_ff(w, p + "mlp.", x), w[p + "norm2"], w[p + "norm2.b"], eps)
    return x


def forward(w, cfg, tokens, dtype=torch.float64, taps=None):
    """Logits [T, vocab]; ``taps``: optional list that collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(w, cfg, i, x)
        if taps is not None:
            taps.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T


# ---- small random models ---------------------------------------------------------------------------------------------
def ssm(heads, vdim, state, groups, conv, norm_groups, **layer):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": None, **layer}


def retain(heads, dim, vdim, base, dims, decay, **layer):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims}, "decay": decay},
            "mlp": None, **layer}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base, scale, **layer):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim}}, "mlp": None, **layer}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def make_config(vocab, width, scale, layers, eps=1e-5):
    """A layer given as a number shares the weights of that layer."""
    out = []
    for L in layers:
        out.append(L if isinstance(L, dict) else {**{k: v for k, v in out[L].items()}, "weights_of": L})
    return {"architecture": "Gudutar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": out}


def make_weights(cfg, seed=0):
    """Random bf16 tensors; every norm weight, bias, tap and skip differs from 1 and 0, so that leaving one out shows."""
    g = torch.Generator().manual_seed(seed)
    w, d = {}, cfg["width"]

    def put(name, *shape, s=None, mean=0.0):
        w[name] = (mean + torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if s is None else s)).to(torch.bfloat16)

    def norm(name):
        put(name, d, s=0.3, mean=1.0)
        put(name + ".b", d, s=0.3)
    put("embed", cfg["vocab"], d, s=1.0 / cfg["embedding"]["scale"])
    put("head", cfg["vocab"], d)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        if "weights_of" in L:
            continue
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        norm(p + "norm1")
        if L["type"] == "mamba2":
            inner, ch = m["heads"] * m["vdim"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            put(q + "in", inner + ch + m["heads"], d)
            put(q + "conv", ch, m["conv"], s=0.6)
            put(q + "conv.b", ch, s=0.3)
            put(q + "dt_bias", m["heads"], s=1.0, mean=-2.0)
            put(q + "A_log", m["heads"], s=1.0, mean=-1.0)      # decays from a few tokens to hundreds
            put(q + "D", m["heads"], s=0.5, mean=0.5)
            put(q + "norm", inner, s=0.3, mean=1.0)
            put(q + "o", d, inner)
        elif L["type"] == "retention":
            for n, r in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                put(q + n, m["heads"] * r, d)
            put(q + "o", d, m["heads"] * m["vdim"])
        else:
            put(q + "q", m["heads"] * (m["dim"] + m["rot_dim"]), d, s=1.5 * d ** -0.5)
            put(q + "dkv", m["kv_rank"] + m["rot_dim"], d)
            put(q + "dkv.norm", m["kv_rank"], s=0.3, mean=1.2)
            put(q + "uk", m["heads"] * m["dim"], m["kv_rank"])
            put(q + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            put(q + "o", d, m["heads"] * m["vdim"])
        if L.get("mlp"):
            norm(p + "norm2")
            put(p + "mlp.gate", L["mlp"]["ff"], d); put(p + "mlp.up", L["mlp"]["ff"], d); put(p + "mlp.down", d, L["mlp"]["ff"])
    return w
