"""Plain, slow implementation of the Lifulorn design, one function per mechanism, on the CPU.

Nothing here is shared with the product path: weights are a dict of tensors under their file names, the configuration is the
parsed ``config.json`` dict, and every function spells its equation out over a whole sequence (no cache, no chunks, no batching).
``dtype`` chooses the arithmetic (float64 for a sharp oracle)."""
from __future__ import annotations

import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


# ---- rotation -----------------------------------------------------------------------------------------------------------
def wavelength_frequencies(base, dims, sc):
    """Frequencies kept where the wavelength is short, divided by the factor where it is long, blended in between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        wave = 2 * math.pi / f
        if wave < sc["original"] / sc["high"]:
            out.append(f)
        elif wave > sc["original"] / sc["low"]:
            out.append(f / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1 - s) * f / sc["factor"] + s * f)
    return out, 1.0


def yarn_frequencies(base, dims, sc):
    """Frequencies divided by the factor along a ramp over the dimensions; cosine and sine are scaled too."""
    def where(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, freqs, gain):
    """x [T, heads, dim] at positions 0..T-1: dimension i turns with dimension i + half, the rest pass."""
    x, half = x.clone(), len(freqs)
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(t * f) * gain, math.sin(t * f) * gain
            u, v = x[t, :, i].clone(), x[t, :, i + half].clone()
            x[t, :, i], x[t, :, i + half] = u * c - v * s, v * c + u * s
    return x


# ---- attention ----------------------------------------------------------------------------------------------------------
def window_softmax(q, k, v, scale, window, sink, cap=None):
    """One head: q, k [T, d], v [T, P]; position i sees i - window + 1 .. i; exp(sink) is in the denominator only."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    if cap is not None:
        s = cap * torch.tanh(s / cap)
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = s.masked_fill((back < 0) | (back >= window), float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return (e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))) @ v


def attention(w, p, m, h, first):
    """``first``: a list that holds the values of the first mixing layer (empty before it)."""
    H, G, dim, vdim, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, dim)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, dim)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, vdim)
    rot = m["rot"]
    freqs, gain = (yarn_frequencies if "fast" in rot["scaling"] else wavelength_frequencies)(rot["base"], rot["dims"], rot["scaling"])
    q, k = rotate(q, freqs, gain), rotate(k, freqs, gain)
    if m.get("v_mix"):
        if first:
            lam = w[p + "vmix"]
            v = (1 - lam) * v + lam * first[0]
        else:
            first.append(v)
    out = [window_softmax(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], m["mask"]["size"], w[p + "sink"][a], m.get("softcap"))
           for a in range(H)]
    return torch.cat(out, 1) @ w[p + "o"].T


# ---- gated delta rule ---------------------------------------------------------------------------------------------------
def causal_conv(x, w):
    """x [T, C], w [C, taps], last column = the current token; zeros before token 0."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, decay, beta, S=None):
    """One head: S decays, takes beta times what it does not yet say about k, and is read by q.  Returns (out [T, P], S [N, P])."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if S is None else S.clone()
    out = torch.empty(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def delta(w, p, m, h, eps):
    H, G, N, P, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    short = lambda n: silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    q = unit(short("q").view(T, G, N)) * N ** -0.5
    k = unit(short("k").view(T, G, N))
    v = short("v").view(T, H, P)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    out = torch.empty(T, H, P, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = delta_rule(q[:, g], k[:, g], v[:, a], decay[:, a], beta[:, a])[0]
    out = unit_rms(out, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, P)
    return out.reshape(T, H * P) @ w[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def expert(w, p, h, limit):
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z, top):
    """Chosen experts of one row and their weights: softmax over the chosen logits only."""
    ids = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    e = torch.exp(z[ids] - z[ids].max())
    return ids, e / e.sum()


def mixture(w, p, m, h, margins=None):
    """``margins``: optional list that collects how far every row's last choice is ahead of the next expert."""
    z = h @ w[p + "router"].T
    if margins is not None and m["router"]["top"] < z.shape[1]:
        best = z.sort(descending=True).values
        margins.append(best[:, m["router"]["top"] - 1] - best[:, m["router"]["top"]])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, wt = route(z[t], m["router"]["top"])
        for i, a in zip(ids, wt):
            y[t] += a * expert(w, f"{p}e{i}.", h[t], m["expert"]["limit"])
    if m.get("shared"):
        y = y + sigmoid(h @ w[p + "shared.sg"].T) * expert(w, p + "shared.", h, m["shared"]["limit"])
    return y


# ---- the model ----------------------------------------------------------------------------------------------------------
def token_input(w, p, i, dim, x, tokens, eps):
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    return unit_rms((gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T, eps) * w[p + "side.norm"]


def layer(w, cfg, i, x, tokens, first, margins=None):
    L, eps, m, p = cfg["layers"][i], cfg["norm"]["eps"], cfg["residual_mult"], f"l{i}."
    h = unit_rms(x, eps) * w[p + "norm1"]
    y = delta(w, p + "mix.", L["mixer"], h, eps) if L["type"] == "delta" else attention(w, p + "mix.", L["mixer"], h, first)
    x = x + m * y * w[p + "ls1"]
    if L.get("mlp"):
        x = x + m * mixture(w, p + "mlp.", L["mlp"], unit_rms(x, eps) * w[p + "norm2"], margins) * w[p + "ls2"]
    return x + m * token_input(w, p, i, cfg["token_side"]["dim"], x, tokens, eps)


def forward(w, cfg, tokens, dtype=torch.float64, taps=None, margins=None):
    """Logits [T, vocab]; ``taps``: optional list that collects the residual after every layer; ``margins``: see mixture."""
    w, tokens, first = {k: v.to(dtype) for k, v in w.items()}, torch.tensor(tokens), []
    x = w["embed"][tokens]
    for i in range(len(cfg["layers"])):
        x = layer(w, cfg, i, x, tokens, first, margins)
        if taps is not None:
            taps.append(x.clone())
    return (unit_rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T


# ---- small random models ---------------------------------------------------------------------------------------------
def wave(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attend(heads, kv_heads, dim, vdim, window, base, dims, scaling, scale, v_mix=True, softcap=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window},
         "rot": {"base": base, "dims": dims, "scaling": scaling}}
    if v_mix is not None:
        m["v_mix"] = v_mix
    if softcap is not None:
        m["softcap"] = softcap
    return {"type": "attention" if softcap is None else "attention_2", "mixer": m, "mlp": mlp}


def rule(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def moe(experts, top, ff, limit, shared_ff, shared_limit):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared_ff:
        out["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return out


def make_config(vocab, width, side, mult, layers, eps=1e-5):
    return {"architecture": "Lifulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "token_side": {"dim": side},
            "layers": layers}


def make_weights(cfg, seed=0):
    """Random bf16 tensors; every norm weight, scale, bias, sink and share differs from 1 and 0, so that leaving one out shows."""
    g = torch.Generator().manual_seed(seed)
    w, d, side = {}, cfg["width"], cfg["token_side"]["dim"]

    def put(name, *shape, s=None, mean=0.0):
        w[name] = (mean + torch.randn(*shape, generator=g) * (shape[-1] ** -0.5 if s is None else s)).to(torch.bfloat16)

    def expert(p, ff):
        put(p + "gate", ff, d, s=1.5 * d ** -0.5); put(p + "up", ff, d, s=1.5 * d ** -0.5); put(p + "down", d, ff)
    put("embed", cfg["vocab"], d, s=1.0)
    put("head", cfg["vocab"], d)
    put("final.norm", d, s=0.3, mean=1.0)
    put("side.embed", cfg["vocab"], side * len(cfg["layers"]), s=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q, H, G, dim, vdim = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "ls1", "side.norm"):
            put(p + n, d, s=0.3, mean=1.0)
        put(p + "side.gate", side, d); put(p + "side.proj", d, side)
        put(q + "o", d, H * vdim)
        if L["type"] == "delta":
            for n, rows in (("q", G * dim), ("k", G * dim), ("v", H * vdim)):
                put(q + n, rows, d)
                put(q + n + ".conv", rows, m["conv"], s=0.6)
            put(q + "g", H * vdim, d); put(q + "a", H, d); put(q + "b", H, d)
            put(q + "norm", vdim, s=0.3, mean=1.0)
            put(q + "dt_bias", H, s=1.0, mean=-2.0)
            put(q + "A_log", H, s=1.0, mean=-1.0)      # decays from a few tokens to hundreds
        else:
            for n, rows in (("q", H * dim), ("k", G * dim), ("v", G * vdim)):
                put(q + n, rows, d, s=(1.5 if n == "q" else 1.0) * d ** -0.5)
                put(q + n + ".b", rows, s=0.3)
            put(q + "sink", H, s=1.0, mean=1.0)
            if m.get("v_mix"):
                w[q + "vmix"] = torch.tensor(0.2 + 0.6 * float(torch.rand(1, generator=g))).to(torch.bfloat16)
        if L.get("mlp"):
            r = L["mlp"]
            put(p + "norm2", d, s=0.3, mean=1.0); put(p + "ls2", d, s=0.3, mean=1.0)
            put(p + "mlp.router", r["router"]["experts"], d, s=2 * d ** -0.5)
            for e in range(r["router"]["experts"]):
                expert(f"{p}mlp.e{e}.", r["expert"]["ff"])
            if r.get("shared"):
                expert(p + "mlp.shared.", r["shared"]["ff"])
                put(p + "mlp.shared.sg", 1, d)
    return w
