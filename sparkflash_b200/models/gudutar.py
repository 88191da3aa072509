"""Gudutar: a small decoder whose layers mix tokens with state-space duality, retention, or latent attention in a window.  A norm
(layer norm) sits on every sublayer's output only, the sublayers read the residual itself; a layer may have no feed-forward, and
layers may share another layer's weights, each with its own cache or state.

This file is the design's configuration, its tensor names and its order of operations.  The mechanisms are models/mixers.py and
ops/rows.py; lanes, cache, state, batching and sampling are models/layered.py.

    input       x = embedding[token] * scale
    a layer     x += LN1(mixer(x)); x += LN2(ff(x))
    head        LN(x) times the output table
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops import rows as R
from .layered import CONFIG_META, LayeredModel, check_keys
from .mixers import DenseFF, LatentAttention, RetentionMixer, StateSpaceMixer, W

ARCHITECTURE = "Gudutar"
FF_ACT = "gelu_tanh"

_TOP = {"architecture", "vocab", "width", "norm", "embedding", "layers"}
_MIXERS = {
    "mamba2": {"heads", "vdim", "state", "groups", "conv", "norm_groups"},
    "retention": {"heads", "dim", "vdim", "rot", "decay"},
    "latent_attention": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask", "rot"},
}


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    ff: int | None            # dense feed-forward width, None: no feed-forward
    weights: int              # layer whose tensors are used


@dataclass
class GudutarConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "gudutar"
    eos_id: int = -1

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, d: dict) -> "GudutarConfig":
        check_keys(d, _TOP, "top level", CONFIG_META)
        if d["architecture"] != ARCHITECTURE:
            raise ValueError(f"config.json: architecture {d['architecture']!r} is not {ARCHITECTURE}")
        check_keys(d["norm"], {"eps"}, "norm")
        check_keys(d["embedding"], {"scale"}, "embedding")
        layers = []
        for i, L in enumerate(d["layers"]):
            check_keys(L, {"type", "mixer", "mlp", "weights_of"}, f"layer {i}", {"mlp", "weights_of"})
            m = L["mixer"]
            if L["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown type {L['type']!r}")
            check_keys(m, _MIXERS[L["type"]], f"layer {i} mixer")
            _check_mixer(L["type"], m, f"layer {i}")
            ff = L.get("mlp")
            if ff is not None:
                check_keys(ff, {"kind", "ff"}, f"layer {i} mlp")
                if ff["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown mlp kind {ff['kind']!r}")
            layers.append(LayerSpec(L["type"], m, ff["ff"] if ff is not None else None, i))
        for i, L in enumerate(d["layers"]):
            j, hops = i, 0
            while d["layers"][j].get("weights_of") is not None:
                j, hops = d["layers"][j]["weights_of"], hops + 1
                if not 0 <= j < len(layers) or hops > len(layers):
                    raise ValueError(f"layer {i}: weights_of does not lead to a layer with tensors")
            a, b = layers[i], layers[j]
            if (a.type, a.mixer, a.ff) != (b.type, b.mixer, b.ff):
                raise ValueError(f"layer {i} differs from layer {j}, whose weights it uses")
            a.weights = j
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["embedding"]["scale"]), layers, d.get("name", "gudutar"),
                   d.get("eos_token_id", -1))

    def shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint."""
        d = self.width
        out = {"embed": (self.vocab, d), "head": (self.vocab, d), "final.norm": (d,), "final.norm.b": (d,)}
        for i, L in enumerate(self.layers):
            if L.weights != i:
                continue
            p, m = f"l{i}.", L.mixer
            for n in ("norm1",) + (("norm2",) if L.ff is not None else ()):
                out[p + n], out[p + n + ".b"] = (d,), (d,)
            q, H = p + "mix.", m["heads"]
            inner = H * m["vdim"]
            out[q + "o"] = (d, inner)
            if L.type == "mamba2":
                ch = inner + 2 * m["groups"] * m["state"]
                out[q + "in"], out[q + "conv"], out[q + "conv.b"] = (inner + ch + H, d), (ch, m["conv"]), (ch,)
                out[q + "dt_bias"] = out[q + "A_log"] = out[q + "D"] = (H,)
                out[q + "norm"] = (inner,)
            elif L.type == "retention":
                out[q + "q"] = out[q + "k"] = (H * m["dim"], d)
                out[q + "v"] = out[q + "g"] = (inner, d)
            else:
                r = m["kv_rank"]
                out[q + "q"], out[q + "dkv"], out[q + "dkv.norm"] = (H * (m["dim"] + m["rot_dim"]), d), (r + m["rot_dim"], d), (r,)
                out[q + "uk"], out[q + "uv"] = (H * m["dim"], r), (inner, r)
            if L.ff is not None:
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (L.ff, d)
                out[p + "mlp.down"] = (d, L.ff)
        return out


def _check_mixer(kind: str, m: dict, where: str) -> None:
    def need(ok: bool, what: str) -> None:
        if not ok:
            raise ValueError(f"{where}: {what}")
    if kind == "mamba2":
        need(m["heads"] % m["groups"] == 0, "heads must be a multiple of groups")
        need(m["heads"] * m["vdim"] % m["norm_groups"] == 0, "heads x vdim must be a multiple of norm_groups")
        need(1 <= m["conv"] <= R.MAX_TAPS, f"convolutions of 1..{R.MAX_TAPS} taps are implemented")
        R.state_pad(m["state"])
    elif kind == "retention":
        check_keys(m["rot"], {"base", "dims"}, f"{where} rot")
        need(len(m["decay"]) == m["heads"], "one decay per head")
        need(m["rot"]["dims"] % 2 == 0 and 0 <= m["rot"]["dims"] <= m["dim"], "rot.dims must be even and at most dim")
        R.state_pad(m["dim"])
    else:
        check_keys(m["rot"], {"base", "dims"}, f"{where} rot")
        check_keys(m["mask"], {"size"}, f"{where} mask")
        need(m["rot"]["dims"] == m["rot_dim"] and m["rot_dim"] % 2 == 0, "rot.dims must be rot_dim, and even")
        need(m["mask"]["size"] >= 1, "a window sees at least its own position")


def random_tensors(cfg: GudutarConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights of the right shapes (benchmarks, tests, ``--synthetic``), bf16 as a checkpoint stores them."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g, device=device)
        if leaf == "b":
            t = r * 0.1
        elif leaf in ("norm", "norm1", "norm2", "D"):
            t = 1 + 0.1 * r
        elif leaf == "dt_bias":
            t = -3 + r
        elif leaf == "A_log":
            t = r
        elif leaf == "embed":
            t = r / cfg.embed_scale
        elif leaf == "conv":
            t = r * 0.4
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    def __init__(self, t, i: int, spec: LayerSpec, cfg: GudutarConfig, dtype, device, max_context: int):
        w = W(t, f"l{i}.", dtype, device)
        mix = w.sub("mix.")
        if spec.type == "mamba2":
            self.mixer = StateSpaceMixer(mix, spec.mixer, cfg.eps)
        elif spec.type == "retention":
            self.mixer = RetentionMixer(mix, spec.mixer, cfg.eps, max_context)
        else:
            self.mixer = LatentAttention(mix, spec.mixer, cfg.eps, max_context)
        self.ff = DenseFF(w.sub("mlp."), FF_ACT) if spec.ff is not None else None
        self.norm = {n: (w.f32(n), w.f32(n + ".b")) for n in ("norm1",) + (("norm2",) if self.ff is not None else ())}


class Gudutar(LayeredModel):
    """The model as models/layered.py drives it."""

    config_class = GudutarConfig

    def __init__(self, cfg: GudutarConfig, tensors: dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device="cuda",
                 max_context: int = 4096):
        self._load(cfg, tensors, dtype, device)
        own = {i: _Layer(tensors, i, L, cfg, dtype, device, max_context) for i, L in enumerate(cfg.layers) if L.weights == i}
        self.layers = [own[L.weights] for L in cfg.layers]
        top = W(tensors, "", dtype, device)
        self.embed, self.head, self.final = top.act("embed"), top.act("head"), (top.f32("final.norm"), top.f32("final.norm.b"))
        self.kv_runs = [L.mixer.kv_run for L in self.layers if L.mixer.kv_run is not None]
        latent = [L.mixer for L in self.layers if isinstance(L.mixer, LatentAttention)]
        self.tc_attention = bool(latent) and all(m.tc for m in latent)
        for m in latent:
            m.tc = self.tc_attention               # a step's runs are cut once for all layers
        self.windows = tuple(sorted({m.window for m in latent})) if self.tc_attention else ()
        cores = [L.mixer.core for L in self.layers if hasattr(L.mixer, "core")]
        self.tc_state = bool(cores) and all(c.tc for c in cores)
        for c in cores:
            c.tc = self.tc_state

    # ---- layered engine -----------------------------------------------------------------------------------------------
    def bind(self, e) -> None:
        n, d = e.max_rows, self.width
        e.scratch.reserve("x", n * d, torch.float32)
        for name in ("h", "y"):
            e.scratch.reserve(name, n * d, self.dtype)
        self.run_state, kv = [], 0
        for i, L in enumerate(self.layers):
            L.mixer.reserve(e)
            if L.ff is not None:
                L.ff.reserve(e)
            self.run_state.append(L.mixer.bind_run(e, f"layer{i}", kv))
            kv += L.mixer.kv_run is not None
        self.engine = e

    def forward(self, s):
        n, d = s.n, self.width
        s.engine = self.engine
        x, h = s.scratch.get("x", n, d), s.scratch.get("h", n, d)
        common = dict(eps=self.cfg.eps, status=s.status)
        R.seam(x, n, h=h, embed=self.embed, tokens=s.tokens, from_embed=True, embed_scale=self.cfg.embed_scale, **common)
        for i, L in enumerate(self.layers):
            update = dict(y=L.mixer.run(s, h, self.run_state[i])[0], post=L.norm["norm1"])
            if L.ff is not None:
                R.seam(x, n, h=h, **update, **common)
                update = dict(y=L.ff.run(s, h), post=L.norm["norm2"])
            if s.taps is not None:
                update["tap"] = torch.empty((n, d), dtype=torch.float32, device=x.device)
                s.taps.append(update["tap"])
            if i + 1 < len(self.layers):
                R.seam(x, n, h=h, **update, **common)
            elif s.nhead or s.taps is not None:
                rows = s.head_rows if s.taps is None else None
                m = n if rows is None else s.nhead
                hf = s.scratch.get("h", m, d)
                R.seam(x, m, h=hf, norm=self.final, row_map=rows, **update, **common)
                if rows is None and s.head_rows is not None:
                    hf = hf[s.head_rows.long()]
        if not s.nhead:
            return None
        V = self.vocab
        out = s.scratch.get("logits", s.nhead, V) if s.single else torch.empty((s.nhead, V), dtype=torch.float32, device=x.device)
        return R.head(hf, self.head, out)
