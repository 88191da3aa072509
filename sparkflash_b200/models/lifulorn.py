"""Lifulorn: a small decoder whose layers mix tokens with the gated delta rule or with one of two kinds of attention in a sliding window
(a learned sink per head, scaled rotations, values mixed with the first such layer's; the second kind caps its scores).  RMS norm ahead of
every sublayer, whose output is scaled element by element; a mixture of experts as feed-forward, or none; every layer ends with an
input of its own that depends on the token.

This file is the design's configuration, its tensor names and its order of operations.  The mechanisms are models/mixers.py and
ops/rows.py; lanes, cache, state, batching and sampling are models/layered.py.

    a layer     x += m ls1 mixer(RMS1(x));  x += m ls2 ff(RMS2(x));  x += m RMS(W_proj (gelu(W_gate x) * table[token]))
    head        RMS(x) times the output table
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops import rows as R
from .layered import CONFIG_META, LayeredModel, check_keys
from .mixers import DeltaMixer, MixtureFF, RotaryAttention, TokenInput, ValueMix, W

ARCHITECTURE = "Lifulorn"
GATE_ALPHA = 1.702        # of the experts' gate g sigmoid(alpha g)

_TOP = {"architecture", "vocab", "width", "norm", "residual_mult", "token_side", "layers"}
_ATT = {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"}
_MIXERS = {"attention": (_ATT, {"v_mix"}), "attention_2": (_ATT | {"softcap"}, {"v_mix"}), "delta": ({"heads", "kv_heads", "dim", "vdim", "conv"}, set())}
_SCALING = {"attention": {"factor", "low", "high", "original"}, "attention_2": {"factor", "original", "fast", "slow"}}


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None          # mixture of experts, None: no feed-forward
    mix: bool                 # takes part in the value mixing


@dataclass
class LifulornConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    side_dim: int
    layers: list[LayerSpec] = field(default_factory=list)
    name: str = "lifulorn"
    eos_id: int = -1

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, d: dict) -> "LifulornConfig":
        check_keys(d, _TOP, "top level", CONFIG_META)
        if d["architecture"] != ARCHITECTURE:
            raise ValueError(f"config.json: architecture {d['architecture']!r} is not {ARCHITECTURE}")
        check_keys(d["norm"], {"eps"}, "norm")
        check_keys(d["token_side"], {"dim"}, "token_side")
        layers, mixed = [], set()
        for i, L in enumerate(d["layers"]):
            check_keys(L, {"type", "mixer", "mlp"}, f"layer {i}", {"mlp"})
            m = L["mixer"]
            if L["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown type {L['type']!r}")
            keys, optional = _MIXERS[L["type"]]
            check_keys(m, keys | optional, f"layer {i} mixer", optional)
            _check_mixer(L["type"], m, f"layer {i}")
            if m.get("v_mix"):
                mixed.add((m["kv_heads"], m["vdim"]))
            if L.get("mlp") is not None:
                _check_mixture(L["mlp"], f"layer {i} mlp")
            layers.append(LayerSpec(L["type"], m, L.get("mlp"), bool(m.get("v_mix"))))
        if len(mixed) > 1:
            raise ValueError(f"config.json: layers that mix values differ in their sizes: {sorted(mixed)}")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["residual_mult"]), d["token_side"]["dim"], layers, d.get("name", "lifulorn"),
                   d.get("eos_token_id", -1))

    def shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint."""
        d, side = self.width, self.side_dim
        out = {"embed": (self.vocab, d), "head": (self.vocab, d), "final.norm": (d,), "side.embed": (self.vocab, side * len(self.layers))}

        def expert(p, ff):
            out[p + "gate"] = out[p + "up"] = (ff, d)
            out[p + "down"] = (d, ff)
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            q, H, G, dim, vdim = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[p + "norm1"] = out[p + "ls1"] = out[p + "side.norm"] = (d,)
            out[p + "side.gate"], out[p + "side.proj"] = (side, d), (d, side)
            out[q + "o"] = (d, H * vdim)
            if L.type == "delta":
                for n, rows in (("q", G * dim), ("k", G * dim), ("v", H * vdim)):
                    out[q + n], out[q + n + ".conv"] = (rows, d), (rows, m["conv"])
                out[q + "g"], out[q + "norm"] = (H * vdim, d), (vdim,)
                out[q + "a"] = out[q + "b"] = (H, d)
                out[q + "A_log"] = out[q + "dt_bias"] = (H,)
            else:
                for n, rows in (("q", H * dim), ("k", G * dim), ("v", G * vdim)):
                    out[q + n], out[q + n + ".b"] = (rows, d), (rows,)
                out[q + "sink"] = (H,)
                if L.mix:
                    out[q + "vmix"] = ()
            if L.mlp is not None:
                out[p + "norm2"] = out[p + "ls2"] = (d,)
                out[p + "mlp.router"] = (L.mlp["router"]["experts"], d)
                for e in range(L.mlp["router"]["experts"]):
                    expert(f"{p}mlp.e{e}.", L.mlp["expert"]["ff"])
                if L.mlp.get("shared") is not None:
                    expert(p + "mlp.shared.", L.mlp["shared"]["ff"])
                    out[p + "mlp.shared.sg"] = (1, d)
        return out


def _need(ok: bool, where: str, what: str) -> None:
    if not ok:
        raise ValueError(f"{where}: {what}")


def _check_mixer(kind: str, m: dict, where: str) -> None:
    _need(m["heads"] % m["kv_heads"] == 0, where, "heads must be a multiple of kv_heads")
    if kind == "delta":
        _need(1 <= m["conv"] <= R.MAX_TAPS, where, f"convolutions of 1..{R.MAX_TAPS} taps are implemented")
        R.state_pad(m["dim"])
        return
    check_keys(m["mask"], {"size"}, f"{where} mask")
    _need(m["mask"]["size"] >= 1, where, "a window sees at least its own position")
    rot = m["rot"]
    check_keys(rot, {"base", "dims", "scaling"}, f"{where} rot", {"scaling"})
    _need(rot["dims"] % 2 == 0 and 0 < rot["dims"] <= m["dim"], where, "rot.dims must be even and at most dim")
    if rot.get("scaling") is not None:
        check_keys(rot["scaling"], _SCALING[kind], f"{where} rot.scaling")
    _need(kind == "attention" or m["softcap"] > 0, where, "softcap must be above 0")


def _check_mixture(m: dict, where: str) -> None:
    check_keys(m, {"kind", "router", "expert", "shared"}, where, {"shared"})
    if m["kind"] != "moe":
        raise ValueError(f"{where}: unknown kind {m['kind']!r}")
    check_keys(m["router"], {"experts", "top"}, f"{where} router")
    check_keys(m["expert"], {"ff", "limit"}, f"{where} expert")
    if m.get("shared") is not None:
        check_keys(m["shared"], {"ff", "limit"}, f"{where} shared")
    r = m["router"]
    _need(1 <= r["top"] <= min(r["experts"], R.MOE_MAX_TOP) and r["experts"] <= R.MOE_MAX_EXPERTS, where,
          f"up to {R.MOE_MAX_EXPERTS} experts and {R.MOE_MAX_TOP} choices, no more choices than experts")


def random_tensors(cfg: LifulornConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights of the right shapes (benchmarks, tests, ``--synthetic``), bf16 as a checkpoint stores them."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g, device=device)
        if leaf == "b" and not name.endswith(".mix.b"):
            t = r * 0.1
        elif leaf in ("norm", "norm1", "norm2", "ls1", "ls2"):
            t = 1 + 0.1 * r
        elif leaf == "dt_bias":
            t = -3 + r
        elif leaf in ("A_log", "embed", "sink"):
            t = r
        elif leaf == "vmix":
            t = 0.5 + 0.1 * r
        elif leaf == "conv":
            t = r * 0.4
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    def __init__(self, t, i: int, spec: LayerSpec, cfg: LifulornConfig, dtype, device, max_context: int, table: torch.Tensor, mix: ValueMix | None):
        w, m = W(t, f"l{i}.", dtype, device), cfg.residual_mult
        if spec.type == "delta":
            self.mixer = DeltaMixer(w.sub("mix."), spec.mixer, cfg.eps)
        else:
            self.mixer = RotaryAttention(w.sub("mix."), spec.mixer, max_context, mix if spec.mix else None)
        self.ff = MixtureFF(w.sub("mlp."), spec.mlp, GATE_ALPHA) if spec.mlp is not None else None
        self.side = TokenInput(w.sub("side."), table, i * cfg.side_dim)
        self.norm1, self.ls1, self.side_norm = w.f32("norm1"), m * w.f32("ls1"), m * w.f32("side.norm")
        self.norm2, self.ls2 = (w.f32("norm2"), m * w.f32("ls2")) if self.ff is not None else (None, None)


class Lifulorn(LayeredModel):
    """The model as models/layered.py drives it."""

    config_class = LifulornConfig

    def __init__(self, cfg: LifulornConfig, tensors: dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device="cuda",
                 max_context: int = 4096):
        self._load(cfg, tensors, dtype, device)
        top = W(tensors, "", dtype, device)
        self.embed, self.head, self.final, self.table = top.act("embed"), top.act("head"), top.f32("final.norm"), top.act("side.embed")
        mixed = [L.mixer for L in cfg.layers if L.mix]
        mix = ValueMix(mixed[0]["kv_heads"] * mixed[0]["vdim"]) if mixed else None
        self.layers = [_Layer(tensors, i, L, cfg, dtype, device, max_context, self.table, mix) for i, L in enumerate(cfg.layers)]
        self.kv_runs = [L.mixer.kv_run for L in self.layers if L.mixer.kv_run is not None]
        att = [L.mixer for L in self.layers if isinstance(L.mixer, RotaryAttention)]
        self.tc_attention = bool(att) and all(m.tc for m in att)
        for m in att:
            m.tc = self.tc_attention               # a step's runs are cut once for all layers
        cores = [L.mixer.core for L in self.layers if isinstance(L.mixer, DeltaMixer)]
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
            L.side.reserve(e)
            if L.ff is not None:
                L.ff.reserve(e)
            self.run_state.append(L.mixer.bind_run(e, f"layer{i}", kv))
            kv += L.mixer.kv_run is not None
        self.engine = e

    def forward(self, s):
        n, d = s.n, self.width
        s.engine = self.engine
        x, h = s.scratch.get("x", n, d), s.scratch.get("h", n, d)
        common = dict(eps=self.cfg.eps, status=s.status, norm_kind="rms")
        R.seam(x, n, h=h, embed=self.embed, tokens=s.tokens, from_embed=True, norm=(self.layers[0].norm1, None), **common)
        for i, L in enumerate(self.layers):
            update = dict(y=L.mixer.run(s, h, self.run_state[i])[0], post=(L.ls1, None), post_kind="scale")
            if L.ff is not None:
                R.seam(x, n, h=h, norm=(L.norm2, None), **update, **common)
                parts, wts = L.ff.run(s, h)
                update = dict(y=parts, parts_w=wts, post=(L.ls2, None), post_kind="scale")
            R.seam(x, n, h=h, **update, **common)              # h: the residual itself
            update = dict(y=L.side.run(s, h), post=(L.side_norm, None), post_kind="rms")
            if s.taps is not None:
                update["tap"] = torch.empty((n, d), dtype=torch.float32, device=x.device)
                s.taps.append(update["tap"])
            if i + 1 < len(self.layers):
                R.seam(x, n, h=h, norm=(self.layers[i + 1].norm1, None), **update, **common)
            elif s.nhead or s.taps is not None:
                rows = s.head_rows if s.taps is None else None
                m = n if rows is None else s.nhead
                hf = s.scratch.get("h", m, d)
                R.seam(x, m, h=hf, norm=(self.final, None), row_map=rows, **update, **common)
                if rows is None and s.head_rows is not None:
                    hf = hf[s.head_rows.long()]
        if not s.nhead:
            return None
        V = self.vocab
        out = s.scratch.get("logits", s.nhead, V) if s.single else torch.empty((s.nhead, V), dtype=torch.float32, device=x.device)
        return R.head(hf, self.head, out)
