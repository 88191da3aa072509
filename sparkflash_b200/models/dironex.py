"""Dironex: a small decoder whose layers mix tokens with latent attention (queries out of a latent of their own, halves rotated at YaRN
frequencies, a gate on the output) or with grouped-query attention in a sliding window (heads normed, no rotation).  The residual is several
streams, which every sublayer reads as a weighted sum and writes back through a matrix; a short convolution on each sublayer's input; dense
feed-forwards with xIELU or a mixture of experts with squared relu, chosen group by group; a range of layers run several times.

This file is the design's configuration, its tensor names and its order of operations.  The mechanisms are models/mixers.py and
ops/rows.py; lanes, cache, state, batching and sampling are models/layered.py.

    runs         layers 0 .. start-1, then start .. stop-1 ``times`` times, then the rest; every run of a layer has its own cache and state
    a sublayer   h = RMS(sum_s in[s] x_s); h += conv(h); y = f(h); x_t = sum_s mix[s, t] x_s + m out[t] y, with f the mixer, then the feed-forward
    head         RMS(sum_s x_s) times the output table
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch
import torch.nn.functional as F

from ..ops import rows as R
from .layered import CONFIG_META, LayeredModel, check_keys, check_loop, loop_runs
from .mixers import HeadNormAttention, LatentAttention, MixtureFF, SingleFF, StreamMix, W

ARCHITECTURE = "Dironex"

_TOP = {"architecture", "vocab", "width", "norm", "embedding", "residual_mult", "streams", "canon", "layers", "loop"}
_MIXERS = {"attention": {"heads", "kv_heads", "dim", "vdim", "scale", "mask"},
           "latent_attention": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot"}}


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None          # dense or mixture of experts, None: no feed-forward


@dataclass
class DironexConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    residual_mult: float
    streams: int
    taps: int
    layers: list[LayerSpec] = field(default_factory=list)
    loop: dict | None = None
    name: str = "dironex"
    eos_id: int = -1

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, d: dict) -> "DironexConfig":
        check_keys(d, _TOP, "top level", CONFIG_META | {"loop"})
        if d["architecture"] != ARCHITECTURE:
            raise ValueError(f"config.json: architecture {d['architecture']!r} is not {ARCHITECTURE}")
        check_keys(d["norm"], {"eps"}, "norm")
        check_keys(d["embedding"], {"scale"}, "embedding")
        check_keys(d["canon"], {"taps"}, "canon")
        layers = []
        for i, L in enumerate(d["layers"]):
            check_keys(L, {"type", "mixer", "mlp"}, f"layer {i}", {"mlp"})
            if L["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown type {L['type']!r}")
            check_keys(L["mixer"], _MIXERS[L["type"]], f"layer {i} mixer")
            _check_mixer(L["type"], L["mixer"], f"layer {i}")
            if L.get("mlp") is not None:
                _check_mlp(L["mlp"], f"layer {i} mlp")
            layers.append(LayerSpec(L["type"], L["mixer"], L.get("mlp")))
        loop = d.get("loop")
        if loop:
            check_loop(loop, len(layers))
        _need(1 <= d["streams"] <= R.MAX_STREAMS, "config.json", f"up to {R.MAX_STREAMS} streams are implemented")
        _need(1 <= d["canon"]["taps"] <= R.MAX_TAPS, "config.json", f"convolutions of 1..{R.MAX_TAPS} taps are implemented")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["residual_mult"]), d["streams"], d["canon"]["taps"],
                   layers, loop or None, d.get("name", "dironex"), d.get("eos_token_id", -1))

    def runs(self) -> list[int]:
        """Layers in the order they run."""
        return [i for i, _ in loop_runs(len(self.layers), self.loop)]

    def shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint."""
        d, s = self.width, self.streams
        out = {"embed": (self.vocab, d), "head": (self.vocab, d), "final.norm": (d,)}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            q, H, dim, vdim = p + "mix.", m["heads"], m["dim"], m["vdim"]
            for k in (1, 2) if L.mlp is not None else (1,):
                out[f"{p}norm{k}"], out[f"{p}canon{k}"] = (d,), (d, self.taps)
                out[f"{p}hc{k}.in"] = out[f"{p}hc{k}.out"] = (s,)
                out[f"{p}hc{k}.mix"] = (s, s)
            out[q + "o"] = (d, H * vdim)
            if L.type == "attention":
                G = m["kv_heads"]
                out[q + "q"], out[q + "k"], out[q + "v"] = (H * dim, d), (G * dim, d), (G * vdim, d)
                out[q + "q.norm"] = out[q + "k.norm"] = (dim,)
            else:
                r, qr, rot = m["kv_rank"], m["q_rank"], m["rot_dim"]
                out[q + "dq"], out[q + "dq.norm"], out[q + "uq"] = (qr, d), (qr,), (H * (dim + rot), qr)
                out[q + "dkv"], out[q + "dkv.norm"] = (r + rot, d), (r,)
                out[q + "uk"], out[q + "uv"], out[q + "g"] = (H * dim, r), (H * vdim, r), (H * vdim, d)
            if L.mlp is None:
                continue
            if L.mlp["kind"] == "dense":
                out[p + "mlp.up"], out[p + "mlp.down"], out[p + "mlp.act"] = (L.mlp["ff"], d), (d, L.mlp["ff"]), (2,)
            else:
                E, ff = L.mlp["router"]["experts"], L.mlp["expert"]["ff"]
                out[p + "mlp.router"], out[p + "mlp.correction"] = (E, d), (E,)
                for e in range(E):
                    out[f"{p}mlp.e{e}.up"], out[f"{p}mlp.e{e}.down"] = (ff, d), (d, ff)
        return out


def _need(ok: bool, where: str, what: str) -> None:
    if not ok:
        raise ValueError(f"{where}: {what}")


def _check_mixer(kind: str, m: dict, where: str) -> None:
    if kind == "attention":
        check_keys(m["mask"], {"size"}, f"{where} mask")
        _need(m["heads"] % m["kv_heads"] == 0, where, "heads must be a multiple of kv_heads")
        _need(m["mask"]["size"] >= 1, where, "a window sees at least its own position")
        return
    rot = m["rot"]
    check_keys(rot, {"base", "dims", "scaling"}, f"{where} rot", {"scaling"})
    _need(rot["dims"] == m["rot_dim"] and m["rot_dim"] % 2 == 0 and m["rot_dim"] > 0, where, "rot.dims must be rot_dim, even and above 0")
    if rot.get("scaling") is not None:
        check_keys(rot["scaling"], {"factor", "original", "fast", "slow"}, f"{where} rot.scaling")


def _groups(router: dict) -> dict:
    return router.get("groups") or {"count": 1, "keep": 1}


def _check_mlp(m: dict, where: str) -> None:
    if m.get("kind") == "dense":
        check_keys(m, {"kind", "ff"}, where)
        return
    if m.get("kind") != "moe":
        raise ValueError(f"{where}: unknown kind {m.get('kind')!r}")
    check_keys(m, {"kind", "router", "expert"}, where)
    check_keys(m["expert"], {"ff"}, f"{where} expert")
    r = m["router"]
    check_keys(r, {"experts", "top", "groups", "scale"}, f"{where} router", {"groups"})
    g = _groups(r)
    check_keys(g, {"count", "keep"}, f"{where} router.groups")
    _need(1 <= r["top"] <= min(r["experts"], R.MOE_MAX_TOP) and r["experts"] <= R.MOE_MAX_EXPERTS, where,
          f"up to {R.MOE_MAX_EXPERTS} experts and {R.MOE_MAX_TOP} choices, no more choices than experts")
    _need(1 <= g["keep"] <= g["count"] <= R.MOE_MAX_GROUPS and r["experts"] % g["count"] == 0, where,
          f"up to {R.MOE_MAX_GROUPS} equal groups of experts, no more kept than there are")
    _need(r["top"] <= r["experts"] // g["count"] * g["keep"], where, "the groups kept hold fewer experts than are chosen")


def random_tensors(cfg: DironexConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights of the right shapes (benchmarks, tests, ``--synthetic``), bf16 as a checkpoint stores them."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g, device=device)
        if leaf in ("norm", "norm1", "norm2"):
            t = 1 + 0.1 * r
        elif leaf in ("in", "out"):
            t = 1 / cfg.streams + 0.2 * r if leaf == "in" else 1 + 0.2 * r
        elif leaf == "mix":
            t = torch.eye(cfg.streams, device=device) + 0.1 * r
        elif leaf == "embed":
            t = r / cfg.embed_scale
        elif leaf == "correction":
            t = 0.1 * r
        elif leaf == "act":
            t = r
        elif leaf in ("canon1", "canon2"):
            t = 0.3 * r
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    def __init__(self, t, i: int, spec: LayerSpec, cfg: DironexConfig, dtype, device, max_context: int):
        w = W(t, f"l{i}.", dtype, device)
        mix, mlp = w.sub("mix."), w.sub("mlp.")
        if spec.type == "attention":
            self.mixer = HeadNormAttention(mix, spec.mixer, cfg.eps, max_context)
        else:
            self.mixer = LatentAttention(mix, spec.mixer, cfg.eps, max_context, halves=True, gated=True)
        self.ff = None
        if spec.mlp is not None and spec.mlp["kind"] == "dense":
            p, q = F.softplus(mlp.f32("act").double(), threshold=50.0).tolist()
            self.ff = SingleFF(mlp, "xielu", p, 0.5 + q)
        elif spec.mlp is not None:
            r = spec.mlp["router"]
            g = _groups(r)
            self.ff = MixtureFF(mlp, spec.mlp, act="relu2", choice=R.Choice(mlp.f32("correction"), g["count"], g["keep"], float(r["scale"])))
        subs = (1, 2) if self.ff is not None else (1,)
        self.norm = [w.f32(f"norm{k}") for k in subs]
        self.canon = [w.taps(f"canon{k}") for k in subs]
        self.streams = [StreamMix(w.sub(f"hc{k}."), cfg.residual_mult) for k in subs]


class Dironex(LayeredModel):
    """The model as models/layered.py drives it."""

    config_class = DironexConfig

    def __init__(self, cfg: DironexConfig, tensors: dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device="cuda",
                 max_context: int = 4096):
        self._load(cfg, tensors, dtype, device)
        self.layers = [_Layer(tensors, i, L, cfg, dtype, device, max_context) for i, L in enumerate(cfg.layers)]
        top = W(tensors, "", dtype, device)
        self.embed, self.head, self.final = top.act("embed"), top.act("head"), top.f32("final.norm")
        self.order = cfg.runs()
        self.kv_runs = [self.layers[i].mixer.kv_run for i in self.order]
        self.tc_attention = any(L.mixer.tc for L in self.layers)
        self.windows = tuple(sorted({L.mixer.window for L in self.layers if isinstance(L.mixer, LatentAttention) and L.mixer.tc}))

    # ---- layered engine -----------------------------------------------------------------------------------------------
    def bind(self, e) -> None:
        n, d, dt = e.max_rows, self.width, self.dtype
        e.scratch.reserve("x", n * self.cfg.streams * d, torch.float32)
        for name in ("h", "hc", "y"):
            e.scratch.reserve(name, n * d, dt)
        for L in self.layers:
            L.mixer.reserve(e)
            if L.ff is not None:
                L.ff.reserve(e)
        self.run_state = []
        for r, i in enumerate(self.order):
            L = self.layers[i]
            st = L.mixer.bind_run(e, f"run{r}", r)
            st["canon"] = [e.state.add(f"run{r}.canon{k}", (self.cfg.taps - 1, d), dt) for k in range(len(L.canon))]
            self.run_state.append(st)
        self.engine = e

    def forward(self, s):
        cfg, n, d = self.cfg, s.n, self.width
        s.engine = self.engine
        x, h = s.scratch.get("x", n, cfg.streams, d), s.scratch.get("h", n, d)
        common = dict(eps=cfg.eps, status=s.status)

        def enter(r, k, **update):
            """The streams take the last output; sublayer k of run r reads them: norm and input convolution."""
            L, hist = self.layers[self.order[r]], self.run_state[r]["canon"][k]
            args = dict(h=h, norm=L.norm[k], into=L.streams[k].into, **update, **common)
            if s.single:
                R.stream_seam(x, n, conv=(L.canon[k], hist, s.seg_src, s.seg_dst), **args)
                return h
            R.stream_seam(x, n, **args)
            hc = s.scratch.get("hc", n, d)
            R.conv(h, L.canon[k], None, hc, hist, s, n, R.CONV_RESIDUAL)
            return hc
        update = dict(embed=self.embed, tokens=s.tokens, embed_scale=cfg.embed_scale)
        for r, i in enumerate(self.order):
            L = self.layers[i]
            y, _ = L.mixer.run(s, enter(r, 0, **update), self.run_state[r])
            update = dict(y=y, mix=L.streams[0].mix, out=L.streams[0].out)
            if L.ff is not None:
                y = L.ff.run(s, enter(r, 1, **update))
                y, wts = y if isinstance(y, tuple) else (y, None)
                update = dict(y=y, parts_w=wts, mix=L.streams[1].mix, out=L.streams[1].out)
            if s.taps is not None:
                update["tap"] = torch.empty((n, d), dtype=torch.float32, device=x.device)
                s.taps.append(update["tap"])
        if not s.nhead and s.taps is None:
            return None
        rows = s.head_rows if s.taps is None else None
        m = n if rows is None else s.nhead
        hf = s.scratch.get("hc", m, d)
        R.stream_seam(x, m, h=hf, norm=self.final, row_map=rows, keep=False, **update, **common)
        if not s.nhead:
            return None
        if rows is None and s.head_rows is not None:
            hf = hf[s.head_rows.long()]
        V = self.vocab
        out = s.scratch.get("logits", s.nhead, V) if s.single else torch.empty((s.nhead, V), dtype=torch.float32, device=x.device)
        return R.head(hf, self.head, out)
