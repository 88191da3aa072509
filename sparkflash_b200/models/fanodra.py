"""Fanodra: a small decoder whose layers mix tokens with a real-gated linear recurrence, or with attention and such a recurrence
side by side; layer norm before and after every sublayer, a short input convolution, looped layers, tied embedding.

This file is the design's configuration, its tensor names and its order of operations.  The mechanisms are models/mixers.py and
ops/rows.py; lanes, cache, state, batching and sampling are models/layered.py.

    runs        layers 0 .. start-1, then start .. stop-1 ``times`` times, then the rest; every run of a layer has its own cache
                and state.  Before pass t of the loop: x += embedding (t > 0), x += step[t].
    a layer     h = LN1(x); h += conv(h); x += LN1b(mixer(h)); x += LN2b(ff(LN2(x)))
    head        LN(x) times the embedding table
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops import rows as R
from .layered import CONFIG_META, LayeredModel, check_keys, check_loop, loop_runs
from .mixers import DenseFF, ParallelMixer, RecurrentMixer, W

ARCHITECTURE = "Fanodra"
DECAY_C = 8.0             # log a = -DECAY_C * r * softplus(lam)

_TOP = {"architecture", "vocab", "width", "norm", "canon", "layers", "loop"}
_REC = {"width", "blocks", "conv"}
_ATT = {"heads", "kv_heads", "dim", "vdim", "scale"}


@dataclass
class LayerSpec:
    type: str                 # "rglru" or "parallel"
    mixer: dict
    ff: int | None            # dense feed-forward width, None: no feed-forward


@dataclass
class FanodraConfig:
    vocab: int
    width: int
    eps: float
    taps: int
    layers: list[LayerSpec] = field(default_factory=list)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0       # 0: no loop
    name: str = "fanodra"
    eos_id: int = -1

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, d: dict) -> "FanodraConfig":
        check_keys(d, _TOP, "top level", CONFIG_META | {"loop"})
        if d["architecture"] != ARCHITECTURE:
            raise ValueError(f"config.json: architecture {d['architecture']!r} is not {ARCHITECTURE}")
        check_keys(d["norm"], {"eps"}, "norm")
        check_keys(d["canon"], {"taps"}, "canon")
        layers = []
        for i, L in enumerate(d["layers"]):
            check_keys(L, {"type", "mixer", "mlp"}, f"layer {i}", {"mlp"})
            m = L["mixer"]
            if L["type"] == "parallel":
                check_keys(m, {"left", "right"}, f"layer {i} mixer")
                check_keys(m["left"], _ATT, f"layer {i} left")
                if m["left"]["heads"] % m["left"]["kv_heads"]:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            elif L["type"] != "rglru":
                raise ValueError(f"layer {i}: unknown type {L['type']!r}")
            rec = m["right"] if L["type"] == "parallel" else m
            check_keys(rec, _REC, f"layer {i} recurrence")
            if rec["width"] % rec["blocks"]:
                raise ValueError(f"layer {i}: recurrence width must be a multiple of blocks")
            if not 1 <= rec["conv"] <= R.MAX_TAPS:
                raise ValueError(f"layer {i}: convolutions of 1..{R.MAX_TAPS} taps are implemented")
            ff = L.get("mlp")
            if ff is not None:
                check_keys(ff, {"kind", "ff"}, f"layer {i} mlp")
                if ff["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown mlp kind {ff['kind']!r}")
            layers.append(LayerSpec(L["type"], m, ff["ff"] if ff is not None else None))
        loop = d.get("loop") or {"start": 0, "stop": 0, "times": 0}
        if loop["times"]:
            check_loop(loop, len(layers))
        if not 1 <= d["canon"]["taps"] <= R.MAX_TAPS:
            raise ValueError(f"convolutions of 1..{R.MAX_TAPS} taps are implemented")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), d["canon"]["taps"], layers, loop["start"], loop["stop"], loop["times"],
                   d.get("name", "fanodra"), d.get("eos_token_id", -1))

    def runs(self) -> list[tuple[int, int | None]]:
        """(layer, pass that begins right before it or None) in the order the layers run."""
        order = loop_runs(len(self.layers), {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times} if self.loop_times else None)
        return [(i, t if i == self.loop_start else None) for i, t in order]

    def shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint."""
        d, out = self.width, {"embed": (self.vocab, self.width), "final.norm": (self.width,), "final.norm.b": (self.width,)}
        if self.loop_times:
            out["loop.step"] = (self.loop_times, d)

        def rec(p, m):
            w, nb = m["width"], m["blocks"]
            for n in ("y", "x"):
                out[p + n], out[p + n + ".b"] = (w, d), (w,)
            out[p + "conv"], out[p + "conv.b"], out[p + "lam"], out[p + "o"] = (w, m["conv"]), (w,), (w,), (d, w)
            for n in ("ra", "ri"):
                out[p + n], out[p + n + ".b"] = (nb, w // nb, w // nb), (nb, w // nb)
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L.ff is not None else ()):
                out[p + n], out[p + n + ".b"] = (d,), (d,)
            out[p + "canon1"] = (d, self.taps)
            if L.type == "rglru":
                rec(p + "mix.", L.mixer)
            else:
                m, q = L.mixer["left"], p + "mix.left."
                for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                    out[q + n], out[q + n + ".b"] = (rows, d), (rows,)
                out[q + "q.norm"], out[q + "k.norm"] = (m["heads"] * m["dim"],), (m["kv_heads"] * m["dim"],)
                out[q + "r1"] = out[q + "r2"] = (m["heads"],)
                out[q + "o"], out[q + "o.b"], out[q + "out"] = (d, m["heads"] * m["vdim"]), (d,), (d,)
                rec(p + "mix.right.", L.mixer["right"])
                out[p + "mix.right.out"] = (d,)
            if L.ff is not None:
                out[p + "mlp.gate"] = out[p + "mlp.up"] = (L.ff, d)
                out[p + "mlp.down"] = (d, L.ff)
        return out


def random_tensors(cfg: FanodraConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random weights of the right shapes (benchmarks, tests, ``--synthetic``), bf16 as a checkpoint stores them."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in cfg.shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g, device=device)
        if name.endswith(".b"):
            t = r * 0.1
        elif leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b", "out"):
            t = 1 + 0.1 * r
        elif leaf in ("r1", "r2"):
            t = 0.2 + r.abs()
        elif leaf == "lam":
            t = -2 + r
        elif leaf == "embed" or leaf == "step":
            t = r
        elif leaf in ("conv", "canon1"):
            t = r * 0.4
        else:
            t = r * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


class _Layer:
    def __init__(self, t, i: int, spec: LayerSpec, cfg: FanodraConfig, dtype, device, max_context: int):
        w = W(t, f"l{i}.", dtype, device)
        if spec.type == "rglru":
            self.mixer = RecurrentMixer(w.sub("mix."), spec.mixer, DECAY_C)
        else:
            self.mixer = ParallelMixer(w.sub("mix."), spec.mixer, cfg.eps, DECAY_C, max_context)
        self.ff = DenseFF(w.sub("mlp.")) if spec.ff is not None else None
        names = ("norm1", "norm1b") + (("norm2", "norm2b") if self.ff is not None else ())
        self.norm = {n: (w.f32(n), w.f32(n + ".b")) for n in names}
        self.canon = w.taps("canon1")


class Fanodra(LayeredModel):
    """The model as models/layered.py drives it."""

    config_class = FanodraConfig

    def __init__(self, cfg: FanodraConfig, tensors: dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16, device="cuda",
                 max_context: int = 4096):
        self._load(cfg, tensors, dtype, device)
        self.layers = [_Layer(tensors, i, spec, cfg, dtype, device, max_context) for i, spec in enumerate(cfg.layers)]
        top = W(tensors, "", dtype, device)
        self.embed = top.act("embed")
        self.final = (top.f32("final.norm"), top.f32("final.norm.b"))
        self.step_vec = list(top.f32("loop.step")) if cfg.loop_times else []
        self.order = cfg.runs()
        self.kv_runs = [self.layers[i].mixer.kv_run for i, _ in self.order if self.layers[i].mixer.kv_run is not None]
        self.tc_attention = any(L.mixer.att.tc for L in self.layers if isinstance(L.mixer, ParallelMixer))

    # ---- layered engine -----------------------------------------------------------------------------------------------
    def bind(self, e) -> None:
        n, d, dt = e.max_rows, self.width, self.dtype
        e.scratch.reserve("x", n * d, torch.float32)
        for name in ("h", "hc", "y", "y2"):
            e.scratch.reserve(name, n * d, dt)
        for L in self.layers:
            L.mixer.reserve(e)
            if L.ff is not None:
                L.ff.reserve(e)
        self.run_state, kv = [], 0
        for r, (i, _) in enumerate(self.order):
            m = self.layers[i].mixer
            st = m.bind_run(e, f"run{r}", kv)
            kv += m.kv_run is not None
            st["canon"] = e.state.add(f"run{r}.canon", (self.cfg.taps - 1, d), dt)
            self.run_state.append(st)
        self.engine = e

    def _begin(self, r: int) -> dict:
        """What run ``r`` adds to the residual before its first norm."""
        t = self.order[r][1]
        return {} if t is None else {"step_vec": self.step_vec[t], "add_embed": t > 0}

    def forward(self, s):
        cfg, n, d = self.cfg, s.n, self.width
        s.engine = self.engine
        x, h = s.scratch.get("x", n, d), s.scratch.get("h", n, d)
        common = dict(eps=cfg.eps, status=s.status, embed=self.embed, tokens=s.tokens)

        def enter(r, **update):
            """Residual update, run r's additions, its first norm and input convolution: the mixer's input."""
            L, st = self.layers[self.order[r][0]], self.run_state[r]
            if s.single:
                R.seam(x, n, h=h, norm=L.norm["norm1"], conv=(L.canon, st["canon"], s.seg_src, s.seg_dst), **self._begin(r), **update, **common)
                return h
            R.seam(x, n, h=h, norm=L.norm["norm1"], **self._begin(r), **update, **common)
            hc = s.scratch.get("hc", n, d)
            R.conv(h, L.canon, None, hc, st["canon"], s, n, R.CONV_RESIDUAL)
            return hc
        h_in = enter(0, from_embed=True)
        for r, (i, _) in enumerate(self.order):
            L = self.layers[i]
            y, y2 = L.mixer.run(s, h_in, self.run_state[r])
            update = dict(y=y, y2=y2, merge_w=L.mixer.merge if y2 is not None else (None, None), post=L.norm["norm1b"])
            if L.ff is not None:
                R.seam(x, n, h=h, norm=L.norm["norm2"], **update, **common)
                update = dict(y=L.ff.run(s, h), post=L.norm["norm2b"])
            if s.taps is not None:
                update["tap"] = torch.empty((n, d), dtype=torch.float32, device=x.device)
                s.taps.append(update["tap"])
            if r + 1 < len(self.order):
                h_in = enter(r + 1, **update)
            elif s.nhead or s.taps is not None:
                rows = s.head_rows if s.taps is None else None
                m = n if rows is None else s.nhead
                hf = s.scratch.get("hc", m, d)
                R.seam(x, m, h=hf, norm=self.final, row_map=rows, **update, **common)
                if rows is None and s.head_rows is not None:
                    hf = hf[s.head_rows.long()]
        if not s.nhead:
            return None
        V = self.vocab
        out = s.scratch.get("logits", s.nhead, V) if s.single else torch.empty((s.nhead, V), dtype=torch.float32, device=x.device)
        return R.head(hf, self.embed, out)
