"""Rows engine of the layered decoders: models that are a list of layers with a paged key/value cache, recurrent state, or both.

A *rows step* takes token rows of any mix of lanes: whole prompts, portions of prompts cut anywhere, and single decoded
tokens, each lane's rows consecutive.  The engine owns what does not depend on the model - lanes, cache pages
(kv/paged.py), state versions (kv/state.py), the step's index arrays, scratch buffers, CUDA graphs of decode steps, the head's
row selection and the sampler - and speaks the contract of serve/driver.py.  A model supplies

    vocab, width, dtype, device        sizes; ``dtype`` is the activation type (bfloat16, or float32 for true 32-bit)
    kv_runs                            (kv_heads, dim, vdim) of every attention layer run
    tc_attention, tc_state             long runs of rows go to the tensor-core arms of attention / of the matrix-state recurrence
    windows                            window lengths whose keys are multiplied out for a step's long runs
    bind(engine)                       reserve scratch, register state tensors
    forward(step) -> [head rows, vocab] float32 logits (None without a head)

and writes no loop, cache or batching of its own (models/fanodra.py, models/gudutar.py, models/lifulorn.py and models/dironex.py; ``LayeredModel`` has
what they share).
"""
from __future__ import annotations

import gc
import json
import os
import warnings

import torch

from ..kv.paged import PAGE, PagedKV
from ..kv.state import StateSlots
from ..ops import rows as R
from ..ops.sampling import candidate_choice

TC_MIN_ROWS = 32          # runs of at least this many rows go to the tensor-core attention (csrc/k_rows_attn_tc.cu)
TC_TILE = 256             # query rows per block there
STATE_CHUNK = 128         # rows of a chunk of the tensor-core recurrence (csrc/k_rows_state_tc.cu)
TARGET_BLOCKS = 592       # blocks that fill the machine (148 SMs x 4): how far a row's keys are split
MAX_SPLITS = 64


class Scratch:
    """Flat buffers by name, reserved for the largest use before any graph is captured; ``get`` returns a [n, cols] view."""

    def __init__(self, device):
        self.device, self.need, self.buf = device, {}, {}

    def reserve(self, name: str, numel: int, dtype: torch.dtype) -> None:
        old = self.need.get(name)
        if old is not None and old[1] != dtype:
            raise ValueError(f"scratch {name!r} reserved with two dtypes")
        self.need[name] = (max(numel, old[0] if old else 0), dtype)

    def allocate(self) -> None:
        for name, (numel, dtype) in self.need.items():
            self.buf[name] = torch.zeros((numel,), dtype=dtype, device=self.device)

    def get(self, name: str, *shape: int) -> torch.Tensor:
        n = 1
        for s in shape:
            n *= s
        b = self.buf[name]
        if n > b.numel():
            raise ValueError(f"scratch {name!r}: {n} elements asked, {b.numel()} reserved")
        return b[:n].view(*shape)

    def nbytes(self) -> int:
        return sum(b.numel() * b.element_size() for b in self.buf.values())


class Step:
    """Device index arrays of one step (int32), as the kernels take them.

    rows: ``tokens``, ``row_pos``, ``row_lane``, ``row_seg``; segments: ``seg_row0``, ``seg_len``, ``seg_src``, ``seg_dst``;
    scan chunks: ``chunk_*``; attention: ``short_rows`` (rows for the exact arm, None = all), ``tiles`` ((row0, rows) pairs of
    the tensor-core arm, longest first); matrix-state recurrence: ``short_segs`` (segments for the row arm, None = all, ``nshort`` of
    them), ``long_*`` (``nchunks`` chunks of the ``nlong`` others, see _stage); ``expand``: per window the pages whose keys the
    tensor-core arm needs, how many they are, and every tile's page offset among them; head: ``head_rows`` (None = all rows, in order)."""

    single = False            # every segment is one row (a decode step)
    taps: list | None = None  # debug: collects the residual after every layer run

    def single_rows(self, tc: bool):
        """(rows, count) that a sublayer takes one by one: all of them, or those that its tensor-core arm does not (None: all, in order)."""
        return (self.short_rows, self.short) if tc else (None, self.n)


def loop_runs(layers: int, loop: dict | None) -> list[tuple[int, int | None]]:
    """Layers in the order they run, each with its pass (None outside the loop): layers start .. stop - 1 run ``times`` times."""
    if not loop:
        return [(i, None) for i in range(layers)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return [(i, None) for i in range(a)] + [(i, t) for t in range(times) for i in range(a, b)] + [(i, None) for i in range(b, layers)]


def check_loop(loop: dict, layers: int) -> None:
    check_keys(loop, {"start", "stop", "times"}, "loop")
    if not (0 <= loop["start"] < loop["stop"] <= layers and loop["times"] >= 1):
        raise ValueError("config.json: loop out of range")


class LayeredModel:
    """What the models of the engine share: a checkpoint of named tensors whose shapes the configuration knows."""

    config_class: type
    tc_attention = False
    tc_state = False
    windows: tuple[int, ...] = ()

    def _load(self, cfg, tensors: dict[str, torch.Tensor], dtype: torch.dtype, device) -> None:
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("activation type must be bfloat16 or float32")
        shapes = cfg.shapes()
        for name, shape in shapes.items():
            if name not in tensors:
                raise ValueError(f"checkpoint lacks {name}")
            if tuple(tensors[name].shape) != shape:
                raise ValueError(f"{name}: shape {tuple(tensors[name].shape)}, expected {shape}")
        extra = set(tensors) - set(shapes)
        if extra:
            warnings.warn(f"checkpoint tensors that the configuration does not use: {sorted(extra)[:4]}")
        self.cfg, self.vocab, self.width, self.dtype, self.device = cfg, cfg.vocab, cfg.width, dtype, device

    @classmethod
    def from_dir(cls, path: str, dtype: torch.dtype = torch.bfloat16, device="cuda", max_context: int = 4096):
        from ..weights.files import load_checkpoint_dir
        with open(os.path.join(path, "config.json")) as f:
            cfg = cls.config_class.from_dict(json.load(f))
        tensors, files = load_checkpoint_dir(path)
        model = cls(cfg, tensors, dtype, device, max_context)
        if torch.device(device).type == "cuda":
            torch.cuda.synchronize()          # the copies out of the mapped files have been made
        for f in files:
            f.close()
        return model

    def nbytes(self) -> int:
        seen, total, todo = set(), 0, [self]
        while todo:
            o = todo.pop()
            if id(o) in seen:
                continue
            seen.add(id(o))
            if isinstance(o, torch.Tensor):
                total += o.numel() * o.element_size()
            elif isinstance(o, (list, tuple)):
                todo += o
            elif isinstance(o, dict):
                todo += o.values()
            elif type(o).__module__.startswith("sparkflash_b200.models"):
                todo += [v for k, v in vars(o).items() if k not in ("engine", "run_state")]
        return total


def check_keys(d: dict, want: set, where: str, optional: set = frozenset()) -> None:
    """A part of config.json has exactly these keys: what is not implemented is refused."""
    missing, extra = want - set(d) - optional, set(d) - want - optional
    if missing or extra:
        raise ValueError(f"config.json: {where}: missing {sorted(missing)}, unknown {sorted(extra)}")


# keys of a config.json that do not describe the computation
CONFIG_META = {"model_type", "architectures", "dtype", "torch_dtype", "transformers_version", "name", "bos_token_id", "eos_token_id", "pad_token_id"}


class LayeredEngine:
    supports_mask = True
    supports_filter = True
    supports_headless = True
    supports_head_last = True
    ring_slack = 0            # a recurrent state cannot be rewound past its latest step: a lane's prefix is reused whole or not at all
    page = PAGE

    def __init__(self, model, max_lanes: int = 4, max_context: int = 4096, max_rows: int = 1024, pool_tokens: int | None = None,
                 use_graphs: bool = True):
        """``pool_tokens``: tokens all lanes together may hold (each lane rounded up to pages); by default every lane can be full."""
        self.model, self.cfg, self.vocab = model, model.cfg, model.vocab
        self.dev = torch.device(model.device)
        if self.dev.type == "cuda" and self.dev.index is None:       # the serving thread selects it by number
            self.dev = torch.device("cuda", torch.cuda.current_device())
        self.max_lanes, self.max_context, self.max_rows = max_lanes, max_context, max_rows
        if not 0 < max_rows <= 65535:
            raise ValueError("max_rows must be in 1..65535")
        per_lane = -(-max_context // PAGE)
        self.n_pages = per_lane * max_lanes if pool_tokens is None else -(-pool_tokens // PAGE)
        self.kv = PagedKV(model.kv_runs, self.n_pages, max_lanes, max_context, model.dtype, self.dev)
        self.state = StateSlots(max_lanes, self.dev)
        self.scratch = Scratch(self.dev)
        self.status = torch.zeros((4,), dtype=torch.int32, device=self.dev)
        self.chunk_rows = 32          # rows of a scan chunk
        self.use_graphs = use_graphs
        model.bind(self)
        self.scratch.reserve("logits", max_lanes * model.vocab, torch.float32)
        self.scratch.allocate()
        self._cap = 22 * max_rows + 64 + len(model.windows) * (self.n_pages + max_rows)
        cuda = self.dev.type == "cuda"
        self._host = torch.zeros((self._cap,), dtype=torch.int32, pin_memory=cuda)
        self._np = self._host.numpy()
        self._meta = torch.zeros((self._cap,), dtype=torch.int32, device=self.dev)
        self._iota = torch.arange(max_rows, dtype=torch.int32, device=self.dev)
        self._ones = torch.ones((max_rows,), dtype=torch.int32, device=self.dev)
        self.best_val = torch.zeros((max_rows,), dtype=torch.float32, device=self.dev)
        self.best_id = torch.zeros((max_rows,), dtype=torch.int32, device=self.dev)
        self._out = torch.zeros((max_rows,), dtype=torch.int32, pin_memory=cuda)
        self.mask: torch.Tensor | None = None
        self.logits: torch.Tensor | None = None          # of the latest step, [head rows, vocab]
        self.graphs: dict[tuple, torch.cuda.CUDAGraph] = {}
        self.launches: dict[tuple, int] = {}             # own kernels per captured step
        self._event = torch.cuda.Event() if cuda else None
        self.tap_layers: list | None = None              # set to []: collects the residual after every layer run (no graphs)

    # ---- lanes ------------------------------------------------------------------------------------------------------
    def release_lane(self, lane: int) -> None:
        """Give back everything a finished sequence holds."""
        self.kv.truncate(lane, 0)
        self.state.reset(lane)

    def trim_lanes(self, rows_held: list[int]) -> None:
        """Follow the scheduler's book: lanes keep the pages of the rows it says they hold."""
        for lane, rows in enumerate(rows_held):
            if rows == 0 and self.state.rows(lane):
                self.release_lane(lane)
            else:
                self.kv.truncate(lane, rows)

    # ---- staging ----------------------------------------------------------------------------------------------------
    def _segments(self, tokens, lanes, positions):
        """[(lane, first position, tokens, first input row)] of a step, checked."""
        segs, i, n, seen = [], 0, len(tokens), set()
        if not 0 < n <= self.max_rows:
            raise ValueError(f"rows {n} out of range 1..{self.max_rows}")
        while i < n:
            lane, p0, j = lanes[i], positions[i], i + 1
            while j < n and lanes[j] == lane:
                if positions[j] != positions[j - 1] + 1:
                    raise ValueError(f"lane {lane}: the rows of a step must be consecutive positions")
                j += 1
            if lane in seen or not 0 <= lane < self.max_lanes:
                raise ValueError(f"lane {lane} out of range, or its rows are not together")
            if p0 < 0 or positions[j - 1] >= self.max_context:
                raise ValueError(f"position {positions[j - 1]} beyond the context of {self.max_context}")
            seen.add(lane)
            segs.append((lane, p0, list(tokens[i:j]), i))
            i = j
        bad = [t for t in tokens if not 0 <= t < self.model.vocab]
        if bad:
            raise ValueError(f"token {bad[0]} outside the vocabulary of {self.model.vocab}")
        return segs

    def _stage(self, segs, advs, heads, temps, seeds):
        """Fill the pinned index buffer, copy it to the device once, and return the Step over it."""
        s, at, views = Step(), 0, {}

        def put(name, values, words=1):
            nonlocal at
            m = len(values)
            self._np[at:at + m] = values
            views[name] = (at, m)
            at += m
        rows_tok, rows_pos, rows_lane, rows_seg, row0, length, back = [], [], [], [], [], [], []
        for k, ((lane, p0, toks, first), adv) in enumerate(zip(segs, advs)):
            run = adv.replay + toks
            row0.append(len(rows_tok)); length.append(len(run))
            rows_tok += run
            rows_pos += range(adv.start, adv.start + len(run))
            rows_lane += [lane] * len(run)
            rows_seg += [k] * len(run)
            back += range(row0[-1] + len(adv.replay), len(rows_tok))       # device row of every input row, in input order
        n = len(rows_tok)
        if n > self.max_rows:
            raise ValueError(f"{n} rows with the ones to run again, at most {self.max_rows}")
        s.n, s.nseg, s.single, model = n, len(segs), len(segs) == n, self.model
        s.nlong, s.nchunks, s.nshort, s.expand = 0, 0, len(segs), {}
        hrows = [back[i] for i in heads]
        s.nhead = len(hrows)
        all_heads = hrows == list(range(n))
        put("seed", [w for i in heads for w in _words(seeds[i] if seeds is not None else 0)])      # first: 8-byte aligned
        put("temp", [_float_bits(temps[i]) if temps is not None else 0 for i in heads])
        put("hpos", [rows_pos[r] for r in hrows])
        put("tokens", rows_tok); put("row_pos", rows_pos); put("row_lane", rows_lane)
        put("seg_src", [a.src for a in advs]); put("seg_dst", [a.dst for a in advs])
        if not all_heads:
            put("head_rows", hrows)
        s.max_pos = max(rows_pos)
        if s.single:
            s.short, s.ntiles, s.chunks, s.summaries = n, 0, n, 0
        else:
            put("row_seg", rows_seg); put("seg_row0", row0); put("seg_len", length)
            cs, cr, cn, cf = [], [], [], []
            for k in range(len(segs)):
                f = len(cs)
                for r in range(0, length[k], self.chunk_rows):
                    cs.append(k); cr.append(row0[k] + r); cn.append(min(self.chunk_rows, length[k] - r)); cf.append(f)
            put("chunk_seg", cs); put("chunk_row0", cr); put("chunk_rows", cn); put("chunk_first", cf)
            s.chunks, s.summaries = len(cs), int(len(cs) > len(segs))
            short, tiles = [], []
            for k in range(len(segs)):
                if model.tc_attention and length[k] >= TC_MIN_ROWS:
                    tiles += [(rows_pos[row0[k] + r], row0[k] + r, min(TC_TILE, length[k] - r)) for r in range(0, length[k], TC_TILE)]
                else:
                    short += range(row0[k], row0[k] + length[k])
            tiles.sort(reverse=True)           # most keys first: the short blocks fill the tail of the launch
            s.short, s.ntiles = len(short), len(tiles)
            put("tiles", [x for _, r, m in tiles for x in (r, m)])
            if tiles:
                put("short_rows", short)
            if model.windows and tiles:
                for w in model.windows:
                    pages, base = [], {}
                    for k in range(len(segs)):
                        if length[k] >= TC_MIN_ROWS:
                            p0 = rows_pos[row0[k]]
                            lo, hi = max(0, p0 - w + 1) // PAGE, (p0 + length[k] - 1) // PAGE + 1
                            base[k] = len(pages) - lo
                            pages += self.kv.pages[segs[k][0]][lo:hi]
                    put(f"pages{w}", pages)
                    put(f"offs{w}", [base[rows_seg[r]] for _, r, _ in tiles])
            if model.tc_state:
                long = [k for k in range(len(segs)) if length[k] >= TC_MIN_ROWS]
                put("short_segs", [k for k in range(len(segs)) if length[k] < TC_MIN_ROWS])
                chunks, first = [], []
                for k in long:
                    first.append(len(chunks))
                    chunks += [(row0[k] + r, min(STATE_CHUNK, length[k] - r)) for r in range(0, length[k], STATE_CHUNK)]
                put("long_seg", long); put("long_first", first + [len(chunks)])
                put("long_row0", [c[0] for c in chunks]); put("long_rows", [c[1] for c in chunks])
                s.nlong, s.nchunks, s.nshort = len(long), len(chunks), len(segs) - len(long)
        self._meta[:at].copy_(self._host[:at], non_blocking=True)
        self.kv.upload()
        if self._event is not None:
            self._event.record()
        for name, (a, m) in views.items():
            setattr(s, name, self._meta[a:a + m])
        if s.single:
            s.row_seg = s.seg_row0 = s.chunk_seg = s.chunk_row0 = s.chunk_first = self._iota[:n]
            s.seg_len = s.chunk_rows = self._ones[:n]
        if "short_rows" not in views:
            s.short_rows = None
        if "short_segs" not in views:
            s.short_segs = None
        s.expand = {w: (getattr(s, f"pages{w}"), views[f"pages{w}"][1], getattr(s, f"offs{w}")) for w in model.windows if f"pages{w}" in views}
        if all_heads:
            s.head_rows = None
        s.seed, s.temp = s.seed.view(torch.int64), s.temp.view(torch.float32)
        s.table, s.status, s.scratch = self.kv.table, self.status, self.scratch
        s.pages = _bucket(s.max_pos // PAGE + 1)
        s.taps = self.tap_layers
        return s

    # ---- the step ---------------------------------------------------------------------------------------------------
    def step(self, tokens, lanes, positions, temperature=None, seeds=None, sync: bool = True, masks: dict | None = None,
             filters: dict | None = None, head: bool | str | list = True, sample: bool = True):
        """Run one rows step.  ``head``: True (every row), "last" (the last row), False (none: a portion of a prompt that is not
        sampled) or a list of rows.  Returns the next token of every row (rows without a head: 0) as a host tensor when
        ``sync`` and ``sample``; the logits of the head rows are ``self.logits``, in the order asked."""
        n = len(tokens)
        if self._event is not None:
            self._event.synchronize()         # the previous step's copies have left the pinned buffers
        segs = self._segments(tokens, lanes, positions)
        heads = list(range(n)) if head is True else [] if head is False else [n - 1] if head == "last" else list(head)
        advs = [self.state.plan(lane, p0) for lane, p0, _, _ in segs]
        for (lane, p0, toks, _), adv in zip(segs, advs):
            self.kv.ensure(lane, p0 + len(toks))
        s = self._stage(segs, advs, heads, temperature, seeds)
        mask = self._stage_masks(masks, heads) if masks else None
        if s.single and heads == list(range(n)) and self.use_graphs and mask is None and self.tap_layers is None:
            self._replay(s, sample)
        else:
            self._run(s, sample, mask)
        for (lane, p0, toks, _), adv in zip(segs, advs):
            self.state.commit(adv, adv.replay + toks)
        if not sample or not heads or not sync:
            return self.best_id[:len(heads)] if sample and heads else None if not sync else torch.zeros((n,), dtype=torch.int32)
        self._out[:len(heads)].copy_(self.best_id[:len(heads)], non_blocking=True)
        torch.cuda.current_stream().synchronize()
        out = torch.zeros((n,), dtype=torch.int32)
        out[heads] = self._out[:len(heads)]
        for r, (top_k, top_p) in (filters or {}).items():
            k = heads.index(r)
            lg = self.logits[k] if mask is None else self.logits[k].masked_fill(mask[k] == 0, float("-inf"))
            out[r] = candidate_choice(lg, 0, 1, top_k, top_p, float(temperature[r]), int(seeds[r]) if seeds is not None else 0, positions[r])
        return out

    def _run(self, s: Step, sample: bool = True, mask=None) -> None:
        with R.exact_matmul():
            self.logits = self.model.forward(s)
        if sample and s.nhead:
            R.sample(self.logits, s.hpos, s.temp, s.seed, mask, self.best_val, self.best_id, s.nhead)

    def _replay(self, s: Step, sample: bool) -> None:
        """Decode steps: one CUDA graph per (rows, context bucket).  The index buffer is packed the same way for the same row
        count, and a repeated step writes what it wrote before, so the warm-up run, the capture and the replay agree."""
        key = (s.n, s.pages, sample)
        g = self.graphs.get(key)
        if g is None:
            from ..runtime.segments import recording
            with recording() as log:
                self._run(s, sample)
            self.launches[key] = sum(x not in ("linear", "block_gates", "head") for x in log.items)
            torch.cuda.current_stream().synchronize()
            g, collecting = torch.cuda.CUDAGraph(), gc.isenabled()
            gc.disable()                  # the collector may not release another engine's graphs while this one is captured
            try:
                with torch.cuda.graph(g):
                    self._run(s, sample)
            finally:
                if collecting:
                    gc.enable()
            self.graphs[key] = g
        self.logits = self.scratch.get("logits", s.n, self.model.vocab)
        g.replay()

    def _stage_masks(self, masks: dict, heads: list[int]):
        import numpy as np
        V = self.model.vocab
        if self.mask is None or self.mask.shape[0] < len(heads):
            self.mask = torch.ones((max(len(heads), self.max_lanes), V), dtype=torch.uint8, device=self.dev)
        self.mask[:len(heads)] = 1
        for r, words in masks.items():
            if r in heads:
                bits = np.unpackbits(np.asarray(words, dtype=np.uint64).view(np.uint8), bitorder="little")[:V]
                self.mask[heads.index(r)].copy_(torch.from_numpy(bits))
        return self.mask[:len(heads)]

    # ---- conveniences of the engine contract ------------------------------------------------------------------------
    def vocab_slice(self) -> tuple[int, int]:
        return 0, self.model.vocab

    def check_status(self) -> None:
        st = self.status.tolist()
        if st[0] != 0:
            raise RuntimeError(f"device status code={st[0]} where={st[1]} detail=({st[2]}, {st[3]})")

    def nbytes(self) -> dict:
        return {"weights": self.model.nbytes(), "kv": self.kv.nbytes(), "state": self.state.nbytes(), "scratch": self.scratch.nbytes()}

    def close(self) -> None:
        torch.cuda.synchronize()
        self.graphs.clear()

    def short_rows(self, tc: bool) -> int:
        """Most rows of a step that do not go to the tensor-core arm."""
        return self.max_lanes * TC_MIN_ROWS if tc else self.max_rows

    def state_chunks(self) -> int:
        """Most chunks of the tensor-core recurrence in a step: a run's last one may be short."""
        return self.max_rows // STATE_CHUNK + min(self.max_lanes, max(1, self.max_rows // TC_MIN_ROWS))

    def expanded_rows(self, window: int) -> int:
        """Most positions whose keys the long runs of a step need: their own and a window before each run, in whole pages."""
        runs = min(self.max_lanes, max(1, self.max_rows // TC_MIN_ROWS))
        return PAGE * min(self.n_pages, self.max_rows // PAGE + runs * (window // PAGE + 3))

    def splits(self, s: Step, rows: int, blocks_per_row: int, window: int = 2 ** 31 - 1) -> int:
        """Ranges a row's pages are cut into so that ``rows`` single rows fill the machine."""
        return max(1, min(s.pages, window // PAGE + 2, MAX_SPLITS, TARGET_BLOCKS // max(1, rows * blocks_per_row)))

    def generate(self, prompt: list[int], n_new: int, lane: int = 0, temperature: float = 0.0, seed: int = 0, chunk: int | None = None):
        """Prefill ``prompt`` in portions of ``chunk`` rows, then decode ``n_new`` tokens one row at a time."""
        chunk, pos, out = chunk or self.max_rows, 0, []
        while pos < len(prompt):
            c = prompt[pos:pos + chunk]
            r = self.step(c, [lane] * len(c), list(range(pos, pos + len(c))), [temperature] * len(c), [seed] * len(c),
                          head="last" if pos + len(c) >= len(prompt) else False)
            pos += len(c)
        nxt = int(r[-1])
        for _ in range(n_new):
            out.append(nxt)
            if len(out) == n_new:
                break
            nxt = int(self.step([nxt], [lane], [pos], [temperature], [seed])[0])
            pos += 1
        self.check_status()
        return out


def _bucket(n: int) -> int:
    b = 16
    while b < n:
        b *= 2
    return b


def _words(seed: int) -> tuple[int, int]:
    seed &= 0xFFFFFFFFFFFFFFFF
    lo, hi = seed & 0xFFFFFFFF, seed >> 32
    return (lo - (1 << 32) if lo >> 31 else lo, hi - (1 << 32) if hi >> 31 else hi)


def _float_bits(x: float) -> int:
    import struct
    return struct.unpack("<i", struct.pack("<f", x))[0]
