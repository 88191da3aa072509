"""Fanodra on the layered engine: whole prompts, portions, decoding, mixed batches, reused pages and slots, generation through the
scheduler, rejected draft rows, and the trace replay, against the plain implementation of tests/oracles/plain_fanodra.py."""
import functools
import io
import json
import random
import types

import pytest
import torch

from oracles import plain_fanodra as P
from sparkflash_b200.models.fanodra import Fanodra, FanodraConfig
from sparkflash_b200.models.layered import LayeredEngine

pytestmark = pytest.mark.gpu

CONFIGS = {
    # grouped heads, unequal head sizes, a loop in the middle, a layer without feed-forward
    "mid": P.make_config(203, 96, 4, [("rglru", P.recurrent(72, 2, 5), 64), ("parallel", P.attending(4, 2, 40, 24, 0.3), P.recurrent(60, 3, 2), 56),
                                      ("rglru", P.recurrent(96, 1, 3), None), ("parallel", P.attending(2, 1, 16, 32, 0.1), P.recurrent(48, 4, 4), None)],
                         loop=(1, 3, 3)),
    # no loop; odd sizes everywhere: no vector loads, no tensor-core attention
    "odd": P.make_config(61, 37, 2, [("parallel", P.attending(3, 3, 10, 7, 0.5), P.recurrent(15, 5, 1), 19), ("rglru", P.recurrent(22, 2, 7), 11)],
                         eps=1e-3),
    # loop over everything, once; single tap
    "once": P.make_config(128, 64, 1, [("parallel", P.attending(4, 1, 64, 64, 0.125), P.recurrent(64, 2, 4), 128), ("rglru", P.recurrent(64, 1, 4), 64)],
                          loop=(0, 2, 1)),
    "loops": P.make_config(90, 80, 3, [("rglru", P.recurrent(40, 1, 2), 48), ("parallel", P.attending(5, 5, 24, 48, 0.2), P.recurrent(32, 2, 3), 40)],
                           loop=(1, 2, 4)),
}
# recurrence only: no attention anywhere; the first layer looped, the same state shapes in every pass
CONFIGS["rec"] = P.make_config(97, 48, 4, [("rglru", P.recurrent(56, 7, 4), None), ("rglru", P.recurrent(32, 1, 8), 36)], loop=(0, 1, 3))
CONFIGS["gen"] = CONFIGS["loops"]       # for greedy decoding: no constant directions in the residual, so that the text varies
CONFIGS["far"] = CONFIGS["mid"]         # for far keys: sharp scores and hardly any distance bias
TOL = {torch.float32: 2e-4, torch.bfloat16: 0.12}      # rms of the logits' difference over the logits' spread


@functools.lru_cache(None)
def weights(name):
    w = P.make_weights(CONFIGS[name], seed=len(name))
    if name == "gen":
        for k in w:
            if k.endswith(".b") and "norm" in k or k.startswith("loop"):
                w[k] = torch.zeros_like(w[k])
        w["embed"] = w["embed"] * 0.25
    if name == "far":
        for k in w:
            if k.endswith(".q.norm"):
                w[k] = w[k] * 2
            if k.endswith(".r1"):
                w[k] = w[k] * 0.02
    return w


@functools.lru_cache(None)
def tokens(name, n, seed=0):
    return tuple(torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist())


@functools.lru_cache(None)
def expected(name, toks):
    return P.forward(weights(name), CONFIGS[name], list(toks), torch.float64).float()


def engine(name, dt=torch.float32, **kw):
    kw = {"max_context": 640, "max_rows": 640, **kw}
    return LayeredEngine(Fanodra(FanodraConfig.from_dict(CONFIGS[name]), weights(name), dt, max_context=kw["max_context"]), **kw)


def error(got, want):
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.std(-1).mean()).max().item()


def feed(eng, lane, toks, at, cuts):
    """Run tokens in portions; logits of every row."""
    out = []
    for c in cuts:
        part = toks[at:at + c]
        eng.step(part, [lane] * len(part), list(range(at, at + len(part))), sample=False)
        out.append(eng.logits.cpu())
        at += len(part)
    eng.check_status()
    return torch.cat(out)


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", ["mid", "odd", "once", "loops", "rec"])
def test_whole_prompt_and_layers(name, dt):
    toks = tokens(name, 333)
    eng = engine(name, dt)
    taps, eng.tap_layers = [], []
    P.forward(weights(name), CONFIGS[name], list(toks[:30]), torch.float64, taps)
    eng.step(toks[:30], [1] * 30, list(range(30)))
    assert len(taps) == len(eng.tap_layers) == len(eng.model.order)
    for i, (a, b) in enumerate(zip(eng.tap_layers, taps)):
        assert (a.cpu() - b.float()).abs().max() < (1e-4 if dt == torch.float32 else 0.5), (i, (a.cpu() - b.float()).abs().max())
    eng.tap_layers = None
    assert error(feed(eng, 0, toks, 0, [333]), expected(name, toks)) < TOL[dt]


@pytest.mark.parametrize("name", ["mid", "odd", "once", "loops", "rec"])
def test_portions_and_token_by_token_match_the_whole(name):
    toks = tokens(name, 200)
    want = expected(name, toks)
    for dt in TOL:
        eng = engine(name, dt)
        whole = feed(eng, 0, toks, 0, [200])
        ref = want if dt == torch.float32 else whole
        for lane, cuts in enumerate(([2] * 100, [1] * 200, [64, 64, 64, 8], [3, 61, 1, 65, 33, 2, 2, 32, 1])):
            got = feed(eng, lane, toks, 0, cuts)
            assert error(got, ref) < (2e-4 if dt == torch.float32 else 0.08), (dt, cuts[:4], error(got, ref))
            assert error(got, want) < TOL[dt]


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("n,key", [(300, 0), (300, 1), (300, 63), (300, 64), (257, 128), (321, 255)])
def test_a_far_token_reaches_prompt_and_decoded_rows(n, key, dt):
    """One token changed long before the row: the change of the logits is the plain implementation's, in a portion and decoded."""
    a = list(tokens("far", n))
    b = list(a)
    b[key] = (b[key] + 17) % 203
    eng = engine("far", dt)
    want = expected("far", tuple(b))[-1] - expected("far", tuple(a))[-1]
    for cuts in ([n], [n - 40] + [1] * 40, [50, n - 52, 2]):
        got = feed(eng, 0, b, 0, cuts)[-1] - feed(eng, 1, a, 0, cuts)[-1]
        rel = ((got - want).pow(2).mean() / want.pow(2).mean()).sqrt().item()
        assert rel < (0.02 if dt == torch.float32 else 0.6), (cuts[:2], rel, want.pow(2).mean().sqrt())


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", ["mid", "odd"])
def test_mixed_batches_with_reused_pages_and_slots(name, dt):
    """Random schedules over a pool too small for the sum of the requests: portions beside single tokens, requests that pause,
    finish and make room for others; every position's logits match the request alone."""
    rng = random.Random(5)
    eng = engine(name, dt, max_lanes=3, pool_tokens=512)
    todo = [(tokens(name, n, s), s) for s, n in enumerate((150, 90, 1, 64, 65, 127, 40, 128, 33, 2))]
    live, worst, reused, seen = {}, 0.0, 0, set()
    while todo or live:
        for lane in range(3):
            if lane not in live and todo and rng.random() < 0.8:
                live[lane] = [todo.pop(0)[0], 0]
        if not live:
            continue
        rows, who = [], []
        for lane, (toks, at) in live.items():
            if rng.random() < 0.2 and len(live) > 1:
                continue                                        # left out of this step
            n = min(len(toks) - at, rng.choice([1, 1, 1, 2, 3, 17, 40, 64, 70]))
            rows += [(toks[at + i], lane, at + i) for i in range(n)]
            who.append((lane, at, n))
        if not rows:
            continue
        eng.step(*map(list, zip(*rows)), sample=False)
        got = eng.logits.split([n for _, _, n in who])
        for (lane, at, n), g in zip(who, got):
            worst = max(worst, error(g, expected(name, live[lane][0])[at:at + n]))
            live[lane][1] += n
            pages = set(eng.kv.pages[lane])
            if live[lane][1] == len(live[lane][0]):
                reused += len(pages & seen)
                seen |= pages
                eng.release_lane(lane)
                del live[lane]
    eng.check_status()
    assert worst < TOL[dt] and reused > 4 and eng.kv.free_pages == eng.n_pages


@pytest.mark.parametrize("dt", list(TOL))
def test_long_decoding_crosses_pages_and_graph_buckets(dt):
    toks = tokens("mid", 420)
    eng = engine("mid", dt)
    got = feed(eng, 2, toks, 0, [50] + [1] * 370)
    assert error(got, expected("mid", toks)) < TOL[dt]
    assert len(eng.graphs) >= 1


@pytest.mark.parametrize("rows", [3, 20])
def test_batched_decoding_matches_each_alone(rows):
    """Few single rows take the fused recurrence kernel, many the separate ones; both through captured steps."""
    eng = engine("mid", max_lanes=rows, max_context=128, max_rows=256)
    reqs = [tokens("mid", 40 + s % 7, s) for s in range(rows)]
    for s, t in enumerate(reqs):
        eng.step(t[:20], [s] * 20, list(range(20)), head=False)
    for p in range(20, 40):
        eng.step([t[p] for t in reqs], list(range(rows)), [p] * rows, sample=False)
        for s in (0, 1, rows - 1):
            assert error(eng.logits[s:s + 1], expected("mid", reqs[s])[p:p + 1]) < 2e-4
    eng.check_status()


def greedy(name, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(P.forward(weights(name), CONFIGS[name], toks, torch.float64)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    from sparkflash_b200.serve.driver import generate_all
    prompts = [list(tokens("gen", n, s)) for s, n in enumerate((9, 30, 1, 17, 5))]
    want = [greedy("gen", p, 8) for p in prompts]
    # two lanes and a pool of three pages for five requests: they wait for lanes and pages, and get them again
    eng = engine("gen", max_lanes=2, max_context=128, max_rows=16, pool_tokens=192)
    assert generate_all(eng, prompts, 8) == want
    assert eng.generate(prompts[1], 8, chunk=7) == want[1]
    sampled = generate_all(eng, prompts[:2], 8, temperature=0.8, seed=3)
    assert sampled == [generate_all(eng, [p], 8, temperature=0.8, seed=3)[0] for p in prompts[:2]]      # keyed on (seed, position)


def test_a_reused_prefix_continues_from_the_lane_state():
    import asyncio
    from sparkflash_b200.serve.driver import DeviceDriver, _IdTokenizer
    from sparkflash_b200.serve.engine_api import EngineRequest
    eng = engine("gen", max_lanes=1, max_context=256, max_rows=64)
    drv = DeviceDriver(eng, _IdTokenizer(), prefix_reuse_min=8).start()

    async def ask(prompt, n):
        return [e[1] async for e in drv.generate(EngineRequest("r", "m", list(prompt), max_tokens=n, temperature=0.0)) if e[0] == "token"]
    try:
        p = list(tokens("gen", 40))
        first = asyncio.run(ask(p, 6))
        longer = p + first[:5] + [3, 4, 5]                       # the lane holds exactly p + first[:5]
        assert asyncio.run(ask(longer, 5)) == greedy("gen", longer, 5)
        assert drv.stats()["prefix_hits"] == 1
        shorter = p[:20] + [1]                                   # a state cannot be rewound: computed from the start
        assert asyncio.run(ask(shorter, 5)) == greedy("gen", shorter, 5)
        assert drv.stats()["prefix_hits"] == 1
    finally:
        drv.shutdown(1.0)


def test_rejected_draft_rows_leave_no_trace():
    """A drafter that is mostly wrong: the output stays the model's own, because a state is run again from before the step."""
    from sparkflash_b200.serve.driver import generate_all

    class Drafter:
        depth = 3

        def __init__(self, right):
            self.right, self.k = right, 0

        def propose(self, history):
            self.k += 1
            at = len(history) - 12
            good = self.right[at:at + 3]
            return (good[:self.k % 4] + [7, 7, 7])[:3], [1.0] * 3
    prompt = list(tokens("gen", 12))
    want = greedy("gen", prompt, 20)
    eng = engine("gen", max_lanes=2, max_context=128, max_rows=32)
    assert generate_all(eng, [prompt], 20, drafter=Drafter(want)) == [want]
    with pytest.raises(ValueError, match="cannot continue"):
        eng.step([1], [0], [3])


def test_sampling_filters_and_masks():
    eng = engine("odd", max_context=64, max_rows=16)
    V = eng.model.vocab
    words = [0] * -(-V // 64)
    words[0] = 1 << 5
    assert eng.step([1, 2, 3], [0] * 3, [0, 1, 2], [0.0] * 3, [0] * 3, masks={2: words}, head="last")[2] == 5
    assert int(eng.step([4], [0], [3], [1.0], [9], filters={0: (1, 1.0)})[0]) == int(eng.logits[0].argmax())


def test_replay_writes_the_wanted_logits(tmp_path):
    from sparkflash_b200.serve import replay
    from sparkflash_b200.weights.files import write_safetensors
    cfg = {k: v for k, v in CONFIGS["mid"].items() if v is not None}
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), weights("mid"))
    a, b = tokens("mid", 90, 1), tokens("mid", 70, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:4], "want": []}, {"id": "a", "tokens": a[64:65], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:], "want": [65, 2]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[65:], "want": [24]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "c", "tokens": b, "want": []}], "end": ["c"]}]
    out = io.StringIO()
    args = types.SimpleNamespace(model=str(tmp_path), dtype="float32", out=str(tmp_path), max_tokens=256)
    assert replay.run(args, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), out) == 0
    assert out.getvalue().split("\n")[:-1] == [f"done {i}" for i in range(5)]
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 203)
    A, B = expected("mid", a), expected("mid", b)
    for i, want in ((0, A[[0, 63]]), (1, A[[64]]), (2, B[[69, 6]]), (3, A[[89]])):
        assert error(read(i), want) < 2e-4
    assert not (tmp_path / "4.f32").exists()


def test_small_engines_and_a_pool_of_one_page():
    """A portion as large as the whole engine (fewer rows than a query tile), in bf16 through the tensor-core attention."""
    toks = tokens("once", 64)
    eng = engine("once", torch.bfloat16, max_lanes=1, max_context=64, max_rows=64)
    assert error(feed(eng, 0, toks, 0, [40, 24]), expected("once", toks)) < TOL[torch.bfloat16]
    eng.release_lane(0)
    assert error(feed(eng, 0, toks, 0, [64]), expected("once", toks)) < TOL[torch.bfloat16]
    with pytest.raises(ValueError, match="beyond the context"):
        eng.step([1], [0], [64])
    with pytest.raises(ValueError, match="vocabulary"):
        eng.step([128], [0], [0])


def test_command_line_and_serving_builders(tmp_path, capsys):
    import asyncio
    from sparkflash_b200 import cli
    from sparkflash_b200.config import Settings
    from sparkflash_b200.serve import launch
    from sparkflash_b200.serve.driver import DeviceDriver
    from sparkflash_b200.serve.engine_api import ApiError, EngineRequest
    from sparkflash_b200.serve.tokenizer import load_tokenizer
    from sparkflash_b200.weights.files import write_safetensors
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["gen"]))
    write_safetensors(str(tmp_path / "model.safetensors"), weights("gen"))
    a, b = list(tokens("gen", 9)), list(tokens("gen", 14, 1))
    assert cli.main(["generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "6", "--max-context", "128", "--max-rows", "64",
                     "--tokens", ",".join(map(str, a)), "--tokens", ",".join(map(str, b))]) == 0
    got = [json.loads(x)["tokens"] for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert got == [greedy("gen", a, 6), greedy("gen", b, 6)]
    st = Settings()
    st.engine.max_lanes = 2
    args = types.SimpleNamespace(model=str(tmp_path), dtype="float32", max_context=128, pool_tokens=256, weights=None, synthetic=None)
    eng = launch.build_engine(args, st, 0, 1)
    tok = load_tokenizer(None, eng.cfg.vocab_size)
    drv = DeviceDriver(eng, tok, model_id="m", eos_id=-1).start()
    try:
        with pytest.raises(ApiError):
            drv.validate(EngineRequest("x", "m", [eng.vocab], max_tokens=4))

        async def ask():
            return [e[1] async for e in drv.generate(EngineRequest("r", "m", a, max_tokens=6, temperature=0.0)) if e[0] == "token"]
        assert asyncio.run(ask()) == greedy("gen", a, 6)
    finally:
        drv.shutdown(1.0)
