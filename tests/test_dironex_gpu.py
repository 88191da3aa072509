"""Dironex on the layered engine: whole prompts, portions, decoding, mixed batches, reused pages and slots, window edges and far keys, generation
through the scheduler, rejected draft rows and the trace replay, against the plain implementation of tests/oracles/plain_dironex.py."""
import functools
import io
import json
import random
import types

import pytest
import torch

from oracles import plain_dironex as P
from sparkflash_b200.models.dironex import Dironex, DironexConfig
from sparkflash_b200.models.layered import LayeredEngine

pytestmark = pytest.mark.gpu

CONFIGS = {
    # no size in common: groups, a looped middle, layers with and without a feed-forward, a latent layer beyond the tensor-core arms
    "mix": P.make_config(203, 96, 2, 3, 0.6, 1.7, [
        P.windowed(4, 2, 24, 16, 50, 0.25, P.moe(12, 3, 40, 4, 2, 1.4)), P.latent(3, 20, 12, 24, 40, 28, 0.2, 700.0, (4.0, 128, 16.0, 1.0), P.ff(72)),
        P.latent(5, 16, 8, 40, 24, 56, 0.25, 1e4), P.windowed(6, 3, 16, 24, 21, 0.3, P.moe(6, 2, 56, 2, 2, 0.8)), P.windowed(2, 1, 32, 8, 300, 0.2, P.ff(40))],
        loop=(1, 3, 2)),
    # everything on the tensor-core arms
    "tc": P.make_config(128, 128, 4, 4, 0.8, 1.0, [
        P.latent(4, 64, 32, 64, 64, 48, 0.12, 1e5, (8.0, 64, 32.0, 1.0), P.moe(16, 4, 72, 4, 2, 1.0)), P.windowed(4, 2, 32, 64, 70, 0.2, P.ff(136)),
        P.latent(18, 40, 16, 24, 128, 72, 0.15, 2e4, (2.0, 256, 8.0, 2.0), P.ff(64)), P.windowed(8, 2, 64, 32, 200, 0.15, P.moe(8, 2, 24, 2, 1, 2.0)),
        P.windowed(4, 1, 96, 64, 33, 0.12, P.ff(48))], loop=(0, 2, 2), eps=1e-6),
    # odd sizes everywhere: no vector loads, no tensor-core arms, a single tap, a window of one, many streams
    "odd": P.make_config(61, 37, 5, 1, 0.9, 3.0, [
        P.windowed(3, 1, 5, 7, 9, 0.5, P.moe(9, 2, 11, 3, 1, 1.1)), P.latent(2, 7, 2, 5, 13, 9, 0.4, 30.0, (2.0, 30, 3.0, 0.4), P.ff(15)), P.windowed(2, 2, 6, 3, 1, 0.5),
        P.latent(3, 3, 6, 9, 11, 5, 0.4, 20.0, None, P.moe(5, 5, 7, 1, 1, 0.7))], loop=(3, 4, 3), eps=1e-3),
    # one stream, no loop, every row uses every expert, so that bf16 turns no choice over; tensor-core arms
    "full": P.make_config(112, 96, 1, 5, 0.75, 0.8, [
        P.latent(2, 48, 24, 56, 80, 40, 0.15, 3e3, (8.0, 96, 16.0, 2.0), P.moe(4, 4, 56, 2, 2, 1.5)), P.windowed(6, 2, 48, 32, 90, 0.2, P.ff(120)),
        P.latent(6, 32, 8, 32, 48, 64, 0.2, 500.0, None, P.moe(3, 3, 40, 1, 1, 0.9))]),
    # windowed attention only, no carried convolution inputs: a token's reach is the window
    "win": P.make_config(90, 64, 3, 1, 1.0, 1.0, [P.windowed(6, 2, 32, 32, 100, 0.5, P.ff(96))]),
    # latent attention only
    "lat": P.make_config(97, 64, 3, 2, 0.7, 1.0, [P.latent(4, 32, 16, 32, 64, 32, 0.3, 1e3, (4.0, 100, 8.0, 1.0), P.ff(64)), P.latent(2, 24, 8, 16, 40, 24, 0.3, 100.0)]),
}
NAMES = list(CONFIGS)
CLOSE = {torch.float32: 2e-6, torch.bfloat16: 0.05}    # choice scores closer than this may swap
TOL = {torch.float32: 5e-5, torch.bfloat16: 0.08}      # rms of the logits' difference over the logits' spread


@functools.lru_cache(None)
def weights(name, dt=torch.float32):
    """In bf16 the experts' corrections lie far apart: a choice turned over would change its row and, through the convolutions, the next ones."""
    return P.make_weights(CONFIGS[name], seed=14 + len(name), spread=dt == torch.bfloat16)


@functools.lru_cache(None)
def tokens(name, n, seed=0):
    return tuple(torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist())


@functools.lru_cache(None)
def expected(name, toks, dt=torch.float32):
    margins = []
    out = P.forward(CONFIGS[name], weights(name, dt), list(toks), margins=margins).float()
    assert not margins or torch.stack(margins).min() > CLOSE[dt]
    return out


def engine(name, dt=torch.float32, **kw):
    kw = {"max_context": 640, "max_rows": 640, **kw}
    return LayeredEngine(Dironex(DironexConfig.from_dict(CONFIGS[name]), weights(name, dt), dt, max_context=kw["max_context"]), **kw)


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
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt_and_layers(name, dt):
    toks = tokens(name, 333)
    eng = engine(name, dt)
    assert eng.model.tc_attention == (dt == torch.bfloat16 and name != "odd")
    taps, eng.tap_layers = [], []
    P.forward(CONFIGS[name], weights(name, dt), list(toks[:40]), taps)
    eng.step(toks[:40], [1] * 40, list(range(40)))
    assert len(taps) == len(eng.tap_layers) == len(P.order(CONFIGS[name]))
    for i, (a, b) in enumerate(zip(eng.tap_layers, taps)):
        off = (a.cpu() - b.float()).pow(2).mean().sqrt() / b.float().pow(2).mean().sqrt()
        assert off < (1e-5 if dt == torch.float32 else 0.05), (i, off)
    eng.tap_layers = None
    assert error(feed(eng, 0, toks, 0, [333]), expected(name, toks, dt)) < TOL[dt]


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", NAMES)
def test_portions_and_token_by_token_match_the_whole(name, dt):
    toks = tokens(name, 200)
    want = expected(name, toks, dt)
    eng = engine(name, dt)
    whole = feed(eng, 0, toks, 0, [200])
    ref = want if dt == torch.float32 else whole
    for lane, cuts in enumerate(([2] * 100, [1] * 200, [64, 64, 64, 8], [3, 61, 1, 65, 33, 2, 2, 32, 1])):
        got = feed(eng, lane, toks, 0, cuts)
        assert error(got, ref) < TOL[dt], (cuts[:4], error(got, ref))
        assert error(got, want) < TOL[dt]


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("key", [0, 63, 64, 99])
def test_a_token_reaches_its_windows_last_row_and_not_the_next(key, dt):
    """Windowed attention is the only mixer: a changed token changes the rows up to window - 1 behind it, in a portion and decoded, and no other."""
    n, window = key + 108, CONFIGS["win"]["layers"][0]["mixer"]["mask"]["size"]
    a = list(tokens("win", n))
    b = list(a)
    b[key] = (b[key] + 7) % 90
    want = expected("win", tuple(b)) - expected("win", tuple(a))
    eng = engine("win", dt)
    last = key + window - 1
    assert (want[last].abs().max() > 1e-4) and (want[last + 1:] == 0).all()
    for cuts in ([n], [last - 40] + [1] * (n - last + 40) if last > 40 else [1] * n, [last, 2, n - last - 2], [last + 1, n - last - 1]):
        got = feed(eng, 0, b, 0, cuts) - feed(eng, 1, a, 0, cuts)
        assert (got[:key] == 0).all() and (got[last + 1:] == 0).all() and got[last].abs().max() > 0, cuts[:2]
        if dt == torch.float32:
            assert (got - want).abs().max() < 1e-3 * want.abs().max()


@functools.lru_cache(None)
def sharp_weights():
    """Latent attention whose first layer looks for one key: position 0's token (number 1, which no other position has) stands out in the latent,
    every query asks for it, and its value is large."""
    w = {k: v.clone() for k, v in weights("lat").items()}
    m = CONFIGS["lat"]["layers"][0]["mixer"]
    w["embed"][1] = 0
    w["embed"][1, 0] = 8.0
    w["embed"][:, 0] = torch.where(torch.arange(97) == 1, 8.0, 0.0).to(torch.bfloat16)
    w["embed"][:, 1] = 3.0                                # the same in every token
    q = "l0.mix."
    w["l0.canon1"].zero_()
    w[q + "uv"] *= 4
    w[q + "g"].zero_()
    for n in ("dq", "dkv", "uq", "uk"):
        w[q + n] *= 0.2
    w[q + "dkv"][0], w[q + "dq"][0] = 0, 0
    w[q + "dkv"][0, 0], w[q + "dq"][0, 1] = 4.0, 4.0      # latent 0: the token's mark; the queries' latent 0: on everywhere
    uk, uq = w[q + "uk"].view(m["heads"], m["dim"], -1), w[q + "uq"].view(m["heads"], m["dim"] + m["rot_dim"], -1)
    uk[:, 0], uq[:, 0] = 0, 0
    uk[:, 0, 0], uq[:, 0, 0] = 2.0, 2.0
    return w


@pytest.mark.parametrize("dt", list(TOL))
def test_one_far_key_stands_out_in_prompts_and_decoding(dt):
    """The key at position 0 carries nearly all the weight at every distance, across pages, portions, and the blocks that decoding cuts keys into."""
    n, cfg, w = 600, CONFIGS["lat"], sharp_weights()
    a = [1] + [2 + t % 95 for t in tokens("lat", n - 1)]
    want = P.forward(cfg, w, a).float()
    without = P.forward(cfg, w, [5] + a[1:]).float()
    assert (want - without)[[1, 63, 64, 128, 400, 599]].std(-1).min() > 0.15 * want.std()
    for cuts in ([n], [63] + [1] * 70 + [n - 133], [256, 300] + [1] * 44, [40, 2, 2, 84, 129, n - 257]):
        eng = LayeredEngine(Dironex(DironexConfig.from_dict(cfg), w, dt, max_context=640), max_context=640, max_rows=640)
        assert error(feed(eng, 0, a, 0, cuts), want) < TOL[dt], cuts[:3]


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", ["mix", "tc", "odd", "full"])
def test_mixed_batches_with_reused_pages_and_slots(name, dt):
    """Random schedules over a pool too small for the sum of the requests: portions beside single tokens, requests that pause,
    finish and make room for others; every position's logits match the request alone."""
    rng = random.Random(5)
    eng = engine(name, dt, max_lanes=3, pool_tokens=512)
    todo = [tokens(name, n, s) for s, n in enumerate((150, 90, 1, 64, 65, 127, 40, 128, 33, 2))]
    live, worst, reused, seen = {}, 0.0, 0, set()
    while todo or live:
        for lane in range(3):
            if lane not in live and todo and rng.random() < 0.8:
                live[lane] = [todo.pop(0), 0]
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
        for (lane, at, n), g in zip(who, eng.logits.split([n for _, _, n in who])):
            worst = max(worst, error(g, expected(name, live[lane][0], dt)[at:at + n]))
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
@pytest.mark.parametrize("name", ["mix", "tc", "full"])
def test_long_decoding_crosses_pages_windows_and_graph_buckets(name, dt):
    toks = tokens(name, 420)
    eng = engine(name, dt)
    assert error(feed(eng, 2, toks, 0, [50] + [1] * 370), expected(name, toks, dt)) < TOL[dt]
    assert len(eng.graphs) >= 1


@pytest.mark.parametrize("rows", [3, 70])
def test_batched_decoding_matches_each_alone(rows):
    """Few single rows take the streaming products, many the separate kernels (and latent attention in slices of rows)."""
    for dt in TOL:
        eng = engine("tc", dt, max_lanes=rows, max_context=128, max_rows=256)
        reqs = [tokens("tc", 40 + s % 7, s) for s in range(rows)]
        for s, t in enumerate(reqs):
            eng.step(t[:20], [s] * 20, list(range(20)), head=False)
        for p in range(20, 40):
            eng.step([t[p] for t in reqs], list(range(rows)), [p] * rows, sample=False)
            if p % 6 == 1:
                for s in (0, 1, rows - 1):
                    assert error(eng.logits[s:s + 1], expected("tc", reqs[s], dt)[p:p + 1]) < TOL[dt]
        eng.check_status()


def test_a_request_does_not_see_what_a_slot_or_page_held_before():
    """Bit by bit: a request on fresh pages and slots, and on ones that another request has left."""
    a, b = tokens("tc", 130), tokens("tc", 200, 1)
    eng = engine("tc", torch.bfloat16, max_lanes=1, max_context=256, max_rows=256)
    cuts = [70, 33] + [1] * 27
    fresh = feed(eng, 0, a, 0, cuts)
    eng.release_lane(0)
    feed(eng, 0, b, 0, [200])
    eng.release_lane(0)
    assert torch.equal(feed(eng, 0, a, 0, cuts), fresh)


def greedy(name, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(P.forward(CONFIGS[name], weights(name), toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    from sparkflash_b200.serve.driver import generate_all
    prompts = [list(tokens("mix", n, s)) for s, n in enumerate((9, 30, 1, 17, 5))]
    want = [greedy("mix", p, 8) for p in prompts]
    # two lanes and a pool of three pages for five requests: they wait for lanes and pages, and get them again
    eng = engine("mix", max_lanes=2, max_context=128, max_rows=16, pool_tokens=192)
    assert generate_all(eng, prompts, 8) == want
    assert eng.generate(prompts[1], 8, chunk=7) == want[1]
    sampled = generate_all(eng, prompts[:2], 8, temperature=0.8, seed=3)
    assert sampled == [generate_all(eng, [p], 8, temperature=0.8, seed=3)[0] for p in prompts[:2]]      # keyed on (seed, position)


def test_rejected_draft_rows_leave_no_trace():
    """A drafter that is mostly wrong: the output stays the model's own, because the convolutions' inputs come from before the step."""
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
    prompt = list(tokens("mix", 12))
    want = greedy("mix", prompt, 16)
    eng = engine("mix", max_lanes=2, max_context=128, max_rows=32)
    assert generate_all(eng, [prompt], 16, drafter=Drafter(want)) == [want]


def test_small_engines_and_a_pool_of_one_page():
    toks, dt = tokens("full", 64), torch.bfloat16
    eng = engine("full", dt, max_lanes=1, max_context=64, max_rows=64)
    assert error(feed(eng, 0, toks, 0, [40, 24]), expected("full", toks, dt)) < TOL[dt]
    eng.release_lane(0)
    assert error(feed(eng, 0, toks, 0, [64]), expected("full", toks, dt)) < TOL[dt]
    with pytest.raises(ValueError, match="beyond the context"):
        eng.step([1], [0], [64])


def test_replay_generate_and_serving_builders(tmp_path, capsys):
    import asyncio
    from sparkflash_b200 import cli
    from sparkflash_b200.config import Settings
    from sparkflash_b200.serve import launch, replay
    from sparkflash_b200.serve.driver import DeviceDriver
    from sparkflash_b200.serve.engine_api import EngineRequest
    from sparkflash_b200.serve.tokenizer import load_tokenizer
    from sparkflash_b200.weights.files import write_safetensors
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["mix"]))
    write_safetensors(str(tmp_path / "model.safetensors"), weights("mix"))
    a, b = tokens("mix", 90, 1), tokens("mix", 70, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:4], "want": []}, {"id": "a", "tokens": a[64:65], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:], "want": [65, 2]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[65:], "want": [24]}], "end": ["a"]}]
    args = types.SimpleNamespace(model=str(tmp_path), dtype="float32", out=str(tmp_path), max_tokens=256)
    assert replay.run(args, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), io.StringIO()) == 0
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, 203)
    A, B = expected("mix", a), expected("mix", b)
    for i, want in ((0, A[[0, 63]]), (1, A[[64]]), (2, B[[69, 6]]), (3, A[[89]])):
        assert error(read(i), want) < 2e-4
    x, y = list(tokens("mix", 9)), list(tokens("mix", 14, 1))
    assert cli.main(["generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new", "6", "--max-context", "128", "--max-rows", "64",
                     "--tokens", ",".join(map(str, x)), "--tokens", ",".join(map(str, y))]) == 0
    got = [json.loads(t)["tokens"] for t in capsys.readouterr().out.splitlines() if t.startswith("{")]
    assert got == [greedy("mix", x, 6), greedy("mix", y, 6)]
    st = Settings()
    st.engine.max_lanes = 2
    eng = launch.build_engine(types.SimpleNamespace(model=str(tmp_path), dtype="float32", max_context=128, pool_tokens=256, weights=None, synthetic=None), st, 0, 1)
    drv = DeviceDriver(eng, load_tokenizer(None, eng.cfg.vocab_size), model_id="m", eos_id=-1).start()
    try:
        async def ask():
            return [e[1] async for e in drv.generate(EngineRequest("r", "m", x, max_tokens=6, temperature=0.0)) if e[0] == "token"]
        assert asyncio.run(ask()) == greedy("mix", x, 6)
    finally:
        drv.shutdown(1.0)
