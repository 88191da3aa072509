"""Lifulorn on the layered engine: whole prompts, portions, decoding, mixed batches, reused pages and slots, window edges, generation
through the scheduler, rejected draft rows and the trace replay, against the plain implementation of tests/oracles/plain_lifulorn.py."""
import functools
import io
import json
import random
import types

import pytest
import torch

from oracles import plain_lifulorn as P
from sparkflash_b200.models.lifulorn import Lifulorn, LifulornConfig
from sparkflash_b200.models.layered import LayeredEngine

pytestmark = pytest.mark.gpu

CONFIGS = {
    # no size in common: groups, partly rotated heads, layers with and without a feed-forward or mixed values
    "mix": P.make_config(203, 96, 20, 0.6, [
        P.rule(4, 2, 20, 24, 4, P.moe(7, 3, 40, 1.0, 24, 2.0)), P.attend(4, 2, 24, 16, 50, 1e4, 16, P.wave(4.0, 1.0, 4.0, 256), 0.25),
        P.attend(6, 2, 16, 16, 21, 500.0, 16, P.yarn(6.0, 200, 16.0, 1.0), 0.3, softcap=4.0, mlp=P.moe(4, 1, 56, 0.7, 16, 1.0)),
        P.rule(3, 3, 32, 8, 2), P.attend(2, 1, 32, 24, 300, 1e5, 8, P.yarn(2.0, 100, 8.0, 1.0), 0.2, v_mix=False, softcap=9.0, mlp=P.moe(9, 2, 32, 3.0, 0, 0))]),
    # everything on the tensor-core arms, two kinds of attention that mix values, long and short windows
    "tc": P.make_config(128, 128, 24, 1.0, [
        P.rule(4, 2, 48, 40, 4, P.moe(6, 2, 72, 1.0, 64, 1.5)), P.attend(4, 2, 32, 24, 70, 500.0, 32, P.wave(8.0, 1.0, 4.0, 128), 0.2, mlp=P.moe(5, 2, 136, 2.0, 40, 1.0)),
        P.attend(8, 2, 64, 24, 200, 2e4, 48, P.yarn(4.0, 64, 32.0, 1.0), 0.15, softcap=3.0), P.rule(2, 2, 128, 72, 3, P.moe(20, 4, 24, 0.6, 24, 9.0)),
        P.attend(2, 2, 64, 24, 33, 2e4, 64, P.yarn(4.0, 64, 32.0, 1.0), 0.15, softcap=30.0)], eps=1e-6),
    # odd sizes everywhere: no vector loads, no tensor-core arms, a single tap, a window of one
    "odd": P.make_config(61, 37, 5, 0.9, [
        P.rule(3, 1, 7, 10, 1, P.moe(3, 2, 11, 0.9, 5, 1.1)), P.attend(3, 1, 5, 7, 9, 50.0, 2, P.wave(3.0, 1.0, 2.0, 20), 0.5),
        P.attend(2, 2, 6, 3, 1, 20.0, 4, P.yarn(2.0, 30, 3.0, 0.4), 0.5, v_mix=None, softcap=1.5, mlp=P.moe(2, 1, 3, 2.0, 7, 0.5)),
        P.attend(1, 1, 3, 7, 14, 20.0, 2, P.yarn(2.0, 30, 3.0, 0.4), 0.4, softcap=8.0)], eps=1e-3),
    # recurrences only
    "rule": P.make_config(97, 48, 8, 0.8, [P.rule(2, 1, 64, 16, 3, P.moe(4, 2, 24, 1.0, 16, 1.0)), P.rule(4, 4, 16, 40, 4), P.rule(2, 2, 32, 24, 2, P.moe(3, 1, 16, 1.0, 0, 0))]),
    # every row uses every expert, so that bf16 turns no choice over; tensor-core arms
    "full": P.make_config(112, 96, 16, 0.75, [
        P.rule(2, 1, 64, 48, 5, P.moe(3, 3, 56, 1.5, 48, 2.0)), P.attend(6, 2, 48, 32, 90, 3e3, 24, P.wave(4.0, 1.0, 2.0, 96), 0.2, mlp=P.moe(2, 2, 40, 0.8, 0, 0)),
        P.attend(4, 2, 96, 32, 45, 1e4, 96, P.yarn(8.0, 96, 16.0, 2.0), 0.12, softcap=6.0, mlp=P.moe(4, 4, 24, 7.0, 136, 1.0)), P.rule(6, 3, 16, 8, 2)]),
    # attention only
    "att": P.make_config(90, 64, 16, 1.0, [P.attend(6, 2, 32, 32, 100, 1000.0, 16, P.wave(2.0, 1.0, 4.0, 512), 0.5)]),
}
NAMES = list(CONFIGS)
CLOSE = 0.15              # router logits closer than this may swap in bf16
TOL = {torch.float32: 5e-5, torch.bfloat16: 0.18}      # rms of the logits' difference over the logits' spread


def tol(name, dt):
    return TOL[dt] if dt == torch.float32 or name not in ("full", "att") else 0.06


@functools.lru_cache(None)
def weights(name):
    return P.make_weights(CONFIGS[name], seed=len(name))


@functools.lru_cache(None)
def tokens(name, n, seed=0):
    return tuple(torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist())


@functools.lru_cache(None)
def oracle(name, toks):
    """Expected logits, and every row's smallest margin between a chosen expert and one that is not."""
    margins = []
    out = P.forward(weights(name), CONFIGS[name], list(toks), torch.float64, margins=margins).float()
    return out, torch.stack(margins).amin(0) if margins else torch.full((len(toks),), float("inf"))


def expected(name, toks):
    return oracle(name, toks)[0]


def clear(name, toks, dt):
    """Rows whose choice of experts no rounding turns over."""
    return oracle(name, toks)[1] > (CLOSE if dt == torch.bfloat16 else 1e-4)


def engine(name, dt=torch.float32, **kw):
    kw = {"max_context": 640, "max_rows": 640, **kw}
    return LayeredEngine(Lifulorn(LifulornConfig.from_dict(CONFIGS[name]), weights(name), dt, max_context=kw["max_context"]), **kw)


def error(got, want, rows=None):
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / want.std(-1).mean()
    if rows is not None:
        assert rows.numel() < 20 or rows.float().mean() > 0.3
        e = e[rows]
    return e.max().item() if e.numel() else 0.0


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
    assert (eng.model.tc_attention, eng.model.tc_state) == ((name in ("mix", "tc", "full", "att"), name in ("tc", "full", "rule")) if dt == torch.bfloat16 else (False, False))
    taps, eng.tap_layers = [], []
    P.forward(weights(name), CONFIGS[name], list(toks[:40]), torch.float64, taps)
    rows = clear(name, toks[:40], dt)
    eng.step(toks[:40], [1] * 40, list(range(40)))
    assert len(taps) == len(eng.tap_layers) == len(CONFIGS[name]["layers"])
    for i, (a, b) in enumerate(zip(eng.tap_layers, taps)):
        off = (a.cpu() - b.float())[rows].pow(2).mean().sqrt() / b.float().pow(2).mean().sqrt()
        assert off < (1e-5 if dt == torch.float32 else 0.05), (i, off)
    eng.tap_layers = None
    assert error(feed(eng, 0, toks, 0, [333]), expected(name, toks), clear(name, toks, dt)) < tol(name, dt)


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", NAMES)
def test_portions_and_token_by_token_match_the_whole(name, dt):
    toks = tokens(name, 200)
    want = expected(name, toks)
    eng = engine(name, dt)
    whole = feed(eng, 0, toks, 0, [200])
    ref, rows = want if dt == torch.float32 else whole, clear(name, toks, dt)
    for lane, cuts in enumerate(([2] * 100, [1] * 200, [64, 64, 64, 8], [3, 61, 1, 65, 33, 2, 2, 32, 1])):
        got = feed(eng, lane, toks, 0, cuts)
        assert error(got, ref, rows) < tol(name, dt), (cuts[:4], error(got, ref, rows))
        assert error(got, want, rows) < tol(name, dt)


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("key", [0, 63, 64, 99])
def test_a_token_reaches_its_windows_last_row_and_not_the_next(key, dt):
    """Attention is the only mixer: a changed token changes the rows up to window - 1 behind it, in a portion and decoded, and no other."""
    n, window = key + 108, CONFIGS["att"]["layers"][0]["mixer"]["mask"]["size"]
    a = list(tokens("att", n))
    b = list(a)
    b[key] = (b[key] + 7) % 90
    want = expected("att", tuple(b)) - expected("att", tuple(a))
    eng = engine("att", dt)
    last = key + window - 1
    assert (want[last].abs().max() > 1e-4) and (want[last + 1:] == 0).all()
    for cuts in ([n], [last - 40] + [1] * (n - last + 40) if last > 40 else [1] * n, [last, 2, n - last - 2], [last + 1, n - last - 1]):
        got = feed(eng, 0, b, 0, cuts) - feed(eng, 1, a, 0, cuts)
        assert (got[:key] == 0).all() and (got[last + 1:] == 0).all() and got[last].abs().max() > 0, cuts[:2]
        if dt == torch.float32:
            assert (got - want).abs().max() < 1e-3 * want.abs().max()


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("n,key", [(300, 0), (300, 1), (300, 127), (300, 128), (257, 64), (321, 255)])
def test_a_far_token_reaches_prompt_and_decoded_rows(n, key, dt):
    """The recurrences carry a token on past every chunk and portion: the change of the logits is the plain implementation's."""
    a = list(tokens("rule", n))
    b = list(a)
    b[key] = (b[key] + 17) % 97
    eng = engine("rule", dt)
    want = expected("rule", tuple(b)) - expected("rule", tuple(a))
    rows = [key + 1, key + 5, min(key + 40, n - 1)]
    for cuts in ([n], [n - 40] + [1] * 40, [50, n - 52, 2]):
        got = feed(eng, 0, b, 0, cuts) - feed(eng, 1, a, 0, cuts)
        rel = ((got[rows] - want[rows]).pow(2).mean() / want[rows].pow(2).mean()).sqrt().item()
        assert rel < (0.02 if dt == torch.float32 else 0.6), (cuts[:2], rel)


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
            worst = max(worst, error(g, expected(name, live[lane][0])[at:at + n], clear(name, live[lane][0], dt)[at:at + n]))
            live[lane][1] += n
            pages = set(eng.kv.pages[lane])
            if live[lane][1] == len(live[lane][0]):
                reused += len(pages & seen)
                seen |= pages
                eng.release_lane(lane)
                del live[lane]
    eng.check_status()
    assert worst < tol(name, dt) and reused > 4 and eng.kv.free_pages == eng.n_pages


@pytest.mark.parametrize("dt", list(TOL))
@pytest.mark.parametrize("name", ["mix", "tc", "full"])
def test_long_decoding_crosses_pages_windows_and_graph_buckets(name, dt):
    toks = tokens(name, 420)
    eng = engine(name, dt)
    assert error(feed(eng, 2, toks, 0, [50] + [1] * 370), expected(name, toks), clear(name, toks, dt)) < tol(name, dt)
    assert len(eng.graphs) >= 1


@pytest.mark.parametrize("rows", [3, 70])
def test_batched_decoding_matches_each_alone(rows):
    """Few single rows take the recurrence with its convolution, many the separate kernels (and attention in slices of rows)."""
    for dt in TOL:
        eng = engine("tc", dt, max_lanes=rows, max_context=128, max_rows=256)
        reqs = [tokens("tc", 40 + s % 7, s) for s in range(rows)]
        for s, t in enumerate(reqs):
            eng.step(t[:20], [s] * 20, list(range(20)), head=False)
        for p in range(20, 40):
            eng.step([t[p] for t in reqs], list(range(rows)), [p] * rows, sample=False)
            if p % 6 == 1:
                for s in (0, 1, rows - 1):
                    assert error(eng.logits[s:s + 1], expected("tc", reqs[s])[p:p + 1], clear("tc", reqs[s], dt)[p:p + 1]) < TOL[dt]
        eng.check_status()


def greedy(name, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(P.forward(weights(name), CONFIGS[name], toks, torch.float64)[-1].argmax()))
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
    prompt = list(tokens("mix", 12))
    want = greedy("mix", prompt, 16)
    eng = engine("mix", max_lanes=2, max_context=128, max_rows=32)
    assert generate_all(eng, [prompt], 16, drafter=Drafter(want)) == [want]


def test_small_engines_and_a_pool_of_one_page():
    toks = tokens("tc", 64)
    eng = engine("tc", torch.bfloat16, max_lanes=1, max_context=64, max_rows=64)
    rows = clear("tc", toks, torch.bfloat16)
    assert error(feed(eng, 0, toks, 0, [40, 24]), expected("tc", toks), rows) < TOL[torch.bfloat16]
    eng.release_lane(0)
    assert error(feed(eng, 0, toks, 0, [64]), expected("tc", toks), rows) < TOL[torch.bfloat16]
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
