"""Host side of the layered decoders: configuration, registry, page pool, state versions, scheduler pages; and the plain
implementation's own invariances."""
import copy
import json

import pytest
import torch

from oracles import plain_fanodra as P
from sparkflash_b200.kv.paged import PAGE, PagedKV, PagesExhausted
from sparkflash_b200.kv.state import StateSlots
from sparkflash_b200.models import registry
from sparkflash_b200.models.fanodra import Fanodra, FanodraConfig
from sparkflash_b200.sched.core import PHASE_IDLE, PHASE_PREFILL, Scheduler
from sparkflash_b200.weights.files import write_safetensors

CFG = P.make_config(50, 24, 3, [("rglru", P.recurrent(12, 3, 2), 20), ("parallel", P.attending(4, 2, 8, 6, 0.3), P.recurrent(10, 1, 4), None)],
                    loop=(1, 2, 2))


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    c = FanodraConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.taps, c.eps) == (50, 24, 3, 1e-5)
    assert c.runs() == [(0, None), (1, 0), (1, 1)] and c.layers[1].ff is None
    assert {n: tuple(t.shape) for n, t in P.make_weights(CFG).items()} == c.shapes()
    plain = copy.deepcopy(CFG)
    del plain["loop"]
    assert FanodraConfig.from_dict(plain).runs() == [(0, None), (1, None)]

    def broken(edit):
        d = copy.deepcopy(CFG)
        edit(d)
        with pytest.raises(ValueError, match="config.json|layer|taps"):
            FanodraConfig.from_dict(d)
    broken(lambda d: d.update(rope_theta=1.0))
    broken(lambda d: d["layers"][0]["mixer"].update(gate=1))
    broken(lambda d: d["layers"][0].update(type="mamba"))
    broken(lambda d: d["layers"][0]["mixer"].update(blocks=5))
    broken(lambda d: d["layers"][1]["mixer"]["left"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda d: d["loop"].update(stop=3))
    broken(lambda d: d["canon"].update(taps=99))
    broken(lambda d: d.update(architecture="Other"))


def test_registry_chooses_the_class_and_the_loader_checks_shapes(tmp_path):
    w = P.make_weights(CFG)
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert registry.architecture(str(tmp_path)) == "Fanodra" and "fanodra" in registry.MODELS
    assert registry.layered_class("Fanodra") is Fanodra
    with pytest.raises(ValueError, match="layered engine"):
        registry.layered_class("deepseek_v41")
    m = Fanodra.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)
    assert torch.equal(m.embed, w["embed"].float()) and m.kv_runs == [(2, 8, 6)] * 2
    d = torch.arange(64)
    assert torch.allclose(m.layers[1].mixer.att.bias[2], w["l1.mix.left.r1"][2].float() * torch.log(1 + w["l1.mix.left.r2"][2].float() * d), atol=1e-5)
    w["l0.mix.o"] = w["l0.mix.o"][:, :-1]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(ValueError, match="l0.mix.o: shape"):
        Fanodra.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)


def test_page_pool_gives_back_and_runs_out():
    kv = PagedKV([(2, 4, 4)], 5, 3, 4 * PAGE, torch.float32, "cpu")
    kv.ensure(0, 1)
    kv.ensure(1, PAGE + 1)
    kv.ensure(0, PAGE)
    assert kv.held(0) == 1 and kv.held(1) == 2 and kv.free_pages == 2
    with pytest.raises(PagesExhausted):
        kv.ensure(2, 3 * PAGE)
    assert kv.held(2) == 0
    kv.upload()
    assert kv.table[1, :2].tolist() == kv.pages[1] and not set(kv.pages[0]) & set(kv.pages[1])
    old = list(kv.pages[1])
    kv.truncate(1, PAGE)
    kv.ensure(2, 3 * PAGE)
    kv.upload()
    assert kv.free_pages == 0 and old[1] in kv.pages[2] and kv.table[2, :3].tolist() == kv.pages[2]
    with pytest.raises(ValueError):
        kv.ensure(0, 4 * PAGE + 1)


def test_state_versions_continue_undo_and_start_over():
    st = StateSlots(2, "cpu")
    st.add("s", (3,), torch.float32)
    a = st.plan(1, 0)
    assert (a.src, a.replay) == (-1, []) and a.dst in (2, 3)
    st.commit(a, [5, 6, 7])
    b = st.plan(1, 3)
    assert b.src == a.dst and b.dst != b.src
    st.commit(b, [8, 9, 10, 11])
    # back into the latest step: the same source, its first tokens again, the same destination
    c = st.plan(1, 5)
    assert (c.src, c.dst, c.start, c.replay) == (b.src, b.dst, 3, [8, 9])
    st.commit(c, c.replay + [1])
    assert st.rows(1) == 6 and st.plan(1, 6).src == b.dst
    with pytest.raises(ValueError, match="cannot continue"):
        st.plan(1, 2)
    d = st.plan(1, 0)                       # a new sequence on the same lane reads nothing
    assert d.src == -1 and d.dst != b.dst
    st.reset(1)
    assert st.rows(1) == 0 and st.rows(0) == 0


def test_scheduler_places_by_pages_and_drops_held_prefixes():
    s = Scheduler(max_lanes=3, max_rows=64, prefill_chunk=64, prefill_chunk_busy=64, prefix_reuse_min=8, max_context=512)
    s.set_pages(64, 4)
    s.set_ring_slack(0)
    assert s.submit(1, list(range(100)), 20) == 0           # two pages
    assert s.submit(2, list(range(200, 290)), 60) == 0      # three: has to wait, although lanes are free
    assert s.submit(3, list(range(300)), 1) == 2            # five: never fits
    for want in (64, 36):
        phase, rows = s.tick()
        assert phase == PHASE_PREFILL and {r.seq for r in rows} == {1} and len(rows) == want
        s.commit(1, len(rows), [7] if want == 36 else [], -1)
    assert s.lane_rows().count(0) == 2 and s.info(2)["state"] == "waiting"
    s.cancel(1)                                             # its lane keeps 100 rows (two pages) for reuse ...
    assert sorted(s.lane_rows()) == [0, 0, 100]
    phase, rows = s.tick()                                  # ... until the pages are needed
    assert {r.seq for r in rows} == {2} and sorted(s.lane_rows()) == [0, 0, 0]
    s.cancel(2)
    assert s.tick()[0] == PHASE_IDLE


def test_plain_implementation_is_causal_and_sees_far_tokens():
    w = P.make_weights(CFG, 3)
    toks = torch.randint(0, 50, (40,), generator=torch.Generator().manual_seed(1)).tolist()
    full = P.forward(w, CFG, toks)
    assert torch.allclose(P.forward(w, CFG, toks[:25]), full[:25], atol=1e-9)
    other = list(toks)
    other[0] = (other[0] + 1) % 50
    assert (P.forward(w, CFG, other)[39] - full[39]).abs().max() > 1e-6
    # one pass of the recurrence from a carried state equals the whole
    u, lam = torch.randn(9, 4, dtype=torch.float64), torch.randn(4, dtype=torch.float64)
    r, i = torch.rand(9, 4, dtype=torch.float64), torch.rand(9, 4, dtype=torch.float64)
    S = P.gated_recurrence(u, r, i, lam)
    assert torch.allclose(P.gated_recurrence(u[5:], r[5:], i[5:], lam, S[4]), S[5:])
