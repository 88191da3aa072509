"""Host side of Gudutar: configuration, shared weights, loader, what the engine stages for windows and long runs; and the plain
implementation's own invariances."""
import copy
import json

import pytest
import torch

from oracles import plain_gudutar as P
from sparkflash_b200.models import registry
from sparkflash_b200.models.gudutar import Gudutar, GudutarConfig, random_tensors
from sparkflash_b200.models.layered import LayeredEngine
from sparkflash_b200.weights.files import write_safetensors

CFG = P.make_config(50, 24, 2.5, [P.ssm(4, 6, 5, 2, 3, 2), P.retain(2, 8, 6, 100.0, 4, [0.9, 0.99]), P.latent(3, 4, 2, 5, 7, 6, 50.0, 0.3, mlp=P.dense(20)),
                                  0, 2, P.latent(2, 8, 4, 6, 9, 11, 60.0, 0.2)])


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    c = GudutarConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.eps, c.embed_scale) == (50, 24, 1e-5, 2.5)
    assert [L.weights for L in c.layers] == [0, 1, 2, 0, 2, 5] and [L.ff for L in c.layers] == [None, None, 20, None, 20, None]
    assert {n: tuple(t.shape) for n, t in P.make_weights(CFG).items()} == c.shapes() == {n: tuple(t.shape) for n, t in random_tensors(c).items()}
    chain = copy.deepcopy(CFG)
    chain["layers"][4]["weights_of"] = 4 - 2
    chain["layers"].append({**copy.deepcopy(CFG["layers"][0]), "weights_of": 3})       # a layer that shares may be shared in turn
    assert GudutarConfig.from_dict(chain).layers[-1].weights == 0

    def broken(edit):
        d = copy.deepcopy(CFG)
        edit(d)
        with pytest.raises(ValueError, match="config.json|layer|states"):
            GudutarConfig.from_dict(d)
    broken(lambda d: d.update(rope_theta=1.0))
    broken(lambda d: d["embedding"].update(tied=True))
    broken(lambda d: d["layers"][0].update(type="mamba"))
    broken(lambda d: d["layers"][0]["mixer"].update(groups=3))
    broken(lambda d: d["layers"][0]["mixer"].update(norm_groups=5))
    broken(lambda d: d["layers"][0]["mixer"].update(conv=99))
    broken(lambda d: d["layers"][0]["mixer"].update(state=1000))
    broken(lambda d: d["layers"][1]["mixer"].update(decay=[0.5]))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=10))
    broken(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=4))
    broken(lambda d: d["layers"][2]["mixer"]["mask"].update(kind="causal"))
    broken(lambda d: d["layers"][2]["mlp"].update(kind="moe"))
    broken(lambda d: d["layers"][3].update(weights_of=3))
    broken(lambda d: d["layers"][3].update(weights_of=1))
    broken(lambda d: d["layers"][4].update(mixer={**d["layers"][4]["mixer"], "scale": 0.31}))
    broken(lambda d: d.update(architecture="Other"))


def test_registry_loader_and_shared_layers(tmp_path):
    w = P.make_weights(CFG)
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert registry.layered_class(registry.architecture(str(tmp_path))) is Gudutar and "gudutar" in registry.MODELS
    m = Gudutar.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)
    assert m.layers[3] is m.layers[0] and m.layers[4] is m.layers[2] and m.kv_runs == [(1, 9, 0), (1, 9, 0), (1, 13, 0)]
    assert m.layers[0].mixer.w_in.shape[0] % 8 == 0 and torch.equal(m.layers[0].mixer.w_in[:w["l0.mix.in"].shape[0]], w["l0.mix.in"].float())
    assert m.windows == () and not m.tc_state                  # true 32-bit: no tensor-core arms
    w["l1.mix.g"] = w["l1.mix.g"][:-1]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(ValueError, match="l1.mix.g: shape"):
        Gudutar.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)


def test_staged_windows_and_long_runs():
    """Pages whose keys a step's long runs need, every tile's offset among them, and the recurrence's chunks."""
    cfg = P.make_config(40, 32, 1.0, [P.latent(2, 16, 8, 16, 24, 70, 50.0, 0.2), P.latent(2, 16, 8, 16, 24, 300, 50.0, 0.2), P.ssm(2, 16, 16, 1, 4, 1)])
    c = GudutarConfig.from_dict(cfg)
    eng = LayeredEngine(Gudutar(c, random_tensors(c), torch.bfloat16, "cpu", max_context=1024), max_lanes=3, max_context=1024, max_rows=600)
    assert eng.model.windows == (70, 300) and eng.model.tc_state
    rows = [(0, 0, 500), (1, 0, 130), (2, 0, 3)]
    for lane, p0, n in rows:
        eng.kv.ensure(lane, p0 + n)

    def stage(parts):
        toks, lanes, pos = [], [], []
        for lane, p0, n in parts:
            toks += [1] * n; lanes += [lane] * n; pos += range(p0, p0 + n)
            eng.kv.ensure(lane, p0 + n)
        segs = eng._segments(toks, lanes, pos)
        for lane, p0, n in parts:
            eng.state.lanes[lane].rows = p0
        return eng._stage(segs, [eng.state.plan(x, p0) for x, p0, _, _ in segs], [], None, None)
    s = stage([(2, 3, 1), (0, 500, 300), (1, 130, 32)])
    assert s.short == 1 and s.nshort == 1 and s.short_segs.tolist() == [0] and s.short_rows.tolist() == [0]
    assert s.long_seg.tolist() == [1, 2] and s.long_first.tolist() == [0, 3, 4]
    assert list(zip(s.long_row0.tolist(), s.long_rows.tolist())) == [(1, 128), (129, 128), (257, 44), (301, 32)]
    tiles = s.tiles.view(-1, 2).tolist()
    assert sorted(tiles) == [[1, 256], [257, 44], [301, 32]]
    for w in (70, 300):
        pages, count, offs = s.expand[w]
        lo0, lo1 = max(0, 500 - w + 1) // 64, max(0, 130 - w + 1) // 64
        assert pages.tolist() == eng.kv.pages[0][lo0:13] + eng.kv.pages[1][lo1:3] and count == len(pages)
        assert {t[0]: o for t, o in zip(tiles, offs.tolist())} == {1: -lo0, 257: -lo0, 301: 13 - lo0 - lo1}
    s = stage([(0, 800, 1), (1, 162, 1)])
    assert s.single and s.ntiles == s.nlong == 0 and s.nshort == 2 and s.short_segs is None and not s.expand


def test_plain_implementation_is_causal_and_its_windows_end():
    w, toks = P.make_weights(CFG, 3), torch.randint(0, 50, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = P.forward(w, CFG, toks)
    assert torch.allclose(P.forward(w, CFG, toks[:17]), full[:17], atol=1e-9)
    other = [(toks[0] + 1) % 50] + toks[1:]
    assert (P.forward(w, CFG, other)[29] - full[29]).abs().max() > 1e-9
    only = P.make_config(50, 24, 1.0, [P.latent(2, 4, 4, 5, 7, 6, 50.0, 0.9)])
    w = P.make_weights(only, 4)
    d = (P.forward(w, only, other) - P.forward(w, only, toks)).abs().amax(1)
    assert (d[:6] > 1e-6).all() and (d[6:] == 0).all()
    # a recurrence carried on equals the whole
    q, k, v, la = torch.randn(9, 4).double(), torch.randn(9, 4).double(), torch.randn(9, 3).double(), -torch.rand(9).double()
    a, S = P.decayed_sum(q[:5], k[:5], v[:5], la[:5])
    assert torch.allclose(torch.cat([a, P.decayed_sum(q[5:], k[5:], v[5:], la[5:], S)[0]]), P.decayed_sum(q, k, v, la)[0])
