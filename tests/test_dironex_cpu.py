"""Host side of Dironex: configuration, loader, layer runs; and the plain implementation's own invariances."""
import copy
import json
import math

import pytest
import torch

from oracles import plain_dironex as P
from sparkflash_b200.models import registry
from sparkflash_b200.models.dironex import Dironex, DironexConfig, random_tensors
from sparkflash_b200.models.layered import LayeredEngine
from sparkflash_b200.models.mixers import rotation_frequencies, rotation_table
from sparkflash_b200.weights.files import write_safetensors

YARN = (3.0, 30, 4.0, 0.5)
CFG = P.make_config(50, 24, 3, 2, 0.6, 2.5, [P.windowed(4, 2, 5, 6, 7, 0.3, P.moe(6, 2, 10, 3, 2, 1.3)), P.latent(3, 8, 4, 5, 10, 7, 0.2, 60.0, YARN, P.ff(14)),
                                             P.latent(2, 6, 2, 9, 8, 12, 0.3, 90.0), P.windowed(2, 1, 4, 3, 2, 0.5, P.ff(9))], loop=(1, 3, 2))


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    c = DironexConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.eps, c.residual_mult, c.embed_scale, c.streams, c.taps) == (50, 24, 1e-5, 0.6, 2.5, 3, 2)
    assert c.runs() == [0, 1, 2, 1, 2, 3] == P.order(CFG) and [L.mlp is None for L in c.layers] == [False, False, True, False]
    assert {n: tuple(t.shape) for n, t in P.make_weights(CFG).items()} == c.shapes() == {n: tuple(t.shape) for n, t in random_tensors(c).items()}
    for loop in (None, {"start": 0, "stop": 4, "times": 1}):
        assert DironexConfig.from_dict({**CFG, "loop": loop}).runs() == [0, 1, 2, 3]
    assert DironexConfig.from_dict({**CFG, "loop": {"start": 3, "stop": 4, "times": 3}}).runs() == [0, 1, 2, 3, 3, 3]

    def broken(edit):
        d = copy.deepcopy(CFG)
        edit(d)
        with pytest.raises(ValueError, match="config.json|layer|taps"):
            DironexConfig.from_dict(d)
    mixer = lambda d, i: d["layers"][i]["mixer"]
    broken(lambda d: d.update(rope_theta=1.0))
    broken(lambda d: d.pop("residual_mult"))
    broken(lambda d: d.update(streams=0))
    broken(lambda d: d.update(streams=99))
    broken(lambda d: d["canon"].update(taps=99))
    broken(lambda d: d["loop"].update(stop=5))
    broken(lambda d: d["loop"].update(start=3))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d["layers"][0].update(type="attention_2"))
    broken(lambda d: mixer(d, 0).update(kv_heads=3))
    broken(lambda d: mixer(d, 0).update(rot={"base": 1.0, "dims": 2}))
    broken(lambda d: mixer(d, 0)["mask"].update(size=0))
    broken(lambda d: mixer(d, 1).pop("q_rank"))
    broken(lambda d: mixer(d, 1)["rot"].update(dims=2))
    broken(lambda d: mixer(d, 1)["rot"]["scaling"].update(low=1.0))
    broken(lambda d: mixer(d, 1).update(mask={"size": 3}))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="glu"))
    broken(lambda d: d["layers"][1]["mlp"].update(limit=3.0))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=5))                # two groups of two hold four
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4))
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda d: d["layers"][0]["mlp"]["expert"].update(limit=1.0))
    broken(lambda d: d["layers"][0]["mlp"].update(shared={"ff": 3}))
    broken(lambda d: d.update(architecture="Other"))


def test_registry_and_loader(tmp_path):
    w = P.make_weights(CFG)
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert registry.layered_class(registry.architecture(str(tmp_path))) is Dironex and "dironex" in registry.MODELS
    m = Dironex.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)
    assert m.kv_runs == [(2, 5, 6), (1, 14, 0), (1, 10, 0), (1, 14, 0), (1, 10, 0), (1, 4, 3)] and not m.tc_attention and m.windows == ()
    a, lat, moe, ff = m.layers[0].mixer, m.layers[1].mixer, m.layers[0].ff, m.layers[1].ff
    assert a.window == 7 and lat.window == 64 and lat.gated and lat.halves and m.layers[2].ff is None and len(m.layers[2].canon) == 1
    # the stacked projection: gate, latent and shared key part, the queries' latent
    assert torch.equal(lat.w_in[:15], w["l1.mix.g"].float()) and torch.equal(lat.w_in[lat.col_c:lat.col_cq], w["l1.mix.dkv"].float())
    assert torch.equal(lat.w_in[lat.col_cq:lat.col_cq + 7], w["l1.mix.dq"].float())
    assert torch.equal(m.layers[3].streams[1].out, 0.6 * w["l3.hc2.out"].float()) and torch.equal(m.layers[0].canon[1], w["l0.canon2"].float().t())
    p, q = w["l1.mlp.act"].double().tolist()
    assert (ff.a, ff.b) == pytest.approx((math.log1p(math.exp(p)), 0.5 + math.log1p(math.exp(q))), rel=1e-12)
    assert moe.w_in.shape == (6, 10, 24) and torch.equal(moe.w_out[4], w["l0.mlp.e4.down"].float()) and (moe.choice.groups, moe.choice.keep, moe.choice.scale) == (3, 2, 1.3)
    e = LayeredEngine(m, max_lanes=2, max_context=64, max_rows=32)
    assert len(e.state.tensors) == 10 and e.nbytes()["weights"] > sum(t.numel() for t in w.values()) * 4       # two per run, one where there is no feed-forward
    w["l1.mix.g"] = w["l1.mix.g"][:-1]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(ValueError, match="l1.mix.g: shape"):
        Dironex.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)


def test_plain_implementation_is_causal_and_its_windows_end():
    w, toks = P.make_weights(CFG, 3), torch.randint(0, 50, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = P.forward(CFG, w, toks)
    assert torch.allclose(P.forward(CFG, w, toks[:17]), full[:17], atol=1e-9)
    other = [(toks[0] + 1) % 50] + toks[1:]
    assert (P.forward(CFG, w, other)[29] - full[29]).abs().max() > 1e-9
    # windowed attention alone: a window of 6 and one more row per carried input of either convolution
    for taps, reach in ((1, 6), (3, 10)):
        only = P.make_config(50, 24, 2, taps, 0.5, 1.0, [P.windowed(2, 1, 4, 5, 6, 0.9, P.ff(8))])
        w = P.make_weights(only, 4)
        d = (P.forward(only, w, other) - P.forward(only, w, toks)).abs().amax(1)
        assert (d[:reach] > 1e-7).all() and (d[reach:] == 0).all()


def test_plain_choice_of_experts():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0}
    # choice scores all below 0: the experts of groups that are left out must not come in as zeros; the pair's sum decides, not the best one
    corr = torch.tensor([-1.5, -3.0, -2.0, -2.0, -4.0, -4.0])
    ids, wts = P.route(torch.zeros(1, 6), corr, r)
    assert ids == [[2, 3]] and wts[0].tolist() == [1.0, 1.0]
    ids, wts = P.route(torch.tensor([[9.0, 0.0, 0.0, 2.0, 0.0, 0.0]]), torch.tensor([0.0, -2.0, 0.0, 0.0, 0.0, 0.0]), r)
    s = [1 / (1 + math.exp(-2.0)), 0.5]
    assert ids == [[3, 2]] and wts[0].tolist() == pytest.approx([2 * s[0] / sum(s), 2 * s[1] / sum(s)], rel=1e-6)


def test_plain_streams_and_activation():
    X = torch.randn(3, 4, 5, dtype=torch.float64)
    mix, out, y = torch.randn(3, 3, dtype=torch.float64), torch.randn(3, dtype=torch.float64), torch.randn(4, 5, dtype=torch.float64)
    new = P.spread(X, mix, out, 0.5, y)
    assert torch.allclose(new, torch.einsum("st,snd->tnd", mix, X) + 0.5 * out[:, None, None] * y)
    assert torch.allclose(P.collapse(X, out), torch.einsum("s,snd->nd", out, X))
    z = torch.tensor([-3.0, -1e-3, 0.0, 2.0], dtype=torch.float64)
    got = P.xielu(z, torch.tensor(0.3, dtype=torch.float64), torch.tensor(-0.4, dtype=torch.float64))
    a, b = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.4))
    assert got.tolist() == pytest.approx([b * (math.exp(-3) + 2) - 1.5, b * (math.expm1(-1e-3) + 1e-3) - 5e-4, 0.0, 4 * a + 1], rel=1e-9)


@pytest.mark.parametrize("scaling", [None, (5.0, 200, 9.0, 0.5), (3.0, 4000, 600.0, 590.0), (1.0, 64, 32.0, 1.0)])
@pytest.mark.parametrize("dims", [2, 20, 64])
def test_rotation_tables(scaling, dims):
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    freqs, gain = P.frequencies(500.0, dims, sc)
    got, g = rotation_frequencies(500.0, dims, sc)
    assert got == pytest.approx(freqs, rel=1e-12) and g == pytest.approx(gain, rel=1e-12)
    x = torch.randn(40, 1, dims, dtype=torch.float64)
    t = rotation_table(500.0, dims, 40, "cpu", sc).double()
    u, v = x[:, 0, :dims // 2], x[:, 0, dims // 2:]
    assert (torch.cat([u * t[..., 0] - v * t[..., 1], v * t[..., 0] + u * t[..., 1]], 1) - P.turn(x, 500.0, dims, sc)[:, 0]).abs().max() < 1e-5
