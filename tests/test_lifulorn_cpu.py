"""Host side of Lifulorn: configuration, loader, which layers mix values; and the plain implementation's own invariances."""
import copy
import json

import pytest
import torch

from oracles import plain_lifulorn as P
from sparkflash_b200.models import registry
from sparkflash_b200.models.layered import LayeredEngine
from sparkflash_b200.models.lifulorn import Lifulorn, LifulornConfig, random_tensors
from sparkflash_b200.models.mixers import rotation_frequencies, rotation_table
from sparkflash_b200.weights.files import write_safetensors

MOE = P.moe(5, 2, 12, 1.0, 7, 2.0)
CFG = P.make_config(50, 24, 6, 0.7, [P.rule(4, 2, 5, 6, 3, MOE), P.attend(4, 2, 8, 5, 6, 100.0, 4, P.wave(4.0, 1.0, 3.0, 40), 0.3),
                                     P.attend(2, 1, 6, 10, 3, 60.0, 6, P.yarn(3.0, 30, 4.0, 0.5), 0.2, v_mix=None, softcap=2.0, mlp=P.moe(3, 3, 4, 0.5, 0, 0)),
                                     P.attend(6, 2, 4, 5, 9, 50.0, 2, P.yarn(3.0, 30, 4.0, 0.5), 0.4, softcap=5.0, mlp=MOE), P.rule(1, 1, 8, 4, 1)])


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    c = LifulornConfig.from_dict(CFG)
    assert (c.vocab, c.width, c.eps, c.residual_mult, c.side_dim) == (50, 24, 1e-5, 0.7, 6)
    assert [L.mix for L in c.layers] == [False, True, False, True, False] and [L.mlp is None for L in c.layers] == [False, True, False, False, True]
    assert {n: tuple(t.shape) for n, t in P.make_weights(CFG).items()} == c.shapes() == {n: tuple(t.shape) for n, t in random_tensors(c).items()}

    def broken(edit):
        d = copy.deepcopy(CFG)
        edit(d)
        with pytest.raises(ValueError, match="config.json|layer|states"):
            LifulornConfig.from_dict(d)
    mixer = lambda d, i: d["layers"][i]["mixer"]
    broken(lambda d: d.update(rope_theta=1.0))
    broken(lambda d: d.pop("residual_mult"))
    broken(lambda d: d["token_side"].update(act="silu"))
    broken(lambda d: d["layers"][0].update(type="delta_2"))
    broken(lambda d: mixer(d, 0).update(kv_heads=3))
    broken(lambda d: mixer(d, 0).update(conv=99))
    broken(lambda d: mixer(d, 0).update(dim=1000))
    broken(lambda d: mixer(d, 1).update(softcap=3.0))
    broken(lambda d: mixer(d, 1)["rot"].update(dims=9))
    broken(lambda d: mixer(d, 1)["rot"]["scaling"].update(fast=3.0))
    broken(lambda d: mixer(d, 1)["mask"].update(size=0))
    broken(lambda d: mixer(d, 3).pop("softcap"))
    broken(lambda d: mixer(d, 3).update(softcap=0.0))
    broken(lambda d: mixer(d, 3).update(vdim=6))               # cannot mix with layer 1's values
    broken(lambda d: d["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mlp"]["expert"].update(bias=True))
    broken(lambda d: d.update(architecture="Other"))


def test_registry_and_loader(tmp_path):
    w = P.make_weights(CFG)
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    assert registry.layered_class(registry.architecture(str(tmp_path))) is Lifulorn and "lifulorn" in registry.MODELS
    m = Lifulorn.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)
    assert m.kv_runs == [(2, 8, 5), (1, 6, 10), (2, 4, 5)] and not m.tc_attention and not m.tc_state
    att = [m.layers[i].mixer for i in (1, 2, 3)]
    assert [a.mix is not None for a in att] == [True, False, True] and att[0].lam is None and float(att[2].lam) == float(w["l3.mix.vmix"])
    assert [a.cap for a in att] == [0.0, 2.0, 5.0] and [a.window for a in att] == [6, 3, 9]
    assert torch.equal(m.layers[0].ls1, 0.7 * w["l0.ls1"].float()) and m.layers[3].side.col0 == 18
    ff = m.layers[0].ff
    assert torch.equal(ff.w_in[3, 12:], w["l0.mlp.e3.up"].float()) and torch.equal(ff.router[5], w["l0.mlp.shared.sg"][0].float()) and ff.slots == 3
    e = LayeredEngine(m, max_lanes=2, max_context=64, max_rows=32)
    assert e.nbytes()["state"] > 0 and e.nbytes()["weights"] > sum(t.numel() for t in w.values()) * 4
    w["l1.mix.sink"] = w["l1.mix.sink"][:-1]
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    with pytest.raises(ValueError, match="l1.mix.sink: shape"):
        Lifulorn.from_dir(str(tmp_path), torch.float32, "cpu", max_context=64)


def test_plain_implementation_is_causal_and_its_windows_end():
    w, toks = P.make_weights(CFG, 3), torch.randint(0, 50, (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = P.forward(w, CFG, toks)
    assert torch.allclose(P.forward(w, CFG, toks[:17]), full[:17], atol=1e-9)
    other = [(toks[0] + 1) % 50] + toks[1:]
    assert (P.forward(w, CFG, other)[29] - full[29]).abs().max() > 1e-9
    only = P.make_config(50, 24, 6, 0.5, [P.attend(2, 1, 4, 5, 6, 50.0, 4, P.wave(2.0, 1.0, 2.0, 20), 0.9)])
    w = P.make_weights(only, 4)
    d = (P.forward(w, only, other) - P.forward(w, only, toks)).abs().amax(1)
    assert (d[:6] > 1e-6).all() and (d[6:] == 0).all()
    # a recurrence carried on equals the whole, and a repeated key writes only what is new
    q, k, v = torch.randn(9, 4).double(), P.unit(torch.randn(9, 4).double()), torch.randn(9, 3).double()
    decay, beta = torch.rand(9).double(), torch.rand(9).double()
    a, S = P.delta_rule(q[:5], k[:5], v[:5], decay[:5], beta[:5])
    assert torch.allclose(torch.cat([a, P.delta_rule(q[5:], k[5:], v[5:], decay[5:], beta[5:], S)[0]]), P.delta_rule(q, k, v, decay, beta)[0])
    one = torch.ones(2, dtype=torch.float64)
    key = torch.tensor([[1.0, 0.0], [1.0, 0.0]], dtype=torch.float64)
    assert torch.allclose(P.delta_rule(key, key, v[:2], one, one)[0], v[:2])


def test_plain_choice_and_clamps():
    ids, a = P.route(torch.tensor([0.0, 3.0, -1.0, 3.0, 1.0]), 3)
    assert ids == [1, 3, 4] and abs(float(a.sum()) - 1) < 1e-6 and float(a[0]) == float(a[1]) > float(a[2])
    w = {"gate": torch.eye(2), "up": torch.eye(2), "down": torch.eye(2)}
    y = P.expert(w, "", torch.tensor([[5.0, -5.0]]), 1.5)
    assert torch.allclose(y, torch.tensor([[1.5 / (1 + torch.exp(torch.tensor(-1.702 * 1.5))) * 2.5, -5 / (1 + torch.exp(torch.tensor(1.702 * 5))) * -0.5]]))


SCALINGS = {"plain": None, "wave": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 300}, "yarn": {"factor": 5.0, "original": 200, "fast": 9.0, "slow": 0.5},
            "step": {"factor": 3.0, "original": 4000, "fast": 600.0, "slow": 590.0}}


@pytest.mark.parametrize("kind", list(SCALINGS))
@pytest.mark.parametrize("dims", [2, 20, 64])
def test_rotation_tables(kind, dims):
    sc = SCALINGS[kind]
    freqs, gain = ([500.0 ** (-2.0 * i / dims) for i in range(dims // 2)], 1.0) if sc is None else (P.yarn_frequencies if "fast" in sc else P.wavelength_frequencies)(500.0, dims, sc)
    got, g = rotation_frequencies(500.0, dims, sc)
    assert got == pytest.approx(freqs, rel=1e-12) and g == pytest.approx(gain, rel=1e-12)
    x = torch.randn(40, 1, dims + 3, dtype=torch.float64)
    t = rotation_table(500.0, dims, 40, "cpu", sc).double()
    u, v = x[:, 0, :dims // 2], x[:, 0, dims // 2:dims]
    want = P.rotate(x, freqs, gain)[:, 0]
    assert (torch.cat([u * t[..., 0] - v * t[..., 1], v * t[..., 0] + u * t[..., 1], x[:, 0, dims:]], 1) - want).abs().max() < 1e-5
