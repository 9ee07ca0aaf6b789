"""Vudezen's configuration and model description, on the CPU: every size and constant comes from config.json, what a
layer leaves out is left out, blended values come from the first layer that blends, the members of a pair of mixers share
one stacked projection and one output matrix, and what cannot run is refused with the key's name."""
import copy
import math

import pytest
import torch

import plain_vudezen as plain
import tiny_vudezen as tv
from atom_b200.config.model_config import ConfigError, config_from_dict
from atom_b200.models.model import Model
from atom_b200.models.registry import build_model_spec
from atom_b200.parts.base import ProjectedMixer
from atom_b200.parts.rope import RotaryYarn
from atom_b200.weights.loader import expected_tensors, load_weights

F = torch.float64


@pytest.mark.parametrize("name", list(tv.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    cfg = config_from_dict(tv.CONFIGS[name])
    assert cfg.architecture == "Vudezen"
    assert config_from_dict(cfg.to_dict()) == cfg
    want = expected_tensors(Model(build_model_spec(cfg)))
    have = tv.random_tensors(tv.CONFIGS[name], 1)
    assert set(want) == set(have)
    for n, (_, _, _, shape, _) in want.items():
        assert tuple(have[n].shape) == tuple(shape), n


def test_what_every_layer_keeps():
    needs = Model(build_model_spec(config_from_dict(tv.CONFIGS["A"]))).cache_needs()
    assert [needs[i].kind for i in range(4)] == ["pages"] * 4
    assert [needs[i].window for i in range(4)] == [24, None, 24, None]
    assert {e.name: e.shape for e in needs[0].entries} == {"k": (2, 16), "v": (2, 24)}
    assert {e.name: (e.shape, e.dtype) for e in needs[0].states} == {
        "right.S": ((6, 12, 8), "float32"), "right.conv": ((2, 6 * 8 + 2 * 3 * 12), "compute")}
    assert not needs[1].states
    needs = Model(build_model_spec(config_from_dict(tv.CONFIGS["B"]))).cache_needs()
    assert {e.name for e in needs[1].states} == {"right.S"}                   # one tap keeps no rows


def test_values_are_blended_with_the_first_layer_that_blends():
    mix = lambda name: [L.parts["mixer"].args.get("value_mix") for L in build_model_spec(config_from_dict(tv.CONFIGS[name])).layers]
    assert mix("A") == [None, "first", None, "mixed"]
    assert mix("B") == [None, None, "first", None]                            # v_mix false is no such layer
    assert mix("C") == ["first", None, "mixed", "mixed", None]


def test_segments_of_multiples_of_eight_come_first_and_the_width_is_rounded_up():
    names, where, width = ProjectedMixer.layout({"a": (3, 2), "b": (16, 8), "c": (4,), "d": (8,)})
    assert names == ["b", "d", "a", "c"] and width == 48
    assert where == {"b": (0, 24), "d": (24, 8), "a": (32, 5), "c": (37, 4)}


def test_stacked_projection_and_output_matrix_of_a_pair(tmp_path):
    cfg = tv.CONFIGS["A"]
    tv.write_model(cfg, str(tmp_path), 7)
    model = Model(build_model_spec(config_from_dict(cfg)))
    got = load_weights(model, str(tmp_path), torch.float32, "cpu")
    W = {k: v.float() for k, v in tv.read_model(str(tmp_path))[1].items()}
    L = "l0.mix."
    # q, k, v (64 + 32 + 48 rows) and the right member's rows (174) and the gate's (4)
    want = torch.cat([W[L + "left.q"], W[L + "left.k"], W[L + "left.v"], W[L + "left.g"], W[L + "right.in"]])
    stacked = got["layers.0.mixer.in.weight"]
    assert stacked.shape[0] % 8 == 0 and torch.equal(stacked[:want.shape[0]], want) and not stacked[want.shape[0]:].any()
    assert torch.equal(got["layers.0.mixer.o.weight"], torch.cat([W[L + "left.o"], W[L + "right.o"]], dim=1))
    assert got["layers.3.mixer.vmix"].shape == (1,) and got["layers.3.mixer.vmix"][0] == W["l3.mix.vmix"]


def test_options_left_out_of_the_config():
    c = copy.deepcopy(tv.CONFIGS["A"])
    del c["logit_softcap"], c["logit_scale"], c["residual_mult"]
    c["layers"][1]["mlp"]["router"].pop("scale")
    cfg = config_from_dict(c)
    assert cfg.logit_softcap is None and cfg.logit_scale == 1.0 and cfg.residual_mult == 1.0
    assert cfg.layers[1].moe.scale == 1.0
    c["logit_softcap"] = 0
    assert config_from_dict(c).logit_softcap is None
    moe = config_from_dict(tv.CONFIGS["B"]).layers[0].moe
    assert moe.identity == 0 and moe.groups is None and config_from_dict(tv.CONFIGS["B"]).layers[2].moe.shared is None


def test_norms_of_a_layer_without_feed_forward_may_be_present(tmp_path):
    from safetensors.torch import load_file, save_file
    cfg = tv.CONFIGS["A"]
    tv.write_model(cfg, str(tmp_path), 7)
    f = str(tmp_path / "model.safetensors")
    t = load_file(f)
    for n in ("norm2", "norm2.b", "norm2b", "norm2b.b"):
        t["l2." + n] = torch.zeros(cfg["width"], dtype=torch.bfloat16)
    save_file(t, f)
    load_weights(Model(build_model_spec(config_from_dict(cfg))), str(tmp_path), torch.bfloat16, "cpu")


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),       # more than the head holds
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),        # odd
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(v_mix=True), "v_mix"),
    (lambda c: c["layers"][3].update(mixer=dict(c["layers"][3]["mixer"], vdim=16)), "v_mix"),                         # values of another size
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "router.groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "router.top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.'size'"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_refusals_name_the_key(edit, word):
    c = copy.deepcopy(tv.CONFIGS["A"])
    edit(c)
    with pytest.raises(ConfigError, match=word.replace(".", r"\.")):
        config_from_dict(c)


def test_yarn_frequencies_against_plain():
    rot = {"base": 50000.0, "dims": 48, "scaling": {"factor": 6.0, "original": 300, "fast": 16.0, "slow": 2.0}}
    part = RotaryYarn(48, 50000.0, rot["scaling"], neighbours=True)
    f, mag = plain.pair_frequencies(rot)
    assert part.neighbours and part.magnitude == pytest.approx(mag, rel=1e-12)
    assert torch.allclose(torch.tensor(part._f, dtype=F), f, rtol=1e-12)
    assert float(f[0]) == 1.0 and float(f[-1]) == pytest.approx(50000.0 ** (-46 / 48) / 6.0)


def test_plain_mechanisms_are_what_the_formulas_say():
    """The plain implementation itself on cases small enough to do by hand."""
    x = torch.tensor([[1.0, 3.0]], dtype=F)
    assert torch.allclose(plain.layer_norm(x, torch.tensor([2.0, 1.0], dtype=F), torch.tensor([0.5, 0.0], dtype=F), 0.0),
                          torch.tensor([[-1.5, 1.0]], dtype=F))
    r = plain.rotate_neighbours(torch.tensor([[[1.0, 0.0, 5.0]], [[1.0, 0.0, 5.0]]], dtype=F), {"dims": 2, "base": 100.0})
    assert torch.allclose(r[1, 0], torch.tensor([math.cos(1.0), math.sin(1.0), 5.0], dtype=F))
    r = plain.rotate_neighbours(torch.tensor([[[0.0, 0.0, 1.0, 0.0]]] * 3, dtype=F), {"dims": 4, "base": 4.0})
    assert torch.allclose(r[2, 0], torch.tensor([0.0, 0.0, math.cos(1.0), math.sin(1.0)], dtype=F))     # 2 * 4^(-1/2)
    assert plain.visible(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    one = torch.ones(2, 1, 1, dtype=F)
    o = plain.sink_attention(one, one * 0, torch.tensor([2.0, 4.0], dtype=F).view(2, 1, 1), 1.0, torch.tensor([math.log(2.0)], dtype=F), None)
    assert torch.allclose(o.flatten(), torch.tensor([2.0 / 3, 6.0 / 4], dtype=F))
    u = torch.tensor([[1.0], [2.0], [3.0]], dtype=F)
    assert plain.biased_conv(u, torch.tensor([[10.0, 1.0]], dtype=F), torch.tensor([0.5], dtype=F)).flatten().tolist() == [1.5, 12.5, 23.5]
    # decay exp(-dt) with dt = log 2: S halves, then takes log 2 * B x
    y = plain.state_space(torch.tensor([1.0, 2.0], dtype=F).view(2, 1, 1), one, one, torch.full((2, 1), math.log(2.0), dtype=F),
                          torch.zeros(1, dtype=F), torch.tensor([3.0], dtype=F))
    assert torch.allclose(y.flatten(), torch.tensor([math.log(2.0) + 3.0, 2.5 * math.log(2.0) + 6.0], dtype=F))
    assert torch.allclose(plain.grouped_rms_norm(torch.tensor([[3.0, 4.0, 1.0, 1.0]], dtype=F), torch.ones(4, dtype=F), 2, 0.0),
                          torch.tensor([[3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 1.0, 1.0]], dtype=F))
    s = torch.tensor([0.5, 0.1, 0.3, 0.1], dtype=F)
    assert plain.choose(s, torch.tensor([-1.0, -0.2, -0.9, -0.9], dtype=F), {"top": 2, "groups": {"count": 2, "keep": 1}}) == [1, 0]
    assert plain.choose(s, torch.zeros(4, dtype=F), {"top": 2}) == [0, 2]
    e = plain.clamped_expert(torch.tensor([[1.0]], dtype=F), {"gate": torch.tensor([[9.0]], dtype=F), "up": torch.tensor([[-9.0]], dtype=F),
                                                             "down": torch.tensor([[1.0]], dtype=F)}, "", 2.0)
    assert float(e) == pytest.approx(2.0 / (1 + math.exp(-3.404)) * -1.0)
