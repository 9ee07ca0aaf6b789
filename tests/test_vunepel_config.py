"""Vunepel's configuration and model description, on the CPU: every size and constant comes from config.json or a tensor's
shape, layers that share keys share a cache that reaches as far back as its readers look, and what cannot run is refused
with the key's name."""
import copy

import pytest
import torch

import plain_vunepel as plain
import tiny_vunepel as tv
from atom_b200.cache import CacheManager
from atom_b200.config.model_config import ConfigError, config_from_dict, load_model_config
from atom_b200.models.model import Model
from atom_b200.models.registry import build_model_spec
from atom_b200.parts.spec import CacheNeed
from atom_b200.weights.loader import expected_tensors, load_weights


@pytest.mark.parametrize("name", list(tv.CONFIGS))
def test_config_round_trip_and_tensor_names(name, tmp_path):
    cfg = config_from_dict(tv.CONFIGS[name])
    assert cfg.architecture == "Vunepel" and config_from_dict(cfg.to_dict()) == cfg
    want = expected_tensors(Model(build_model_spec(cfg)))
    have = tv.random_tensors(tv.CONFIGS[name], 1)
    assert set(want) == set(have)
    for n, (_, _, _, shape, _) in want.items():
        assert tuple(have[n].shape) == tuple(shape), n
    tv.write_model(tv.CONFIGS[name], str(tmp_path), 1)          # (the folder's config.json has no ranks)
    assert load_model_config(str(tmp_path)) == cfg


def test_run_order_and_what_every_layer_keeps():
    spec = build_model_spec(config_from_dict(tv.CONFIGS["A"]))
    assert [(e.layer, e.cache, e.writes_cache) for e in spec.run_order] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 1, False)]
    needs = Model(spec).cache_needs()
    assert sorted(needs) == [0, 1, 2]
    assert {e.name: (e.shape, e.dtype) for e in needs[0].states} == {
        "S": ((4, 16, 24), "float32"), "conv": ((3, 2 * 2 * 16 + 4 * 24), "compute")}
    assert {e.name: e.shape for e in needs[1].entries} == {"k": (4, 16), "v": (2, 24)}
    assert (needs[1].window, needs[1].chunked) == (40, False)         # chunks of 24 and of 40 read these keys
    needs = Model(build_model_spec(config_from_dict(tv.CONFIGS["B"]))).cache_needs()
    assert needs[0].window is None                                    # two of three readers look at everything
    assert (needs[3].window, needs[3].chunked) == (16, True)
    assert {e.name for e in needs[1].states} == {"S"}                 # one tap keeps no rows
    needs = Model(build_model_spec(config_from_dict(tv.CONFIGS["D"]))).cache_needs()
    assert (needs[1].window, needs[1].chunked) == (100, True)
    assert all(n.kind == "state" for n in Model(build_model_spec(config_from_dict(tv.CONFIGS["E"]))).cache_needs().values())


def test_pages_of_a_chunk_that_is_over_go_back():
    need = CacheNeed("pages", num_kv_heads=1, head_dim=8, window=24, chunked=True)
    m = CacheManager({0: need}, 8, 20, 2)
    m.admit("a")
    for n, held in ((8, 1), (23, 3), (24, 0), (25, 1), (47, 3), (48, 0), (60, 2)):
        m.extend("a", n)
        m.commit("a", n)
        assert m.groups[0].pool.num_used == held, n
    m.check()
    m.release("a")
    assert m.groups[0].pool.num_used == 0
    # pages that straddle a chunk's border stay until the later chunk is over too
    m = CacheManager({0: CacheNeed("pages", num_kv_heads=1, head_dim=8, window=20, chunked=True)}, 8, 20, 2)
    m.admit("a")
    for n, held in ((20, 1), (24, 1), (39, 3), (40, 0)):
        m.extend("a", n)
        m.commit("a", n)
        assert m.groups[0].pool.num_used == held, n
    sliding = CacheNeed("pages", num_kv_heads=1, head_dim=8, window=24)
    assert sliding.group_key() != need.group_key()


def test_loaded_tensors_stand_where_the_parts_expect_them(tmp_path):
    cfg = tv.CONFIGS["C"]
    tv.write_model(cfg, str(tmp_path), 3)
    model = Model(build_model_spec(load_model_config(str(tmp_path))))
    got = load_weights(model, str(tmp_path), torch.float32, "cpu")
    raw = tv.random_tensors(cfg, 3)
    part = model.blocks[0].mixer
    _, where, width = part.layout(part.segments())
    w = got["layers.0.mixer.in.weight"]
    assert w.shape == (width, 100) and width % 8 == 0
    for seg, names in (("qkv", "qkv"), ("a", ("a1",)), ("g", ("g1",)), ("b", ("b",))):
        a, n = where[seg]
        assert torch.equal(w[a:a + n], torch.cat([raw[f"l0.mix.{x}"] for x in names]).float()), seg
    assert torch.equal(got["layers.0.mixer.conv.weight"], torch.cat([raw[f"l0.mix.{x}.conv"] for x in "qkv"]).float())
    assert torch.equal(got["layers.1.mixer.lambdas"][2], raw["l1.mix.lq2"].float())
    assert torch.equal(got["layers.3.ffn.router.weight"][-1:], raw["l3.mlp.shared.sg"].float())
    assert float(got["layers.0.norm.alpha"]) == float(raw["l0.norm1.alpha"])


def test_weight_of_the_second_map():
    from atom_b200.parts import registry
    from atom_b200.parts.spec import PartSpec

    part = registry.build("mixer", PartSpec("differential_attention", dict(
        hidden_size=16, num_heads=2, num_kv_heads=1, key_dim=4, value_dim=4, scale=0.5, diff=0.3, norm_eps=1e-5, qk_norm=False)))
    lam = torch.randn(4, 4, generator=torch.Generator().manual_seed(1))
    part.w_lambdas = lam
    part.after_load()
    P = dict(zip(("lq1", "lk1", "lq2", "lk2"), lam.double()))
    assert abs(part._lambda - float(plain.two_map_weight(P, 0.3))) < 1e-12


def _broken(path, value, name="A"):
    d = copy.deepcopy(tv.CONFIGS[name])
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is None:
        at.pop(path[-1])
    else:
        at[path[-1]] = value
    return d


@pytest.mark.parametrize("path,value,says", [
    (("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "conv"), 0, "conv"), (("layers", 0, "mixer", "decay_rank"), None, "decay_rank"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"), (("layers", 1, "mixer", "diff"), None, "diff"),
    (("layers", 3, "mixer", "kv_from"), 2, "kv_from"), (("layers", 3, "mixer", "kv_from"), 3, "kv_from"),
    (("layers", 3, "mixer", "kv_from"), 9, "kv_from"), (("layers", 3, "mixer", "vdim"), 16, "sizes"),
    (("layers", 0, "mlp", "limit"), None, "limit"), (("layers", 0, "mlp", "kind"), "glu", "kind"),
    (("layers", 1, "mlp", "router", "top"), 7, "top"), (("layers", 1, "mlp", "shared", "ff"), 0, "ff"),
    (("norm", "eps"), 0, "eps"), (("width",), 0, "width"), (("layers",), [], "layers")])
def test_what_cannot_run_is_refused(path, value, says):
    with pytest.raises(ConfigError, match=says.replace(".", r"\.")):
        config_from_dict(_broken(path, value))


def test_plain_chunks_and_shared_keys_differ_from_a_sliding_window():
    seen = plain.visible(10, 4)
    assert [int(r.sum()) for r in seen] == [1, 2, 3, 4, 1, 2, 3, 4, 1, 2]
    assert bool(seen[7, 4]) and not bool(seen[8, 7])
