"""Vipovik's configuration, its tensor declarations, the cache's kept pages and the plain implementation's own consistency
(no GPU)."""
import copy
import json
import os

import numpy as np
import pytest
import torch

import plain_vipovik as pv
from vipovik_helpers import MIXED, ODD, ONE_LAYER, REAL, WIDE, as_numpy, make_weights, tokens_of


def test_round_trip_and_registry():
    import cbis_b200 as cb
    for cfgd in (MIXED, ODD, WIDE, REAL, *ONE_LAYER.values()):
        c = cb.config_from_dict(cfgd)
        assert type(c).__name__ == "VipovikConfig" and cb.config_from_dict(c.to_dict()) == c
        spec = c.model_spec()
        loop = cfgd.get("loop")
        runs = len(cfgd["layers"]) + ((loop["times"] - 1) * (loop["stop"] - loop["start"]) if loop else 0)
        assert len(spec.layers) == runs == len(pv.run_order(len(cfgd["layers"]), loop))
        assert spec.max_positions == 0 and spec.head_spec().params["tensor"] is None
        assert spec.embedding_spec().params["multiplier"] == cfgd.get("embedding", {}).get("scale", 1.0)
    assert cb.config_from_dict(MIXED).to_dict()["layers"][0] == MIXED["layers"][0]


def test_layers_that_run_several_times_share_weights_and_nothing_else():
    import cbis_b200 as cb
    from cbis_b200.cache import cache_groups_of
    from cbis_b200.models import Model
    m = Model(cb.config_from_dict(MIXED).model_spec())
    assert [l.spec.prefix for l in m.layers] == ["l0."] + ["l1.", "l2.", "l3."] * 3 + ["l4."]
    assert [l.spec.pass_input for l in m.layers] == [None, (0, 0), None, None, (0, 1), None, None, (0, 2), None, None, None]
    assert m.layers[4].mixer is m.layers[1].mixer is m.layers[7].mixer and m.layers[5].mixer is not m.layers[1].mixer
    assert m.layers[4].block is not m.layers[1].block
    names = [d.name for d in m.declared()]
    assert len(names) == len(set(names)) and "loop.in" in names and names.count("l2.norm1") == 1
    assert sorted(i for g in cache_groups_of(m, 8) for i in g.layers) == list(range(11))        # a cache for every run
    groups = {(g.need.window, g.need.keep_first): g.layers for g in cache_groups_of(m, 8)}
    assert groups[(21, 5)] == [0] and groups[(13, 9)] == [1, 4, 7] and groups[(6, 33)] == [10] and groups[(40, 0)] == [3, 6, 9]


def test_parts_and_their_constants():
    import cbis_b200 as cb
    layers = cb.config_from_dict(MIXED).model_spec().layers
    assert {l.mixer.kind for l in layers} == {"side_by_side"} and {l.arrangement for l in layers} == {"pre_norm_scaled"}
    p = layers[0].mixer.params
    a, b = p["left"].params, p["right"].params
    assert (p["left_scale"], p["right_scale"]) == (0.8, 1.3)
    assert (a["window"], a["keep_first"], a["cap"], a["scale"], a["rot_dims"], a["rot_blend"]) == (21, 5, 3.0, 0.4, 12, (3.0, 60.0, 12.0, 0.7))
    assert a["turned_norm"] and (b["heads"], b["dim"], b["rank"]) == (3, 20, 10)
    assert layers[1].mixer.params["left"].params["cap"] == 0.0 and layers[2].mixer.params["left"].params["rot_blend"] is None
    f = layers[3].feed_forward.params
    assert (f["limit"], f["beta"], f["up_shift"], f["top"], f["renormalize"], f["renorm_eps"], f["score"]) == (0.7, 1.702, 1.0, 3, True, 1e-20, "softmax")
    assert layers[0].feed_forward.params["activation"] == "gelu_erf" and layers[2].feed_forward.kind == "nothing"


def test_declared_tensors_follow_the_sizes():
    import cbis_b200 as cb
    from cbis_b200.models import Model
    decl = {d.name: tuple(d.shape) for d in Model(cb.config_from_dict(MIXED).model_spec()).declared()}
    assert decl["embed"] == (90, 64) and decl["final.norm"] == (64,) and "head" not in decl
    assert decl["loop.in"] == (64, 128) and decl["loop.step"] == (3, 64)
    assert decl["l0.mix.left.q"] == (64, 64) and decl["l0.mix.left.k"] == (32, 64) and decl["l0.mix.left.v"] == (48, 64)
    assert decl["l0.mix.left.o"] == (64, 96) and decl["l0.mix.right.o"] == (64, 60) and decl["l0.mix.right.g"] == (60, 64)
    assert decl["l0.mix.right.w1"] == (10, 64) and decl["l0.mix.right.w2"] == (60, 10) and decl["l0.mix.right.w0"] == (60,)
    assert decl["l0.mix.right.u"] == (3, 20) and decl["l0.mix.right.norm"] == (60,) and decl["l0.mix.right.mu.w"] == (64,)
    assert decl["l1.mlp.router"] == (5, 64) and decl["l1.mlp.e4.down"] == (64, 24) and decl["l0.mlp.up"] == (72, 64)
    assert "l2.norm2" not in decl and "l5.norm1" not in decl


def test_a_size_that_only_the_tensors_tell(tmp_path):
    """A folder whose config.json does not give the rows of the decays' narrow matrices: the tensors' shapes do."""
    import cbis_b200 as cb
    from cbis_b200.models import load_model
    from cbis_b200.weights.safetensors_io import write_safetensors
    bare = copy.deepcopy(MIXED)
    for l in bare["layers"]:
        del l["mixer"]["right"]["decay_rank"]
    w = make_weights(MIXED, 5)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(bare, f)
    write_safetensors(os.path.join(tmp_path, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})
    m = load_model(str(tmp_path), "float32", "cpu")
    assert [l.mixer.right.rank for l in m.layers[:4]] == [10, 24, 8, 12] and m.config == cb.config_from_dict(MIXED)
    with pytest.raises(cb.ConfigError, match="decay_rank"):
        cb.config_from_dict(bare).model_spec()


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="serial"), "is not one of"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "integer >= 1"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "integer >= 0"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-2.0), "positive"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "'right' is missing"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "exceeds"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "is not one of"),
    (lambda c: c["loop"].update(stop=6), "name no run"),
    (lambda c: c["loop"].update(start=4), "name no run"),
    (lambda c: c["loop"].update(times=0), "integer >= 1"),
    (lambda c: c["norm"].pop("eps"), "'eps' is missing"),
])
def test_what_a_configuration_refuses(change, message):
    import cbis_b200 as cb
    cfgd = copy.deepcopy(MIXED)
    change(cfgd)
    with pytest.raises(cb.ConfigError, match=message):
        cb.config_from_dict(cfgd)


def test_what_parts_and_models_refuse():
    import dataclasses

    import cbis_b200 as cb
    from cbis_b200.config import PartSpec
    from cbis_b200.models import Model
    from cbis_b200.parts.base import make_mixer
    base = {"width": 32, "n_head": 4, "n_kv_head": 2, "head_dim": 8, "v_head_dim": 8, "scale": 1.0}
    mix = PartSpec("time_mixing", {"width": 32, "heads": 2, "dim": 8, "rank": 4, "eps": 1e-5})
    with pytest.raises(ValueError, match="needs a window"):
        make_mixer(PartSpec("rotary_attention", {**base, "keep_first": 4}))
    with pytest.raises(ValueError, match="turned_norm"):
        make_mixer(PartSpec("rotary_attention", {**base, "turned_norm": True, "qk_norm": True}))
    with pytest.raises(ValueError, match="outside"):
        make_mixer(PartSpec("time_mixing", {"width": 32, "heads": 1, "dim": 513, "rank": 4, "eps": 1e-5}))
    rot = PartSpec("rotary_attention", base)
    with pytest.raises(ValueError, match="keep a cache"):
        make_mixer(PartSpec("side_by_side", {"width": 32, "left": rot, "right": rot}))
    with pytest.raises(ValueError, match="keep a state"):
        make_mixer(PartSpec("side_by_side", {"width": 32, "left": mix, "right": mix}))
    with pytest.raises(ValueError, match="does not offer"):
        make_mixer(PartSpec("side_by_side", {"width": 32, "left": PartSpec("gated_attention", base), "right": mix}))
    spec = cb.config_from_dict(MIXED).model_spec()
    layers = list(spec.layers)
    layers[4] = dataclasses.replace(layers[4], weights_from=6)
    with pytest.raises(ValueError, match="no earlier layer"):
        Model(dataclasses.replace(spec, layers=tuple(layers)))


def test_pages_of_the_first_tokens_stay_while_others_behind_the_window_go_back():
    from cbis_b200.kernels.library import host
    h = host()
    for ps, window, keep in ((4, 6, 5), (8, 3, 8), (4, 1, 0), (16, 40, 1), (4, 5, 30)):
        m = h.CacheManager([h.GroupSpec(ps, 64, window, keep)], 2)
        assert m.keep_first(0) == keep
        s = m.admit(1)
        for length in range(1, 90):
            assert m.append(s, 1)
            m.release_out_of_window(s)
            table = m.block_table(s, 0)
            for lp, page in enumerate(table):
                keys = range(lp * ps, min((lp + 1) * ps, length))
                needed = any(j < keep or length - j < window for j in keys) or (lp + 1) * ps > length
                assert (page >= 0) == needed or (page >= 0 and lp * ps < keep), (ps, window, keep, length, lp)
            assert m.check() == ""
        m.release(s)
        assert m.free_pages(0) == 64
    # what a request of n tokens may hold at a time: the window, the portion, a page of rounding, the kept pages
    small = h.CacheManager([h.GroupSpec(4, 6, 8, 5)], 1)
    assert small.fits_at_all(1000, 4) and not small.fits_at_all(1000, 8)


def test_the_plain_implementation_agrees_with_itself():
    """Rows of a prompt do not depend on what follows; the recurrence can be cut anywhere; a mask's edges; a cap that is far
    away caps nothing; a rotation depends on distances alone."""
    w = as_numpy(make_weights(MIXED, 3))
    toks = tokens_of(MIXED, 50, 1)
    full, streams, _ = pv.forward(MIXED, w, toks)
    part, _, _ = pv.forward(MIXED, w, toks[:31])
    assert np.abs(full[:31] - part).max() < 1e-9 and streams.shape == (11, 50, 64)
    g = np.random.default_rng(0)
    r, k, v = (g.normal(size=(20, 2, 5)) for _ in range(3))
    wd, u = g.uniform(0.2, 1.0, size=(20, 2, 5)), g.normal(size=(2, 5))
    o, S = pv.recurrence(r, k, v, wd, u)
    o1, S1 = pv.recurrence(r[:7], k[:7], v[:7], wd[:7], u)
    o2, S2 = pv.recurrence(r[7:], k[7:], v[7:], wd[7:], u, S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    kv = [np.einsum("hk,hv->hkv", k[t], v[t]) for t in range(3)]
    by_hand = np.einsum("hkv,hk->hv", wd[1][:, :, None] * kv[0] + kv[1] + u[:, :, None] * kv[2], r[2])
    assert np.allclose(o[2], by_hand)
    ok = pv.seen(np.arange(12), {"size": 4, "keep_first": 2})
    assert ok[9].tolist() == [True, True, False, False, False, False, True, True, True, True, False, False]
    rot = {"base": 50.0, "dims": 6, "scaling": {"factor": 2.0, "original": 40, "fast": 4.0, "slow": 0.5}}
    q, kk = g.normal(size=(1, 1, 8)), g.normal(size=(1, 1, 8))
    dots = [float((pv.rotate(q, [p + 3], rot) * pv.rotate(kk, [p], rot)).sum()) for p in (0, 5, 200)]
    assert np.allclose(dots, dots[0])
    f, length = pv.frequencies(rot)
    assert length == pytest.approx(1 + 0.1 * np.log(2)) and f[0] == 1.0 and f[-1] == pytest.approx(50.0 ** (-2 / 3) / 2)
    assert np.allclose(pv.soft_cap(np.array([0.3, -2.0]), 1e6), [0.3, -2.0])
