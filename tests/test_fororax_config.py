"""Fororax's configuration, its tensor declarations and the plain implementation's own consistency (no GPU)."""
import copy

import numpy as np
import pytest

import plain_fororax as pf
from fororax_helpers import MIXED, ODD, ONE_LAYER, REAL, WIDE, as_numpy, make_weights, tokens_of


def test_round_trip_and_registry():
    import cbis_b200 as cb
    for cfgd in (MIXED, ODD, WIDE, REAL, *ONE_LAYER.values()):
        c = cb.config_from_dict(cfgd)
        assert type(c).__name__ == "FororaxConfig" and cb.config_from_dict(c.to_dict()) == c
        spec = c.model_spec()
        assert [l.arrangement for l in spec.layers] == ["post_norm"] * len(cfgd["layers"])
        assert all(l.stream_scale == cfgd.get("postln_alpha", 1.0) for l in spec.layers)
        assert spec.max_positions == cfgd["max_positions"] and spec.vocab_size == cfgd["vocab"]
        assert spec.head_spec().params["soft_cap"] == cfgd.get("logit_softcap", 0.0)
        assert spec.embedding_spec().params["multiplier"] == cfgd.get("embedding", {}).get("scale", 1.0)
        assert spec.position.kind == "learned"
    assert cb.config_from_dict(MIXED).to_dict()["layers"][0] == MIXED["layers"][0]


def test_parts_and_their_constants():
    import cbis_b200 as cb
    layers = cb.config_from_dict(MIXED).model_spec().layers
    assert [l.mixer.kind for l in layers] == ["gated_attention"] * 6
    assert [l.cache_source for l in layers] == [None, None, 0, None, 1, None]
    a, b = layers[0].mixer.params, layers[1].mixer.params
    assert a["log_bias"] and a["qk_norm"] and not (a["sinks"] or a["talk"] or a["qkv_bias"] or a["out_bias"]) and a["gate"] is None
    assert b["sinks"] and b["talk"] and b["qkv_bias"] and b["out_bias"] and b["gate"] == "element" and not b["log_bias"]
    assert (a["head_dim"], a["v_head_dim"], a["scale"], a["own_kv"]) == (16, 24, 0.25, True)
    assert not layers[2].mixer.params["own_kv"] and not layers[4].mixer.params["own_kv"]
    f = layers[4].feed_forward.params
    assert (f["limit"], f["shared_limit"], f["beta"], f["up_shift"], f["identity"], f["top"]) == (2.0, 1.7, 1.702, 1.0, 0, 4)
    assert f["score"] == "softmax" and not f["renormalize"] and f["weight_on"] == "output" and f["correction"] and f["shared_gate"]
    assert layers[1].feed_forward.params["shared_inner"] == 0 and layers[3].feed_forward.kind == "nothing"


def test_declared_tensors_follow_the_sizes():
    import cbis_b200 as cb
    from cbis_b200.models import Model
    decl = {d.name: tuple(d.shape) for d in Model(cb.config_from_dict(MIXED).model_spec()).declared()}
    assert decl["embed"] == (90, 64) and decl["pos"] == (320, 64) and decl["head"] == (90, 64) and decl["final.norm"] == (64,)
    assert decl["l0.mix.q"] == (64, 64) and decl["l0.mix.k"] == (32, 64) and decl["l0.mix.v"] == (48, 64)
    assert decl["l0.mix.q.norm"] == (16,) and decl["l0.mix.k.norm"] == (16,) and decl["l0.mix.o"] == (64, 96)
    assert decl["l0.mix.r1"] == (4,) and decl["l0.mix.r2"] == (4,)
    assert not any(n in decl for n in ("l0.mix.q.b", "l0.mix.g", "l0.mix.sink", "l0.mix.talk", "l1.mix.r1", "l1.mix.g.b"))
    assert decl["l1.mix.q.b"] == (144,) and decl["l1.mix.k.b"] == (72,) and decl["l1.mix.v.b"] == (48,) and decl["l1.mix.o.b"] == (64,)
    assert decl["l1.mix.talk"] == (6, 6) and decl["l1.mix.sink"] == (6,) and decl["l1.mix.g"] == (96, 64)
    assert not any(n in decl for n in ("l2.mix.k", "l2.mix.v", "l2.mix.k.norm", "l4.mix.v")) and decl["l2.mix.q.norm"] == (16,)
    assert decl["l0.mlp.router"] == (7, 64) and decl["l0.mlp.correction"] == (7,) and decl["l0.mlp.e4.down"] == (64, 24)
    assert "l0.mlp.e5.down" not in decl and decl["l0.mlp.shared.sg"] == (1, 64) and decl["l0.mlp.shared.up"] == (40, 64)
    assert "l1.mlp.shared.sg" not in decl and "l3.norm2" not in decl and "l3.mlp.router" not in decl


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "is not one of"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "keeps no keys and values"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "differs from layer 0"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "exceeds"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "is not one of"),
    (lambda c: c.pop("max_positions"), "'max_positions' is missing"),
    (lambda c: c.update(logit_softcap=-1.0), "positive"),
])
def test_what_a_configuration_refuses(change, message):
    import cbis_b200 as cb
    cfgd = copy.deepcopy(MIXED)
    change(cfgd)
    with pytest.raises(cb.ConfigError, match=message):
        cb.config_from_dict(cfgd)


def test_what_parts_refuse():
    from cbis_b200.parts.base import make_block, make_mixer, make_norm
    from cbis_b200.parts.dense import NoFeedForward
    from cbis_b200.config import PartSpec
    base = {"width": 32, "n_head": 4, "n_kv_head": 2, "head_dim": 8, "v_head_dim": 8, "scale": 1.0}
    with pytest.raises(ValueError, match="one distance bias"):
        make_mixer(PartSpec("gated_attention", {**base, "slope_power": 8.0, "log_bias": True}))
    with pytest.raises(ValueError, match="gate"):
        make_mixer(PartSpec("gated_attention", {**base, "gate": "row"}))
    mixer = make_mixer(PartSpec("gated_attention", base))
    ln = make_norm(PartSpec("layernorm", {"width": 32, "eps": 1e-5}))
    with pytest.raises(ValueError, match="root-mean-square"):
        make_block("post_norm", mixer, NoFeedForward(32), ln, ln)


def test_the_plain_implementation_agrees_with_itself():
    """Rows of a prompt do not depend on what follows; an identity matrix mixes nothing; without a rate the bias is none;
    a sink takes its share; an identity expert hands its input on."""
    w = as_numpy(make_weights(MIXED, 3))
    toks = tokens_of(MIXED, 50, 1)
    full, streams, _ = pf.forward(MIXED, w, toks)
    part, _, _ = pf.forward(MIXED, w, toks[:31])
    assert np.abs(full[:31] - part).max() < 1e-9 and streams.shape == (6, 50, 64)
    g = np.random.default_rng(0)
    q, k, v = g.normal(size=(30, 4, 5)), g.normal(size=(30, 2, 5)), g.normal(size=(30, 2, 3))
    pos = np.arange(30)
    bare = pf.attention_rows(q, k, v, 0.5, pos)
    assert np.allclose(pf.attention_rows(q, k, v, 0.5, pos, talk=np.eye(4)), bare)
    assert np.allclose(pf.attention_rows(q, k, v, 0.5, pos, r1=np.ones(4), r2=np.zeros(4)), bare)
    assert np.allclose(bare[0], v[0][[0, 0, 1, 1]])
    lone = pf.attention_rows(q[:1], k[:1], v[:1], 0.5, pos[:1], sinks=np.log([1.0, 3.0, 1.0, 3.0]))
    e = np.exp(0.5 * np.array([q[0, h] @ k[0, h // 2] for h in range(4)]))
    assert np.allclose(lone[0], v[0][[0, 0, 1, 1]] * (e / (e + np.array([1.0, 3.0, 1.0, 3.0])))[:, None])
    # heads mixed: what one head puts on a key, another may take to its own key/value head's value
    swap = np.zeros((4, 4))
    swap[0, 3] = 1.0
    own = pf.causal_weights(np.stack([q[:, h] @ k[:, h // 2].T for h in range(4)]) * 0.5, pos)
    assert np.allclose(pf.attention_rows(q, k, v, 0.5, pos, talk=swap)[:, 0], own[3] @ v[:, 0])
    h = g.normal(size=(6, 8))
    f = {"router": {"experts": 1, "identity": 2, "top": 2}, "expert": {"ff": 4, "limit": 1.0}}
    t = {"m.router": g.normal(size=(3, 8)), "m.correction": np.array([-9.0, 0.0, 0.0])}
    out, _ = pf.routed_ff(f, t, "m.", h)
    z = np.exp(h @ t["m.router"].T)
    assert np.allclose(out, h * ((z[:, 1] + z[:, 2]) / z.sum(1))[:, None])
