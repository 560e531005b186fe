"""The Buludra configuration on the host: what config.json gives, what is refused, what may be absent, layers that run
with another layer's weights, the tensors and cache groups the specification asks for, and controls that the plain
implementation would notice a wrong reading."""
import copy

import numpy as np
import pytest

import buludra_models as bm
from helpers import rel_err
from mynah_slm_b200.config.keys import ConfigError
from mynah_slm_b200.engine.model import Model
from mynah_slm_b200.registry import known_architectures, parse_config
from plain import buludra as plain


def test_registered_and_round_trips():
    assert "Buludra" in known_architectures()
    for cfg in bm.CONFIGS.values():
        typed = parse_config(cfg)
        assert parse_config(typed.to_dict()).to_dict() == typed.to_dict()
        back = typed.to_dict()
        assert back["layers"] == cfg["layers"] and back.get("logit_softcap") == cfg.get("logit_softcap")


def test_layers_that_run_again():
    spec = parse_config(bm.HYBRID).model_spec()
    assert [L.prefix for L in spec.layers] == ["l0.", "l1.", "l2.", "l3.", "l4."]
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 4, 0, 1, 2, 4]
    assert all(e.cache_from is None for e in spec.schedule)               # a cache and a state of its own, every time
    # a layer may name one that stands behind it, or one that itself names another
    layers = [bm.bare(bm.gla(2, 8, 8, 4.0)), bm.bare(bm.gla(2, 8, 8, 4.0)), bm.bare(bm.gla(2, 8, 8, 4.0))]
    layers[0]["weights_of"], layers[2]["weights_of"] = 1, 0
    spec = parse_config(bm.config(32, 50, layers)).model_spec()
    assert [L.prefix for L in spec.layers] == ["l1."] and [e.layer for e in spec.schedule] == [0, 0, 0]


def test_tensors_and_cache_groups():
    for name, cfg in bm.CONFIGS.items():
        model = Model(parse_config(cfg).model_spec())
        want = bm.tensor_shapes(cfg, rank=-1)                             # the narrow size is the checkpoint's
        got = {ts.name: tuple(ts.shape) for _, ts in model.tensor_specs() if not ts.ignorable}
        assert got == want, name
    plan = Model(parse_config(bm.HYBRID).model_spec()).cache_plan()
    # keys and values lie in heads of 64 (the tensor-core kernels' widths); (kv heads, key width, value width) -> runs kept there
    groups = {(g.kv_heads, g.head_dim, g.v_head_dim): list(g.entries) for g in plan.groups}
    assert groups == {(2, 64, 64): [1, 6], (3, 64, 64): [2, 4, 7, 8], (1, 64, 64): [3]}
    assert all(g.window is None for g in plan.groups)
    states = [sorted(e.state) if e.state else None for e in plan.entries]
    assert states == [["S"], ["1"], None, None, ["1"], ["S"], ["1"], None, ["1"]]
    assert {k: tuple(v.shape) for k, v in plan.entries[6].state["1"].items()} == {"S": (2, 8, 16), "n": (2, 8), "m": (2,)}


def _broken(path, value, base=bm.HYBRID):
    cfg = copy.deepcopy(base)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    return cfg


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "tau"), None, "tau"), (("layers", 0, "mixer", "tau"), 0.0, "tau"),
    (("layers", 1, "mixer", "left_scale"), None, "left_scale"), (("layers", 1, "mixer", "left", "rot"), None, "rot"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 18, "rot.dims"), (("layers", 1, "mixer", "right", "gate_cap"), None, "gate_cap"),
    (("layers", 2, "mixer", "kv_heads"), 4, "kv_heads"), (("layers", 2, "mixer", "q_temp", "every"), 0, "every"),
    (("layers", 3, "mixer", "scale"), None, "scale"), (("layers", 1, "mlp", "router", "groups", "count"), 4, "groups"),
    (("layers", 1, "mlp", "router", "top"), 5, "top"), (("layers", 1, "mlp", "shared", "ff"), None, "ff"),
    (("layers", 4, "mlp", "kind"), "sparse", "kind"), (("layers", 5, "weights_of"), 5, "weights_of"),
    (("layers", 5, "weights_of"), 9, "weights_of"), (("layers", 5, "weights_of"), 3, "not like"), (("norm",), None, "norm"),
    (("logit_softcap",), -1.0, "logit_softcap"), (("vocab",), 2.5, "vocab")])
def test_refusals_name_the_key(path, value, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(path, value))
    assert word in str(e.value)


def test_what_may_be_absent():
    spec = parse_config(bm.HYBRID).model_spec()
    ffn = spec.layers[2].ffn
    assert (ffn["groups"], ffn["keep"], ffn["shared"]) == (1, 1, 24)
    assert spec.layers[3].mixer["q_temp"] is None and spec.layers[3].ffn is None and "ffn" not in spec.layers[3].norms
    assert parse_config(bm.ODD).model_spec().head["logit_softcap"] is None
    assert parse_config(bm.ODD).model_spec().layers[0].ffn["shared"] is None


# ------------------------------------------------------------------ controls on the plain implementation
def _logits(cfg, W, n=90, seed=3):
    toks = np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()
    return plain.forward(cfg, W, toks)


def test_the_plain_implementation_notices_a_wrong_reading():
    cfg, W = bm.HYBRID, bm.as_numpy(bm.weights_of("hybrid"))
    ref = _logits(cfg, W)
    for layers, path, value in (((0, 5), ("mixer", "tau"), 7.0), ((1, 6), ("mixer", "left_scale"), 0.9), ((1, 6), ("mixer", "right_scale"), 1.2),
                                ((1, 6), ("mixer", "left", "rot", "base"), 400.0), ((1, 6), ("mixer", "left", "rot", "dims"), 16),
                                ((1, 6), ("mixer", "right", "gate_cap"), 2.0), ((2, 7), ("mixer", "q_temp", "every"), 19),
                                ((2, 7), ("mixer", "q_temp", "coef"), 0.5), ((1, 6), ("mlp", "router", "groups", "keep"), 1),
                                ((2, 7), ("mlp", "router", "top"), 2), ((3,), ("mixer", "scale"), 0.35)):
        other = cfg
        for i in layers:
            other = _broken(("layers", i) + path, value, other)
        assert rel_err(ref, _logits(other, W)) > 1e-3, path
    assert rel_err(ref, _logits(_broken(("logit_softcap",), 15.0), W)) > 1e-3
    for name in ("l0.mix.a2.b", "l0.mix.norm", "l1.mix.right.f.b", "l1.mix.right.i.b", "l1.mix.right.norm", "l2.mix.q.norm",
                 "l1.mlp.shared.sg", "l1.mlp.router"):
        Wo = dict(W)
        Wo[name] = W[name] * 1.5 + 0.05
        assert rel_err(ref, _logits(cfg, Wo)) > 1e-4, name
    before = plain.softmax_rows
    plain.softmax_rows = lambda s, null=False: before(s)
    try:
        assert rel_err(ref, _logits(cfg, W)) > 1e-2, "a missing null key goes unseen"
    finally:
        plain.softmax_rows = before
    # a layer that runs again has a state of its own: without the second run of layer 0 the logits are others
    fewer = copy.deepcopy(cfg)
    del fewer["layers"][5]
    assert rel_err(ref, _logits(fewer, W)) > 1e-2


def test_null_key_and_unit_norms_in_the_plain_implementation():
    s = np.array([[-2.0, 9.0], [0.5, 1.5]])
    p = plain.softmax_rows(s, null=True)
    assert np.allclose(p[0], [np.exp(-2.0) / (1 + np.exp(-2.0)), 0.0])
    assert np.allclose(p[1], np.exp([0.5, 1.5]) / (1 + np.exp(0.5) + np.exp(1.5)))
    assert np.allclose(plain.softmax_rows(s)[1].sum(), 1.0)
    x = np.random.default_rng(0).normal(size=(5, 2, 8))                  # a turn leaves the mean square alone
    rot = {"dims": 6, "base": 50.0}
    assert np.allclose(plain.rms_unit(plain.turn_halves(x, rot), 1e-5), plain.turn_halves(plain.rms_unit(x, 1e-5), rot))


def test_groups_leave_better_experts_out():
    """The second best expert sits outside the best group: with one group kept it is left out, with two it comes back;
    the weights are softmax scores over ALL experts."""
    W = {"router": np.array([[3.0], [0.0], [2.0], [1.9], [-1.0], [-1.0]])}
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    picked, weights = plain.pick_experts(np.ones((1, 1)), W, "", router)
    z = np.exp(W["router"][:, 0])
    assert picked[0].tolist() == [0, 1] and np.allclose(weights[0], z[[0, 1]] / z.sum())
    router["groups"]["keep"] = 2
    assert plain.pick_experts(np.ones((1, 1)), W, "", router)[0][0].tolist() == [0, 2]


def test_query_temperature_steps():
    t = plain.query_temperature(10, {"coef": 0.5, "every": 4})
    assert np.allclose(t[:3], 1.0) and np.allclose(t[3:7], 1.0 + 0.5 * np.log(2.0)) and np.allclose(t[7:], 1.0 + 0.5 * np.log(3.0))
    from mynah_slm_b200.parts.attention_capped import query_temperatures
    for every in (1, 3, 7, 64, 0.7):
        assert np.allclose(query_temperatures(3000, -0.3, every, "cpu").numpy(), plain.query_temperature(3000, {"coef": -0.3, "every": every}), atol=1e-6)
