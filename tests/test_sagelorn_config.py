"""The Sagelorn configuration on the host: what config.json gives, what is refused, what may be absent, the tensors, states
and cache groups the specification asks for (keys borrowed through another mask), and controls that the plain
implementation would notice a wrong reading."""
import copy

import numpy as np
import pytest

import sagelorn_models as sm
from helpers import rel_err
from mynah_slm_b200.config.keys import ConfigError
from mynah_slm_b200.engine.model import Model
from mynah_slm_b200.registry import known_architectures, parse_config
from plain import sagelorn as plain


def test_registered_and_round_trips():
    assert "Sagelorn" in known_architectures()
    for cfg in sm.CONFIGS.values():
        assert parse_config(cfg).to_dict() == cfg


def test_tensors():
    for name, cfg in sm.CONFIGS.items():
        model = Model(parse_config(cfg).model_spec())
        want = sm.tensor_shapes(cfg, q_rank=-1)                           # a size the configuration does not name is the tensors'
        got = {ts.name: tuple(ts.shape) for _, ts in model.tensor_specs() if not ts.ignorable}
        assert got == want, name


def test_borrowed_keys_and_cache_groups():
    spec = parse_config(sm.HYBRID).model_spec()
    assert [e.cache_from for e in spec.schedule] == [None, None, 0, None, None, None, 0, None]
    plan = Model(spec).cache_plan()
    groups = {(g.kv_heads, g.head_dim, g.v_head_dim, g.window): list(g.entries) for g in plan.groups}
    # layer 0 looks 40 back, but layer 2 reads its keys 70 back: that is what is kept
    assert groups == {(2, 64, 64, 70): [0], (1, 64, 0, 24): [1], (1, 64, 64, None): [4], (1, 64, 0, None): [7]}
    assert [e.source for e in plan.entries] == [None, None, 0, None, None, None, 0, None]
    assert {k: tuple(v.shape) for k, v in plan.entries[3].state.items()} == {"S": (3, 24, 16)}
    assert tuple(plan.embedding_state.shape) == ()
    # a reader without a window needs every key
    cfg = copy.deepcopy(sm.HYBRID)
    del cfg["layers"][6]["mixer"]["mask"]
    assert Model(parse_config(cfg).model_spec()).cache_plan().groups[0].window is None
    # readers that look less far change nothing
    cfg = copy.deepcopy(sm.HYBRID)
    cfg["layers"][2]["mixer"]["mask"]["size"] = 39
    assert Model(parse_config(cfg).model_spec()).cache_plan().groups[0].window == 40


def _broken(path, value, base=sm.HYBRID):
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
    (("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "scale"), None, "scale"), (("layers", 0, "mixer", "rot"), None, "rot"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 0, "mixer", "rot", "scaling", "low"), None, "low"),
    (("layers", 0, "mixer", "rot", "scaling", "low"), 4.0, "low and high"), (("layers", 0, "mixer", "mask", "size"), 0, "size"),
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 1, "mixer", "kv_rank"), None, "kv_rank"),
    (("layers", 1, "mixer", "rot", "dims"), 10, "rot.dims"), (("layers", 1, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 6, "mixer", "kv_from"), 2, "kv_from"), (("layers", 6, "mixer", "kv_from"), 4, "differs"),
    (("layers", 3, "mixer", "decay"), [0.5], "decay"), (("layers", 3, "mixer", "decay"), [0.5, 0.5, -0.1], "decay"),
    (("layers", 1, "mlp", "router", "top"), 7, "top"), (("layers", 1, "mlp", "shared", "ff"), None, "ff"),
    (("layers", 4, "mlp", "kind"), "sparse", "kind"), (("norm",), None, "norm"), (("logit_scale",), None, "logit_scale"),
    (("embedding", "bigram", "buckets"), 0, "buckets"), (("embedding", "bigram", "mul_cur"), None, "mul_cur"), (("vocab",), 2.5, "vocab")])
def test_refusals_name_the_key(path, value, word):
    with pytest.raises(ConfigError) as e:
        parse_config(_broken(path, value))
    assert word in str(e.value)


def test_what_may_be_absent():
    spec = parse_config(sm.HYBRID).model_spec()
    assert spec.layers[3].ffn is None and "ffn" not in spec.layers[3].norms
    assert spec.layers[5].ffn["shared"] is None and spec.layers[7].mixer["q_rank"] == -1 and spec.layers[7].mixer["window"] is None
    assert spec.layers[4].mixer["rot"]["scaling"] is None


# ------------------------------------------------------------------ controls on the plain implementation
def _logits(cfg, W, n=90, seed=3):
    toks = np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()
    return plain.forward(cfg, W, toks)


def test_the_plain_implementation_notices_a_wrong_reading():
    cfg, W = sm.HYBRID, sm.as_numpy(sm.weights_of("hybrid"))
    ref = _logits(cfg, W)
    for path, value in ((("layers", 0, "mixer", "mask", "size"), 39), (("layers", 1, "mixer", "mask", "size"), 25),
                        (("layers", 2, "mixer", "mask", "size"), 69), (("layers", 6, "mixer", "mask", "size"), 10),
                        (("layers", 0, "mixer", "rot", "scaling", "factor"), 3.0), (("layers", 0, "mixer", "rot", "scaling", "high"), 6.0),
                        (("layers", 1, "mixer", "rot", "base"), 200.0), (("layers", 2, "mixer", "scale"), 0.42),
                        (("layers", 3, "mixer", "decay"), [0.9, 0.98, 0.995]), (("layers", 2, "mlp", "router", "top"), 2),
                        (("logit_scale",), 0.71), (("embedding", "bigram", "mul_prev"), 28), (("embedding", "bigram", "buckets"), 96)):
        assert rel_err(ref, _logits(_broken(path, value), W)) > 1e-3, path
    for name in ("l0.mix.sink", "l6.mix.sink", "l2.mix.q.norm", "l0.mix.k.norm", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l1.mix.g",
                 "l3.norm1", "final.norm", "l1.mlp.router", "l1.mlp.shared.up", "l5.mlp.e1.down"):
        Wo = dict(W)
        Wo[name] = W[name] * 1.3 + 0.05
        assert rel_err(ref, _logits(cfg, Wo)) > 1e-4, name
    Wo = dict(W, bigram=W["bigram"].copy())
    Wo["bigram"][-1] += 1.0                                              # the row of a sequence's first token
    assert rel_err(ref[:1], _logits(cfg, Wo)[:1]) > 1e-2


def test_sinks_take_their_share():
    s = np.array([[-2.0, 9.0], [0.5, 1.5]])
    see = plain.visible(2, None)
    p = plain.softmax_rows(s, see, 0.7)
    assert np.allclose(p[0], [np.exp(-2.0) / (np.exp(0.7) + np.exp(-2.0)), 0.0])
    assert np.allclose(p[1], np.exp([0.5, 1.5]) / (np.exp(0.7) + np.exp(0.5) + np.exp(1.5)))
    assert np.allclose(plain.softmax_rows(s, see, -1e4)[1], plain.softmax_rows(s, see)[1])


def test_windows_and_pair_rows():
    assert plain.visible(6, {"size": 3}).sum(-1).tolist() == [1, 2, 3, 3, 3, 3]
    assert plain.visible(4, {"size": 1}).sum(-1).tolist() == [1, 1, 1, 1]
    rows = plain.pair_rows([5, 9, 0, 9], {"buckets": 13, "mul_prev": 3, "mul_cur": 7})
    assert rows.tolist() == [13, (15 + 63) % 13, 27 % 13, 63 % 13]


def test_the_weight_stands_on_the_experts_input():
    """With a squared activation a weight on the input counts twice: half the input gives a quarter of the output."""
    W = {"router": np.zeros((1, 2)), "e0.up": np.eye(2), "e0.down": np.eye(2)}
    mlp = {"router": {"experts": 1, "top": 1}}
    out = plain.routed_ff(np.array([[2.0, -3.0]]), W, "", mlp)            # sigmoid(0) = 1/2
    assert np.allclose(out, [[1.0, 0.0]])


def test_frequencies_against_the_rotation_part():
    from mynah_slm_b200.parts.position import rotary_frequencies
    for dims, base, scaling in ((20, 400000.0, (3.0, 1.0, 4.0, 128)), (12, 500.0, (8.0, 0.5, 6.0, 60)), (8, 300.0, None)):
        rot = sm.rotation(dims, base, scaling)
        sc = {"kind": "wavelength", **rot["scaling"]} if scaling else None
        got, mult = rotary_frequencies(dims, base, sc)
        assert mult == 1.0 and np.allclose(got, plain.pair_frequencies(rot), rtol=1e-14)
    f, f0 = plain.pair_frequencies(sm.rotation(20, 400000.0, (3.0, 1.0, 4.0, 128))), plain.pair_frequencies(sm.rotation(20, 400000.0))
    kinds = {"kept": np.isclose(f, f0), "divided": np.isclose(f, f0 / 3.0)}
    assert kinds["kept"].any() and kinds["divided"].any() and (~kinds["kept"] & ~kinds["divided"]).any()
