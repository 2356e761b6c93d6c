"""Nufavik without a device: the configuration's round trip and its errors, what the layers keep per request, the
declared tensors, and the plain model's own properties."""

import copy

import numpy as np
import pytest

import nufavik_helpers as nf
import plain_nufavik as plain
from mini_llm_b200.config import ConfigError, config_from_dict, describe_model
from mini_llm_b200.engine.model import Model
from mini_llm_b200.parts.base import build_part
from mini_llm_b200.parts.spec import FixedState, PagedKV, PartSpec


def test_round_trip():
    raw = nf.full_stack()
    parsed = config_from_dict(raw)
    assert parsed.architecture == "Nufavik" and parsed.embedding_scale == 3.0
    assert parsed.to_dict() == raw
    assert config_from_dict(parsed.to_dict()) == parsed


def _changed(raw, path, value):
    raw = copy.deepcopy(raw)
    node = raw
    for key in path[:-1]:
        node = node[key]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return raw


@pytest.mark.parametrize("path, value, named", [
    (["width"], None, "width"), (["vocab"], -3, "vocab"), (["norm", "eps"], None, "norm.eps"),
    (["embedding", "scale"], None, "embedding.scale"), (["embedding"], None, "embedding"), (["layers"], [], "layers"),
    (["layers", 0, "type"], "hyena", "layers[0].type"), (["layers", 0, "mixer"], 7, "layers[0].mixer"),
    (["layers", 0, "mixer", "conv"], None, "layers[0].mixer.conv"), (["layers", 0, "mixer", "conv"], 0, "layers[0].mixer.conv"),
    (["layers", 1, "mixer", "heads"], 5, "layers[1].mixer.heads"), (["layers", 1, "mixer", "scale"], "x", "layers[1].mixer.scale"),
    (["layers", 1, "mixer", "rot", "dims"], 18, "layers[1].mixer.rot.dims"), (["layers", 1, "mixer", "rot", "dims"], 7, "layers[1].mixer.rot.dims"),
    (["layers", 1, "mixer", "rot", "base"], 1.0, "layers[1].mixer.rot.base"),
    (["layers", 2, "mixer", "mask", "size"], 0, "layers[2].mixer.mask.size"),
    (["layers", 2, "mixer", "mask", "keep_first"], -1, "layers[2].mixer.mask.keep_first"),
    (["layers", 2, "mixer", "mask", "keep_first"], None, "layers[2].mixer.mask.keep_first"),
    (["layers", 0, "mlp", "kind"], "dense", "layers[0].mlp.kind"), (["layers", 0, "mlp", "router", "top"], 8, "layers[0].mlp.router.top"),
    (["layers", 0, "mlp", "router", "identity"], -1, "layers[0].mlp.router.identity"),
    (["layers", 0, "mlp", "router", "scale"], None, "layers[0].mlp.router.scale"),
    (["layers", 0, "mlp", "expert", "ff"], 0, "layers[0].mlp.expert.ff"),
])
def test_errors_name_their_key(path, value, named):
    with pytest.raises(ConfigError) as error:
        config_from_dict(_changed(nf.full_stack(), path, value))
    assert f"'{named}'" in str(error.value)


def test_what_the_layers_keep():
    spec = describe_model(config_from_dict(nf.full_stack()))
    model = Model(spec)
    needs = model.cache_needs()
    assert needs[0] == {"mixer.kv": PagedKV(2, 16, 11, value_size=24, keep_first=3),
                        "mixer.taps": FixedState((2, 64 + 32 + 48), "float32")}
    assert needs[1]["mixer.kv"] == PagedKV(2, 16, 5, value_size=24) and needs[1]["mixer.taps"] == FixedState((1, 144), "float32")
    assert needs[2] == {"mixer.kv": PagedKV(3, 8, 30, value_size=8, keep_first=9)}                  # one tap: no state
    assert needs[3]["mixer.kv"].keep_first == 17
    names = {w.name: tuple(w.shape) for part in model.parts() for w in part.weight_specs()}
    assert names["embed"] == (211, 96) and "head" not in names
    assert names["l0.mix.v.conv"] == (48, 3) and names["l0.mix.k.b"] == (32,) and names["l0.mix.o"] == (96, 96) and "l0.mix.o.b" not in names
    assert names["l0.mlp.router"] == (7, 96) and names["l0.mlp.correction"] == (7,)
    assert names["l0.mlp.e4.up"] == (24, 96) and names["l0.mlp.e4.down"] == (96, 24)
    assert not any(n.startswith(("l0.mlp.e5", "l1.mlp")) or n.endswith((".gate", "norm2", ".sink")) for n in names)
    assert model.graph_safe


def test_parts_refuse_what_does_not_go_together():
    def experts(**kw):
        return PartSpec("routed_experts", "m", {"width": 8, "n_experts": 2, "top": 1, "expert_inner": 4, **kw})
    for bad in (experts(n_identity=1), experts(correction=True), experts(form="tanh"), experts(router_scale=2.0),
                experts(weights="softmax_of_all", n_identity=1, top=4)):
        with pytest.raises(ValueError):
            build_part(bad)
    rotation = PartSpec("banded_rotary", "m", {"base": 10.0, "dims": 4})
    for bad in ({"sink": "one"}, {"window": 4, "keep_first": -1}):
        with pytest.raises(ValueError):
            build_part(PartSpec("normed_attention", "m", {"width": 8, "n_heads": 2, "n_kv_heads": 1, "key_size": 8, "value_size": 8,
                                                          "score_scale": 1.0, "eps": 0.0, "position": rotation, "norm": None, **bad}))


# ---- the plain model's own properties ---------------------------------------------------------------

def test_plain_visibility():
    assert plain.visible(3, 5, 2) == [0, 1, 2, 3]
    assert plain.visible(9, 3, 2) == [0, 1, 7, 8, 9]
    assert plain.visible(9, 3, 8) == list(range(10))
    assert plain.visible(9, 1, 0) == [9]


def test_plain_sink_and_choice():
    np.testing.assert_allclose(plain.sink_weights(np.zeros(3)), [0.25] * 3)
    np.testing.assert_allclose(plain.sink_weights(np.array([50.0, -50.0])).sum(), 1.0)
    assert plain.sink_weights(np.array([-40.0])).sum() < 1e-15
    chosen, weights = plain.choose(np.log([0.5, 0.3, 0.2]), np.array([-1.0, 0.0, 0.2]), 2, 3.0)
    assert chosen.tolist() == [2, 1]                                   # the correction ranks, it does not weigh
    np.testing.assert_allclose(weights, [1.2, 1.8])


def test_plain_convolution_and_rotation():
    u = np.arange(4.0)[:, None]
    np.testing.assert_allclose(plain.short_convolution(u, np.array([[100.0, 10.0, 1.0]]))[:, 0], [0, 1, 12, 123])
    x = np.zeros((1, 1, 6))
    x[0, 0, 0] = 1.0
    turned = plain.rotate_half(x, [2], 7.0, 4)
    np.testing.assert_allclose(turned[0, 0], [np.cos(2.0), 0, np.sin(2.0), 0, 0, 0], atol=1e-12)


def test_plain_is_causal_and_every_mechanism_shows(tmp_path):
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=1, matrix_scale=2.0)
    tokens = np.random.default_rng(0).integers(0, 211, 40).tolist()
    full = nf.plain_logits(folder, tokens)
    np.testing.assert_allclose(full[:25], nf.plain_logits(folder, tokens[:25]), atol=1e-9)
    for mechanism in ("keep_first", "sink", "correction", "identity", "taps"):
        assert np.abs(full[-1] - nf.plain_logits(folder, tokens, drop=(mechanism,))[-1]).max() > 0.02, mechanism
