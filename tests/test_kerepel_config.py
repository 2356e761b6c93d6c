"""Kerepel without a device: the configuration's round trip and its errors, what the layers keep per request, the
declared tensors, and the plain model's own properties."""

import copy

import numpy as np
import pytest

import kerepel_helpers as kp
import plain_kerepel as plain
from mini_llm_b200.config import ConfigError, config_from_dict, describe_model
from mini_llm_b200.engine.model import Model
from mini_llm_b200.parts.base import build_part
from mini_llm_b200.parts.spec import FixedState, PagedKV, PartSpec


def test_round_trip():
    raw = kp.full_stack()
    parsed = config_from_dict(raw)
    assert parsed.architecture == "Kerepel" and parsed.logit_scale == 1.7 and parsed.bigram["buckets"] == 37 and parsed.side_dim == 12
    assert config_from_dict(parsed.to_dict()) == parsed
    written = parsed.to_dict()
    for index, (mine, given) in enumerate(zip(written["layers"], raw["layers"])):
        assert mine["mixer"] == given["mixer"], index
    plainer = config_from_dict(kp.config([kp.latent(mlp=None)], side=None) | {"embedding": {}})
    assert plainer.bigram is None and plainer.side_dim is None and config_from_dict(plainer.to_dict()) == plainer


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


MIX0, MIX1, MOE1 = ["layers", 0, "mixer"], ["layers", 1, "mixer"], ["layers", 1, "mlp"]


@pytest.mark.parametrize("path, value, named", [
    (["width"], None, "width"), (["vocab"], -3, "vocab"), (["norm", "eps"], None, "norm.eps"), (["logit_scale"], None, "logit_scale"),
    (["embedding", "bigram", "buckets"], 0, "embedding.bigram.buckets"), (["embedding", "bigram", "mul_prev"], None, "embedding.bigram.mul_prev"),
    (["embedding", "bigram", "mul_cur"], -1, "embedding.bigram.mul_cur"), (["token_side", "dim"], 0, "token_side.dim"), (["layers"], [], "layers"),
    (["layers", 0, "type"], "hyena", "layers[0].type"), (["layers", 0, "mixer"], 7, "layers[0].mixer"),
    (MIX0 + ["conv"], None, "layers[0].mixer.conv"), (MIX0 + ["heads"], 5, "layers[0].mixer.heads"), (MIX0 + ["scale"], "x", "layers[0].mixer.scale"),
    (MIX0 + ["mask", "size"], 0, "layers[0].mixer.mask.size"), (MIX0 + ["softcap"], -2.0, "layers[0].mixer.softcap"),
    (["layers", 2, "mixer", "kv_from"], 2, "layers[2].mixer.kv_from"), (["layers", 2, "mixer", "kv_from"], 1, "layers[2].mixer.kv_from"),
    (["layers", 4, "mixer", "kv_from"], 2, "layers[4].mixer.kv_from"), (["layers", 2, "mixer", "vdim"], 8, "layers[2].mixer.kv_from"),
    (MIX1 + ["kv_rank"], None, "layers[1].mixer.kv_rank"), (MIX1 + ["rot", "dims"], 6, "layers[1].mixer.rot.dims"),
    (MIX1 + ["rot", "base"], 1.0, "layers[1].mixer.rot.base"), (MIX1 + ["rot", "scaling", "fast"], None, "layers[1].mixer.rot.scaling.fast"),
    (MIX1 + ["rot_dim"], -2, "layers[1].mixer.rot_dim"),
    (["layers", 0, "mlp", "kind"], "gated", "layers[0].mlp.kind"), (["layers", 0, "mlp", "ff"], None, "layers[0].mlp.ff"),
    (MOE1 + ["router", "top"], 5, "layers[1].mlp.router.top"), (MOE1 + ["router", "groups", "count"], 4, "layers[1].mlp.router.groups.count"),
    (MOE1 + ["router", "groups", "keep"], 4, "layers[1].mlp.router.groups.keep"), (MOE1 + ["expert", "limit"], None, "layers[1].mlp.expert.limit"),
    (MOE1 + ["shared", "ff"], 0, "layers[1].mlp.shared.ff"),
])
def test_errors_name_their_key(path, value, named):
    with pytest.raises(ConfigError) as error:
        config_from_dict(_changed(kp.full_stack(), path, value))
    assert f"'{named}'" in str(error.value)


def test_what_the_layers_keep():
    model = Model(describe_model(config_from_dict(kp.full_stack())))
    needs = model.cache_needs()
    # layer 2 reads layer 0's keys over a wider window: they are kept that long
    assert needs[0] == {"mixer.kv": PagedKV(2, 16, 29, value_size=24), "mixer.taps": FixedState((2, 64 + 32 + 48), "float32")}
    assert needs[1] == PagedKV(1, 48, None, has_values=False)
    assert needs[2] == {"mixer.taps": FixedState((1, 64), "float32")}           # a reader keeps its queries' taps only
    assert needs[3]["mixer.kv"] == PagedKV(1, 24, 4, value_size=8)
    assert needs[4] is None                                                     # one tap, another layer's pages
    assert needs[7] == FixedState((1,), "int32") and len(needs) == 8            # the embedding: the last token
    names = {w.name: tuple(w.shape) for part in model.parts() for w in part.weight_specs()}
    assert names["embed"] == (211, 96) and names["bigram"] == (38, 96) and names["side.embed"] == (211, 84) and "head" not in names
    assert names["l0.mix.v.conv"] == (48, 3) and names["l0.mix.k.norm"] == (16,) and names["l0.mix.g"] == (96, 96) and "l0.mix.v.norm" not in names
    assert names["l2.mix.q.conv"] == (64, 2) and "l2.mix.k" not in names and "l2.mix.k.norm" not in names and "l2.mix.v.conv" not in names
    assert names["l1.mix.dkv"] == (48, 96) and names["l1.mix.g"] == (3, 96) and names["l1.mix.uv"] == (72, 40)
    assert names["l1.mlp.correction"] == (6,) and names["l1.mlp.shared.gate"] == (40, 96) and names["l1.mlp.shared.sg"] == (1, 96)
    assert "l2.mlp.shared.sg" not in names and not any(n.startswith(("l3.mlp", "l3.norm2")) for n in names)
    assert names["l3.side.gate"] == (12, 96) and names["l3.side.proj"] == (96, 12) and names["l3.side.norm"] == (96,)
    assert model.graph_safe


def test_a_reader_without_a_window_keeps_every_key():
    layers = [kp.attention(mlp=None), kp.attention(kv_from=0, mlp=None)]
    del layers[1]["mixer"]["mask"]
    assert Model(describe_model(config_from_dict(kp.config(layers)))).cache_needs()[0]["mixer.kv"].window is None


def test_parts_refuse_what_does_not_go_together():
    def experts(**kw):
        return PartSpec("routed_experts", "m", {"width": 8, "n_experts": 6, "top": 2, "expert_inner": 4, "weights": "sigmoid", **kw})
    build_part(experts(groups=(3, 1), correction=True, form="clamped_glu", limit=1.0))
    for bad in (experts(groups=(4, 1)), experts(groups=(3, 4)), experts(groups=(6, 1)), experts(form="clamped_glu"),
                experts(form="clamped_glu", limit=1.0, shared_inner=4)):
        with pytest.raises(ValueError):
            build_part(bad)
    with pytest.raises(ValueError):
        build_part(PartSpec("normed_attention", "m", {"width": 8, "n_heads": 2, "n_kv_heads": 1, "key_size": 8, "value_size": 8,
                                                      "score_scale": 1.0, "eps": 0.0, "distance_slopes": (0.5,)}))
    with pytest.raises(ValueError):
        build_part(PartSpec("token_side_input", "m", {"vocab_size": 9, "width": 8, "dim": 4, "index": 2, "n_layers": 2, "eps": 0.0}))
    with pytest.raises(ValueError):
        build_part(PartSpec("paired_token_embedding", "", {"vocab_size": 9, "width": 8, "buckets": 0, "mul_prev": 1, "mul_cur": 1}))


# ---- the plain model's own properties ---------------------------------------------------------------

def test_plain_pair_rows_and_slopes():
    assert plain.pair_rows([5, 2, 9], 10, 3, 7) == [10, (15 + 14) % 10, (6 + 63) % 10]
    np.testing.assert_allclose(plain.slopes(4), [0.25, 0.0625, 0.015625, 0.00390625])


def test_plain_choice_within_groups():
    # the best single expert (4) lies in a group whose two best sum to less than the others'
    z = np.log(np.array([0.5, 0.5, 0.6, 0.55, 0.9, 0.05]) / (1 - np.array([0.5, 0.5, 0.6, 0.55, 0.9, 0.05])))
    none = np.zeros(6)
    assert plain.choose(z, none, {"top": 2})[0].tolist() == [4, 2]
    chosen, weights = plain.choose(z, none, {"top": 2, "groups": {"count": 3, "keep": 2}})
    assert chosen.tolist() == [2, 3]
    np.testing.assert_allclose(weights, [0.6, 0.55])
    # ranking scores below zero are still chosen ahead of experts outside the kept groups; weights are the scores
    chosen, weights = plain.choose(z, none - 2.0, {"top": 2, "groups": {"count": 3, "keep": 1}})
    assert chosen.tolist() == [2, 3] and weights.min() > 0


def test_plain_frequencies():
    plain_f, one = plain.frequencies({"base": 100.0, "dims": 4})
    assert one == 1.0 and plain_f == [1.0, 0.1]
    # the ramp goes from pair 0 to (where there would be one) pair 2: the first keeps its frequency, the other is halfway
    f, amplitude = plain.frequencies({"base": 100.0, "dims": 4, "scaling": {"factor": 4.0, "original": 200.0, "fast": 16.0, "slow": 1.0}})
    np.testing.assert_allclose(f, [1.0, 0.1 * 0.5 + 0.025 * 0.5], rtol=1e-12)
    np.testing.assert_allclose(amplitude, 0.1 * np.log(4.0) + 1.0)
    turned = plain.rotate_pairs(np.array([[[1.0, 0.0, 0.0, 2.0, 5.0]]]), [3], [0.5, 1.0], 2.0)
    np.testing.assert_allclose(turned[0, 0], [2 * np.cos(1.5), 2 * np.sin(1.5), -4 * np.sin(3.0), 4 * np.cos(3.0), 5.0])


def test_plain_expert_is_clamped():
    w = {"e.gate": np.array([[1.0]]), "e.up": np.array([[-1.0]]), "e.down": np.array([[1.0]])}
    np.testing.assert_allclose(plain.expert(np.array([[7.0]]), w, "e", 2.0), [[2.0 * plain.sigmoid(3.404) * -1.0]])
    np.testing.assert_allclose(plain.expert(np.array([[-7.0]]), w, "e", 2.0), [[-7.0 * plain.sigmoid(-7.0 * 1.702) * 3.0]])


def test_plain_is_causal_and_every_mechanism_shows(tmp_path):
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=6, matrix_scale=2.0)
    tokens = np.random.default_rng(5).integers(0, 211, 40).tolist()
    full = kp.plain_logits(folder, tokens)
    np.testing.assert_allclose(full[:25], kp.plain_logits(folder, tokens[:25]), atol=1e-9)
    for mechanism in kp.MECHANISMS:
        assert np.abs(full[-1] - kp.plain_logits(folder, tokens, drop=(mechanism,))[-1]).max() > 0.02, mechanism
