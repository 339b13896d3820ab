"""Zivazen without a GPU: the configuration reader, the model as data (parts, cache needs, tensor names), and the plain
implementation against itself and on hand-made inputs."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_zivazen as P
import zivazen_cases as C
from etalii.dllm_b200 import architectures  # noqa: F401
from etalii.dllm_b200.config.registry import ConfigError, architecture, config_from_dict
from etalii.dllm_b200.parts import build_part
from etalii.dllm_b200.parts.position import rotary_frequencies
from etalii.dllm_b200.weights.loader import WeightError, expected_tensors, load_weights
from etalii.dllm_b200.weights.random_init import random_tensors, write_model


def _spec(config_dict):
    config = config_from_dict(config_dict)
    return architecture(config.model_type).build_spec(config)


@pytest.mark.parametrize("case", sorted(C.CASES))
def test_config_reads_back_and_names_every_tensor(case, tmp_path):
    config_dict = C.CASES[case]()
    config = config_from_dict(config_dict)
    assert config.model_type == "Zivazen" and config.to_hf() == config_dict
    assert config_from_dict(config.to_hf()) == config
    expected = expected_tensors(_spec(config_dict))
    made = C.make_weights(config_dict)
    assert {name: tuple(param.shape) for name, param in expected.items()} == \
        {name: tuple(value.shape) for name, value in made.items()}
    assert set(random_tensors(config, 3)) == set(expected)
    loaded = load_weights(write_model(str(tmp_path / "model"), config_dict, made), _spec(config_dict))
    assert all(torch.equal(loaded[name], made[name]) for name in made)
    del made["l0.norm1"]
    with pytest.raises(WeightError):
        load_weights(write_model(str(tmp_path / "less"), config_dict, made), _spec(config_dict))


def test_the_model_as_data():
    spec = _spec(C.CASES["mixed"]())
    mix = [layer.parts["mixer"].params.get("value_mix") for layer in spec.layers]
    assert mix == [None, None, "keep", "mix", None, "mix"]  # the first layer that mixes keeps its own
    assert [("feed_forward" in layer.parts) for layer in spec.layers] == [True, True, True, True, False, False]
    first = build_part("mixer", spec.layers[0].parts["mixer"])
    need = first.cache_need()
    assert (need.kv_heads, need.head_dim, need.value_dim, need.chunks(), need.window) == (2, 24, 16, (40,), None)
    assert build_part("mixer", spec.layers[5].parts["mixer"]).cache_need().chunks() == ()
    need = build_part("mixer", spec.layers[1].parts["mixer"]).cache_need()
    keys, state = need.parts
    assert (keys.kind, keys.window) == ("kv", 30)
    assert [part.state_shape for part in state.parts] == [(4, 12, 12), (2, 88)]  # rows of a multiple of four
    need = build_part("mixer", spec.layers[4].parts["mixer"]).cache_need()
    assert need.parts[1].kind == "state" and need.parts[0].value_dim == 14  # one tap keeps no history
    assert spec.layers[1].parts["mixer"].params["left"].kind == "attention"
    assert spec.layers[4].parts["mixer"].params["left"].kind == "sink_attention"
    assert spec.head.names["weight"] == "head" and spec.embedding.names["norm"] == "embed.norm"


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="mamba"), "type 'mamba' is not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "no scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "no low"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=1.0), "high above low"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=20), "cannot be mixed"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "no left_scale"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=3), "not a multiple of 3 groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "no conv"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "mlp.kind"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top 7 of 6"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "no ff"),
    (lambda c: c["norm"].update(eps=0.0), "norm.eps"),
    (lambda c: c.pop("width"), "no width"),
])
def test_refused_configurations(change, text):
    config_dict = copy.deepcopy(C.CASES["mixed"]())
    change(config_dict)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(config_dict)


@pytest.mark.parametrize("case", sorted(C.CASES))
def test_the_plain_model_gives_the_same_logits_however_a_prompt_is_cut(case):
    config = C.CASES[case]()
    weights = C.as_numpy(C.make_weights(config, 3))
    tokens = C.tokens_for(config, [90])[0]
    whole = P.forward(config, weights, tokens)
    for cuts in ([90], [1] * 90, [2, 5, 1, 82], [89, 1]):
        state, at, rows = P.new_state(config), 0, []
        for n in cuts:
            rows.append(P.forward(config, weights, tokens[at:at + n], state, at))
            at += n
        assert np.allclose(np.concatenate(rows), whole, rtol=0, atol=1e-9 * float(np.abs(whole).max()))


@pytest.mark.parametrize("rot", [{"base": 10000.0, "dims": 16}, {"base": 500.0, "dims": 30, "scaling": {
    "factor": 6.0, "low": 1.5, "high": 3.5, "original": 200}}])
def test_the_librarys_frequencies_are_the_plain_ones(rot):
    scaling = rot.get("scaling")
    if scaling:
        scaling = {"rope_type": "llama3", "factor": scaling["factor"], "low_freq_factor": scaling["low"],
                   "high_freq_factor": scaling["high"], "original_max_position_embeddings": scaling["original"]}
    got, want = rotary_frequencies(rot["dims"], rot["base"], scaling), P.frequencies(rot)
    assert np.allclose(got, want, rtol=1e-12)
    if scaling:  # all three branches are taken
        plain = P.frequencies({"base": rot["base"], "dims": rot["dims"]})
        ratio = plain / want
        assert ratio.min() == pytest.approx(1) and ratio.max() == pytest.approx(6) and ((ratio > 1.1) & (ratio < 5.9)).any()


def test_plain_rotation_masks_and_softmax_by_hand():
    x = np.array([[[1.0, 2.0, 3.0, 4.0, 9.0]]])
    a, b = 2.0 * 1.0, 2.0 * 0.1
    assert P.rotate(x, [2], {"base": 100.0, "dims": 4})[0, 0] == pytest.approx(
        [math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b), 3 * math.cos(a) + math.sin(a),
         4 * math.cos(b) + 2 * math.sin(b), 9.0])
    assert [j for j in range(9) if P.same_chunk(7, j, 5)] == [5, 6, 7]
    assert [j for j in range(9) if P.same_chunk(5, j, 5)] == [5] and [j for j in range(9) if P.same_chunk(4, j, 5)] == \
        [0, 1, 2, 3, 4]
    assert [j for j in range(9) if P.in_window(7, j, 3)] == [5, 6, 7]
    s = np.array([[1.0, -2.0, -np.inf]])
    e = np.exp([1.0, -2.0])
    assert P.softmax_plus_one(s)[0] == pytest.approx([*(e / (1 + e.sum())), 0])
    assert P.softmax_plus_one(s - 100)[0] == pytest.approx([0, 0, 0]) and P.softmax(s)[0] == pytest.approx(
        [*(e / e.sum()), 0])
    assert P.mix_values(2.0, 10.0, 0.25) == 4.0


def test_plain_state_space_by_hand():
    """Two tokens of one head with a state of one: the state shrinks, is written with the step size, then read; the token's
    own value is added with its share."""
    x, dt = np.array([[[3.0]], [[5.0]]]), np.array([[0.5], [2.0]])
    b, c = np.array([[[2.0]], [[1.0]]]), np.array([[[7.0]], [[-1.0]]])
    state = np.array([[[4.0]]])
    y = P.state_space_scan(x, b, c, dt, np.array([0.3]), np.array([10.0]), state)
    s1 = 4 * math.exp(-0.15) + 0.5 * 2 * 3
    s2 = s1 * math.exp(-0.6) + 2 * 1 * 5
    assert y[0, 0, 0] == pytest.approx(7 * s1 + 30) and y[1, 0, 0] == pytest.approx(-s2 + 50)
    assert state[0, 0, 0] == pytest.approx(s2)
    y, kept = P.short_convolution(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0, 100.0]]), np.array([0.5]),
                                  np.array([[5.0], [7.0]]))
    assert list(y[:, 0]) == [157.5, 271.5] and list(kept[:, 0]) == [1, 2]
    got = P.gate_then_norm(np.array([[1.0, 2.0, 3.0, 4.0]]), np.full((1, 4), 50.0), np.array([1.0, 1.0, 1.0, 2.0]), 2, 0.0)
    assert got[0] == pytest.approx([50 / math.sqrt(2500 * 2.5), 2 / math.sqrt(2.5), 3 / math.sqrt(12.5),
                                    8 / math.sqrt(12.5)])


def test_plain_choice_by_hand():
    """Groups count by their two best corrected scores, closed experts are out although their scores are higher than the
    (negative) ones of the open groups, and the weights are the scores without the correction."""
    scores = np.array([0.9, 0.1, 0.5, 0.6, 0.3, 0.2])
    correction = np.array([-1.0, -1.0, -1.0, -1.0, -1.0, -1.0])
    router = {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}}
    picked, weights = P.choose(scores, correction, router)
    assert list(picked) == [3, 2] and weights == pytest.approx([3 * 0.6 / 1.1, 3 * 0.5 / 1.1])
    picked, weights = P.choose(scores, np.array([0, 0, 0, 0, 0.9, 0.9]), {"experts": 6, "top": 1, "scale": 1.0})
    assert list(picked) == [4] and weights == pytest.approx([1.0])
    assert list(P.choose(scores, correction, dict(router, groups={"count": 6, "keep": 3}))[0]) == [0, 3]
