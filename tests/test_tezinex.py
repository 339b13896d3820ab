"""Tezinex without a GPU: the configuration reader, the model as data (borrowed cache entries, sizes that the checkpoint
decides, tensor names), and the plain implementation against itself and on hand-made inputs."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_tezinex as P
import tezinex_cases as C
from etalii.dllm_b200 import architectures  # noqa: F401
from etalii.dllm_b200.config.registry import ConfigError, architecture, config_from_dict
from etalii.dllm_b200.parts.spec import FreeSize
from etalii.dllm_b200.weights.loader import WeightError, expected_tensors, load_weights
from etalii.dllm_b200.weights.random_init import random_tensors, write_model


def _spec(config_dict):
    config = config_from_dict(config_dict)
    return architecture(config.model_type).build_spec(config)


@pytest.mark.parametrize("case", sorted(C.CASES))
def test_config_reads_back_and_names_every_tensor(case):
    config_dict = C.CASES[case]()
    config = config_from_dict(config_dict)
    assert config.model_type == "Tezinex" and config.to_hf() == config_dict
    assert config_from_dict(config.to_hf()) == config
    expected = expected_tensors(_spec(config_dict))
    made = C.random_weights(config_dict)
    assert set(expected) == set(made)
    for name in made:
        for have, want in zip(made[name].shape, expected[name].shape):
            assert have == want or isinstance(want, FreeSize)
    assert not any(name.startswith("l2.mix.k") for name in expected) or case != "mixed"


def test_the_checkpoint_decides_the_inner_sizes_of_low_rank_projections(tmp_path):
    config_dict = C.CASES["mixed"]()
    weights = C.random_weights(config_dict)
    spec = _spec(config_dict)
    loaded = load_weights(write_model(str(tmp_path / "a"), config_dict, weights), spec)
    assert loaded["l1.mix.a1"].shape[0] == 8 and loaded["l3.mix.a1"].shape[0] == 14  # (each layer its own)
    assert loaded["l1.mix.g2"].shape == (80, 12)
    wrong = dict(weights)
    wrong["l1.mix.a2"] = torch.zeros(48, 9, dtype=torch.bfloat16)  # eight columns would fit its first matrix
    wrong["l3.mix.g1"] = torch.zeros(6, 90, dtype=torch.bfloat16)  # the width is the configuration's
    with pytest.raises(WeightError) as raised:
        load_weights(write_model(str(tmp_path / "b"), config_dict, wrong), spec)
    assert sorted(name for name, *_ in raised.value.wrong_shape) == ["l1.mix.a2", "l3.mix.g1"]
    made = random_tensors(config_from_dict(config_dict), 3)
    assert made["l1.mix.a1"].shape == (12, 96) and made["l1.mix.g1"].shape == (20, 96)
    assert made["l2.dwa"].shape == (4,) and abs(float(made["l2.dwa"][-1]) - 1) < 0.2 > abs(float(made["l2.dwa"][0]))


def test_layers_that_borrow_keys_share_the_owners_cache_entry():
    spec = _spec(C.CASES["mixed"]())
    order = spec.run_order()
    assert [e.cache for e in order] == [0, 1, 0, 2, 3, 0]
    assert [e.writes_cache for e in order] == [True, True, False, True, True, False]
    from etalii.dllm_b200.parts import build_part

    need = build_part("mixer", spec.layers[0].parts["mixer"]).cache_need()
    assert (need.window, need.keep_first) == (90, 70)  # what any reader of the entry still sees
    assert (need.head_dim, need.value_dim, need.kv_heads) == (24, 16, 2)
    assert build_part("mixer", spec.layers[4].parts["mixer"]).cache_need().window is None
    assert spec.head.names["weight"] == spec.embedding.names["weight"] == "embed"


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="mamba"), "type 'mamba' is not supported"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "no conv"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "no scale"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), "earlier layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "attention layers only"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=2), "no keys and values of its own"),
    (lambda c: c["layers"][2]["mixer"].update(dim=20), "layer 0's dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "mlp.kind"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.pop("residual_mult"), "no residual_mult"),
])
def test_refused_configurations(change, text):
    config_dict = copy.deepcopy(C.CASES["mixed"]())
    change(config_dict)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(config_dict)


@pytest.mark.parametrize("case", sorted(C.CASES))
def test_the_plain_model_gives_the_same_logits_however_a_prompt_is_cut(case):
    config = C.CASES[case]()
    weights = C.as_numpy(C.random_weights(config, 3))
    tokens = C.tokens_for(config, [90])[0]
    whole = P.forward(config, weights, tokens)
    for cuts in ([90], [1] * 90, [2, 5, 1, 82], [89, 1]):
        state, at, rows = P.new_state(config), 0, []
        for n in cuts:
            rows.append(P.forward(config, weights, tokens[at:at + n], state, at))
            at += n
        assert np.allclose(np.concatenate(rows), whole, rtol=0, atol=1e-9 * float(np.abs(whole).max()))


def test_plain_sinusoid_norm_and_average_by_hand():
    assert P.sinusoid([0, 3], 4)[1] == pytest.approx([math.sin(3), math.cos(3), math.sin(0.03), math.cos(0.03)])
    assert list(P.sinusoid([0], 4)[0]) == [0, 1, 0, 1]
    x = np.array([[3.0, -4.0]])
    assert P.zero_centred_norm(x, np.array([0.0, 1.0]), 0.5)[0] == pytest.approx(
        [3 / math.sqrt(13), -8 / math.sqrt(13)])
    assert P.depth_average([2.0, -1.0], [x, 2 * x])[0] == pytest.approx([0, 0])
    assert P.cap(np.array([3.0]), 2.0)[0] == pytest.approx(2 * math.tanh(1.5)) and P.cap(3.0, None) == 3.0


def test_plain_delta_rule_shrinks_rows_writes_and_then_reads():
    """Two key channels with decays of their own; the second token's key is the first's: what the shrunk state answers
    is taken off the new value, and the read-out sees the write."""
    q = k = np.array([[[1.0, 0.0]], [[1.0, 0.0]]])
    v = np.array([[[4.0]], [[10.0]]])
    g = np.array([[[0.3, 0.9]], [[0.5, 0.25]]])
    beta = np.array([[0.5], [0.25]])
    state = np.array([[[8.0], [16.0]]])
    out = P.delta_scan(q, k, v, g, beta, state)
    first = 8 * 0.3 + 0.5 * (4 - 8 * 0.3)
    assert out[0, 0, 0] == pytest.approx(first)
    assert out[1, 0, 0] == pytest.approx(first * 0.5 + 0.25 * (10 - first * 0.5))
    assert state[0, 1, 0] == pytest.approx(16 * 0.9 * 0.25)  # the other channel only shrinks
    y, kept = P.short_convolution(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0, 100.0]]), np.array([[5.0], [7.0]]))
    assert list(y[:, 0]) == [50 + 7 + 100, 70 + 1 + 200] and list(kept[:, 0]) == [1, 2]


def test_plain_sink_cap_and_window_by_hand():
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 2.0, "softcap": 3.0,
         "mask": {"size": 2, "keep_first": 1}}
    one, zero = np.ones((1, 1)), np.zeros(1)
    w = {"q": one, "q.b": zero, "k": one, "k.b": zero, "v": one, "v.b": np.array([4.0]), "o": one,
         "sink": np.array([0.7])}
    h = np.ones((4, 1))
    out, kept = P.attention(w, m, h, None)
    e = math.exp(3 * math.tanh(2 / 3))  # every key scores the same; position 3 sees 0 (kept), 2 and 3
    for i, keys in enumerate((1, 2, 3, 3)):
        assert out[i, 0] == pytest.approx(5 * keys * e / (keys * e + math.exp(0.7)))
    assert [int(j) for j in range(9) if P.visible(8, j, {"size": 3, "keep_first": 2})] == [0, 1, 6, 7, 8]
    borrowed, _ = P.attention(w, dict(m, mask=None), h[3:], None, borrowed=kept)
    assert borrowed[0, 0] == pytest.approx(5 * 4 * e / (4 * e + math.exp(0.7)))
