"""Host-side pieces of the Mizerax family that need no GPU: the registry, config validation (done before a device is touched), the
model-folder round trip, and the oracle's own invariants."""
import json
import math

import numpy as np
import pytest

import mizerax_oracle as O
from xalm_b200 import capi
from xalm_b200 import safetensors_io as ST
from xalm_b200.model import Model

CFG = O.make_config(vocab=19, width=16, max_positions=40, loop=(0, 1, 2), layers=[
    O.attention_layer(4, 2, 6, 5, 0.3, (0.7, 8), mlp=O.moe(6, 3, 2, identity=1, shared=7)),
    O.attention_layer(2, 1, 4, 4, 0.5, None, mlp=None),
    O.attention_layer(3, 3, 5, 5, 0.4, (0.2, 3), mlp=O.moe(4, 2, 1))])


def test_registry_lists_the_family():
    assert {"Llama", "Nabalix", "Bolovik", "Duletar", "Kubolorn", "Mizerax"} <= set(capi.families())


def test_model_folder_roundtrip(tmp_path):
    W = O.random_weights(CFG, 1)
    ST.write_model_dir(str(tmp_path), CFG, W, "BF16")
    back = ST.read_tensors(str(tmp_path / "model.safetensors"))
    assert set(back) == set(W) == set(O.tensor_shapes(CFG))
    for n, (t, shape, raw) in back.items():
        assert np.array_equal(ST.bf16_bits_to_f32(raw.view(np.uint16)).reshape(shape), W[n])   # the test weights are bf16-exact
    assert Model.from_pretrained(str(tmp_path)).config["architecture"] == "Mizerax"
    assert "head" not in W and "l1.ls2" not in W and "l2.mlp.shared.up" not in W              # tied head; optional parts


@pytest.mark.parametrize("edit,needle", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "convolution"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "query heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 0), "query heads"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].__setitem__("every", 0), "q_temp"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].__setitem__("every", 2.5), "q_temp"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "dense"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 5), "experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("identity", -1), "experts"),
    (lambda c: c["layers"][0]["mlp"]["shared"].__setitem__("ff", 0), "shared"),
    (lambda c: c["loop"].__setitem__("stop", 4), "loop"),
    (lambda c: c["loop"].__setitem__("times", 0), "loop"),
    (lambda c: c.__setitem__("max_positions", 0), "max_positions"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c.pop("width"), "width"),
])
def test_bad_configs_are_named_before_any_device_is_touched(edit, needle):
    c = json.loads(json.dumps(CFG))
    edit(c)
    with pytest.raises(capi.XalmError, match=needle):
        Model.from_json(c, {}).cuda()


def test_oracle_cut_into_portions_equals_one_run():
    W = O.random_weights(CFG, 2)
    tokens = np.random.default_rng(0).integers(0, 19, 20).tolist()
    whole, st = O.forward(CFG, W, tokens, {}), {}
    parts = np.concatenate([O.forward(CFG, W, tokens[a:b], st) for a, b in ((0, 7), (7, 9), (9, 10), (10, 20))])
    assert np.allclose(parts, whole, atol=1e-10)


def test_oracle_run_order():
    assert O.layer_runs(CFG) == [(0, True), (0, True), (1, False), (2, False)]
    assert O.layer_runs(O.make_config(5, 4, [{}] * 4, loop=(1, 3, 2))) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert O.layer_runs(O.make_config(5, 4, [{}] * 2)) == [(0, False), (1, False)]


def test_oracle_attention_against_a_matrix_form():
    """With a value of ones the output is the share of the weights that is not the sink's: below one; one lone key of score s gets
    e^s / (1 + e^s); without slopes and with large scores it is plain softmax."""
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 1, 4)), rng.standard_normal((6, 1, 3))
    out = O.biased_attention(q, k, v, 0, 0.5, [0.25, 0.0])
    for h, slope in enumerate((0.25, 0.0)):
        s = (q[:, h] @ k[:, 0].T) * 0.5 - slope * (np.arange(6)[:, None] - np.arange(6)[None, :])
        e = np.exp(np.where(np.tril(np.ones((6, 6))) > 0, s, -np.inf))
        assert np.allclose(out[:, h], (e / (1.0 + e.sum(-1, keepdims=True))) @ v[:, 0])
    share = O.biased_attention(q, k, np.ones((6, 1, 1)), 0, 0.5, [0.25, 0.0])
    assert (share > 0).all() and (share < 1).all()
    s00 = math.exp(0.5 * q[0, 0] @ k[0, 0])
    assert np.isclose(share[0, 0, 0], s00 / (1.0 + s00))


def test_oracle_routing_and_temperature():
    logits = np.log(np.array([[0.5, 0.3, 0.15, 0.05]]))
    idx, wgt = O.route(logits, np.array([0.0, 0.0, 0.4, 0.0]), 2)
    assert idx.tolist() == [[2, 0]] and np.allclose(wgt, [[0.15, 0.5]])            # chosen with the correction, weighted without, not renormalised
    t = {"coef": 0.5, "every": 4}
    assert O.query_temperature(2, t) == 1.0                                         # position 3 completes the first block of four
    assert np.isclose(O.query_temperature(3, t), 1 + 0.5 * math.log(2.0)) and np.isclose(O.query_temperature(11, t), 1 + 0.5 * math.log(4.0))
    assert O.head_slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    x = np.random.default_rng(3).standard_normal((3, 8)) * 5 + 2
    n = O.layer_norm(x, np.ones(8), np.zeros(8), 0.0)
    assert np.allclose(n.mean(-1), 0) and np.allclose((n ** 2).mean(-1), 1)
