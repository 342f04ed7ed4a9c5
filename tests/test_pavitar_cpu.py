"""Host-side pieces of the Pavitar family that need no GPU: the registry, config validation (done before a device is touched), the
model-folder round trip, and the oracle's own invariants."""
import json
import math

import numpy as np
import pytest

import pavitar_oracle as O
from xalm_b200 import capi
from xalm_b200 import safetensors_io as ST
from xalm_b200.model import Model

CFG = O.make_config(vocab=19, width=16, loop=(0, 1, 2), layers=[
    O.latent_layer(4, 6, 5, 9, 12, 7, 0.3, mlp=O.moe(6, 3, 2, shared=7)),
    O.attention_layer(4, 2, 4, 6, 5, 0.5, (100.0, 2), mlp=None),
    O.attention_layer(3, 3, 5, 5, 30, 0.4, (1e4, 4), mlp=O.moe(4, 2, 1))])


def test_registry_lists_the_family():
    assert {"Llama", "Nabalix", "Bolovik", "Duletar", "Kubolorn", "Mizerax", "Pavitar"} <= set(capi.families())


def test_model_folder_roundtrip(tmp_path):
    W = O.random_weights(CFG, 1)
    ST.write_model_dir(str(tmp_path), CFG, W, "BF16")
    back = ST.read_tensors(str(tmp_path / "model.safetensors"))
    assert set(back) == set(W) == set(O.tensor_shapes(CFG))
    for n, (t, shape, raw) in back.items():
        assert np.array_equal(ST.bf16_bits_to_f32(raw.view(np.uint16)).reshape(shape), W[n])   # the test weights are bf16-exact
    assert Model.from_pretrained(str(tmp_path)).config["architecture"] == "Pavitar"
    assert "head" not in W and "l1.norm2" not in W and "l2.mlp.shared.sg" not in W             # tied head; optional parts


@pytest.mark.parametrize("edit,needle", [
    (lambda c: c["layers"][0].__setitem__("type", "convolution"), "convolution"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 3), "query heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 0), "heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_rank", 0), "latent"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "mask"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", -4), "mask"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 3), "rotary"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 6), "rotary"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "dense"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 4), "experts"),
    (lambda c: c["layers"][0]["mlp"]["shared"].__setitem__("ff", 0), "shared"),
    (lambda c: c["loop"].__setitem__("stop", 4), "loop"),
    (lambda c: c["loop"].__setitem__("times", 0), "loop"),
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
    assert O.layer_runs(CFG) == [(0, 1), (0, 2), (1, 0), (2, 0)]
    assert O.layer_runs(O.make_config(5, 4, [{}] * 4, loop=(1, 3, 2))) == [(0, 0), (1, 1), (2, 0), (1, 2), (2, 0), (3, 0)]
    assert O.layer_runs(O.make_config(5, 4, [{}] * 2)) == [(0, 0), (1, 0)]


def test_oracle_masks():
    seen = lambda f, i, size: [j for j in range(12) if f(i, j, size)]
    assert seen(O.sees_window, 7, 3) == [5, 6, 7] and seen(O.sees_window, 1, 3) == [0, 1] and seen(O.sees_window, 4, 1) == [4]
    assert seen(O.sees_chunk, 7, 4) == [4, 5, 6, 7] and seen(O.sees_chunk, 8, 4) == [8] and seen(O.sees_chunk, 9, 100) == list(range(10))


def test_oracle_attention_against_a_matrix_form():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((6, 2, 4)), rng.standard_normal((6, 1, 4)), rng.standard_normal((6, 1, 3))
    i, j = np.indices((6, 6))
    for sees, mask in ((lambda a, b: O.sees_window(a, b, 3), (i - j >= 0) & (i - j < 3)), (lambda a, b: O.sees_chunk(a, b, 4), (j <= i) & (i // 4 == j // 4))):
        out = O.attend(q, k, v, 0, 0.5, sees)
        for h in range(2):
            e = np.where(mask, np.exp((q[:, h] @ k[:, 0].T) * 0.5), 0.0)
            assert np.allclose(out[:, h], (e / e.sum(-1, keepdims=True)) @ v[:, 0])


def test_oracle_rotation_and_routing():
    x = np.random.default_rng(3).standard_normal((3, 2, 8))
    y = O.turn_pairs(x, 5, 50.0, 6)
    assert np.allclose(y[:, :, 6:], x[:, :, 6:]) and np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1))
    z = (x[:, :, 2] + 1j * x[:, :, 3]) * np.exp(1j * (5 + np.arange(3)) * 50.0 ** (-2 / 6))[:, None]    # entries 2 and 3 are the second pair
    assert np.allclose(y[:, :, 2], z.real) and np.allclose(y[:, :, 3], z.imag)
    idx, wgt = O.route(np.array([[0.5, 2.0, -1.0, 2.0]]), 3)
    assert idx.tolist() == [[1, 3, 0]] and np.isclose(wgt.sum(), 1) and np.isclose(wgt[0, 2] / wgt[0, 0], math.exp(-1.5))
