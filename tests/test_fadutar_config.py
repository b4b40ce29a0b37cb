"""Configuration, tensor list and the plain mechanisms of the Fadutar decoder (no GPU)."""
import copy

import numpy as np
import pytest

from fadutar_cases import CASES, random_config, tensor_shapes


def _spec(raw):
    from xeno_rt_b200.config import config_from_dict
    arch, config = config_from_dict(raw)
    return arch, config, arch.build_spec(config)


@pytest.mark.parametrize("name", list(CASES))
def test_the_spec_expects_exactly_the_tensors_of_the_design(name):
    raw = CASES[name][0]
    arch, config, spec = _spec(raw)
    assert arch.name == "Fadutar"
    spec.validate()
    got = {e.name: tuple(e.shape) for e in spec.expected_tensors()}
    assert got == {k: tuple(v) for k, v in tensor_shapes(raw).items()}
    assert config.to_dict() == raw and _spec(config.to_dict())[1] == config


def test_random_configurations_give_their_tensors_too():
    for seed in range(60):
        raw = random_config(np.random.default_rng(seed))
        spec = _spec(raw)[2]
        assert {e.name: tuple(e.shape) for e in spec.expected_tensors()} == {k: tuple(v) for k, v in tensor_shapes(raw).items()}


def test_a_layer_that_reads_another_layers_keys_is_scheduled_on_its_cache():
    spec = _spec(CASES["odd"][0])[2]
    assert [p.cache_from for p in spec.schedule] == [None, None, None, None, 2, None, 2]
    names = {e.name for e in spec.expected_tensors()}
    assert "l2.mix.k" in names and "l4.mix.k" not in names and "l6.mix.v" not in names and "l6.mix.sink" in names
    assert "l2.norm2" not in names and "l3.norm2b" in names   # a layer without a feed-forward has no second pair of norms


def test_every_bad_key_is_reported_in_one_error():
    from xeno_rt_b200.core import ConfigError
    raw = copy.deepcopy(CASES["mixed"][0])
    raw["vocab"] = -1
    raw["norm"] = {}
    raw["layers"][0]["mixer"]["blocks"] = 7                  # 96 channels are no multiple
    raw["layers"][0]["mlp"]["limit"] = 0
    raw["layers"][1]["mixer"]["kv_heads"] = 3                # 4 heads are no multiple
    raw["layers"][1]["mixer"]["mask"] = {"size": 0}
    raw["layers"][1]["mlp"] = {"kind": "moe"}
    raw["layers"][2]["mixer"]["rot"]["dims"] = 4             # a latent layer rotates all of rot_dim
    raw["layers"][2]["mixer"]["mask"] = {"size": 8}
    raw["layers"][3]["mixer"]["kv_from"] = 2                 # a latent layer has no keys to give
    raw["layers"][3]["mixer"]["rot"] = {"dims": 4, "base": 10.0}
    raw["layers"][4]["mixer"].pop("conv")
    raw["layers"].append({"type": "mamba", "mixer": {}, "mlp": None})
    with pytest.raises(ConfigError) as err:
        _spec(raw)
    text = str(err.value)
    for piece in ("vocab", "eps", "7 equal blocks", "limit", "3 kv_heads", "mask.size", "'moe'", "rot.dims 4", "layers[2].mixer.mask",
                  "kv_from", "layers[3].mixer.rot", "layers[4].mixer.conv", "'mamba'"):
        assert piece in text, piece


def test_a_reader_must_match_its_owner_and_come_after_it():
    from xeno_rt_b200.core import ConfigError
    for key, value in (("dim", 32), ("kv_heads", 1), ("vdim", 8), ("kv_from", 3), ("kv_from", 0)):
        raw = copy.deepcopy(CASES["mixed"][0])
        raw["layers"][3]["mixer"][key] = value
        with pytest.raises(ConfigError):
            _spec(raw)
    raw = copy.deepcopy(CASES["odd"][0])
    raw["layers"][6]["mixer"]["kv_from"] = 4                 # layer 4 reads layer 2 itself
    with pytest.raises(ConfigError):
        _spec(raw)


def test_norms_of_layers_without_a_feed_forward_may_lie_in_the_file():
    ignorable = _spec(CASES["mixed"][0])[2].ignorable_tensors
    assert set(ignorable) == {"l2.norm2", "l2.norm2b", "l4.norm2", "l4.norm2b"}


def test_the_plain_chunks_and_sinks():
    from plain import fadutar
    assert list(fadutar.visible(9, 5)) == [5, 6, 7, 8, 9] and list(fadutar.visible(10, 5)) == [10]
    assert list(fadutar.visible(3, None)) == [0, 1, 2, 3] and list(fadutar.visible(7, 1)) == [7]
    assert fadutar.sink_weights([-30.0, -31.0], 0.0).sum() < 1e-12
    assert np.allclose(fadutar.sink_weights([2.0, 2.0, 2.0], 2.0), 0.25)
    assert abs(fadutar.sink_weights([800.0, 799.0], -3.0).sum() - 1) < 1e-12
    assert np.allclose(fadutar.sink_weights([0.0], np.log(3.0)), 0.25)


def test_the_plain_recurrence_and_gate():
    from plain import fadutar
    lam = np.array([-3.0, 0.5])
    u, r, i = np.ones((3, 2)), np.full((3, 2), 0.25), np.full((3, 2), 0.5)
    a = np.exp(-8.0 * 0.25 * np.log1p(np.exp(lam)))
    b = np.sqrt(1 - a * a) * 0.5
    assert np.allclose(fadutar.linear_recurrence(u, r, i, lam), [b, a * b + b, a * (a * b + b) + b])
    g = fadutar.limited_gate(np.array([5.0, -9.0, 0.5]), np.array([-5.0, 9.0, 0.25]), 2.0)
    sig = lambda z: 1 / (1 + np.exp(-z))
    assert np.allclose(g, [2 * sig(3.404) * -1.0, -9 * sig(-9 * 1.702) * 3.0, 0.5 * sig(0.851) * 1.25])
    out = fadutar.short_convolution(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 1.0]]), np.array([0.5]))
    assert np.allclose(out[:, 0], [1.5, 12.5, 24.5])
    w = np.arange(8.0).reshape(2, 2, 2)
    got = fadutar.block_product(np.array([[1.0, 2.0, 3.0, 4.0]]), w, np.zeros((2, 2)))
    assert np.allclose(got, [[2.0, 8.0, 32.0, 46.0]])       # [out, in] matrices, a part each


def test_the_spans_and_launch_shapes_of_chunks():
    """A chunk is a window as far as launch shapes and the blocks that can be given back go."""
    from xeno_rt_b200.parts.attention_bf16 import visible_span
    for chunk in (1, 5, 64, 70, 129):
        for pos in range(600):
            first = pos - pos % chunk
            blocks = pos // 64 - first // 64 + 1
            assert blocks * 64 <= visible_span(1024, chunk)
            assert first > pos - chunk                        # never behind a window of the same size
