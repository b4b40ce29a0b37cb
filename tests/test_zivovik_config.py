"""Configuration, tensor list and the plain mechanisms of the Zivovik decoder (no GPU)."""
import copy

import numpy as np
import pytest

from plain import zivovik as plain
from zivovik_cases import CASES, random_config, tensor_shapes


def _spec(raw):
    from xeno_rt_b200.config import config_from_dict
    arch, config = config_from_dict(raw)
    return arch, config, arch.build_spec(config)


@pytest.mark.parametrize("name", list(CASES))
def test_the_spec_expects_exactly_the_tensors_of_the_design(name):
    raw = CASES[name][0]
    arch, config, spec = _spec(raw)
    assert arch.name == "Zivovik"
    spec.validate()
    got = {e.name: tuple(e.shape) for e in spec.expected_tensors()}
    assert got == {k: tuple(v) for k, v in tensor_shapes(raw).items()}
    assert config.to_dict() == raw and _spec(config.to_dict())[1] == config


def test_random_configurations_give_their_tensors_too():
    for seed in range(60):
        raw = random_config(np.random.default_rng(seed))
        spec = _spec(raw)[2]
        assert {e.name: tuple(e.shape) for e in spec.expected_tensors()} == {k: tuple(v) for k, v in tensor_shapes(raw).items()}


def test_a_looped_stretch_is_scheduled_again_with_the_embedding_added_before_every_pass_but_the_first():
    for name, (raw, _) in CASES.items():
        spec = _spec(raw)[2]
        assert [(p.layer, p.before is not None) for p in spec.schedule] == plain.order(raw), name
        assert all(p.cache_from is None for p in spec.schedule)     # a pass has a cache or state of its own
    assert plain.order(CASES["mixed"][0]) == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False), (4, False)]
    raw = copy.deepcopy(CASES["mixed"][0])
    raw["loop"]["times"] = 1
    once = _spec(raw)[2]
    raw["loop"] = None
    assert [p.layer for p in once.schedule] == [p.layer for p in _spec(raw)[2].schedule] == [0, 1, 2, 3, 4]
    assert not once.stream_parts


def test_the_number_of_positions_may_come_from_the_tables_shape():
    from xeno_rt_b200.config import config_from_dict
    from xeno_rt_b200.core import ConfigError
    raw = copy.deepcopy(CASES["odd"][0])
    del raw["max_positions"]
    arch, config = config_from_dict(raw)
    with pytest.raises(ConfigError, match="max_positions"):
        arch.build_spec(config)
    found = config.with_tensor_shapes({"pos": (77, 36)})
    assert found.max_positions == 77 and arch.build_spec(found).max_positions == 77
    assert config_from_dict(CASES["odd"][0])[1].with_tensor_shapes({"pos": (77, 36)}).max_positions == 420


def test_missing_options_mean_none():
    raw = copy.deepcopy(CASES["mixed"][0])
    del raw["embedding"], raw["residual_mult"], raw["loop"]
    _, config, spec = _spec(raw)
    assert config.embedding_scale == 1.0 and config.residual_mult == 1.0 and config.loop is None
    raw["layers"][1]["mixer"]["q_temp"] = None
    assert _spec(raw)[2].layers[1].parts["mixer"][1].params["q_temp"] is None


def test_every_bad_key_is_reported_in_one_error():
    from xeno_rt_b200.core import ConfigError
    raw = copy.deepcopy(CASES["mixed"][0])
    raw["vocab"] = -1
    raw["norm"] = {}
    raw["embedding"]["scale"] = 0
    raw["residual_mult"] = "much"
    raw["max_positions"] = 0
    raw["loop"]["stop"] = 9
    raw["layers"][0]["mixer"]["decay"] = [0.5]
    raw["layers"][0]["mlp"]["router"]["top"] = 7
    raw["layers"][1]["mixer"]["vdim"] = 8                    # tied values have the keys' size
    raw["layers"][1]["mixer"]["q_temp"]["every"] = 0
    raw["layers"][1]["mlp"] = {"kind": "dense", "ff": 8}
    raw["layers"][2]["mixer"]["left"]["kv_heads"] = 4        # 6 heads are no multiple
    raw["layers"][2]["mixer"]["right"].pop("conv")
    raw["layers"][3]["mixer"]["scale"] = 0
    raw["layers"].append({"type": "mamba", "mixer": {}, "mlp": None})
    with pytest.raises(ConfigError) as err:
        _spec(raw)
    text = str(err.value)
    for piece in ("vocab", "eps", "embedding.scale", "residual_mult", "max_positions", "loop", "1 numbers for 3 heads",
                  "top 7", "vdim 8", "q_temp.every", "'dense'", "4 kv_heads", "right.conv", "layers[3].mixer.scale", "'mamba'"):
        assert piece in text, piece


def test_second_norms_of_layers_without_a_feed_forward_may_lie_in_the_file():
    assert set(_spec(CASES["mixed"][0])[2].ignorable_tensors) == {"l3.norm2", "l4.norm2"}


# ------------------------------------------------------------------------------------------------ the plain mechanisms
def test_the_plain_temperature_steps_where_the_position_does():
    t = {"coef": 0.5, "every": 10}
    assert [plain.temperature(p, t) for p in (0, 8)] == [1.0, 1.0]
    assert np.isclose(plain.temperature(9, t), 1 + 0.5 * np.log(2)) and np.isclose(plain.temperature(18, t), 1 + 0.5 * np.log(2))
    assert np.isclose(plain.temperature(19, t), 1 + 0.5 * np.log(3)) and plain.temperature(500, None) == 1.0


def test_the_plain_recurrences():
    k, v, q = np.array([[1.0, 0.0], [0.0, 2.0]]), np.array([[3.0], [5.0]]), np.array([[2.0, 7.0], [1.0, 1.0]])
    assert np.allclose(plain.constant_decay_scan(q, k, v, 0.5), [[6.0], [1.5 + 10.0]])
    unit = np.array([[1.0, 0.0], [1.0, 0.0]])  # the same key twice: the second write replaces what the first left
    got = plain.delta_scan(unit, unit, v, np.array([1.0, 0.5]), np.array([1.0, 1.0]))
    assert np.allclose(got, [[3.0], [5.0]])
    got = plain.delta_scan(unit, unit, v, np.array([1.0, 0.5]), np.array([1.0, 0.25]))
    assert np.allclose(got, [[3.0], [1.5 + 0.25 * (5.0 - 1.5)]])
    assert np.allclose(plain.head_decay(np.array([[0.3]]), np.array([0.7]), np.array([-1.0])),
                       np.exp(-np.exp(0.7) * np.log1p(np.exp(-0.7))))


def test_the_plain_routing_and_embedding():
    chosen, w = plain.route(np.array([0.0, 3.0, 1.0, 2.0]), 2)
    assert list(chosen) == [1, 3] and np.allclose(w, np.array([np.e, 1.0]) / (np.e + 1.0))
    table, pos = np.arange(6.0).reshape(3, 2), np.array([[100.0, 200.0], [300.0, 400.0]])
    assert np.allclose(plain.embed([2, 0], table, pos, 3.0), [[112.0, 215.0], [300.0, 403.0]])
