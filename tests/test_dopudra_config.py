"""Reading, refusing and laying out Dopudra configurations; runs without a GPU."""

import copy

import pytest
import torch

import dopudra_cases as cases
import plain_dopudra as plain
from stride_b200.config import ConfigError, DopudraConfig, config_from_dict
from stride_b200.engine.loading import _declarations, footprint
from stride_b200.parts.attention import distance_bucket


def completed(case):
    """The configuration as the loader sees it: sizes no key names come from the tensors' shapes."""
    state = cases.case_state(case, 1)
    return config_from_dict(cases.CASES[case], set(state), {k: tuple(v.shape) for k, v in state.items()}), state


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_declarations_are_the_checkpoints_tensors(case):
    config, state = completed(case)
    assert isinstance(config, DopudraConfig)
    declared = _declarations(config)
    assert set(declared) == set(state)
    for name, decl in declared.items():
        assert tuple(decl.shape) == tuple(state[name].shape), name
    assert config_from_dict(config.to_dict()) == config


def test_sizes_that_only_shapes_give():
    d = copy.deepcopy(cases.CASE_A)
    d.pop("max_positions")
    state = cases.case_state("A", 1)
    config = config_from_dict(d, set(state), {k: tuple(v.shape) for k, v in state.items()})
    assert config.max_position_embeddings == 320
    assert [config.layers[i]["mixer"]["left"]["buckets"] for i in (1, 3)] == [8, 20]
    assert [config.layers[i]["mixer"]["right"]["decay_rank"] for i in (1, 3)] == [5, 16]
    # given in config.json they are kept, and a table of another length is then an error of the loader
    d["layers"][1]["mixer"]["left"]["buckets"] = 12
    assert config_from_dict(d, set(state), {k: tuple(v.shape) for k, v in state.items()}).layers[1]["mixer"]["left"]["buckets"] == 12
    with pytest.raises(ValueError, match="number of buckets"):
        _declarations(config_from_dict(cases.CASE_A))           # neither given nor read off a checkpoint


def test_layout():
    config, _ = completed("A")
    spec = config.to_model_spec()
    assert spec.copies == 3 and spec.max_positions == 320 and spec.head_spec().name == "head"
    assert dict(spec.embedding_spec().params) == {"scale": 1.3, "positions": ("pos", 320)}
    assert all(layer.kind == "copies" for layer in spec.layers) and [e.cache for e in spec.schedule] == [0, 1, 2, 3]
    assert dict(spec.layers[0].params) == {"copies": 3, "mixer_copies": "l0.hc1.", "mixer_scale": "l0.ls1"}
    assert dict(spec.layers[1].params)["ffn_copies"] == "l1.hc2." and spec.layers[1].feed_forward.kind == "mlp"
    assert spec.layers[0].feed_forward is None and spec.layers[0].ffn_norm is None
    light = spec.layers[0].mixer
    assert light.kind == "lightning" and dict(light.params)["decay"] == (0.0, 0.93, 1.0)
    (left, ls), (right, rs) = dict(spec.layers[1].mixer.params)["branches"]
    p = dict(left.params)
    assert (ls, rs) == (0.9, 1.3) and left.scale == 0.6 and left.window is None and left.position.kind == "none" and not left.bias
    assert (p["conv"], p["qk_norm"], p["query_factor"], p["distance_table"], p["value_dim"]) == (4, "rows", (0.3, 16), (8, 30, 320), 24)
    p = dict(right.params)
    assert right.kind == "channel_decay" and (p["tau"], p["decay_rank"], p["value_dim"]) == (4.0, 5, 40)


def test_footprint_counts_both_branches_states():
    config, _ = completed("A")
    f = footprint(config, "bfloat16")
    assert f["kv_bytes_per_token"] == 2 * (2 * 16 + 2 * 24 + 3 * 8 + 3 * 8)
    tails = [3 * (6 * 16 + 2 * 16 + 2 * 24), 1 * (9 * 8)]           # taps - 1 projected rows of either attention
    assert f["state_bytes_per_request"] == 4 * (3 * 12 * 20 + tails[0] + 2 * 24 * 40 + 2 * 40 * 16 + tails[1] + 3 * 16 * 8)


def test_distance_buckets():
    """Against the rule as written, over tables of many lengths; at distances where the logarithm is a whole number the bucket
    is the one that the exact value gives."""
    for buckets, largest in ((32, 120), (8, 30), (2, 6), (10, 21), (20, 100), (64, 33), (32, 100000), (6, 4), (7, 50)):
        for n in list(range(0, 3 * largest if largest < 1000 else 3000)):
            assert distance_bucket(n, buckets, largest) == plain.distance_bucket(n, buckets, largest), (buckets, largest, n)
    # 16 buckets, 8 * 2^(k / 2): every second power of sqrt(2) is a distance, and its bucket begins there
    for k in range(0, 8, 2):
        n = 8 * 2 ** (k // 2)
        assert distance_bucket(n, 16, 128) == 8 + k and distance_bucket(n - 1, 16, 128) == (8 + k - 1 if k else 7)
    assert [distance_bucket(n, 16, 128) for n in (126, 127, 128, 129, 10 ** 6)] == [15] * 5


def test_plain_mechanisms_have_the_properties_they_name():
    """The oracle itself: a memory with decay 1 is a running sum, with decay 0 the last token's product alone; a convolution
    with one tap is a factor; equal copies mixed by a matrix of column sums one stay equal."""
    w = {"q": torch.eye(2, dtype=torch.float64), "k": torch.eye(2, dtype=torch.float64), "v": torch.eye(2, dtype=torch.float64),
         "g": torch.full((2, 2), 0.0, dtype=torch.float64), "o": torch.eye(2, dtype=torch.float64), "norm": torch.ones(2, dtype=torch.float64)}
    h = torch.tensor([[1.0, -0.5], [0.3, 2.0], [-1.0, 0.7]], dtype=torch.float64)
    m = {"heads": 1, "dim": 2, "vdim": 2, "decay": [0.0]}
    s = plain.silu(h)
    alone = torch.stack([(s[t] @ s[t]) * s[t] for t in range(3)])
    assert torch.allclose(plain.lightning(h, w, "", m, 0.0), plain.rms_unit(alone, 0.0) * 0.5)
    m["decay"] = [1.0]
    summed = torch.stack([sum((s[t] @ s[j]) * s[j] for j in range(t + 1)) for t in range(3)])
    assert torch.allclose(plain.lightning(h, w, "", m, 0.0), plain.rms_unit(summed, 0.0) * 0.5)
    X = torch.ones(3, 2, 4, dtype=torch.float64)
    mix = torch.tensor([[0.5, 0.1, 0.3], [0.2, 0.6, 0.3], [0.3, 0.3, 0.4]], dtype=torch.float64)
    new = plain.write_copies(X, torch.zeros(2, 4, dtype=torch.float64), {"mix": mix, "out": torch.ones(3, dtype=torch.float64)}, "")
    assert torch.allclose(new, X)


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="wkv"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(decay=[0.5, 0.5]), "decay"),
    (lambda d: d["layers"][0]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda d: d["layers"][0]["mixer"].update(dim=300), "256"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(kv_heads=4), "group"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(vdim=300), "256"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(conv=17), "taps"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(buckets=64), "bias_max"),
    (lambda d: d["layers"][1]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(tau=0), "tau"),
    (lambda d: d["layers"][1]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda d: d["layers"][1]["mlp"].update(kind="moe"), "kind"),
    (lambda d: d.update(streams=17), "streams"),
    (lambda d: d.update(streams=0), "streams"),
    (lambda d: d.pop("embedding"), "embedding"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.pop("max_positions"), "max_positions"),
])
def test_refusals(change, message):
    d = copy.deepcopy(cases.CASE_A)
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)
