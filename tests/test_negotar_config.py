"""Reading, refusing and laying out Negotar configurations; properties of the plain implementation; runs without a GPU."""

import copy
import math

import pytest
import torch

import negotar_cases as cases
import plain_negotar as plain
from stride_b200.config import ConfigError, NegotarConfig, PositionSpec, RopeScaling, config_from_dict, plan_memory
from stride_b200.engine.loading import _declarations, footprint

F64 = torch.float64


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_declarations_are_the_checkpoints_tensors(case):
    config, state = config_from_dict(cases.CASES[case]), cases.seeded_state(cases.CASES[case], 1)
    assert isinstance(config, NegotarConfig)
    declared = _declarations(config)
    assert set(declared) == set(state)
    for name, decl in declared.items():
        assert tuple(decl.shape) == tuple(state[name].shape), name
    assert config.to_dict() == cases.CASES[case] and config_from_dict(config.to_dict()) == config
    assert config.with_max_positions(70000).max_position_embeddings == 70000


def test_layout():
    spec = config_from_dict(cases.CASE_A).to_model_spec()
    assert spec.head_spec().name is None and spec.head_spec().hidden == 72
    assert dict(spec.final_norm.params) == {"tensor": "final.norm", "weight_offset": 1.0, "factor": 1.7}
    assert all(layer.kind == "output_norm" and layer.residual_mult == 1.0 for layer in spec.layers)
    assert dict(spec.layers[0].mixer_norm.params) == {"tensor": "l0.norm1", "weight_offset": 1.0}
    m = spec.layers[0].mixer
    assert (m.kind, m.num_heads, m.head_dim) == ("mamba2", 6, 20)
    assert dict(m.params) == {"groups": 3, "state": 12, "taps": 3, "norm_groups": 2, "norm_eps": 1e-4}
    mixing = [dict(layer.mixer.params).get("value_mix") for layer in spec.layers]
    assert mixing == [None, "first", None, "later"]
    assert [dict(layer.mixer.params).get("softcap") for layer in spec.layers[1:]] == [20.0, None, 3.0]
    position = spec.layers[3].mixer.position
    assert dict(position.params)["rotated"] == 8 and position.scaling == RopeScaling("llama3", 4.0, 2.0, 3.0, 100)
    assert spec.layers[1].mixer.position.scaling is None and spec.layers[1].feed_forward is None and spec.layers[1].ffn_norm is None
    d = copy.deepcopy(cases.CASE_A)
    d["layers"][1]["mixer"]["rot"] = None
    assert dict(config_from_dict(d).to_model_spec().layers[1].mixer.position.params)["rotated"] == 0
    f = spec.layers[3].feed_forward
    assert (f.kind, f.intermediate, f.activation) == ("routed_experts", 16, "silu")
    assert dict(f.params) == {"experts": 7, "top": 4, "router": "sigmoid_scores", "weigh": "inputs"}


def test_footprint_counts_states_and_padded_heads():
    f = footprint(config_from_dict(cases.CASE_A), "float32")
    assert f["kv_bytes_per_token"] == 4 * (2 * (20 + 24) + 1 * (16 + 40) + 2 * (24 + 24))
    assert f["state_bytes_per_request"] == 4 * (6 * 12 * 20 + 3 * (6 * 20 + 2 * 3 * 12))
    # bfloat16: heads of 20 / 24 stay (64 would more than double them), 80 / 64 lie in 128, 128 / 64 in 128
    f = footprint(config_from_dict(cases.CASE_C), "bfloat16")
    assert f["kv_bytes_per_token"] == 2 * (2 * 128 + 2 * 256 + 2 * 256)
    assert footprint(config_from_dict(cases.CASE_A), "bfloat16")["kv_bytes_per_token"] == 2 * (2 * 44 + 56 + 2 * 48)
    assert plan_memory(config_from_dict(cases.CASE_C)).num_blocks > 0


def test_rotation_tables_follow_the_rule():
    """Part of a head, halves paired, frequencies kept, divided and in between; against the rule evaluated in float64."""
    from stride_b200.parts import Runtime, build_part
    rt = Runtime("cpu", torch.float32, 8, 8)
    for rot, dim in ((cases.rotation(12, scaled=False), 20), (cases.rotation(48, base=500000.0, factor=8.0, original=128), 80),
                     (cases.rotation(10, base=37.0, factor=3.0, low=2.0, high=2.0, original=50), 10), (cases.rotation(0, scaled=False), 7)):
        sc = rot.get("scaling")
        scaling = RopeScaling("llama3", sc["factor"], sc["low"], sc["high"], sc["original"]) if sc else None
        part = build_part("position", PositionSpec(kind="rope", head_dim=dim, theta=rot["base"], max_positions=300, scaling=scaling,
                                                   params=(("angles", "float64"), ("rotated", rot["dims"]))), rt)
        cos, sin = part.plain_tables()
        f = torch.tensor(plain.rotation_frequencies(rot), dtype=F64)
        a = torch.arange(300, dtype=F64)[:, None] * f
        assert cos.shape == sin.shape == (300, rot["dims"] // 2) and cos.dtype == torch.float32
        if rot["dims"]:
            assert float((cos.double() - a.cos()).abs().max()) < 1e-7 and float((sin.double() - a.sin()).abs().max()) < 1e-7
    kept, divided = plain.rotation_frequencies(cases.rotation(48, base=500000.0, factor=8.0, original=128, scaled=False)), \
        plain.rotation_frequencies(cases.rotation(48, base=500000.0, factor=8.0, original=128))
    ratio = [b / a for a, b in zip(kept, divided)]
    assert ratio[0] == 1.0 and abs(ratio[-1] - 0.125) < 1e-12 and any(0.13 < r < 0.99 for r in ratio)


def test_plain_mechanisms_have_the_properties_they_name():
    """The oracle itself: with no decay the memory is a running sum; a turn keeps a head's length and scores depend on distances; one
    part per channel norms to signs; a gate in front of a norm is not the gate behind it; a chosen expert's input carries the score."""
    g = torch.Generator().manual_seed(1)
    x, B, C = torch.randn(5, 2, 3, generator=g, dtype=F64), torch.randn(5, 1, 4, generator=g, dtype=F64), torch.randn(5, 1, 4, generator=g, dtype=F64)
    dt = torch.rand(5, 2, generator=g, dtype=F64)
    y = plain.selective_memory(x, B, C, dt, torch.full((2,), -80.0, dtype=F64), torch.tensor([0.0, 2.0], dtype=F64))
    for h in range(2):
        want = torch.stack([sum(float(C[t, 0] @ B[j, 0]) * dt[j, h] * x[j, h] for j in range(t + 1)) for t in range(5)])
        assert torch.allclose(y[:, h], want + (2.0 if h else 0.0) * x[:, h])
    assert torch.allclose(plain.step_size(torch.tensor([-700.0, 0.0, 800.0], dtype=F64), 0.0), torch.tensor([0.0, math.log(2.0), 800.0], dtype=F64))
    rot = cases.rotation(4, original=16)
    q, k = torch.randn(1, 1, 6, generator=g, dtype=F64), torch.randn(1, 1, 6, generator=g, dtype=F64)
    dot = lambda i, j: float((plain.rotate(q, rot, i) * plain.rotate(k, rot, j)).sum())
    assert abs(dot(9, 4) - dot(25, 20)) < 1e-12 and abs(dot(9, 4) - dot(9, 5)) > 1e-6
    assert torch.equal(plain.rotate(q, rot, 31)[..., 4:], q[..., 4:]) and abs(float(plain.rotate(q, rot, 31).norm() - q.norm())) < 1e-12
    z = torch.randn(2, 6, generator=g, dtype=F64)
    y = torch.randn(2, 6, generator=g, dtype=F64)
    assert torch.allclose(plain.gated_group_norm(y, z, torch.ones(6, dtype=F64), 6, 0.0), torch.sign(y * z))
    assert not torch.allclose(plain.gated_group_norm(y, z, torch.ones(6, dtype=F64), 2, 0.0), plain.rms_unit(y.view(2, 2, 3), 0.0).view(2, 6) * plain.silu(z))
    router = torch.tensor([[1.0, 0.0], [3.0, 0.0], [-2.0, 0.0]], dtype=F64)
    ids, scores = plain.route(torch.tensor([1.0, 5.0], dtype=F64), router, 2)
    assert ids == [1, 0] and torch.allclose(scores, torch.sigmoid(torch.tensor([3.0, 1.0], dtype=F64)))


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="wkv"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(groups=4), "groups"),
    (lambda d: d["layers"][0]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda d: d["layers"][0]["mixer"].update(state=257), "256"),
    (lambda d: d["layers"][0]["mixer"].update(conv=17), "taps"),
    (lambda d: d["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), "group"),
    (lambda d: d["layers"][1]["mixer"].update(dim=300), "256"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=300), "256"),
    (lambda d: d["layers"][1]["mixer"].update(v_mix=1), "v_mix"),
    (lambda d: d["layers"][3]["mixer"].update(vdim=20), "cannot be mixed"),
    (lambda d: d["layers"][3]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][1]["mixer"].update(rot=3), "rot"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), "at most"),
    (lambda d: d["layers"][3]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda d: d["layers"][3]["mixer"]["rot"]["scaling"].update(high=1.0), "high"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "experts"),
    (lambda d: d["layers"][0]["mlp"].pop("expert"), "ff"),
    (lambda d: d.pop("logit_scale"), "logit_scale"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_refusals(change, message):
    d = copy.deepcopy(cases.CASE_A)
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)
