"""Legilix on the host: reading config.json, the model spec it turns into, the tensors it declares, the stores of its
layers, refused configurations, the rotation's frequencies, the plain rules, and ``random-model``."""

import copy
import json
import math

import pytest
import torch

from legilix_models import CONFIGS, make_weights
from plain_legilix import (F64, distance_bias, forward, gelu_tanh, grouped_rms_norm, mix_scores, rms_unit, route,
                           routed_feed_forward, silu, window_mask, yarn)


def test_the_registry_finds_the_design_by_its_own_key():
    from zephyr_b200.config import LegelixConfig, LegilixConfig, resolve_architecture

    assert resolve_architecture(CONFIGS["A"]).config_class is LegilixConfig          # and not the one a letter away
    assert resolve_architecture({"architecture": "Legelix"}).config_class is LegelixConfig
    config = LegilixConfig.from_dict(CONFIGS["B"])
    assert LegilixConfig.from_dict(config.to_dict()) == config
    assert json.loads(json.dumps(config.to_dict())) == CONFIGS["B"]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    from zephyr_b200.config import LegilixConfig
    from zephyr_b200.parts import expected_weights

    weights = make_weights(CONFIGS[name], seed=1)
    declared = expected_weights(LegilixConfig.from_dict(CONFIGS[name]).to_model_spec())
    assert set(declared) == set(weights)
    for tensor_name, decl in declared.items():
        assert tuple(weights[tensor_name].shape) == decl.shape, tensor_name


def test_the_spec_names_every_mechanism_with_its_constants():
    from zephyr_b200.cache import PagedCacheSpec
    from zephyr_b200.config import LegilixConfig
    from zephyr_b200.parts import cache_specs

    spec = LegilixConfig.from_dict(CONFIGS["A"]).to_model_spec()
    assert [call.layer for call in spec.run_order] == [0, 1, 2, 3] and [call.caches for call in spec.run_order] == [(0,), (1,), (2,), (3,)]
    assert cache_specs(spec) == [PagedCacheSpec(2, key_dim=24, value_dim=40, window=19, keep_first=5),
                                 PagedCacheSpec(3, key_dim=20, value_dim=12, window=9),
                                 PagedCacheSpec(2, key_dim=20, value_dim=12, window=23, keep_first=30),
                                 PagedCacheSpec(1, key_dim=16, value_dim=32, window=33)]
    assert [layer.block for layer in spec.layers] == ["prenorm_residual"] * 4
    assert all(norm.kind == "rmsnorm" and norm.groups == 3 and norm.eps == 1e-5 for layer in spec.layers for norm in layer.norms.values())
    assert spec.output.params["norm"].groups == 3 and spec.output.params["weight"] == "embed" and spec.output.params["logit_scale"] == 0.7
    assert spec.input.params["scale"] == 3.0 and spec.input.params["float32_stream"]
    first, second = spec.layers[0].mixer, spec.layers[1].mixer
    assert first.kind == second.kind == "attention"
    assert first.params["score_mix"] == "l0.mix.talk" and first.params["keep_first"] == 5 and first.params["scale"] == 0.25
    assert first.params["q_bias"] == "l0.mix.q.b" and first.params["q_norm"] == "l0.mix.q.norm" and "head_gate" not in first.params
    assert first.position.kind == "rope_halves" and first.position.params["dims"] == 16
    assert first.position.params["scaling"] == {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 1.0}
    assert spec.layers[2].mixer.position.params["scaling"] is None
    assert second.position is None and second.params["distance_bias"] == ("l1.mix.r1", "l1.mix.r2")
    assert second.params["head_gate"] == "l1.mix.g" and "q_norm" not in second.params and "score_mix" not in second.params
    assert second.params["v_bias"] == "l1.mix.v.b" and second.params["window"] == 9
    routed, ungated = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert routed.kind == "routed" and routed.params["scores"] == "sigmoid" and routed.params["weigh"] == "inputs"
    assert routed.params["top"] == 2 and len(routed.params["expert_names"]) == 6
    assert ungated.kind == "ungated" and ungated.params["intermediate_size"] == 100
    assert spec.layers[2].feed_forward is None and set(spec.layers[2].norms) == {"mixer"}


def test_keys_that_may_be_left_out():
    from zephyr_b200.config import LegilixConfig

    config = copy.deepcopy(CONFIGS["B"])
    for key in ("embedding", "logit_scale"):
        config.pop(key)
    config["norm"].pop("groups")
    config["layers"][2]["mixer"]["mask"].pop("keep_first")
    config["layers"][1]["mixer"]["rot"].pop("scaling")
    spec = LegilixConfig.from_dict(config).to_model_spec()
    assert spec == LegilixConfig.from_dict(CONFIGS["B"]).to_model_spec()


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown layer type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(fast=0.0), "rot.scaling.fast"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "router.top"),
    (lambda c: c["layers"][1].update(mlp={"kind": "glu", "ff": 8}), "dense or a moe"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["norm"].update(groups=7), "groups"),
    (lambda c: c.update(vocab=0), "vocab"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_bad_configurations_are_refused(change, message):
    from zephyr_b200.config import ConfigError, LegilixConfig

    config = copy.deepcopy(CONFIGS["A"])
    change(config)
    with pytest.raises(ConfigError, match=message):
        LegilixConfig.from_dict(config)


def test_parts_refuse_what_does_not_combine():
    from zephyr_b200.config import ConfigError
    from zephyr_b200.config.spec import FeedForwardSpec, NormSpec
    from zephyr_b200.parts import RMSNorm, RoutedFeedForward

    with pytest.raises(ConfigError, match="groups"):
        RMSNorm(NormSpec("rmsnorm", 10, 1e-6, "w", groups=3), {"w": torch.ones(10)}, torch.float32)
    norm = RMSNorm(NormSpec("rmsnorm", 10, 1e-6, "w", groups=2), {"w": torch.ones(10)}, torch.float32)
    assert norm.as_rms_scale() is None
    with pytest.raises(ConfigError, match="float32 stream"):
        norm.add_forward(torch.zeros(1, 10), torch.zeros(1, 10))
    with pytest.raises(ConfigError, match="identity"):
        RoutedFeedForward(FeedForwardSpec("routed", {"hidden_size": 8, "intermediate_size": 8, "experts": 2, "identity": 1, "top": 1,
                                                     "weigh": "inputs", "router": "r", "expert_names": ()}), {}, torch.float32)


def test_frequencies_masks_and_the_plain_rules():
    freqs, mult = yarn({"base": 100.0, "dims": 8, "scaling": None})
    assert mult == 1.0 and torch.allclose(freqs, torch.tensor([1.0, 100.0 ** -0.25, 0.1, 100.0 ** -0.75], dtype=F64))
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 200, "fast": 8.0, "slow": 0.5}}
    scaled, mult = yarn(rot)
    # turns over 200 positions: d(8) = 8 ln(200 / (16 pi)) / (2 ln 100) = 1.199..., d(0.5) = 3.607...: lo 1, hi 4
    ramp = torch.tensor([0.0, 0.0, 1.0 / 3.0, 2.0 / 3.0], dtype=F64)
    assert torch.allclose(scaled, freqs / 4.0 * ramp + freqs * (1.0 - ramp)) and abs(mult - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    from zephyr_b200.config.spec import PositionSpec
    from zephyr_b200.parts.position import RopeHalves
    part = RopeHalves(PositionSpec("rope_halves", 16, 64, rot), torch.float32, "cpu")
    got, dims, got_mult = part.as_half_frequencies()
    assert dims == 8 and abs(got_mult - mult) < 1e-12 and torch.allclose(got.double(), scaled, rtol=1e-7)
    # a window of 3 that keeps 2 tokens
    assert window_mask(8, 3, 2)[6].nonzero().flatten().tolist() == [0, 1, 4, 5, 6]
    assert window_mask(8, 1)[6].nonzero().flatten().tolist() == [6]
    # each part of a row has a statistic of its own, the scale is one vector over the row
    x = torch.tensor([[3.0, 4.0, 0.0, 0.5]], dtype=F64)
    w = torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=F64)
    expected = torch.tensor([[3.0 / math.sqrt(12.5), 8.0 / math.sqrt(12.5), 0.0, 4.0 * math.sqrt(2.0)]], dtype=F64)
    assert torch.allclose(grouped_rms_norm(x, w, 2, 0.0), expected)
    assert torch.allclose(grouped_rms_norm(x, w, 1, 0.0), rms_unit(x, 0.0) * w)
    # row h of the matrix holds what head h takes of every head's scores
    scores = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    assert mix_scores(scores, torch.tensor([[1.0, 2.0], [0.0, -1.0]], dtype=F64)).flatten().tolist() == [21.0, -10.0]
    bias = distance_bias(4, torch.tensor([2.0], dtype=F64), torch.tensor([0.5], dtype=F64))[0]
    assert bias[2, 2] == 0.0 and abs(float(bias[3, 0]) - 2.0 * math.log(2.5)) < 1e-12
    z = torch.tensor([-3.0, 0.0, 0.7, 5.0], dtype=F64)
    assert torch.allclose(gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_the_router_weighs_inputs_with_scores_that_do_not_add_up_to_one():
    w = {"r.router": torch.eye(3, 2, dtype=F64)}
    for e in range(3):
        w.update({f"r.e{e}.gate": torch.full((1, 2), 1.0 + e, dtype=F64), f"r.e{e}.up": torch.full((1, 2), 0.5, dtype=F64),
                  f"r.e{e}.down": torch.tensor([[1.0], [10.0]], dtype=F64)})
    h = torch.tensor([[2.0, -1.0]], dtype=F64)
    ids, weights, margin = route(h, w, "r", 2)
    assert ids.tolist() == [[0, 2]] and margin.tolist() == [1.0]                     # logits 2, -1, 0
    assert torch.allclose(weights, torch.sigmoid(torch.tensor([[2.0, 0.0]], dtype=F64)))
    total = 0.0
    for e, s in ((0, weights[0, 0]), (2, weights[0, 1])):
        x = s * h[0].sum()
        total = total + silu((1.0 + e) * x) * (0.5 * x)
    assert torch.allclose(routed_feed_forward(h, w, "r", {"router": {"top": 2, "experts": 3}}),
                          total * torch.tensor([[1.0, 10.0]], dtype=F64))


def test_the_plain_model_runs_every_configuration():
    for name, config in CONFIGS.items():
        layers: list = []
        weights = make_weights(config, seed=3)
        tokens = list(range(30))
        logits = forward(config, weights, tokens, layers_out=layers)
        assert logits.shape == (30, config["vocab"]) and torch.isfinite(logits).all() and len(layers) == len(config["layers"])
        # nothing looks ahead
        assert torch.allclose(forward(config, weights, tokens[:17]), logits[:17], atol=1e-9)


def test_random_model_from_the_command_line(tmp_path):
    from zephyr_b200.cli import main
    from zephyr_b200.config import load_model_config
    from zephyr_b200.parts import expected_weights
    from zephyr_b200.weights import Checkpoint
    from zephyr_b200.weights.loader import check_store

    source = tmp_path / "config.json"
    source.write_text(json.dumps(CONFIGS["C"]))
    assert main(["random-model", "--config", str(source), "--out", str(tmp_path / "model"), "--seed", "3"]) == 0
    config = load_model_config(tmp_path / "model")
    assert config.to_dict() == CONFIGS["C"]
    store = Checkpoint(tmp_path / "model")
    check_store(store, expected_weights(config.to_model_spec()))
    assert tuple(store.shape("l1.mix.talk")) == (16, 16) and tuple(store.shape("l4.mix.r1")) == (17,)
