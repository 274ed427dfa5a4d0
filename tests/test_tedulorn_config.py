"""Tedulorn on the host: reading config.json, the model spec it turns into, the tensors it declares, the stores of its
layers, refused configurations, the plain rules, and ``random-model``."""

import copy
import json
import math

import pytest
import torch

from plain_tedulorn import (F64, bounded_expert, decayed_states, forward, frequencies, gelu_tanh, mix_values, rms_norm, rotate_halves,
                            route, softmax_plus_one, token_side, window_mask)
from tedulorn_models import CONFIGS, first_mixing_layer, make_weights


def test_the_registry_finds_the_design_by_its_own_key():
    from zephyr_b200.config import TedulornConfig, resolve_architecture

    assert resolve_architecture(CONFIGS["A"]).config_class is TedulornConfig
    config = TedulornConfig.from_dict(CONFIGS["B"])
    assert TedulornConfig.from_dict(config.to_dict()) == config
    assert json.loads(json.dumps(config.to_dict())) == CONFIGS["B"]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_declared_tensors_are_the_checkpoints(name):
    """All but the first mixing layer's share, which may lie in a checkpoint and is not read."""
    from zephyr_b200.config import TedulornConfig
    from zephyr_b200.parts import expected_weights

    weights = make_weights(CONFIGS[name], seed=1)
    spec = TedulornConfig.from_dict(CONFIGS[name]).to_model_spec()
    declared = expected_weights(spec)
    unread = f"l{first_mixing_layer(CONFIGS[name])}.mix.vmix"
    assert set(declared) == set(weights) - {unread} and unread in spec.ignorable_weights
    for tensor_name, decl in declared.items():
        assert tuple(weights[tensor_name].shape) == decl.shape, tensor_name


def test_the_spec_names_every_mechanism_with_its_constants():
    from zephyr_b200.cache import PagedCacheSpec, StateCacheSpec
    from zephyr_b200.config import TedulornConfig
    from zephyr_b200.parts import cache_specs

    spec = TedulornConfig.from_dict(CONFIGS["A"]).to_model_spec()
    assert [call.caches for call in spec.run_order] == [(0,), (1,), (2,), (3,), (4,)]
    assert cache_specs(spec) == [StateCacheSpec(shape=(3 * 20 * 12,), dtype="float32"),
                                 PagedCacheSpec(2, key_dim=24, value_dim=40, window=19, keep_first=5),
                                 PagedCacheSpec(5, key_dim=16, value_dim=24, window=33),
                                 PagedCacheSpec(2, key_dim=20, value_dim=40, window=9, keep_first=30),
                                 StateCacheSpec(shape=(33 * 50,), dtype="float32")]
    assert [layer.block for layer in spec.layers] == ["prenorm_residual"] * 5
    assert all(norm.kind == "rmsnorm" and norm.eps == 1e-5 for layer in spec.layers for norm in layer.norms.values())
    assert spec.input.params["scale"] == 3.0 and spec.input.params["float32_stream"]
    assert spec.output.params["weight"] == "head" and spec.output.params["norm"].weight == "final.norm"
    kept, seen = spec.layers[0].mixer, spec.layers[1].mixer
    assert kept.kind == "retention" and kept.params["decay"] == (0.5, 0.97, 0.999) and kept.params["norm_eps"] == 1e-5
    assert kept.position.kind == "rope_halves" and kept.position.params == {"base": 300.0, "dims": 8} and kept.position.head_dim == 20
    assert seen.kind == "attention" and seen.params["zero_sinks"] and seen.params["keep_first"] == 5 and seen.params["window"] == 19
    assert seen.params["scale"] == 0.25 and seen.params["head_gate"] == "l1.mix.g" and seen.params["q_norm"] == "l1.mix.q.norm"
    assert seen.params["value_mix"] == {"group": "values", "share": None}
    assert "value_mix" not in spec.layers[2].mixer.params
    assert spec.layers[3].mixer.params["value_mix"] == {"group": "values", "share": "l3.mix.vmix"}
    assert spec.layers[2].feed_forward is None and set(spec.layers[2].norms) == {"mixer"}
    ungated, routed = spec.layers[0].feed_forward, spec.layers[1].feed_forward
    assert ungated.kind == "ungated" and ungated.params["activation"] == "relu_squared" and ungated.params["intermediate_size"] == 100
    p = routed.params
    assert routed.kind == "routed" and p["scores"] == "softmax" and p["normalize"] and p["groups"] == {"count": 3, "keep": 2, "top": 1}
    assert (p["activation"], p["limit"], p["alpha"], p["up_shift"]) == ("clamped_swish", 1.2, 1.702, 1.0)
    assert (p["shared"]["intermediate_size"], p["shared"]["limit"], p["shared"]["gate_proj"]) == (24, 2.0, "l1.mlp.shared.gate")
    assert p["correction"] == "l1.mlp.correction" and len(p["expert_names"]) == 6
    side = spec.layers[3].side
    assert side.kind == "token_gate" and side.params["offset"] == 36 and side.params["dim"] == 12 and side.params["row"] == 60
    assert side.params["norm"].weight == "l3.side.norm"


def test_keys_that_may_be_left_out():
    from zephyr_b200.config import TedulornConfig

    config = copy.deepcopy(CONFIGS["B"])
    config.pop("embedding")
    config["layers"][0]["mlp"]["router"].pop("groups")
    config["layers"][2]["mixer"]["mask"].pop("keep_first")
    config["layers"][0]["mixer"].pop("v_mix")
    spec = TedulornConfig.from_dict(config).to_model_spec()
    full = TedulornConfig.from_dict(CONFIGS["B"]).to_model_spec()
    assert spec.layers[1:] == full.layers[1:] and spec.input == full.input
    assert spec.layers[0].mixer == full.layers[0].mixer and "groups" not in spec.layers[0].feed_forward.params
    config["layers"][2]["mixer"]["mask"] = None
    assert TedulornConfig.from_dict(config).to_model_spec().layers[2].mixer.params["window"] == 0
    config.pop("token_side")
    assert all(layer.side is None for layer in TedulornConfig.from_dict(config).to_model_spec().layers)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="delta"), "unknown layer type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.9, "x"]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), "size"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=20), "mix values"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=8), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0.0), "expert.limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0].update(mlp={"kind": "glu", "ff": 8}), "dense or a moe"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(vocab=0), "vocab"),
])
def test_bad_configurations_are_refused(change, message):
    from zephyr_b200.config import ConfigError, TedulornConfig

    config = copy.deepcopy(CONFIGS["A"])
    change(config)
    with pytest.raises(ConfigError, match=message):
        TedulornConfig.from_dict(config)


def test_parts_refuse_what_does_not_combine():
    from zephyr_b200.config import ConfigError
    from zephyr_b200.config.spec import FeedForwardSpec, LayerSpec, MixerSpec, SideSpec
    from zephyr_b200.parts import RoutedFeedForward, UngatedFeedForward
    from zephyr_b200.parts.model import _layer_classes

    with pytest.raises(ConfigError, match="relu_squared"):
        UngatedFeedForward(FeedForwardSpec("ungated", {"activation": "tanh", "up_proj": "u", "down_proj": "d"}), {}, torch.float32)
    routed = {"hidden_size": 8, "intermediate_size": 8, "experts": 2, "top": 1, "router": "r", "expert_names": ()}
    with pytest.raises(ConfigError, match="positive limit"):
        RoutedFeedForward(FeedForwardSpec("routed", {**routed, "activation": "clamped_swish", "limit": 0.0}), {}, torch.float32)
    with pytest.raises(ConfigError, match="weights on their outputs"):
        RoutedFeedForward(FeedForwardSpec("routed", {**routed, "activation": "clamped_swish", "limit": 1.0, "weigh": "inputs"}), {}, torch.float32)
    with pytest.raises(ConfigError, match="no side part"):
        _layer_classes(LayerSpec("sandwich_residual", MixerSpec("attention", {}), None,
                                 {"mixer": None, "mixer_out": None}, side=SideSpec("token_gate", {})))


def test_the_plain_rules():
    # a window of 3 that keeps 2 tokens
    assert window_mask(8, 3, 2)[6].nonzero().flatten().tolist() == [0, 1, 4, 5, 6]
    assert window_mask(8, 1)[6].nonzero().flatten().tolist() == [6]
    # one joins the denominator, also far from zero
    weights = softmax_plus_one(torch.tensor([[0.0, math.log(2.0), 9.0]], dtype=F64), torch.tensor([[True, True, False]]))
    assert torch.allclose(weights, torch.tensor([[0.25, 0.5, 0.0]], dtype=F64))
    assert float(softmax_plus_one(torch.tensor([[-300.0]], dtype=F64), torch.tensor([[True]]))) < 1e-100
    assert abs(float(softmax_plus_one(torch.tensor([[800.0]], dtype=F64), torch.tensor([[True]]))) - 1.0) < 1e-12
    # the state forgets by its head's factor, the newest token counts in full
    q = torch.ones(3, 2, 1, dtype=F64)
    v = torch.tensor([[[1.0], [1.0]], [[10.0], [10.0]], [[100.0], [100.0]]], dtype=F64)
    o = decayed_states(q, q, v, torch.tensor([0.5, 1.0], dtype=F64))
    assert o[2].flatten().tolist() == [100.0 + 5.0 + 0.25, 111.0]
    # value i < dims / 2 turns with value i + dims / 2, the rest passes
    rot = {"base": 100.0, "dims": 4}
    assert torch.allclose(frequencies(rot), torch.tensor([1.0, 0.1], dtype=F64))
    x = torch.arange(1.0, 7.0, dtype=F64).view(1, 1, 6)
    y = rotate_halves(x, torch.tensor([5]), rot).flatten()
    assert torch.allclose(y[[0, 2]], torch.tensor([math.cos(5.0) - 3.0 * math.sin(5.0), 3.0 * math.cos(5.0) + math.sin(5.0)], dtype=F64))
    assert torch.allclose(y[[1, 3]], torch.tensor([2.0 * math.cos(0.5) - 4.0 * math.sin(0.5), 4.0 * math.cos(0.5) + 2.0 * math.sin(0.5)], dtype=F64))
    assert y[4:].tolist() == [5.0, 6.0]
    assert mix_values(torch.tensor([1.0, 2.0]), torch.tensor([5.0, 5.0]), torch.tensor(0.25)).tolist() == [2.0, 2.75]
    assert mix_values(torch.tensor([1.0]), None, torch.tensor(0.25)).tolist() == [1.0]
    z = torch.tensor([-3.0, 0.0, 0.7, 5.0], dtype=F64)
    assert torch.allclose(gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_a_bounded_expert_and_the_token_gate():
    w = {"e.gate": torch.tensor([[1.0], [1.0]], dtype=F64), "e.up": torch.tensor([[1.0], [-1.0]], dtype=F64),
         "e.down": torch.tensor([[1.0, 10.0]], dtype=F64)}
    y = bounded_expert(torch.tensor([[3.0]], dtype=F64), w, "e", 2.0)         # both bounds reached
    s = 2.0 / (1.0 + math.exp(-3.404))
    assert abs(float(y) - (s * 3.0 + 10.0 * s * -1.0)) < 1e-12
    y = bounded_expert(torch.tensor([[-3.0]], dtype=F64), w, "e", 2.0)        # the gate has no lower bound
    s = -3.0 / (1.0 + math.exp(3.0 * 1.702))
    assert abs(float(y) - (s * -1.0 + 10.0 * s * 3.0)) < 1e-12
    w = {"s.gate": torch.tensor([[1.0, 0.0]], dtype=F64), "s.proj": torch.tensor([[3.0], [4.0]], dtype=F64), "s.norm": torch.tensor([1.0, 2.0], dtype=F64)}
    y = token_side(torch.tensor([[100.0, 7.0]], dtype=F64), torch.tensor([[0.5]], dtype=F64), w, "s", 0.0)     # gelu(100) = 100
    assert torch.allclose(y, torch.tensor([[150.0 / math.sqrt(31250.0), 400.0 / math.sqrt(31250.0)]], dtype=F64))
    assert torch.allclose(rms_norm(torch.tensor([[3.0, 4.0]], dtype=F64), torch.ones(2, dtype=F64), 12.5), torch.tensor([[0.6, 0.8]], dtype=F64))


def test_the_router_looks_at_groups_with_choices_below_zero():
    z = torch.log(torch.tensor([[0.30, 0.10, 0.20, 0.15, 0.05, 0.20]], dtype=F64))
    correction = torch.tensor([-0.9, -0.9, -0.5, -0.9, -0.9, -0.4], dtype=F64)
    # choices -0.6 -0.8 | -0.3 -0.75 | -0.85 -0.2: the first group is out although its best beats others' seconds
    ids, weights, margin = route(z, correction, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert ids.tolist() == [[5, 2, 3]]
    assert torch.allclose(weights, torch.tensor([[0.20, 0.20, 0.15]], dtype=F64) / 0.55)        # scores without the correction
    assert abs(float(margin) - 0.1) < 1e-9                                                      # expert 3 before expert 4
    ids, _, margin = route(z, correction, {"experts": 6, "top": 1, "groups": {"count": 3, "keep": 3}})
    assert ids.tolist() == [[5]] and abs(float(margin) - 0.1) < 1e-9


def test_the_plain_model_runs_every_configuration():
    for name, config in CONFIGS.items():
        layers: list = []
        weights = make_weights(config, seed=3)
        tokens = list(range(30))
        logits = forward(config, weights, tokens, layers_out=layers)
        assert logits.shape == (30, config["vocab"]) and torch.isfinite(logits).all() and len(layers) == len(config["layers"])
        # nothing looks ahead
        assert torch.allclose(forward(config, weights, tokens[:17]), logits[:17], atol=1e-9)
        # the first mixing layer's share is not read; a later one's is
        mixing = [i for i, layer in enumerate(config["layers"]) if layer["mixer"].get("v_mix")]
        other = {**weights, f"l{mixing[0]}.mix.vmix": torch.tensor(0.9)}
        assert torch.equal(forward(config, other, tokens), logits)
        other = {**weights, f"l{mixing[1]}.mix.vmix": torch.tensor(0.9)}
        assert not torch.allclose(forward(config, other, tokens), logits, atol=1e-3)


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
    assert tuple(store.shape("side.embed")) == (64, 6 * 32) and tuple(store.shape("l2.mix.vmix")) == ()
