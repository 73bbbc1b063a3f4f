"""Getozen on the host: configuration, registry, tensor list, schedule, cache plan, the plain mechanisms by hand."""

import json
import math

import pytest
import torch

import getozen_helpers as gh
from paged_attention_engine_b200.cache import plan_cache
from paged_attention_engine_b200.config import ConfigError, GetozenConfig, resolve
from paged_attention_engine_b200.parts import MIXERS
from paged_attention_engine_b200.weights import WeightsError, collect_tensor_specs
from plain import getozen_plain as plain


def test_configuration_round_trip_and_registry():
    for raw, _page, _seed in gh.SMALL.values():
        cfg, spec = resolve(raw)
        assert isinstance(cfg, GetozenConfig)
        assert GetozenConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.to_dict() == raw
        assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"]
        own = [(i, e) for i, e in enumerate(raw["layers"]) if "weights_of" not in e]
        assert len(spec.layers) == len(own) and len(spec.schedule) == len(raw["layers"])
        for layer, (i, entry) in zip(spec.layers, own):
            assert layer.block == ("parallel_two_norms" if entry["mlp"] else "summed_mixer")
            m = entry["mixer"]
            if entry["type"] == "parallel":
                assert layer.mixer.kind == "side_by_side"
                left, right = layer.mixer.params["mixers"]
                assert (left["kind"], left["scale"], right["kind"], right["scale"]) == (
                    "gated_window_attention", m["left_scale"], "retention", m["right_scale"])
                assert left["params"]["pairing"] == "interleaved" and left["params"]["qkv_bias"] and left["params"]["window"] == 0
                scaling = m["left"]["rot"].get("scaling")
                assert left["params"]["position_encoding"]["scaling"] == (dict(scaling, kind="linear") if scaling else None)
                assert right["params"]["pairing"] == "half" and list(right["params"]["decay"]) == m["right"]["decay"]
            else:
                assert layer.mixer.kind == "state_space" and layer.mixer.params["conv_taps"] == m["conv"]
            if entry["mlp"]:
                assert layer.feed_forward.kind == "gated_mlp" and layer.feed_forward.params["activation"] == "relu"
        assert spec.final_norm.kind == "dynamic_tanh"


def test_a_layer_that_uses_anothers_weights_is_a_second_run_of_it():
    _, spec = resolve(gh.SMALL_A)            # layers 0, 1, 2, then 1 and 0 again, then one of its own
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 0, 3]
    names = collect_tensor_specs(spec)
    assert not any(n.startswith(("l3.", "l4.")) for n in names) and "l5.mix.left.q" in names
    plan = plan_cache(spec)
    assert sorted(plan.entry_group) == [0, 4, 5]             # every run of the attention holds its own keys
    assert plan.entry_group[0][0] == plan.entry_group[4][0] and plan.entry_group[0][1] != plan.entry_group[4][1]
    assert sorted(plan.state_needs) == list(range(6))        # and every run its own state


def test_cache_plan_and_states():
    plan = plan_cache(resolve(gh.SMALL_A)[1])
    group = plan.groups[plan.entry_group[0][0]]
    assert (group.num_kv_heads, group.head_dim, group.value_dim, group.window) == (2, 12, 20, 0)
    assert plan.state_needs[0].shape == (3, 10, 6) and plan.state_needs[0].dtype == torch.float32
    # S and the convolution's rows, each from a 16-byte boundary on
    assert plan.state_needs[1].shape == (6 * 10 * 7 + 2 * (60 + 2 * 3 * 7),)
    assert plan.state_needs[2].shape == (4 * 16 * 20 + 4 * (64 + 40),)
    only_states = plan_cache(resolve(gh.config(50, 16, [gh.mamba(1, 5, 3, 1, 1, 1)]))[1])
    assert not only_states.groups and only_states.state_needs[0].shape == (16,)


def test_tensor_names_and_shapes():
    names = collect_tensor_specs(resolve(gh.SMALL_A)[1])
    assert names["l0.mix.left.q"].shape == (48, 64) and names["l0.mix.left.k.b"].shape == (24,) and names["l0.mix.left.v.b"].shape == (40,)
    assert names["l0.mix.left.g"].shape == (80, 64) and names["l0.mix.left.o"].shape == (64, 80) and "l0.mix.left.g.b" not in names
    assert names["l0.mix.right.k"].shape == (30, 64) and names["l0.mix.right.g"].shape == (18, 64) and names["l0.mix.right.o"].shape == (64, 18)
    assert names["l1.mix.in"].shape == (60 + 60 + 42 + 6, 64) and names["l1.mix.conv"].shape == (102, 3) and names["l1.mix.conv.b"].shape == (102,)
    assert names["l1.mix.dt_bias"].shape == names["l1.mix.A_log"].shape == names["l1.mix.D"].shape == (6,)
    assert names["l1.mix.norm"].shape == (60,) and names["l1.mix.o"].shape == (64, 60)
    assert names["l1.mlp.gate"].shape == (24, 64) and names["l1.mlp.down"].shape == (64, 24)
    assert names["l1.norm2.alpha"].shape == () and "l2.norm2" not in names and "l2.mlp.up" not in names


def test_an_absent_branch_may_still_have_its_norm_in_the_checkpoint(tmp_path):
    from safetensors.torch import load_file, save_file

    from paged_attention_engine_b200.weights import load_tensors, write_random_model

    folder = write_random_model(tmp_path / "m", gh.SMALL_A, 3)
    spec = resolve(gh.SMALL_A)[1]
    path = str(folder / "model.safetensors")
    tensors = load_file(path)
    plain_set = set(load_tensors(folder, spec, torch.float32, "cpu"))
    tensors.update({"l2.norm2": torch.ones(64), "l2.norm2.b": torch.zeros(64), "l2.norm2.alpha": torch.ones(())})
    save_file(tensors, path)
    assert set(load_tensors(folder, spec, torch.float32, "cpu")) == plain_set
    tensors["l2.norm3"] = torch.ones(64)
    save_file(tensors, path)
    with pytest.raises(WeightsError, match="l2.norm3"):
        load_tensors(folder, spec, torch.float32, "cpu")


@pytest.mark.parametrize("damage, text", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["layers"][0].update(type="mlstm"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "layers[0].mixer.right"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "layers[0].mixer.left_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "layers[0].mixer.left.heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14), "layers[0].mixer.left.rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("factor"), "left.rot.scaling.factor"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5]), "layers[0].mixer.right.decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, -0.5, 0.1]), "layers[0].mixer.right.decay"),
    (lambda c: c["layers"][0]["mixer"]["right"]["rot"].update(dims=5), "layers[0].mixer.right.rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "layers[1].mixer.state"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "layers[1].mixer.heads"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "layers[1].mixer.norm_groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "layers[0].mlp.kind"),
    (lambda c: c["layers"][3].update(weights_of=4), "layers[3].weights_of"),
    (lambda c: c["layers"][3].update(weights_of=9), "layers[3].weights_of"),
    (lambda c: c["layers"][3].update(weights_of=2), "layers[3] differs"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
])
def test_configuration_errors_name_the_key(damage, text):
    raw = json.loads(json.dumps(gh.SMALL_A))
    damage(raw)
    with pytest.raises(ConfigError, match=text.replace("[", r"\[").replace("]", r"\]").replace(".", r"\.")):
        GetozenConfig.from_dict(raw)


def test_mixers_side_by_side_share_one_cache_and_one_state():
    spec = resolve(gh.SMALL_A)[1].layers[0].mixer
    assert MIXERS.get("side_by_side").cache_need(spec).head_dim == 12
    double = type(spec)(spec.kind, {"mixers": list(spec.params["mixers"]) + [dict(spec.params["mixers"][1], name="third")]}, spec.prefix)
    with pytest.raises(ValueError, match="state_need"):
        MIXERS.get("side_by_side").state_need(double)


def test_plain_mechanisms_on_cases_worked_by_hand():
    f64 = torch.float64
    # neighbours turn together, or channels half a span apart; the factor slows every pair; position 2
    x = torch.tensor([[[1.0, 0.0, 1.0, 0.0, 9.0]]], dtype=f64)
    turned = plain.rotate(x, {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}}, True, first=2)
    assert turned.flatten().tolist() == pytest.approx([math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1), 9.0])
    turned = plain.rotate(torch.tensor([[[1.0, 1.0, 0.0, 0.0, 9.0]]], dtype=f64), {"dims": 4, "base": 100.0}, False, first=2)
    assert turned.flatten().tolist() == pytest.approx([math.cos(2.0), math.cos(0.2), math.sin(2.0), math.sin(0.2), 9.0])
    # softmax over the keys up to the query's own
    ones = torch.ones(2, 1, 1, dtype=f64)
    out = plain.causal_attention(ones, torch.tensor([[[0.0]], [[math.log(3.0)]]], dtype=f64), torch.tensor([[[4.0]], [[8.0]]], dtype=f64), 1.0)
    assert out.flatten().tolist() == pytest.approx([4.0, 7.0])
    # a memory that halves, read after the write
    out, state = plain.decayed_memory(ones, ones, torch.tensor([[[4.0]], [[8.0]]], dtype=f64), torch.full((2, 1), 0.5, dtype=f64))
    assert out.flatten().tolist() == [4.0, 10.0] and state.flatten().tolist() == [10.0]
    # the step multiplies what is written and the rate in the exponent; the skip is added
    y = plain.selective_memory(torch.tensor([[[1.0]], [[2.0]]], dtype=f64), ones, ones, torch.full((2, 1), 3.0, dtype=f64),
                               torch.tensor([math.log(2.0) / 3.0], dtype=f64), torch.tensor([10.0], dtype=f64))
    assert y.flatten().tolist() == pytest.approx([13.0, 27.5])
    # the last tap is the current token's
    taps, bias = torch.tensor([[0.5, 2.0]]), torch.tensor([1.0])
    assert plain.short_convolution(torch.tensor([[3.0], [5.0]], dtype=f64), taps, bias).flatten().tolist() == [7.0, 12.5]
    # both sublayers read the same stream, each through its own norm
    tensors = {"l.norm1": torch.ones(1), "l.norm1.b": torch.zeros(1), "l.norm1.alpha": torch.tensor(1.0), "l.norm2": torch.full((1,), 2.0),
               "l.norm2.b": torch.zeros(1), "l.norm2.alpha": torch.tensor(1.0), "l.mlp.gate": torch.ones(1, 1), "l.mlp.up": torch.ones(1, 1),
               "l.mlp.down": torch.ones(1, 1)}
    saved = plain.mixer
    plain.mixer = lambda h, *rest: 5.0 * h
    try:
        out = plain.layer(torch.tensor([[0.5]], dtype=f64), tensors, "l", {"type": "", "mixer": None, "mlp": {"kind": "dense", "ff": 1}}, 1e-5)
    finally:
        plain.mixer = saved
    t = math.tanh(0.5)
    assert float(out) == pytest.approx(0.5 + 5.0 * t + (2.0 * t) ** 2)


def test_random_models_are_written_and_read_back(tmp_path):
    from paged_attention_engine_b200.weights import write_random_model

    folder = write_random_model(tmp_path / "m", gh.SMALL_A, 3)
    raw, tensors = gh.read_model(folder)
    assert raw["architecture"] == "Getozen" and raw["layers"][3]["weights_of"] == 1
    assert tensors["l0.norm1.alpha"].shape == () and float(tensors["l1.mix.A_log"].float().min()) >= -2.0
    logits = plain.forward(raw, tensors, [1, 2, 3])
    assert logits.shape == (3, 211) and bool(torch.isfinite(logits).all())
