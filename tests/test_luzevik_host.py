"""Luzevik on the host: configuration, registry, tensor list, schedule, cache plan, the plain mechanisms by hand."""

import json
import math

import pytest
import torch

import luzevik_helpers as lh
from paged_attention_engine_b200.cache import plan_cache
from paged_attention_engine_b200.config import ConfigError, LuzevikConfig, resolve
from paged_attention_engine_b200.weights import WeightsError, collect_tensor_specs
from plain import luzevik_plain as plain


def test_configuration_round_trip_and_registry():
    for raw, _page, _seed in lh.SMALL.values():
        cfg, spec = resolve(raw)
        assert isinstance(cfg, LuzevikConfig)
        assert LuzevikConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.to_dict() == raw
        assert spec.vocab_size == raw["vocab"] and spec.hidden_size == raw["width"]
        assert spec.embedding.params["scale"] == raw["embedding"]["scale"] and spec.head.params["tied_to"] == "embed"
        for layer, entry in zip(spec.layers, raw["layers"]):
            assert layer.block == ("post_norm_residual" if entry["mlp"] else "post_norm_residual_mixer")
            m, p = entry["mixer"], layer.mixer.params
            if entry["type"] == "parallel":
                assert layer.mixer.kind == "side_by_side" and p["out_norm_eps"] == raw["norm"]["eps"]
                left, right = p["mixers"]
                assert (left["kind"], left["scale"], right["kind"], right["scale"]) == ("gated_window_attention", 0.5, "gated_delta", 0.5)
                assert left["params"]["pairing"] == "half" and left["params"]["qkv_bias"] and not left["params"]["output_gate"]
                assert left["params"]["scale"] == m["left"]["scale"] and left["params"]["qk_norm_eps"] == raw["norm"]["eps"]
                scaling = m["left"]["rot"].get("scaling")
                assert left["params"]["position_encoding"]["scaling"] == (dict(scaling, kind="linear") if scaling else None)
                assert right["params"]["conv_taps"] == m["right"]["conv"] and right["params"]["num_kv_heads"] == m["right"]["kv_heads"]
            else:
                assert layer.mixer.kind == "latent_attention" and p["learned_sink"] and p["pairing"] == "half"
                assert p["q_rank"] == m["q_rank"] and p["own_latent"] == ("kv_from" not in m)
            if entry["mlp"] and entry["mlp"]["kind"] == "dense":
                assert layer.feed_forward.kind == "gated_mlp" and layer.feed_forward.params["activation"] == "gelu_tanh"
            elif entry["mlp"]:
                assert layer.feed_forward.kind == "routed_experts" and layer.feed_forward.params["score"] == "chosen_softmax"
                assert layer.feed_forward.params["top"] == entry["mlp"]["router"]["top"]
        assert spec.final_norm.kind == "rms_norm"


def test_latents_that_several_layers_read_and_states():
    _, spec = resolve(lh.SMALL_A)
    assert [e.cache_from for e in spec.schedule] == [None, None, 0, None, None, 3, 0]
    plan = plan_cache(spec)
    assert plan.entry_group[0] == plan.entry_group[2] == plan.entry_group[6] and plan.entry_group[3] == plan.entry_group[5]
    latents = plan.groups[plan.entry_group[0][0]]
    assert (latents.num_kv_heads, latents.head_dim, latents.value_dim, latents.window) == (1, 26, 20, 0)
    keys = plan.groups[plan.entry_group[1][0]]
    assert (keys.num_kv_heads, keys.head_dim, keys.value_dim) == (2, 12, 20)
    assert sorted(plan.state_needs) == [1, 4]
    # S and the convolution's rows, each from a 16-byte boundary on
    assert plan.state_needs[1].shape == (6 * 10 * 6 + 2 * (2 * 3 * 10 + 6 * 6),) and plan.state_needs[1].dtype == torch.float32
    assert plan.state_needs[4].shape == (128 + 4 * (2 * 7 + 18),)
    assert plan_cache(resolve(lh.ONES)[1]).state_needs[0].shape == (128,)          # a single tap keeps no rows


def test_tensor_names_and_shapes():
    names = collect_tensor_specs(resolve(lh.SMALL_A)[1])
    shape = lambda n: names[n].shape
    assert shape("l0.mix.dq") == (18, 60) and shape("l0.mix.uq") == (48, 18) and shape("l0.mix.dkv") == (26, 60)
    assert shape("l0.mix.uk") == (30, 20) and shape("l0.mix.uv") == (42, 20) and shape("l0.mix.sink") == (3,) and shape("l0.mix.o") == (60, 42)
    assert "l2.mix.dkv" not in names and "l2.mix.dkv.norm" not in names and shape("l2.mix.uk") == (16, 20)
    assert shape("l1.mix.left.q") == (48, 60) and shape("l1.mix.left.k.b") == (24,) and shape("l1.mix.left.v.b") == (40,)
    assert shape("l1.mix.left.q.norm") == shape("l1.mix.left.k.norm") == (12,) and shape("l1.mix.left.o") == (60, 80)
    assert shape("l1.mix.right.k") == (30, 60) and shape("l1.mix.right.v.conv") == (36, 3) and shape("l1.mix.right.b") == (6, 60)
    assert shape("l1.mix.right.A_log") == shape("l1.mix.right.dt_bias") == (6,) and shape("l1.mix.right.norm") == (6,)
    assert shape("l1.mix.left.out") == shape("l1.mix.right.out") == (60,)
    assert shape("l1.mlp.e4.gate") == (24, 60) and shape("l1.mlp.router") == (5, 60) and shape("l1.mlp.router.b") == (5,)
    assert shape("l0.mlp.down") == (60, 44) and shape("l0.norm2") == (60,) and "l2.norm2" not in names and "head" not in names
    assert "l0.norm" not in names and shape("final.norm") == (60,) and shape("embed") == (211, 60)


def test_an_absent_branch_may_still_have_its_norm_in_the_checkpoint(tmp_path):
    from safetensors.torch import load_file, save_file

    from paged_attention_engine_b200.weights import load_tensors, write_random_model

    folder = write_random_model(tmp_path / "m", lh.SMALL_A, 3)
    spec = resolve(lh.SMALL_A)[1]
    path = str(folder / "model.safetensors")
    tensors = load_file(path)
    read = set(load_tensors(folder, spec, torch.float32, "cpu"))
    tensors["l2.norm2"] = torch.ones(60)
    save_file(tensors, path)
    assert set(load_tensors(folder, spec, torch.float32, "cpu")) == read
    tensors["l2.mix.dkv"] = torch.ones(26, 60)
    save_file(tensors, path)
    with pytest.raises(WeightsError, match="l2.mix.dkv"):
        load_tensors(folder, spec, torch.float32, "cpu")


@pytest.mark.parametrize("damage, text", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("embedding"), "embedding.scale"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0].update(type="attention"), "layers[0].type"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "layers[0].mixer.q_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "layers[0].mixer.rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "layers[2].mixer.kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "layers[2].mixer.kv_from"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=2), "layers[6].mixer.kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=24), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=41.0), "kv_rank, rot_dim or rot"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "layers[1].mixer.right"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "layers[1].mixer.left.heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=4), "layers[1].mixer.right.heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "layers[1].mixer.right.conv"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=14), "layers[1].mixer.left.rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("factor"), "left.rot.scaling.factor"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "layers[1].mlp.kind"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "layers[1].mlp.expert.ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "layers[1].mlp.router.top"),
])
def test_configuration_errors_name_the_key(damage, text):
    raw = json.loads(json.dumps(lh.SMALL_A))
    damage(raw)
    with pytest.raises(ConfigError, match=text.replace("[", r"\[").replace("]", r"\]").replace(".", r"\.")):
        LuzevikConfig.from_dict(raw)


def test_plain_mechanisms_on_cases_worked_by_hand():
    f64 = torch.float64
    # channels half a span apart turn together; the factor slows every pair; the rest passes; position 2
    x = torch.tensor([[[1.0, 1.0, 0.0, 0.0, 9.0]]], dtype=f64)
    turned = plain.rotate(x, {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}}, first=2)
    assert turned.flatten().tolist() == pytest.approx([math.cos(1.0), math.cos(0.1), math.sin(1.0), math.sin(0.1), 9.0])
    # a sink is one more term of the denominator, unscaled
    ones = torch.ones(2, 1, 1, dtype=f64)
    values = torch.tensor([[[4.0]], [[8.0]]], dtype=f64)
    keys = torch.tensor([[[0.0]], [[2.0 * math.log(3.0)]]], dtype=f64)
    assert plain.causal_attention(ones, keys, values, 0.5).flatten().tolist() == pytest.approx([4.0, 7.0])
    sunk = plain.causal_attention(ones, keys, values, 0.5, torch.tensor([math.log(4.0)]))
    assert sunk.flatten().tolist() == pytest.approx([0.8, 28.0 / 8.0])
    # a key written twice: the second value takes the first one's place; the decay comes first, the read-out last
    k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]], dtype=f64)
    o, state = plain.delta_memory(k, k, values, torch.full((2, 1), 0.5, dtype=f64), torch.tensor([[1.0], [0.75]], dtype=f64))
    assert o.flatten().tolist() == [4.0, 6.5] and state.flatten().tolist() == [6.5, 0.0]
    # the last tap is the current token's
    assert plain.short_convolution(torch.tensor([[3.0], [5.0]], dtype=f64), torch.tensor([[0.5, 2.0]])).flatten().tolist() == [6.0, 11.5]
    assert plain.unit(torch.tensor([3.0, 4.0], dtype=f64)).tolist() == pytest.approx([0.6, 0.8])
    # two of three experts, the softmax over the two alone; the lower index first among equals
    order, weights = plain.choose(torch.tensor([0.0, math.log(3.0), -5.0], dtype=f64), 2)
    assert order == [1, 0] and weights.tolist() == pytest.approx([0.75, 0.25])
    assert plain.choose(torch.tensor([1.0, 1.0, 1.0], dtype=f64), 2)[0] == [0, 1]
    assert float(plain.gelu_tanh(torch.tensor(1.0, dtype=f64))) == pytest.approx(0.841192, abs=1e-6)
    assert plain.rms(torch.tensor([3.0, 4.0], dtype=f64), torch.tensor([1.0, 2.0]), 12.5).tolist() == pytest.approx([0.6, 1.6])


def test_the_feed_forward_reads_the_stream_that_the_mixer_left():
    f64 = torch.float64
    tensors = {"l0.norm1": torch.full((1,), 2.0), "l0.norm2": torch.full((1,), 3.0), "l0.mlp.gate": torch.ones(1, 1), "l0.mlp.up": torch.ones(1, 1),
               "l0.mlp.down": torch.ones(1, 1)}
    saved = plain.side_by_side
    plain.side_by_side = lambda h, *rest: -5.0 * h
    try:
        out = plain.layer(torch.tensor([[0.5]], dtype=f64), tensors, 0, {"type": "parallel", "mixer": None, "mlp": lh.dense(1)}, 1e-9, {})
    finally:
        plain.side_by_side = saved
    # 0.5 - 2 * 1, then the feed-forward of -1.5 (negative gate times negative up) over its own size, times 3
    assert float(out) == pytest.approx(0.5 - 2.0 + 3.0)


def test_random_models_are_written_and_read_back(tmp_path):
    from paged_attention_engine_b200.weights import write_random_model

    folder = write_random_model(tmp_path / "m", lh.SMALL_A, 3)
    raw, tensors = lh.read_model(folder)
    assert raw["architecture"] == "Luzevik" and float(tensors["l1.mix.right.A_log"].float().min()) >= -2.0
    logits = plain.forward(raw, tensors, [1, 2, 3])
    assert logits.shape == (3, 211) and bool(torch.isfinite(logits).all())
