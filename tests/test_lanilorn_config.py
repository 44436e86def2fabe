"""The Lanilorn configuration: what it reads, what it refuses, how it is laid out as parts; the plain
implementation's own mechanisms (no GPU)."""

import copy
import math

import numpy as np
import pytest
import torch

import lanilorn_models as lm
import plain_lanilorn as plain
from from_scratch_inference_engine_b200.config import ConfigError, config_from_dict
from from_scratch_inference_engine_b200.parts.difference_attention import query_temperature_table
from from_scratch_inference_engine_b200.parts.model import DecoderModel, tensor_specs
from from_scratch_inference_engine_b200.parts.rope import yarn_rotary_table
from from_scratch_inference_engine_b200.weights.loader import WeightError, check_tensors
from from_scratch_inference_engine_b200.weights.tensor_spec import TensorSpec

F64 = torch.float64


def test_every_test_configuration_reads_and_round_trips():
    for name, data in lm.CONFIGS.items():
        config = config_from_dict(data)
        assert type(config).__name__ == "LanilornConfig"
        assert config_from_dict(config.to_dict()) == config, name
    for seed in range(30):
        DecoderModel(config_from_dict(lm.random_config(seed)).build_spec())


def test_caches_states_and_scales():
    spec = config_from_dict(lm.CONFIGS["all"]).build_spec()
    assert spec.streams == 4 and spec.head_name is None
    assert spec.embedding_scale == 1.5 and spec.logit_scale == 2.0 and spec.logit_softcap == 0.0
    model = DecoderModel(spec)
    assert model.capturable
    needs, states = model.cache_needs(), model.state_needs()
    # a differential layer's two keys are one row of the cache
    assert (needs[0].kv_heads, needs[0].head_dim, needs[0].v_dim, needs[0].window) == (4, 32, 24, 0)
    assert (needs[1].kv_heads, needs[1].head_dim, needs[1].v_dim, needs[1].window) == (1, 16, 16, 21)
    assert (needs[5].kv_heads, needs[5].head_dim, needs[5].v_dim) == (1, 40, 40)
    assert needs[2] is None and needs[4] is None
    assert [None if s is None else s.shape for s in states] == [None, None, (2, 16, 24), None, (3, 8, 8), None]
    assert states[2].dtype is torch.float32


def test_tensor_names_and_shapes():
    every = tensor_specs(config_from_dict(lm.CONFIGS["all"]).build_spec())
    specs = {s.name: tuple(s.shape) for s in every if not s.optional}
    assert specs["embed"] == (131, 64) and specs["final.norm"] == (64,) and "head" not in specs
    assert not any(name.endswith((".norm1.b", ".norm2.b", "norm.b")) for name in specs)
    assert specs["l0.ls1"] == specs["l0.ls2"] == (64,)
    assert specs["l0.hc1.in"] == specs["l0.hc2.out"] == (4,) and specs["l0.hc2.mix"] == (4, 4)
    assert specs["l0.mix.q"] == (128, 64) and specs["l0.mix.k"] == (128, 64) and specs["l0.mix.v"] == (96, 64)
    assert specs["l0.mix.lq1"] == specs["l0.mix.lk2"] == (16,) and specs["l0.mix.g"] == (4, 64)
    assert specs["l0.mix.o"] == (64, 96)
    assert specs["l1.mix.q"] == (64, 64) and specs["l1.mix.k"] == (16, 64) and "l1.mix.v" not in specs
    assert specs["l1.mix.q.norm"] == (64,) and specs["l1.mix.k.norm"] == (16,) and specs["l1.mix.sink"] == (4,)
    assert specs["l2.mix.a1"] == (8, 64) and specs["l2.mix.a2"] == (32, 8) and specs["l2.mix.a2.b"] == (32,)
    assert specs["l2.mix.norm"] == (24,) and specs["l2.mix.g"] == (48, 64)
    assert specs["l0.mlp.up"] == (72, 64) and specs["l0.mlp.down"] == (64, 72)
    # a layer without feed-forward needs nothing of one, and tolerates what is stored all the same
    assert not any(name.startswith(("l2.norm2", "l2.hc2", "l2.ls2", "l2.mlp")) for name in specs)
    assert {"l2.norm2", "l2.ls2", "l2.hc2.in", "l2.hc2.mix"} <= {s.name for s in every if s.optional}


def test_the_checkpoint_decides_the_rank_of_the_decays():
    specs = tensor_specs(config_from_dict(lm.CONFIGS["recurrent"]).build_spec())
    tensors = {s.name: torch.zeros(s.shape) for s in specs if not s.optional}
    tensors["l0.mix.a1"], tensors["l0.mix.a2"] = torch.zeros(11, 40), torch.zeros(30, 11)
    check_tensors(specs, tensors)
    tensors["l0.mix.a1"] = torch.zeros(11, 41)
    with pytest.raises(WeightError, match="l0.mix.a1"):
        check_tensors(specs, tensors)
    assert TensorSpec("t", (4, 5), free=(0,)).fits((9, 5)) and not TensorSpec("t", (4, 5), free=(0,)).fits((9, 6))
    assert not TensorSpec("t", (4, 5), free=(0,)).fits((9,)) and not TensorSpec("t", (4, 5), free=(0,)).fits((0, 5))


def test_refusals_name_the_place():
    def refused(change):
        data = copy.deepcopy(lm.CONFIGS["all"])
        change(data)
        with pytest.raises(ConfigError) as info:
            config_from_dict(data)
        return str(info.value)

    mixer = lambda d, i: d["layers"][i]["mixer"]
    assert "type" in refused(lambda d: d["layers"][1].update(type="mamba"))
    assert "kv_heads" in refused(lambda d: mixer(d, 3).update(heads=4))
    assert "scale" in refused(lambda d: mixer(d, 0).pop("scale"))
    assert "vdim" in refused(lambda d: mixer(d, 1).update(vdim=8))
    assert "mask" in refused(lambda d: mixer(d, 1).update(mask=7))
    assert "mask.size" in refused(lambda d: mixer(d, 1)["mask"].update(size=0))
    assert "rot.dims" in refused(lambda d: mixer(d, 1)["rot"].update(dims=18))
    assert "rot.dims" in refused(lambda d: mixer(d, 1)["rot"].update(dims=3))
    assert "factor" in refused(lambda d: mixer(d, 1)["rot"]["scaling"].pop("factor"))
    assert "original" in refused(lambda d: mixer(d, 1)["rot"]["scaling"].update(original=0))
    assert "base" in refused(lambda d: mixer(d, 1)["rot"].update(base=1.0))
    assert "diff" in refused(lambda d: mixer(d, 0).pop("diff"))
    assert "every" in refused(lambda d: mixer(d, 0)["q_temp"].update(every=0))
    assert "tau" in refused(lambda d: mixer(d, 2).update(tau=0.0))
    assert "dim" in refused(lambda d: mixer(d, 2).pop("dim"))
    assert "kind" in refused(lambda d: d["layers"][0]["mlp"].update(kind="moe"))
    assert "ff" in refused(lambda d: d["layers"][0]["mlp"].pop("ff"))
    assert "streams" in refused(lambda d: d.pop("streams"))
    assert "eps" in refused(lambda d: d.update(norm={}))
    assert "embedding" in refused(lambda d: d.update(embedding=2.0))


def test_what_may_be_absent():
    data = copy.deepcopy(lm.CONFIGS["all"])
    for key in ("embedding", "logit_scale"):
        data.pop(key)
    for key in ("mask", "rot", "vdim", "kv_heads"):
        data["layers"][1]["mixer"].pop(key)
    for key in ("q_temp", "vdim", "kv_heads"):
        data["layers"][0]["mixer"].pop(key)
    for index in (2, 4):
        data["layers"][index]["mixer"].pop("rank")
    data["layers"][0].pop("mlp")
    spec = config_from_dict(data).build_spec()
    assert spec.embedding_scale == spec.logit_scale == 1.0
    params = spec.layers[1].mixer.params
    assert params["window"] == 0 and params["position"].kind == "none" and params["kv_heads"] == 4
    params = spec.layers[0].mixer.params
    assert params["temperature"] is None and params["vdim"] == 16 and params["kv_heads"] == 4
    assert spec.layers[0].feed_forward is None
    DecoderModel(spec)


def test_parts_that_do_not_go_together_are_refused():
    from from_scratch_inference_engine_b200.config import PartSpec
    from from_scratch_inference_engine_b200.parts import build_part
    base = dict(hidden_size=32, heads=4, kv_heads=2, dim=8, vdim=8, scale=1.0, position=PartSpec("none", {}),
                temperature=False, bias=False)

    def build(**change):
        return build_part("mixer", PartSpec("scaled_gqa_attention", dict(base, **change)), "p.")
    build(keys_as_values=True, qk_norm=True, norm_span="projection", sink=True, head_gate=True)
    for change in (dict(keys_as_values=True, vdim=6), dict(keys_as_values=True, bias=True),
                   dict(keys_as_values=True, value_mix="mix"), dict(norm_span="row")):
        with pytest.raises(ValueError):
            build(**change)
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("difference_attention", dict(hidden_size=8, heads=1, kv_heads=1, dim=4, vdim=600,
                                                                  scale=1.0, diff=0.5, eps=1e-5)), "p.")
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("gated_linear_attention", dict(hidden_size=8, heads=1, dim=300, vdim=8, tau=1.0,
                                                                    eps=1e-5)), "p.")
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("plain_mlp", dict(hidden_size=8, intermediate_size=8, activation="silu")), "p.")


def test_tables_of_angles_and_temperatures():
    rot = lm.yarn(5000.0, 12, 4.0, 64, 8.0, 0.5)
    table = yarn_rotary_table(5000.0, 12, 40, 4.0, 64, 8.0, 0.5)
    freq, magnitude = plain.yarn_frequencies(rot)
    for p in (0, 1, 17, 39):
        for i, f in enumerate(freq):
            assert abs(table[p, i] - magnitude * math.cos(p * f)) < 1e-6
            assert abs(table[p, 6 + i] - magnitude * math.sin(p * f)) < 1e-6
    for coef, every in ((0.25, 48), (0.5, 1), (0.2, 7)):
        want = plain.query_temperature(200, {"coef": coef, "every": every}).numpy()
        assert np.abs(query_temperature_table(coef, every, 200) - want).max() < 1e-6
    # the first step of the temperature falls on position every - 1
    assert query_temperature_table(0.25, 48, 70)[46] == 1.0 and query_temperature_table(0.25, 48, 70)[47] > 1.17


def test_plain_mechanisms():
    mask = plain.window_mask(7, 3)
    assert mask[5].tolist() == [False, False, False, True, True, True, False]
    assert mask[0].tolist() == [True] + [False] * 6
    q, k = torch.zeros(2, 1, 4, dtype=F64), torch.zeros(2, 1, 4, dtype=F64)
    v = torch.tensor([[[4.0]], [[8.0]]], dtype=F64)
    out = plain.sink_attention(q, k, v, plain.causal_mask(2), 1.0, torch.tensor([math.log(2.0)], dtype=F64))
    assert abs(float(out[0]) - 4.0 / 3.0) < 1e-12 and abs(float(out[1]) - 3.0) < 1e-12       # e^0 / (e^0 + 2), 12 / 4
    o1, o2 = torch.tensor([[[3.0, 1.0]]], dtype=F64), torch.tensor([[[1.0, 3.0]]], dtype=F64)
    o = plain.difference(o1, o2, 0.5, 0.2, 0.0)[0, 0]                                      # (2.5, -0.5) normed
    assert abs(float(o[0]) - 0.8 * 2.5 / math.sqrt(3.25)) < 1e-12 and abs(float(o[1]) + 0.8 * 0.5 / math.sqrt(3.25)) < 1e-12
    one = torch.ones(1, dtype=F64)
    assert abs(plain.difference_weight(one, one * 2, one, one * 0.5, 0.25) - (math.exp(2) - math.exp(0.5) + 0.25)) < 1e-12
    w = {"a1": torch.ones(1, 1, dtype=F64), "a2": torch.zeros(2, 1, dtype=F64), "a2.b": torch.tensor([0.0, 30.0], dtype=F64)}
    a = plain.key_decays(torch.ones(1, 1, dtype=F64), w, "", 2.0)[0]
    assert abs(float(a[0]) - 0.5 ** 0.5) < 1e-12 and abs(float(a[1]) - 1.0) < 1e-9
    # two key rows with decays of their own: the row that does not decay keeps its first value
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 10.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 1.0]], [[0.0, 0.0]]], dtype=F64)
    v = torch.tensor([[[5.0]], [[7.0]]], dtype=F64)
    decay = torch.tensor([[[0.3, 0.3]], [[0.5, 1.0]]], dtype=F64)
    assert plain.decayed_recurrence(q, k, v, decay)[:, 0, 0].tolist() == [5.0, 52.5]
    x = plain.rotate(torch.tensor([[[1.0, 9.0, 0.0, 5.0]]] * 2, dtype=F64), {"base": 10.0, "dims": 2, "scaling": None})
    assert x[0, 0].tolist() == [1.0, 9.0, 0.0, 5.0]
    assert abs(float(x[1, 0, 0]) - (math.cos(1.0) - 9 * math.sin(1.0))) < 1e-12 and float(x[1, 0, 2]) == 0.0
    streams = [torch.tensor([[1.0, 2.0]], dtype=F64), torch.tensor([[10.0, 20.0]], dtype=F64)]
    mix = torch.tensor([[1.0, 3.0], [0.0, 2.0]], dtype=F64)          # [from, to]
    new = plain.spread_streams(streams, mix, torch.tensor([1.0, 0.0], dtype=F64), torch.tensor([[100.0, 0.0]], dtype=F64))
    assert new[0].tolist() == [[101.0, 2.0]] and new[1].tolist() == [[23.0, 46.0]]
