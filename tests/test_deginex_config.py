"""The Deginex configuration: what it reads, what it refuses, how it is laid out as parts; the plain
implementation's own mechanisms (no GPU)."""

import copy

import pytest
import torch

import deginex_models as dm
import plain_deginex as plain
from from_scratch_inference_engine_b200.config import ConfigError, config_from_dict
from from_scratch_inference_engine_b200.parts.model import DecoderModel, tensor_specs

F64 = torch.float64


def test_every_test_configuration_reads_and_round_trips():
    for name, data in dm.CONFIGS.items():
        config = config_from_dict(data)
        assert type(config).__name__ == "DeginexConfig"
        assert config_from_dict(config.to_dict()) == config, name


def test_run_order_streams_and_cache_needs():
    spec = config_from_dict(dm.CONFIGS["loop"]).build_spec()
    assert [c.layer for c in spec.schedule] == [0, 1, 2, 1, 2, 3]
    assert [entry for _, entry, _ in spec.resolved_schedule()] == list(range(6))    # a cache entry per call
    assert spec.streams == 4 and not spec.inlets and spec.head_name is None
    model = DecoderModel(spec)
    assert model.capturable
    needs = model.cache_needs()
    assert needs[1] == needs[3] and needs[2] == needs[4] and needs[0] == needs[5] and needs[0] != needs[1]
    # pages behind a chunk are given back like pages behind a window of its length
    assert (needs[1].kv_heads, needs[1].head_dim, needs[1].v_dim, needs[1].window) == (2, 12, 20, 40)
    assert model.state_needs() == [None] * 6
    for name, order in (("loop_first", [0, 1]), ("loop_last", [0, 1, 1, 1]), ("chunk", [0])):
        assert [c.layer for c in config_from_dict(dm.CONFIGS[name]).build_spec().schedule] == order
        assert plain.run_order(dm.CONFIGS[name]) == order


def test_tensor_names_and_shapes():
    every = tensor_specs(config_from_dict(dm.CONFIGS["loop"]).build_spec())
    specs = {s.name: tuple(s.shape) for s in every if not s.optional}
    assert specs["embed"] == (131, 64) and "head" not in specs
    assert specs["final.norm"] == (64,) and specs["final.norm.b"] == (64,)
    assert specs["l0.norm1"] == specs["l0.norm1.b"] == specs["l0.norm2"] == specs["l0.norm2.b"] == (64,)
    assert specs["l0.hc1.in"] == specs["l0.hc2.out"] == (4,) and specs["l0.hc2.mix"] == (4, 4)
    assert specs["l1.mix.q"] == (24, 64) and specs["l1.mix.k"] == (24, 64) and specs["l1.mix.v"] == (40, 64)
    assert specs["l1.mix.g"] == (40, 64) and specs["l1.mix.o"] == (64, 40)
    assert not any(name.startswith("l") and name.endswith((".q.b", ".k.b", ".v.b", ".q.norm")) for name in specs)
    assert specs["l0.mlp.gate"] == specs["l0.mlp.up"] == (72, 64) and specs["l0.mlp.down"] == (64, 72)
    assert specs["l1.mlp.router"] == (6, 64) and specs["l1.mlp.router.b"] == (6,)
    assert specs["l1.mlp.e5.gate"] == (24, 64) and specs["l1.mlp.e5.down"] == (64, 24)
    # a layer without feed-forward needs no second norm and no second set of coefficients, and
    # tolerates stored ones
    assert not any(name.startswith(("l2.norm2", "l2.hc2", "l2.mlp")) for name in specs)
    assert {"l2.norm2", "l2.norm2.b", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"} <= {s.name for s in every if s.optional}


def test_refusals_name_the_place():
    def refused(change, name="loop"):
        data = copy.deepcopy(dm.CONFIGS[name])
        change(data)
        with pytest.raises(ConfigError) as info:
            config_from_dict(data)
        return str(info.value)

    assert "type" in refused(lambda d: d["layers"][1].update(type="mamba"))
    assert "kv_heads" in refused(lambda d: d["layers"][0]["mixer"].update(heads=3))
    assert "scale" in refused(lambda d: d["layers"][0]["mixer"].pop("scale"))
    assert "softcap" in refused(lambda d: d["layers"][0]["mixer"].update(softcap=-1.0))
    assert "mask" in refused(lambda d: d["layers"][0]["mixer"].update(mask=7))
    assert "mask.size" in refused(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    assert "streams" in refused(lambda d: d.update(streams=0))
    assert "streams" in refused(lambda d: d.pop("streams"))
    assert "kind" in refused(lambda d: d["layers"][0]["mlp"].update(kind="sparse"))
    assert "ff" in refused(lambda d: d["layers"][0]["mlp"].pop("ff"))
    assert "top" in refused(lambda d: d["layers"][1]["mlp"]["router"].update(top=7))
    assert "loop" in refused(lambda d: d["loop"].update(stop=5))
    assert "loop" in refused(lambda d: d["loop"].update(start=3))
    assert "times" in refused(lambda d: d["loop"].update(times=0))
    assert "eps" in refused(lambda d: d.update(norm={}))


def test_what_may_be_absent():
    data = copy.deepcopy(dm.CONFIGS["loop"])
    data.pop("loop")
    mixer = data["layers"][1]["mixer"]
    for key in ("mask", "softcap", "vdim", "kv_heads"):
        mixer.pop(key)
    spec = config_from_dict(data).build_spec()
    assert [c.layer for c in spec.schedule] == [0, 1, 2, 3]
    params = spec.layers[1].mixer.params
    assert params["chunk"] == 0 and params["softcap"] == 0.0 and params["vdim"] == 12 and params["kv_heads"] == 2


def test_parts_that_do_not_go_together_are_refused():
    from dataclasses import replace
    spec = config_from_dict(dm.CONFIGS["loop"]).build_spec()
    with pytest.raises(ValueError):         # several streams have no place where an inlet could meet them
        from from_scratch_inference_engine_b200.config import PartSpec
        DecoderModel(replace(spec, inlets=((PartSpec("concat_embedding", {"hidden_size": 64}), "x."),)))
    with pytest.raises(TypeError):          # a streams layer in a model with one residual
        DecoderModel(replace(spec, streams=0))


def test_plain_streams_chunks_caps_and_choice():
    streams = [torch.tensor([[1.0, 2.0]], dtype=F64), torch.tensor([[10.0, 20.0]], dtype=F64)]
    assert plain.gather_streams(streams, torch.tensor([2.0, -1.0], dtype=F64)).tolist() == [[-8.0, -16.0]]
    mix = torch.tensor([[1.0, 3.0], [0.0, 2.0]], dtype=F64)          # [from, to]
    new = plain.spread_streams(streams, mix, torch.tensor([1.0, 0.0], dtype=F64), torch.tensor([[100.0, 0.0]], dtype=F64))
    assert new[0].tolist() == [[101.0, 2.0]]                         # stream 1 hands nothing to stream 0
    assert new[1].tolist() == [[23.0, 46.0]]                         # and the old stream 0 is what stream 1 gets
    mask = plain.chunk_mask(7, 3)
    assert mask[5].tolist() == [False, False, False, True, True, True, False]
    assert mask[3].tolist() == [False, False, False, True, False, False, False]
    q, k = torch.full((1, 4), 10.0, dtype=F64), torch.tensor([[1.0] * 4, [1e-4] * 4], dtype=F64)
    s = plain.capped_scores(q, k, 0.5, 2.0)[0].tolist()
    assert abs(s[0] - 2.0) < 1e-6 and abs(s[1] - 0.002) < 1e-8       # flat far out, the identity near zero
    w = {"r.router": torch.zeros(4, 2, dtype=F64), "r.router.b": torch.tensor([0.0, 3.0, 1.0, 2.0], dtype=F64)}
    ids, weights = plain.route(torch.ones(1, 2, dtype=F64), w, "r.", 2)
    assert ids[0].tolist() == [1, 3] and abs(float(weights.sum()) - 1.0) < 1e-12
    assert abs(float(weights[0, 0] / weights[0, 1]) - 2.718281828459045) < 1e-9      # over the chosen alone
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F64)
    y = plain.layer_norm(x, torch.ones(4, dtype=F64), torch.tensor([0.0, 0.0, 0.0, 9.0], dtype=F64), 0.0)
    assert abs(float(y[0, 0]) + 3.0 / 5.0 ** 0.5) < 1e-12 and abs(float(y[0, 3]) - 9.0 - 3.0 / 5.0 ** 0.5) < 1e-12
