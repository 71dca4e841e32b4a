"""The Pukinex configuration without a GPU: reading and writing back, declared tensors, the plan, looped layers with a cache
of their own per pass, table sizes from the checkpoint, distance buckets, refused configurations."""

import copy

import pytest
import torch

import plain_pukinex as plain
from ondeviceinfer_b200.cache import KVNeed, SequenceCache, StateNeed
from ondeviceinfer_b200.config.pukinex import PukinexConfig
from ondeviceinfer_b200.config.specs import (CappedAttentionSpec, LayerNormSpec, MLPSpec, NoPositionSpec, RetentionSpec, RotarySpec,
                                             SideBySideMixersSpec, StreamMixBlockSpec)
from ondeviceinfer_b200.engine.model import DecoderModel
from ondeviceinfer_b200.parts.capped_attention import distance_bucket, distance_entries
from ondeviceinfer_b200.registry import config_from_dict
from ondeviceinfer_b200.weights.tensors import StoredTensor

CONFIGS = {"A": plain.TINY_A, "B": plain.TINY_B, "C": plain.TINY_C, "D": plain.TINY_D, "sharp": plain.SHARP}


@pytest.mark.parametrize("case", sorted(CONFIGS))
def test_reads_and_writes_back(case):
    cfg = CONFIGS[case]
    config = config_from_dict(cfg)
    assert isinstance(config, PukinexConfig) and config.to_dict() == cfg
    assert config_from_dict(config.to_dict()) == config


@pytest.mark.parametrize("case", sorted(CONFIGS))
def test_declares_the_designs_tensors(case):
    cfg = CONFIGS[case]
    model = DecoderModel(config_from_dict(cfg).to_plan())
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == plain.tensor_shapes(cfg)


@pytest.mark.parametrize("seed", range(16))
def test_random_configurations_declare_their_tensors(seed):
    cfg = plain.random_config(seed)
    model = DecoderModel(config_from_dict(cfg).to_plan())
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == plain.tensor_shapes(cfg)


def test_plan_follows_the_configuration():
    plan = config_from_dict(plain.TINY_A).to_plan()
    assert [e.layer for e in plan.order] == [0, 1, 2, 1, 2] and all(e.cache_from is None for e in plan.order)
    assert all(isinstance(b, StreamMixBlockSpec) and (b.streams, b.residual_mult) == (2, 0.6) for b in plan.layers)
    assert plan.layers[0].mixer_names == ("l0.hc1.in", "l0.hc1.out", "l0.hc1.mix") and plan.layers[2].ffn_names is None
    pair, attention = plan.layers[0].mixer, plan.layers[1].mixer
    assert isinstance(pair, SideBySideMixersSpec) and (pair.left_scale, pair.right_scale) == (1.3, 0.6)
    left, right = pair.left, pair.right
    assert isinstance(left, CappedAttentionSpec) and isinstance(right, RetentionSpec)
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.scale, left.sink, left.gate, left.q_temperature,
            left.bias_rows, left.bias_reach, left.unit_norm_eps, left.softcap, left.window) == \
        (6, 2, 32, 24, 0.21, True, "lane", (0.4, 16), 12, 40.0, 1e-5, None, None)
    assert isinstance(left.position, NoPositionSpec) and left.has("v_bias") and left.has("q_norm")
    assert (right.num_heads, right.qk_dim, right.v_dim, right.decay, right.norm_eps) == (3, 24, 40, (0.9, 0.995, 0.5), 1e-5)
    assert right.position == RotarySpec(24, 5000.0, 16, linear_factor=1.0)
    assert (attention.values_are_keys, attention.sink, attention.gate, attention.softcap) == (True, True, "head", 20.0)
    assert attention.position == RotarySpec(32, 3000.0, 20, interleaved=True, linear_factor=4.0)
    assert isinstance(plan.layers[0].ffn, MLPSpec) and plan.layers[0].ffn.activation == "relu2" and plan.layers[2].ffn is None
    assert (plan.embedding.scale, plan.embedding.streams, plan.head.softcap) == (3.0, 2, 15.0)
    assert plan.final_norm == LayerNormSpec(104, 1e-5, "final.norm", "final.norm.b", streams=2, output_scale=0.7)
    assert set(plan.ignored_tensors) == {"l2.norm2", "l2.norm2.b", "l2.hc2.in", "l2.hc2.out", "l2.hc2.mix"}
    bare = config_from_dict(plain.TINY_C).to_plan()
    assert bare.layers[0].mixer_names is None and bare.layers[0].streams == 1 and bare.head.softcap is None
    assert isinstance(bare.layers[0].mixer.position, NoPositionSpec) and bare.layers[0].mixer.softcap is None
    assert bare.layers[1].mixer.left.q_temperature is None


def test_the_checkpoint_gives_the_rows_of_a_distance_table():
    cfg = copy.deepcopy(plain.TINY_A)
    for i, rows in ((0, 12), (2, 10)):
        assert cfg["layers"][i]["mixer"]["left"].pop("bias_rows") == rows
    config = config_from_dict(cfg)
    stored = {name: StoredTensor(shape=shape, dtype=torch.bfloat16) for name, shape in plain.tensor_shapes(plain.TINY_A).items()}
    model = DecoderModel(config.plan_for(stored))
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == plain.tensor_shapes(plain.TINY_A)
    assert config.to_plan().layers[0].mixer.left.bias_rows == 32


def test_one_stream_comes_with_or_without_coefficients():
    cfg = dict(copy.deepcopy(plain.TINY_C), streams=1)
    stored_of = lambda c: {name: StoredTensor(shape=shape, dtype=torch.bfloat16) for name, shape in plain.tensor_shapes(c).items()}
    with_them = config_from_dict(cfg).plan_for(stored_of(cfg))
    assert with_them.layers[0].mixer_names == ("l0.hc1.in", "l0.hc1.out", "l0.hc1.mix")
    assert config_from_dict(cfg).plan_for(stored_of(plain.TINY_C)).layers[0].mixer_names is None
    assert config_from_dict(cfg).to_plan().layers[0].mixer_names is not None


def test_every_pass_of_a_loop_keeps_a_cache_of_its_own():
    model = DecoderModel(config_from_dict(plain.TINY_A).to_plan())
    assert model.layers[0].cache_needs() == (KVNeed(2, 32, None, value_dim=24), StateNeed((3, 24, 40), torch.float32, "retention state"))
    assert model.layers[1].cache_needs() == (KVNeed(2, 32, None, value_dim=32),)
    needs = [model.layers[e.layer].cache_needs() for e in model.plan.order]
    cache = SequenceCache(needs, [None] * len(needs), dtype=torch.float32, device="cpu", max_tokens=256, max_seqs=2)
    assert cache.view(1).keys.data_ptr() != cache.view(3).keys.data_ptr()
    assert cache.view(2).states[0].data_ptr() != cache.view(4).states[0].data_ptr()
    assert cache.max_step_tokens is None


@pytest.mark.parametrize("rows,reach", [(16, 100), (2, 9), (7, 33), (32, 150), (40, 221), (12, 4096.0), (5, 3)])
def test_distance_buckets_follow_the_plain_ones(rows, reach):
    entries = distance_entries(rows, reach)
    assert entries == sorted(entries) and entries[-1] == rows - 1 and len(entries) <= reach + 1
    for n in range(int(reach) + 20):
        want = plain.bucket(n, rows, reach)
        assert distance_bucket(n, rows, reach) == want == entries[min(n, len(entries) - 1)]
    assert entries[:rows // 2] == list(range(rows // 2))


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="latent"), ValueError),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), ValueError),
    (lambda c: c["layers"][0]["mixer"].pop("right"), KeyError),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), KeyError),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("bias_max"), KeyError),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].pop("every"), KeyError),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("decay"), KeyError),
    (lambda c: c["layers"][0]["mixer"]["right"]["rot"].pop("base"), KeyError),
    (lambda c: c["loop"].update(stop=9), ValueError),
    (lambda c: c["loop"].update(times=0), ValueError),
    (lambda c: c["loop"].pop("times"), KeyError),
    (lambda c: c.update(streams=0), ValueError),
    (lambda c: c.update(logit_softcap=-1.0), ValueError),
    (lambda c: c.pop("width"), KeyError),
    (lambda c: c["norm"].update(eps=0.0), ValueError),
    (lambda c: c.update(layers=[]), ValueError),
])
def test_refused_configurations(change, error):
    cfg = copy.deepcopy(plain.TINY_A)
    change(cfg)
    with pytest.raises(error):
        config_from_dict(cfg).to_plan()


@pytest.mark.parametrize("path,value", [((0, "left", "kv_heads"), 4), ((0, "left", "bias_max"), 6), ((0, "left", "bias_rows"), 1),
                                        ((0, "left", "dim"), 513), ((0, "right", "decay"), [0.5]), ((0, "right", "dim"), 1025),
                                        ((0, "left", "q_temp", "every"), 0), ((1, "vdim"), 16), ((1, "rot", "dims"), 34),
                                        ((1, "softcap"), -1.0), ((1, "rot", "scaling", "factor"), 0.0)])
def test_sizes_that_the_kernels_do_not_take_are_refused_when_the_model_is_built(path, value):
    cfg = copy.deepcopy(plain.TINY_A)
    node = cfg["layers"][path[0]]["mixer"]
    for key in path[1:-1]:
        node = node[key]
    node[path[-1]] = value
    with pytest.raises(ValueError):
        DecoderModel(config_from_dict(cfg).to_plan())


def test_streams_need_their_coefficients_and_a_limit():
    cfg = dict(copy.deepcopy(plain.TINY_A), streams=17)
    with pytest.raises(ValueError):
        DecoderModel(config_from_dict(cfg).to_plan())
