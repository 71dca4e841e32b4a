"""The Noganex configuration without a GPU: reading and writing back, declared tensors, the plan, layers that run the
tensors of others on a cache of their own, what the cache keeps for a chunk, refused configurations."""

import copy

import pytest
import torch

import plain_noganex as plain
from ondeviceinfer_b200.cache import KVNeed, SequenceCache, StateNeed, pages_for
from ondeviceinfer_b200.config.noganex import NoganexConfig
from ondeviceinfer_b200.config.specs import (GatedMLPSpec, GatedPostNormBlockSpec, HeadDeltaSpec, MixedAttentionSpec,
                                             NoPositionSpec, RotarySpec, RoutedExpertsSpec)
from ondeviceinfer_b200.engine.model import DecoderModel
from ondeviceinfer_b200.parts.position import ramped_frequencies
from ondeviceinfer_b200.registry import config_from_dict

CONFIGS = {"A": plain.TINY_A, "B": plain.TINY_B, "C": plain.TINY_C, "D": plain.TINY_D, "sharp": plain.SHARP}


@pytest.mark.parametrize("case", sorted(CONFIGS))
def test_reads_and_writes_back(case):
    cfg = CONFIGS[case]
    config = config_from_dict(cfg)
    assert isinstance(config, NoganexConfig) and config.to_dict() == cfg
    assert config_from_dict(config.to_dict()) == config


@pytest.mark.parametrize("case", sorted(CONFIGS))
def test_declares_the_designs_tensors(case):
    cfg = CONFIGS[case]
    model = DecoderModel(config_from_dict(cfg).to_plan())
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == plain.tensor_shapes(cfg)


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations_declare_their_tensors(seed):
    cfg = plain.random_config(seed)
    model = DecoderModel(config_from_dict(cfg).to_plan())
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == plain.tensor_shapes(cfg)


def test_plan_follows_the_layer_list():
    plan = config_from_dict(plain.TINY_A).to_plan()
    assert [(e.layer, e.cache_from) for e in plan.order] == [(0, None), (1, None), (0, None), (1, None), (2, None)]
    assert len(plan.layers) == 3 and all(isinstance(block, GatedPostNormBlockSpec) for block in plan.layers)
    attention, delta = plan.layers[0].mixer, plan.layers[1].mixer
    assert isinstance(attention, MixedAttentionSpec) and isinstance(delta, HeadDeltaSpec)
    assert (attention.num_heads, attention.num_kv_heads, attention.head_dim, attention.value_dim, attention.scale,
            attention.chunk, attention.row_norm_eps) == (6, 2, 32, 24, 0.21, 40, 1e-5)
    assert attention.position == RotarySpec(32, 5000.0, 20, index_ramp=(4.0, 512.0, 16.0, 2.0)) and attention.has("talk")
    assert (delta.num_heads, delta.num_kv_heads, delta.qk_dim, delta.v_dim, delta.conv_taps, delta.unit_eps) == (6, 3, 24, 40, 4, 1e-6)
    experts, dense = plan.layers[0].ffn, plan.layers[1].ffn
    assert isinstance(experts, RoutedExpertsSpec) and isinstance(dense, GatedMLPSpec)
    assert (experts.scoring, experts.expert_form, experts.renormalise, experts.weight_scale, experts.has_correction,
            experts.top_k, experts.num_experts, experts.expert_size, experts.shared_size) == \
        ("sigmoid", "gated_silu", True, 1.7, True, 2, 6, 40, 24)
    assert (dense.activation, dense.intermediate_size) == ("gelu_tanh", 72) and dense.has("gate_bias") and dense.has("down_bias")
    assert plan.layers[2].ffn is None and plan.layers[2].ffn_gate_name is None
    assert set(plan.ignored_tensors) == {"l4.norm2", "l4.rg2", "l4.rg2.b"}
    assert plan.final_norm.output_scale == 0.7 and plan.final_norm.scale_in_fp32 and plan.head.weight_name == "head"
    assert plan.layers[0].mixer_norm.output_scale == 1.0
    bare = config_from_dict(plain.TINY_B).to_plan()
    assert bare.layers[1].mixer.chunk is None and bare.layers[1].mixer.position.index_ramp is None
    unrotated = copy.deepcopy(plain.TINY_B)
    unrotated["layers"][1]["mixer"].pop("rot")
    assert isinstance(config_from_dict(unrotated).to_plan().layers[1].mixer.position, NoPositionSpec)


def test_a_layer_may_borrow_from_a_later_one_and_from_layer_zero():
    plan = config_from_dict(plain.TINY_C).to_plan()
    assert [e.layer for e in plan.order] == [0, 2, 1, 2] and plan.layers[2].mixer.prefix == "l3.mix."
    cfg = copy.deepcopy(plain.TINY_A)
    cfg["layers"][4] = {**cfg["layers"][3], "weights_of": 3}       # of a layer that borrows itself
    assert [e.layer for e in config_from_dict(cfg).to_plan().order] == [0, 1, 0, 1, 1]


def test_every_execution_keeps_a_cache_of_its_own():
    model = DecoderModel(config_from_dict(plain.TINY_A).to_plan())
    assert model.layers[0].cache_needs() == (KVNeed(2, 32, 40, value_dim=32),)        # stored in steps of 16 lanes
    state, taps = model.layers[1].cache_needs()
    assert state == StateNeed((6, 24, 40), torch.float32, "delta state") and taps.shape == (3, 2 * 3 * 24 + 6 * 40)
    assert len(DecoderModel(config_from_dict(plain.TINY_B).to_plan()).layers[0].cache_needs()) == 1      # one tap: no inputs kept
    needs = [model.layers[e.layer].cache_needs() for e in model.plan.order]
    cache = SequenceCache(needs, [None] * len(needs), dtype=torch.float32, device="cpu", max_tokens=256, max_seqs=2)
    assert cache.view(0).keys.data_ptr() != cache.view(2).keys.data_ptr()
    assert cache.view(1).states[0].data_ptr() != cache.view(3).states[0].data_ptr()


def test_a_chunk_keeps_a_ring_of_pages():
    cache = SequenceCache([(KVNeed(2, 16, 130, value_dim=16),)], [None], dtype=torch.float32, device="cpu", max_tokens=4096,
                          max_seqs=1, max_step_tokens=16)
    slot, group = cache.alloc(), cache.kv_groups[0]
    for _ in range(100):
        cache.reserve([slot], [16])
        cache.advance([slot], [16])
    assert len(group.slot_pages[slot]) == group.ring_len == pages_for(130 + 16 - 1) + 1
    # the chunk of any query of a step, and the step's own later tokens, lie on pages of their own
    for p in range(0, 1500):
        pages = {q // 64 for q in range(p - p % 130, p + 16)}
        assert len({page % group.ring_len for page in pages}) == len(pages)


def test_frequencies_slowed_by_a_ramp_follow_the_plain_ones():
    for dims, base, scaling in ((20, 5000.0, (4.0, 512, 16.0, 2.0)), (48, 300.0, (8.0, 64, 3.0, 0.5)), (2, 1e4, (2.0, 256, 32.0, 1.0))):
        want, factor = plain.ramp_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), scaling)))
        exact = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        got, magnitude = ramped_frequencies(exact, base, dims, scaling)
        assert got == pytest.approx(want, rel=1e-12) and magnitude == pytest.approx(factor, rel=1e-12)
        assert want != exact or dims == 2


@pytest.mark.parametrize("change,error", [
    (lambda c: c["layers"][0].update(type="latent"), ValueError),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), ValueError),
    (lambda c: c["layers"][2].update(weights_of=9), ValueError),
    (lambda c: c["layers"][2].update(weights_of=1), ValueError),       # a layer of the other type
    (lambda c: (c["layers"][0].update(weights_of=2), c["layers"][2].update(weights_of=0)), ValueError),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), KeyError),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), KeyError),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), KeyError),
    (lambda c: c.pop("width"), KeyError),
    (lambda c: c["norm"].update(eps=0.0), ValueError),
    (lambda c: c.update(layers=[]), ValueError),
])
def test_refused_configurations(change, error):
    cfg = copy.deepcopy(plain.TINY_A)
    change(cfg)
    with pytest.raises(error):
        config_from_dict(cfg).to_plan()


@pytest.mark.parametrize("path,value", [((0, "mask", "size"), 0), ((0, "rot", "dims"), 40), ((0, "kv_heads"), 4), ((1, "dim"), 600),
                                        ((1, "conv"), 17), ((0, "dim"), 513)])
def test_sizes_that_the_kernels_do_not_take_are_refused_when_the_model_is_built(path, value):
    cfg = copy.deepcopy(plain.TINY_A)
    node = cfg["layers"][path[0]]["mixer"]
    for key in path[1:-1]:
        node = node[key]
    node[path[-1]] = value
    with pytest.raises(ValueError):
        DecoderModel(config_from_dict(cfg).to_plan())
