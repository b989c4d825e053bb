"""Host-side parts of the Mozetar design: its configuration class, the names and shapes of its tensors, the caches and states its
layers ask for, and the plain implementation's own mechanisms on hand-made cases."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_mozetar as plain
from lalamo_b200.config import (
    AttentionSpec, ConfigError, DenseMLPSpec, DifferentialSpec, HyperBlockSpec, InputConvSpec, LinearAttentionSpec, LlamaScaling, MozetarConfig, QueryTemperature,
    RoutedMLPSpec, StreamConnectionSpec, config_from_dict, load_config,
)
from lalamo_b200.parts.model import plan_tensor_decls
from lalamo_b200.weights.loader import WeightsError, load_weights
from tiny_mozetar import CONFIG_A, CONFIG_B, CONFIG_D, CONFIGS, tensor_shapes, write_model


def test_every_size_and_constant_comes_from_the_configuration():
    config = config_from_dict(CONFIG_A)
    assert isinstance(config, MozetarConfig)
    plan = config.to_plan()
    assert (plan.vocab_size, plan.model_dim, plan.streams) == (150, 64, 3) and not plan.head.tied and plan.head.scale == 1.0 and plan.embedding.scale == 1.0
    assert plan.final_norm.exact and plan.final_norm.eps == 1e-5
    assert [entry.cache_from for entry in plan.schedule] == [None, None, None, 0, None]
    for layer in plan.layers:
        assert isinstance(layer, HyperBlockSpec) and layer.pre_mixer_norm.exact and layer.input_conv == InputConvSpec(64, 3)
        assert layer.mixer_connection == StreamConnectionSpec(3) and (layer.ffn is None) == (layer.ffn_connection is None) == (layer.pre_ffn_norm is None)
    windowed, differential, linear, borrower, last = (layer.mixer for layer in plan.layers)
    assert isinstance(windowed, AttentionSpec) and not windowed.borrows_kv
    assert (windowed.num_heads, windowed.num_groups, windowed.head_dim, windowed.value_dim, windowed.window, windowed.scale, windowed.conv_taps) == (6, 2, 16, 24, 19, 0.35, 4)
    assert (windowed.position.rotary_dim, windowed.position.theta, windowed.position.pairing) == (12, 300.0, "interleaved")
    assert windowed.position.scaling == LlamaScaling(factor=5.0, low=1.0, high=3.0, original=48.0)
    assert (differential.num_heads, differential.num_groups, differential.head_dim, differential.value_dim, differential.scale, differential.window) == (4, 2, 16, 40, 0.4, None)
    assert differential.differential == DifferentialSpec(offset=0.3, norm_eps=1e-5, head_gate=True) and differential.position is None
    assert differential.query_temperature == QueryTemperature(0.7, 10)
    assert isinstance(linear, LinearAttentionSpec) and (linear.num_heads, linear.key_dim, linear.value_dim, linear.decay, linear.norm_weight) == (3, 8, 24, "forget", True)
    assert (linear.gate_activation, linear.query_activation, linear.scaled, linear.norm_eps) == ("none", "silu", "none", 1e-5)
    assert borrower.borrows_kv and (borrower.window, borrower.conv_taps, borrower.scale) == (45, 2, 0.25)
    assert last.differential.offset == 0.7 and plan.layers[4].ffn is None
    routed, dense = plan.layers[2].ffn, plan.layers[1].ffn
    assert isinstance(routed, RoutedMLPSpec) and (routed.num_experts, routed.top, routed.hidden_dim, routed.group_count, routed.group_keep) == (8, 3, 16, 4, 3)
    assert (routed.score, routed.renormalize, routed.group_score, routed.gated, routed.activation, routed.shared) == ("softmax", True, "largest", True, "silu", None)
    assert isinstance(dense, DenseMLPSpec) and (dense.hidden_dim, dense.activation, dense.has_bias, dense.norm_eps) == (56, "poly_norm", True, 1e-5)
    other = config_from_dict(CONFIG_B).to_plan()
    assert other.streams == 1 and other.layers[2].mixer.position.scaling is None and other.layers[3].ffn.group_count == 1 and other.final_norm.eps == 1e-6
    assert config.to_json_dict()["architecture"] == "Mozetar"


@pytest.mark.parametrize("path,value,key", [
    (("layers", 0, "type"), "attention_3", "layers[0].type"),
    (("streams",), 0, "config.streams"),
    (("canon", "taps"), None, "config.canon.taps"),
    (("norm", "eps"), None, "config.norm.eps"),
    (("layers", 0, "mixer", "kv_heads"), 4, "layers[0].mixer.kv_heads"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "layers[0].mixer.rot.dims"),
    (("layers", 0, "mixer", "rot", "scaling", "high"), None, "layers[0].mixer.rot.scaling.high"),
    (("layers", 0, "mixer", "mask", "size"), 0, "layers[0].mixer.mask.size"),
    (("layers", 1, "mixer", "diff"), None, "layers[1].mixer.diff"),
    (("layers", 1, "mixer", "q_temp", "every"), 0, "layers[1].mixer.q_temp.every"),
    (("layers", 1, "mixer", "scale"), None, "layers[1].mixer.scale"),
    (("layers", 2, "mixer", "vdim"), None, "layers[2].mixer.vdim"),
    (("layers", 3, "mixer", "kv_from"), 1, "layers[3].mixer.kv_from"),
    (("layers", 3, "mixer", "kv_from"), 3, "layers[3].mixer.kv_from"),
    (("layers", 3, "mixer", "dim"), 24, "layers[3].mixer.kv_from"),
    (("layers", 1, "mlp", "kind"), "sparse", "layers[1].mlp.kind"),
    (("layers", 1, "mlp", "ff"), None, "layers[1].mlp.ff"),
    (("layers", 2, "mlp", "router", "top"), 7, "layers[2].mlp.router.top"),
    (("layers", 2, "mlp", "router", "groups", "count"), 3, "layers[2].mlp.router.groups"),
])
def test_a_bad_configuration_names_its_key(path, value, key):
    raw = copy.deepcopy(CONFIG_A)
    at = raw
    for step in path[:-1]:
        at = at[step]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as caught:
        config_from_dict(raw)
    assert key in str(caught.value)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_tensor_names_and_shapes(tmp_path, name):
    """Every tensor of a model folder written from the design's own names is asked for under that name with that shape, and nothing else is."""
    config = CONFIGS[name]
    folder, _ = write_model(tmp_path / name, config, 3)
    typed = load_config(folder)
    plan = typed.to_plan()
    asked = {typed.checkpoint_names(path, local)[0]: tuple(decl.shape) for (path, local), decl in plan_tensor_decls(plan).items()}
    assert asked == tensor_shapes(config)
    assert len(load_weights(folder, typed, plan)) == len(asked)


def test_a_checkpoint_that_does_not_fit_is_reported_whole(tmp_path):
    from lalamo_b200.weights.safetensors_io import write_safetensors

    folder, weights = write_model(tmp_path / "a", CONFIG_A, 3)
    broken = {name: tensor.to(torch.bfloat16) for name, tensor in weights.items() if name != "l1.mix.lq2"}
    broken["l0.hc1.in"] = torch.zeros(5, dtype=torch.bfloat16)
    broken["l3.mix.k"] = torch.zeros(32, 64, dtype=torch.bfloat16)   # a layer that borrows keys has no projection of its own
    write_safetensors(folder / "model.safetensors", broken)
    with pytest.raises(WeightsError) as caught:
        load_weights(folder, load_config(folder))
    assert caught.value.missing == ["l1.mix.lq2"] and caught.value.unexpected == ["l3.mix.k"] and caught.value.wrong_shape[0][0] == "l0.hc1.in"


def needs_of(config: dict):
    """The cache needs of a configuration's layers as its model would state them, from parts built on the CPU."""
    from lalamo_b200.parts.base import Runtime
    from lalamo_b200.parts.model import DecoderModel
    from tiny_mozetar import random_weights

    typed = config_from_dict(config)
    plan = typed.to_plan()
    tensors = random_weights(config, 5)
    given = {(path, local): tensors[typed.checkpoint_names(path, local)[0]] for path, local in plan_tensor_decls(plan)}
    model = DecoderModel(plan, given, Runtime(torch.device("cpu"), torch.float32))
    return model.cache_needs(), [entry.cache_from for entry in plan.schedule]


def test_caches_and_states_the_layers_ask_for():
    """Pages of keys (both maps' side by side) and values, the convolutions' last inputs, the matrix state; a borrower has states of
    its own but no pages, and the pages it reads stay for as long as its longer window looks back."""
    from lalamo_b200.cache.manager import CacheManager
    from lalamo_b200.parts.base import BorrowedKVNeed, CompositeNeed, PagedKVNeed, SlotStateNeed

    needs, cache_from = needs_of(CONFIG_A)
    canon = SlotStateNeed((2, 64))
    assert needs[0] == CompositeNeed((CompositeNeed((PagedKVNeed(2, 16, window=19, value_dim=24), SlotStateNeed((3, 6 * 16 + 2 * 16 + 2 * 24)))), canon))
    assert needs[1] == CompositeNeed((PagedKVNeed(2, 32, window=None, value_dim=40), canon))
    assert needs[2] == CompositeNeed((SlotStateNeed((3, 8, 24), torch.float32), canon))
    assert needs[3] == CompositeNeed((CompositeNeed((BorrowedKVNeed(window=45), SlotStateNeed((1, 96)))), canon))
    manager = CacheManager(needs, cache_from, None, page_size=16, num_pages=12, num_slots=2)
    assert {group.window: len(group.entries) for group in manager.groups} == {45: 1, None: 2}
    manager.admit("a")
    manager.reserve("a", 100)
    manager.commit("a", 100)
    held = {group.window: sum(page >= 0 for page in manager.requests["a"].blocks[index]) for index, group in enumerate(manager.groups)}
    assert held == {None: 7, 45: 7 - (100 - 45 + 1) // 16}
    manager.release("a")
    manager.check()
    # one tap: no state; an unbounded borrower keeps every page
    needs_b, _ = needs_of(CONFIG_B)
    assert needs_b[2] == CompositeNeed((PagedKVNeed(3, 20, window=1, value_dim=6), None))
    endless = [CompositeNeed((PagedKVNeed(1, 8, window=5), None)), CompositeNeed((BorrowedKVNeed(window=None), SlotStateNeed((1, 8))))]
    assert [group.window for group in CacheManager(endless, [None, 0], None, page_size=16, num_pages=2, num_slots=1).groups] == [None]
    with pytest.raises(ValueError, match="no entry is named"):
        CacheManager(endless, [None, None], None, page_size=16, num_pages=2, num_slots=1)
    with pytest.raises(ValueError, match="exactly one set"):
        CacheManager([SlotStateNeed((1,)), BorrowedKVNeed()], [None, 0], None, page_size=16, num_pages=2, num_slots=1)
    with pytest.raises(ValueError, match="exactly one set"):
        CacheManager([PagedKVNeed(1, 8), BorrowedKVNeed(), BorrowedKVNeed()], [None, 0, 1], None, page_size=16, num_pages=2, num_slots=1)


def test_frequencies_slowed_down_by_wavelength():
    from lalamo_b200.parts.rope import slowed_frequencies

    for scaling in ((8.0, 1.0, 4.0, 512), (3.0, 0.5, 5.0, 100), (5.0, 1.0, 3.0, 48)):
        rot = {"dims": 32, "base": 1e4, "scaling": dict(zip(("factor", "low", "high", "original"), scaling))}
        want = plain.frequencies(rot)
        got = slowed_frequencies(32, 1e4, LlamaScaling(*scaling))
        assert torch.allclose(got.double(), want, rtol=1e-6)
        bare = plain.frequencies({"dims": 32, "base": 1e4})
        assert float(got[0]) == float(bare[0]) and abs(float(got[-1]) * scaling[0] / float(bare[-1]) - 1.0) < 1e-6   # the fastest as it is, the slowest divided
        assert ((want < bare * (1 - 1e-9)) & (want > bare / scaling[0] * (1 + 1e-9))).any()   # and some in between


def test_blocks_and_streams_go_together():
    from dataclasses import replace

    plan = config_from_dict(CONFIG_A).to_plan()
    with pytest.raises(ValueError, match="go together"):
        replace(plan, streams=0)
    from lalamo_b200.parts.base import Runtime
    from lalamo_b200.parts.streams import InputConv, StreamConnection
    runtime = Runtime(torch.device("cpu"), torch.float32)
    with pytest.raises(ValueError, match="1 to 8 residual streams"):
        StreamConnection(StreamConnectionSpec(9), {"read": torch.ones(9), "mix": torch.eye(9), "write": torch.ones(9)}, runtime)
    with pytest.raises(ValueError, match="1 to 17 taps"):
        InputConv(InputConvSpec(4, 18), {"weight": torch.ones(4, 18)}, runtime)


def test_the_plain_mechanisms_on_hand_made_cases():
    # a convolution of three taps: the last column is the token's own
    u = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=torch.float64)
    assert plain.causal_conv(u, torch.tensor([[3.0, 2.0, 1.0]], dtype=torch.float64)).flatten().tolist() == [1.0, 12.0, 123.0, 1230.0]
    # streams: `mix` is indexed from, to
    X = torch.tensor([[[1.0], [10.0]]], dtype=torch.float64)
    fresh = plain.write_streams(X, torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=torch.float64), torch.tensor([100.0, 200.0], dtype=torch.float64), torch.ones(1, 1, dtype=torch.float64))
    assert fresh.flatten().tolist() == [1.0 + 30.0 + 100.0, 2.0 + 40.0 + 200.0]
    assert plain.read_streams(X, torch.tensor([2.0, 0.5], dtype=torch.float64)).item() == 7.0
    # the temperature steps where position + 1 reaches a multiple of `every`
    t = plain.query_temperature(torch.tensor([0, 2, 3, 6, 7]), {"coef": 0.5, "every": 4})
    assert torch.allclose(t, 1.0 + 0.5 * torch.log(torch.tensor([1.0, 1.0, 2.0, 2.0, 3.0], dtype=torch.float64)))
    # two maps combined
    w = {name: torch.tensor(value, dtype=torch.float64) for name, value in (("lq1", [0.5, 1.0]), ("lk1", [1.0, 0.5]), ("lq2", [0.2, 0.0]), ("lk2", [1.0, 9.0]))}
    assert abs(plain.differential_lambda(w, 0.3) - (math.exp(1.0) - math.exp(0.2) + 0.3)) < 1e-12
    a1, a2 = torch.tensor([[[3.0, 1.0]]], dtype=torch.float64), torch.tensor([[[1.0, 1.0]]], dtype=torch.float64)
    out = plain.combine_maps(a1, a2, 2.0, 0.25, torch.zeros(1, 1, dtype=torch.float64), 0.0)
    assert torch.allclose(out, torch.tensor([[[1.0, -1.0]]], dtype=torch.float64) * 0.75 * 0.5)
    # the forget gate says what is written: with f = 1/2 throughout, S_t = v_t / 2 + v_(t-1) / 4 + ...
    q, f = torch.ones(3, 1, 1, dtype=torch.float64), torch.full((3, 1, 1), 0.5, dtype=torch.float64)
    out, state = plain.forget_recurrence(q, f, torch.tensor([8.0, 0.0, 4.0], dtype=torch.float64).reshape(3, 1, 1))
    assert out.flatten().tolist() == [4.0, 2.0, 3.0] and state.item() == 3.0
    assert plain.forget_gate(torch.zeros(1, dtype=torch.float64), torch.tensor([0.2], dtype=torch.float64)).item() == pytest.approx(0.6)
    # a polynomial of normed powers
    z = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    parts = [z / math.sqrt(2.5), z**2 / math.sqrt(8.5), z**3 / math.sqrt(32.5)]
    assert torch.allclose(plain.poly_norm(z, torch.tensor([1.0, 2.0, 3.0, 4.0], dtype=torch.float64), 0.0), parts[0] + 2 * parts[1] + 3 * parts[2] + 4.0)
    # groups by their largest expert: {0.3, 0.3} loses against {0.4, 0.0}, though its sum is larger
    scores = torch.tensor([0.3, 0.29, 0.4, 0.01], dtype=torch.float64)
    assert plain.choose_experts(scores, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}}) == [2, 3]
    assert plain.choose_experts(scores, {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 2}}) == [2, 0]
    # neighbours turn as pairs
    x = torch.tensor([[[1.0, 0.0, 5.0]]], dtype=torch.float64)
    turned = plain.rotate_neighbours(x, torch.tensor([2]), {"dims": 2, "base": 10.0})
    assert torch.allclose(turned, torch.tensor([[[math.cos(2.0), math.sin(2.0), 5.0]]], dtype=torch.float64))
