"""Host-side parts of the Zevetar design: its configuration class, the names and shapes of its tensors, the caches and states its
layers ask for, and the plain implementation's own mechanisms on hand-made cases."""

from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_zevetar as plain
from lalamo_b200.config import (
    ConfigError, GatedMLPSpec, LatentAttentionSpec, LayerScaleSpec, LinearAttentionSpec, ParallelBlockSpec, RMSNormSpec, RoutedMLPSpec, YarnScaling, ZevetarConfig,
    config_from_dict, load_config,
)
from lalamo_b200.parts.model import plan_tensor_decls
from lalamo_b200.weights.loader import WeightsError, load_weights
from tiny_zevetar import CONFIG_A, CONFIG_B, CONFIGS, random_weights, tensor_shapes, write_model


def test_every_size_and_constant_comes_from_the_configuration():
    config = config_from_dict(CONFIG_A)
    assert isinstance(config, ZevetarConfig)
    plan = config.to_plan()
    assert (plan.vocab_size, plan.model_dim, plan.streams) == (150, 64, 0)
    assert plan.head.tied and (plan.head.scale, plan.head.softcap, plan.embedding.scale) == (1.5, 20.0, 4.0)
    assert plan.final_norm == RMSNormSpec(dim=64, eps=1e-5, exact=True)
    assert [entry.cache_from for entry in plan.schedule] == [None, None, 0, None, 0]
    for layer in plan.layers:
        assert isinstance(layer, ParallelBlockSpec) and layer.norm == RMSNormSpec(dim=64, eps=1e-5, exact=True)
        assert layer.mixer_scale == LayerScaleSpec(64) and layer.ffn_scale == (LayerScaleSpec(64) if layer.ffn is not None else None)
    owner, linear, borrower, last_linear, last = (layer.mixer for layer in plan.layers)
    assert isinstance(owner, LatentAttentionSpec) and not owner.borrows_kv and owner.gated and not owner.sink
    assert (owner.num_heads, owner.head_dim, owner.rope_dim, owner.value_dim, owner.query_rank, owner.latent_dim, owner.window, owner.scale) == (4, 16, 8, 24, 40, 32, 19, 0.35)
    assert (owner.position.rotary_dim, owner.position.theta, owner.position.pairing, owner.position.exact) == (8, 300.0, "interleaved", True)
    assert owner.position.scaling == YarnScaling(factor=5.0, original=48.0, fast=4.0, slow=0.5)
    assert owner.query_norm == RMSNormSpec(dim=40, eps=1e-5, exact=True) and owner.latent_norm == RMSNormSpec(dim=32, eps=1e-5, exact=True)
    assert borrower.borrows_kv and (borrower.num_heads, borrower.head_dim, borrower.value_dim, borrower.query_rank, borrower.window, borrower.scale) == (6, 24, 16, 24, 45, 0.25)
    assert isinstance(linear, LinearAttentionSpec) and (linear.num_heads, linear.key_dim, linear.value_dim, linear.decay, linear.scaled) == (4, 16, 24, "fixed", "key")
    assert (linear.norm_weight, linear.norm_eps, linear.gate_activation, linear.position.rotary_dim, linear.position.theta, linear.position.pairing) == (False, 1e-5, "silu", 12, 100.0, "half")
    assert last_linear.decay_values == (0.9, 0.995) and plan.layers[3].ffn is None and last.window == 7
    routed, dense = plan.layers[2].ffn, plan.layers[1].ffn
    assert isinstance(routed, RoutedMLPSpec) and (routed.num_experts, routed.top, routed.hidden_dim, routed.score, routed.renormalize) == (5, 3, 16, "sigmoid", False)
    assert routed.weigh_input and routed.gated and routed.shared_gate and routed.shared == GatedMLPSpec(64, 24)
    assert dense == GatedMLPSpec(64, 56)
    other = config_from_dict(CONFIG_B).to_plan()
    assert other.head.softcap == 0.0 and other.layers[0].ffn.shared is None and not other.layers[0].ffn.shared_gate and other.layers[1].mixer.window is None
    assert other.layers[0].mixer.position.scaling is None and other.layers[2].mixer.position is None and other.final_norm.eps == 1e-6
    assert config.to_json_dict()["architecture"] == "Zevetar" and config_from_dict(config.to_json_dict()).to_plan() == plan


@pytest.mark.parametrize("path,value,key", [
    (("layers", 0, "type"), "attention", "layers[0].type"),
    (("width",), 0, "config.width"),
    (("norm", "eps"), None, "config.norm.eps"),
    (("logit_softcap",), -1.0, "logit_softcap"),
    (("layers", 0, "mixer", "q_rank"), None, "layers[0].mixer.q_rank"),
    (("layers", 0, "mixer", "scale"), None, "layers[0].mixer.scale"),
    (("layers", 0, "mixer", "rot", "dims"), 6, "layers[0].mixer.rot.dims"),
    (("layers", 0, "mixer", "rot", "scaling", "slow"), None, "layers[0].mixer.rot.scaling.slow"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "layers[0].mixer.rot.scaling"),
    (("layers", 0, "mixer", "rot", "base"), 1.0, "layers[0].mixer.rot.base"),
    (("layers", 0, "mixer", "mask", "size"), 0, "layers[0].mixer.mask.size"),
    (("layers", 1, "mixer", "decay"), [0.5], "layers[1].mixer.decay"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "layers[1].mixer.rot.dims"),
    (("layers", 2, "mixer", "kv_from"), 1, "layers[2].mixer.kv_from"),
    (("layers", 2, "mixer", "kv_from"), 2, "layers[2].mixer.kv_from"),
    (("layers", 4, "mixer", "kv_from"), 2, "layers[4].mixer.kv_from"),
    (("layers", 2, "mixer", "kv_rank"), 48, "layers[2].mixer.kv_from"),
    (("layers", 2, "mixer", "rot", "base"), 301.0, "layers[2].mixer.kv_from"),
    (("layers", 1, "mlp", "kind"), "sparse", "layers[1].mlp.kind"),
    (("layers", 1, "mlp", "ff"), None, "layers[1].mlp.ff"),
    (("layers", 2, "mlp", "router", "top"), 6, "layers[2].mlp.router.top"),
    (("layers", 2, "mlp", "shared", "ff"), 0, "layers[2].mlp.shared.ff"),
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
    broken = {name: tensor.to(torch.bfloat16) for name, tensor in weights.items() if name != "l4.ls1"}
    broken["l0.mix.dq.norm"] = torch.zeros(39, dtype=torch.bfloat16)
    broken["l2.mix.dkv"] = torch.zeros(40, 64, dtype=torch.bfloat16)   # a layer that borrows rows has no projection of its own
    broken["l3.ls2"] = torch.zeros(64, dtype=torch.bfloat16)   # without a feed-forward its scale has no effect
    write_safetensors(folder / "model.safetensors", broken)
    with pytest.raises(WeightsError) as caught:
        load_weights(folder, load_config(folder))
    assert caught.value.missing == ["l4.ls1"] and caught.value.unexpected == ["l2.mix.dkv"] and caught.value.wrong_shape[0][0] == "l0.mix.dq.norm"


def build_model(config: dict):
    """A configuration's model from parts built on the CPU (nothing runs)."""
    from lalamo_b200.parts.base import Runtime
    from lalamo_b200.parts.model import DecoderModel

    typed = config_from_dict(config)
    plan = typed.to_plan()
    tensors = random_weights(config, 5)
    given = {(path, local): tensors[typed.checkpoint_names(path, local)[0]] for path, local in plan_tensor_decls(plan)}
    return DecoderModel(plan, given, Runtime(torch.device("cpu"), torch.float32))


def test_caches_and_states_the_layers_ask_for():
    """One row a token for the owner of latents, nothing for its borrowers (whose longest window the pages outlive), a 32-bit state."""
    from lalamo_b200.cache.manager import CacheManager
    from lalamo_b200.parts.base import BorrowedKVNeed, PagedKVNeed, SlotStateNeed

    model = build_model(CONFIG_A)
    needs, cache_from = model.cache_needs(), [entry.cache_from for entry in model.plan.schedule]
    assert needs[0] == PagedKVNeed(1, 40, window=19, value_dim=32, values_in_keys=True)
    assert needs[1] == SlotStateNeed((4, 16, 24), torch.float32) and needs[3] == SlotStateNeed((2, 8, 16), torch.float32)
    assert needs[2] == BorrowedKVNeed(window=45) and needs[4] == BorrowedKVNeed(window=7)
    manager = CacheManager(needs, cache_from, None, page_size=16, num_pages=12, num_slots=2)
    assert [(group.window, len(group.entries)) for group in manager.groups] == [(45, 1)]
    manager.admit("a")
    manager.reserve("a", 100)
    manager.commit("a", 100)
    assert sum(page >= 0 for page in manager.requests["a"].blocks[0]) == 7 - (100 - 45 + 1) // 16
    manager.release("a")
    manager.check()


def test_parts_refuse_what_they_do_not_support():
    from dataclasses import replace

    from lalamo_b200.parts.base import Runtime, build_part, part_type
    from lalamo_b200.parts.block import block_tensor_decls, build_block

    runtime = Runtime(torch.device("cpu"), torch.float32)
    plan = config_from_dict(CONFIG_A).to_plan()
    linear = plan.layers[1].mixer
    tensors = {name: torch.zeros(decl.shape) for name, decl in part_type(linear).tensor_decls(linear).items()}
    with pytest.raises(ValueError, match="in halves"):
        build_part(replace(linear, position=replace(linear.position, pairing="interleaved")), tensors, runtime)
    with pytest.raises(ValueError, match="not supported"):
        build_part(replace(linear, query_activation="silu"), tensors, runtime)
    block = replace(plan.layers[3], ffn_scale=LayerScaleSpec(64))
    with pytest.raises(ValueError, match="no scale for one"):
        build_block(block, {key: torch.zeros(decl.shape) for key, decl in block_tensor_decls(block).items()}, runtime)


def test_exact_frequencies_and_stretched_ones():
    from lalamo_b200.config import RopeSpec
    from lalamo_b200.parts.base import Runtime, build_part, part_type

    runtime = Runtime(torch.device("cpu"), torch.float32)
    for dims, base, scaling in ((64, 1e6, None), (10, 20.0, None), (32, 2.5e5, (4.0, 1000, 32.0, 1.0)), (16, 50.0, (7.0, 40, 2.0, 0.3)), (6, 1e4, (2.0, 10, 100.0, 50.0))):
        rot = {"dims": dims, "base": base}
        if scaling is not None:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
        want, factor = plain.pair_frequencies(rot)
        spec = RopeSpec(dims, base, "half", None if scaling is None else YarnScaling(*scaling), exact=True)
        part = build_part(spec, {}, runtime)
        assert torch.equal(part.inv_freq, want.to(torch.float32)) and part.magnitude == pytest.approx(factor, rel=1e-12)


def test_the_plain_mechanisms_on_hand_made_cases():
    one = torch.ones(1, 1, dtype=torch.float64)
    # retention: with decay 1/2 and k = v = q = 1 the state is 1, 3/2, 7/4 before the norm takes the size away; two channels show it
    q = torch.tensor([[1.0], [1.0], [1.0]], dtype=torch.float64)
    w = {"q": one, "k": one, "v": torch.tensor([[1.0], [0.0]], dtype=torch.float64), "g": torch.full((2, 1), 50.0, dtype=torch.float64), "o": torch.eye(2, dtype=torch.float64)}
    out = plain.retention(q, w, {"heads": 1, "dim": 1, "vdim": 2, "decay": [0.5]}, 0.0)
    assert torch.allclose(out, torch.tensor([[math.sqrt(2.0), 0.0]] * 3, dtype=torch.float64) * 50.0)
    # pairs of halves and of neighbours turn by the position; what lies behind passes
    x = torch.tensor([[[1.0, 0.0, 5.0]]], dtype=torch.float64)
    for turn in (plain.rotate_halves, plain.rotate_neighbours):
        assert torch.allclose(turn(x, torch.tensor([2]), {"dims": 2, "base": 10.0}), torch.tensor([[[math.cos(2.0), math.sin(2.0), 5.0]]], dtype=torch.float64))
    four = torch.tensor([[[1.0, 2.0, 0.0, 0.0]]], dtype=torch.float64)
    halves = plain.rotate_halves(four, torch.tensor([1]), {"dims": 4, "base": 100.0})
    assert torch.allclose(halves, torch.tensor([[[math.cos(1.0), 2 * math.cos(0.1), math.sin(1.0), 2 * math.sin(0.1)]]], dtype=torch.float64))
    neighbours = plain.rotate_neighbours(four, torch.tensor([1]), {"dims": 4, "base": 100.0})
    assert torch.allclose(neighbours, torch.tensor([[[math.cos(1.0) - 2 * math.sin(1.0), 2 * math.cos(1.0) + math.sin(1.0), 0.0, 0.0]]], dtype=torch.float64))
    # stretching puts its factor on sines and cosines
    turned = plain.rotate_neighbours(x, torch.tensor([0]), {"dims": 2, "base": 10.0, "scaling": {"factor": math.e, "original": 100, "fast": 32.0, "slow": 1.0}})
    assert torch.allclose(turned, torch.tensor([[[1.1, 0.0, 5.0]]], dtype=torch.float64))
    # an expert's weight goes in at its input: silu(w g) (w u), not w silu(g) u
    h = torch.tensor([[2.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[-9.0], [0.0]], dtype=torch.float64), **{f"e{e}.{n}": one for e in (0, 1) for n in ("gate", "up", "down")}}
    got = plain.routed_experts(h, w, {"router": {"experts": 2, "top": 1}, "expert": {"ff": 1}})
    assert got.item() == pytest.approx(1.0 / (1.0 + math.exp(-1.0)))   # score 1/2: silu(1) * 1
