"""Small Zevetar configurations for the tests, and a writer of model folders whose tensor names and shapes are spelled
out here from the configuration (not taken from the package), with weights large enough that every mechanism matters
in the logits."""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

from lalamo_b200.weights.safetensors_io import write_safetensors


def latent(heads=4, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scale=0.3, size=21, base=10000.0, scaling=(4.0, 64, 8.0, 1.0), kv_from=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    entry = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if size is not None:
        entry["mask"] = {"size": size}
    if kv_from is not None:
        entry["kv_from"] = kv_from
    return entry


def retention(heads=4, dim=16, vdim=16, decay=None, dims=16, base=10000.0):
    entry = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** (-2 - h) for h in range(heads)]}
    if dims:
        entry["rot"] = {"dims": dims, "base": base}
    return entry


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared_ff=32):
    entry = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared_ff is not None:
        entry["shared"] = {"ff": shared_ff}
    return entry


def layer(kind, mix, mlp):
    return {"type": kind, "mixer": mix, "mlp": mlp}


def model(vocab, width, layers, eps=1e-5, scale=4.0, logit_scale=1.5, cap=20.0):
    return {"architecture": "Zevetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "logit_scale": logit_scale,
            "logit_softcap": cap, "layers": layers}


# A: both mixers with every kind of feed-forward; a borrower that looks further back than the rows' owner and one that looks less far, with
# heads, value sizes and query latents of their own; part of each head rotated in the retention; more than one expert a token.
CONFIG_A = model(150, 64, [
    layer("latent_attention", latent(heads=4, dim=16, rot_dim=8, vdim=24, q_rank=40, kv_rank=32, scale=0.35, size=19, base=300.0, scaling=(5.0, 48, 4.0, 0.5)), moe(6, 2, 24, 32)),
    layer("retention", retention(heads=4, dim=16, vdim=24, dims=12, base=100.0), dense(56)),
    layer("latent_attention", latent(heads=6, dim=24, rot_dim=8, vdim=16, q_rank=24, kv_rank=32, scale=0.25, size=45, base=300.0, scaling=(5.0, 48, 4.0, 0.5), kv_from=0), moe(5, 3, 16, 24)),
    layer("retention", retention(heads=2, dim=8, vdim=16, decay=[0.9, 0.995], dims=8, base=5000.0), None),
    layer("latent_attention", latent(heads=2, dim=16, rot_dim=8, vdim=40, q_rank=64, kv_rank=32, scale=0.3, size=7, base=300.0, scaling=(5.0, 48, 4.0, 0.5), kv_from=0), dense(40)),
])

# B: sizes that fit no kernel's favourite shape (odd ranks, value sizes and widths), one head, one expert of two, no stretching, no rotation of
# the retention, a window of one, no window at all, decays of a half and of one.
CONFIG_B = model(131, 70, [
    layer("latent_attention", latent(heads=1, dim=12, rot_dim=6, vdim=10, q_rank=13, kv_rank=27, scale=0.5, size=1, base=50.0, scaling=None), moe(2, 1, 20, None)),
    layer("latent_attention", latent(heads=3, dim=9, rot_dim=10, vdim=7, q_rank=33, kv_rank=20, scale=0.4, size=None, base=20.0, scaling=(2.0, 30, 3.0, 0.7)), None),
    layer("retention", retention(heads=3, dim=12, vdim=20, decay=[0.5, 0.97, 1.0], dims=0), moe(7, 3, 9, 11)),
    layer("latent_attention", latent(heads=2, dim=5, rot_dim=6, vdim=6, q_rank=8, kv_rank=27, scale=0.6, size=11, base=50.0, scaling=None, kv_from=0), dense(20)),
    layer("retention", retention(heads=1, dim=10, vdim=6, decay=[0.93], dims=4, base=7.0), moe(4, 4, 8, 6)),
], eps=1e-6, scale=1.0, logit_scale=1.0, cap=0.0)

# C: the sizes the tensor-core kernels take (latents, rotated parts and heads in multiples of 16, widths of 64s), windows like a real model's
# in small, heads of the recurrence long portions of which run as chunks.
CONFIG_C = model(256, 128, [
    layer("latent_attention", latent(heads=4, dim=64, rot_dim=32, vdim=64, q_rank=96, kv_rank=128, scale=0.102, size=64, base=1e5, scaling=(8.0, 128, 16.0, 1.0)), dense(256)),
    layer("retention", retention(heads=2, dim=64, vdim=128, dims=64, base=1e4), moe(8, 1, 64, 64)),
    layer("latent_attention", latent(heads=4, dim=64, rot_dim=32, vdim=64, q_rank=64, kv_rank=128, scale=0.13, size=80, base=1e5, scaling=(8.0, 128, 16.0, 1.0), kv_from=0), moe(8, 2, 64, 128)),
    layer("retention", retention(heads=4, dim=32, vdim=64, dims=16, base=1e3), dense(192)),
])

# D: other tensor-core shapes: a latent wider than one CTA's columns, seven heads, a window longer than most prompts.
CONFIG_D = model(200, 96, [
    layer("latent_attention", latent(heads=7, dim=32, rot_dim=16, vdim=48, q_rank=56, kv_rank=272, scale=0.15, size=130, base=5e5, scaling=(3.0, 100, 32.0, 1.0)), moe(9, 4, 32, 40)),
    layer("retention", retention(heads=6, dim=48, vdim=32, dims=48, base=5e4), dense(88)),
])

# E, F: one mixer each without a feed-forward; G: each kind of feed-forward behind the smallest mixer.
CONFIG_E = model(96, 64, [layer("latent_attention", latent(heads=4, dim=16, rot_dim=16, vdim=16, q_rank=32, kv_rank=48, size=20), None)])
CONFIG_F = model(96, 64, [layer("retention", retention(heads=4, dim=16, vdim=8, decay=[0.8, 0.9, 0.99, 0.999]), None)])
CONFIG_G = model(96, 64, [layer("retention", retention(heads=1, dim=8, vdim=8, decay=[0.9], dims=8), dense(72)),
                          layer("retention", retention(heads=2, dim=8, vdim=8, dims=4), moe(12, 3, 24, 16))], cap=5.0)

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E, "F": CONFIG_F, "G": CONFIG_G}


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    width = config["width"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (config["vocab"], width), "final.norm": (width,)}
    for index, entry in enumerate(config["layers"]):
        root = f"l{index}."
        shapes[root + "norm1"] = shapes[root + "ls1"] = (width,)
        mix, p = entry["mixer"], root + "mix."
        heads, dim, vdim = mix["heads"], mix["dim"], mix["vdim"]
        shapes[p + "g"] = (heads * vdim, width)
        shapes[p + "o"] = (width, heads * vdim)
        if entry["type"] == "retention":
            shapes[p + "q"] = shapes[p + "k"] = (heads * dim, width)
            shapes[p + "v"] = (heads * vdim, width)
        else:
            shapes[p + "dq"], shapes[p + "dq.norm"] = (mix["q_rank"], width), (mix["q_rank"],)
            shapes[p + "uq"] = (heads * (dim + mix["rot_dim"]), mix["q_rank"])
            if mix.get("kv_from") is None:
                shapes[p + "dkv"], shapes[p + "dkv.norm"] = (mix["kv_rank"] + mix["rot_dim"], width), (mix["kv_rank"],)
            shapes[p + "uk"] = (heads * dim, mix["kv_rank"])
            shapes[p + "uv"] = (heads * vdim, mix["kv_rank"])
        mlp = entry["mlp"]
        if mlp is None:
            continue
        shapes[root + "ls2"] = (width,)
        m = root + "mlp."

        def gated(prefix: str, ff: int) -> None:
            shapes[prefix + "gate"] = shapes[prefix + "up"] = (ff, width)
            shapes[prefix + "down"] = (width, ff)

        if mlp["kind"] == "dense":
            gated(m, mlp["ff"])
            continue
        for e in range(mlp["router"]["experts"]):
            gated(m + f"e{e}.", mlp["expert"]["ff"])
        shapes[m + "router"] = (mlp["router"]["experts"], width)
        if mlp.get("shared") is not None:
            gated(m + "shared.", mlp["shared"]["ff"])
            shapes[m + "shared.sg"] = (1, width)
    return shapes


def random_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors: matrices N(0, 1/in); norm weights around one; layer scales of unequal size and either sign; queries and keys whose
    scores spread; routers whose scores do."""
    generator = np.random.default_rng(seed)
    tensors: dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        normal = generator.standard_normal(shape)
        if last in ("norm", "norm1"):
            values = 1.0 + 0.2 * normal
        elif last in ("ls1", "ls2"):
            values = np.where(generator.random(shape) < 0.2, -1.0, 1.0) * (1.0 + 0.4 * np.abs(normal))
        elif last == "embed":
            values = normal / config["embedding"]["scale"]
        elif last == "router":
            values = 3.0 * normal / np.sqrt(shape[1])
        elif last in ("uq", "uk", "dkv") or (last in ("q", "k") and ".mix." in name):
            values = 1.4 * normal / np.sqrt(shape[1])
        else:
            values = normal / np.sqrt(shape[-1])
        tensors[name] = torch.from_numpy(np.asarray(values)).to(torch.bfloat16)
    return tensors


def write_model(directory: Path, config: dict, seed: int) -> tuple[Path, dict[str, torch.Tensor]]:
    """Writes the folder; returns it and the weights in float64 (the bfloat16 values) for the plain implementation."""
    directory = Path(directory)
    directory.mkdir(parents=True, exist_ok=True)
    tensors = random_weights(config, seed)
    (directory / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(directory / "model.safetensors", tensors)
    return directory, {name: tensor.to(torch.float64) for name, tensor in tensors.items()}
