"""Small Mozetar configurations for the tests, and a writer of model folders whose tensor names and shapes are spelled
out here from the configuration (not taken from the package), with weights large enough that every mechanism matters
in the logits."""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

from lalamo_b200.weights.safetensors_io import write_safetensors


def differential(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, diff=0.4, coef=0.6, every=16):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "q_temp": {"coef": coef, "every": every}}


def window(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3, conv=3, size=21, dims=8, base=10000.0, scaling=(4.0, 1.0, 4.0, 64), kv_from=None):
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    entry = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "mask": {"size": size}, "rot": rot}
    if kv_from is not None:
        entry["kv_from"] = kv_from
    return entry


def hgrn2(heads=2, dim=16, vdim=24):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, count=3, keep=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def layer(kind, mix, mlp):
    return {"type": kind, "mixer": mix, "mlp": mlp}


def model(vocab, width, streams, taps, layers, eps=1e-5):
    return {"architecture": "Mozetar", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps}, "norm": {"eps": eps}, "layers": layers}


# A: every kind of mixer and feed-forward; the borrower of keys and values looks further back than their owner, with a convolution of
# another length and another scale; three streams.
CONFIG_A = model(150, 64, 3, 3, [
    layer("attention_2", window(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.35, conv=4, size=19, dims=12, base=300.0, scaling=(5.0, 1.0, 3.0, 48)), moe(6, 2, 24, 3, 2)),
    layer("attention", differential(heads=4, kv_heads=2, dim=16, vdim=40, scale=0.4, diff=0.3, coef=0.7, every=10), dense(56)),
    layer("hgrn2", hgrn2(heads=3, dim=8, vdim=24), moe(8, 3, 16, 4, 3)),
    layer("attention_2", window(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.25, conv=2, size=45, dims=12, base=300.0, scaling=(5.0, 1.0, 3.0, 48), kv_from=0), dense(40)),
    layer("attention", differential(heads=3, kv_heads=1, dim=24, vdim=16, scale=0.3, diff=0.7, coef=0.2, every=7), None),
])

# B: sizes that fit no kernel's favourite shape, one stream, one tap in the input convolution, one head, no rotation scaling, a window of
# one, an expert per group.
CONFIG_B = model(131, 72, 1, 1, [
    layer("attention", differential(heads=1, kv_heads=1, dim=12, vdim=10, scale=0.5, diff=0.2, coef=1.5, every=3), moe(2, 1, 20, 2, 1)),
    layer("hgrn2", hgrn2(heads=1, dim=12, vdim=20), None),
    layer("attention_2", window(heads=3, kv_heads=3, dim=20, vdim=6, scale=0.4, conv=1, size=1, dims=20, base=50.0, scaling=None), dense(20)),
    layer("attention_2", window(heads=3, kv_heads=3, dim=20, vdim=6, scale=0.6, conv=3, size=11, dims=20, base=50.0, scaling=None, kv_from=2), moe(7, 3, 8, 1, 1)),
], eps=1e-6)

# C: the sizes the tensor-core kernels take (heads of 64 with values of 128, widths in multiples of 64), windows like a real model's in small.
CONFIG_C = model(256, 128, 4, 4, [
    layer("attention", differential(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.125, diff=0.35, coef=0.5, every=64), dense(256)),
    layer("attention_2", window(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15, conv=4, size=64, dims=64, base=1000.0, scaling=(8.0, 1.0, 4.0, 128)), moe(8, 2, 64, 4, 2)),
    layer("hgrn2", hgrn2(heads=2, dim=64, vdim=128), dense(192)),
    layer("attention_2", window(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15, conv=4, size=80, dims=64, base=1000.0, scaling=(8.0, 1.0, 4.0, 128), kv_from=1), moe(8, 2, 64, 2, 1)),
    layer("attention", differential(heads=8, kv_heads=2, dim=32, vdim=64, scale=0.2, diff=0.55, coef=0.4, every=50), None),
])

# D: other tensor-core shapes: key heads of 48 and 96 channels, values of 96 and 40, two streams, a convolution longer than the special kernels.
CONFIG_D = model(200, 96, 2, 6, [
    layer("attention_2", window(heads=4, kv_heads=1, dim=96, vdim=40, scale=0.12, conv=5, size=33, dims=32, base=5e5, scaling=(3.0, 0.5, 5.0, 100)), dense(88)),
    layer("attention", differential(heads=6, kv_heads=3, dim=48, vdim=96, scale=0.18, diff=0.8, coef=0.3, every=31), moe(9, 4, 32, 3, 2)),
])

# E, F, G: one mixer each without a feed-forward; H: a feed-forward of each kind behind the smallest mixer.
CONFIG_E = model(96, 64, 2, 2, [layer("attention", differential(heads=4, kv_heads=1, dim=16, vdim=16, diff=0.5), None)])
CONFIG_F = model(96, 64, 2, 2, [layer("attention_2", window(heads=4, kv_heads=2, dim=16, vdim=32, conv=3, size=20, dims=10), None)])
CONFIG_G = model(96, 64, 5, 2, [layer("hgrn2", hgrn2(heads=4, dim=16, vdim=8), None)])
CONFIG_H = model(96, 64, 2, 2, [layer("hgrn2", hgrn2(heads=1, dim=8, vdim=8), dense(72)), layer("hgrn2", hgrn2(heads=2, dim=8, vdim=8), moe(12, 3, 24, 4, 2))])

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E, "F": CONFIG_F, "G": CONFIG_G, "H": CONFIG_H}


def tensor_shapes(config: dict) -> dict[str, tuple[int, ...]]:
    width, streams = config["width"], config["streams"]
    shapes: dict[str, tuple[int, ...]] = {"embed": (config["vocab"], width), "final.norm": (width,), "head": (config["vocab"], width)}

    def connection(root: str) -> None:
        shapes[root + "in"] = shapes[root + "out"] = (streams,)
        shapes[root + "mix"] = (streams, streams)

    for index, entry in enumerate(config["layers"]):
        root = f"l{index}."
        shapes[root + "norm1"] = (width,)
        shapes[root + "canon1"] = (width, config["canon"]["taps"])
        connection(root + "hc1.")
        mix, p = entry["mixer"], root + "mix."
        heads, dim, vdim = mix["heads"], mix["dim"], mix["vdim"]
        shapes[p + "o"] = (width, heads * vdim)
        if entry["type"] == "hgrn2":
            shapes[p + "q"] = shapes[p + "f"] = (heads * dim, width)
            shapes[p + "f.b"] = shapes[p + "lower"] = (heads * dim,)
            shapes[p + "v"] = (heads * vdim, width)
            shapes[p + "norm"] = (vdim,)
        else:
            maps = 2 if entry["type"] == "attention" else 1
            shapes[p + "q"] = (heads * maps * dim, width)
            if mix.get("kv_from") is None:
                shapes[p + "k"] = (mix["kv_heads"] * maps * dim, width)
                shapes[p + "v"] = (mix["kv_heads"] * vdim, width)
            if maps == 2:
                shapes[p + "g"] = (heads, width)
                for name in ("lq1", "lk1", "lq2", "lk2"):
                    shapes[p + name] = (dim,)
            else:
                for name in ("q", "k", "v"):
                    if p + name in shapes:
                        shapes[p + name + ".conv"] = (shapes[p + name][0], mix["conv"])
        mlp = entry["mlp"]
        if mlp is None:
            continue
        shapes[root + "norm2"] = (width,)
        connection(root + "hc2.")
        m = root + "mlp."
        if mlp["kind"] == "dense":
            shapes[m + "up"], shapes[m + "up.b"] = (mlp["ff"], width), (mlp["ff"],)
            shapes[m + "down"], shapes[m + "down.b"] = (width, mlp["ff"]), (width,)
            shapes[m + "act"] = (4,)
            continue
        for e in range(mlp["router"]["experts"]):
            shapes[m + f"e{e}.gate"] = shapes[m + f"e{e}.up"] = (mlp["expert"]["ff"], width)
            shapes[m + f"e{e}.down"] = (width, mlp["expert"]["ff"])
        shapes[m + "router"] = (mlp["router"]["experts"], width)
    return shapes


def random_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 tensors: matrices N(0, 1/in); norm weights around one; queries and keys whose scores spread; forget gates that forget over tens of tokens above lower bounds between zero and a half;
    streams read and written with unequal weights of either sign, mixing matrices near the identity."""
    generator = np.random.default_rng(seed)
    tensors: dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        normal = generator.standard_normal(shape)
        if last in ("norm", "norm1", "norm2"):
            values = 1.0 + 0.2 * normal
        elif ".hc" in name:
            values = np.eye(shape[0]) + 0.2 * normal if last == "mix" else (1.0 if last == "out" else 1.0 / shape[0]) + 0.3 * normal
        elif name.endswith("f.b"):
            values = 2.5 + normal
        elif last == "lower":
            values = 0.5 * generator.random(shape)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            values = 0.8 * normal / np.sqrt(shape[0])
        elif last == "act":
            values = np.array([0.8, -0.5, 0.6, 0.1]) + 0.2 * normal
        elif last == "canon1" or last == "conv":
            values = 0.4 * normal
        elif last == "b":
            values = 0.3 * normal
        elif last == "embed":
            values = normal
        elif last == "router":
            values = 3.0 * normal / np.sqrt(shape[1])
        elif last in ("q", "k") and ".mix." in name:
            values = 1.3 * normal / np.sqrt(shape[1])
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
