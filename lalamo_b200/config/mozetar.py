"""Typed configuration of the Mozetar architecture (``"architecture": "Mozetar"`` in ``config.json``).

A pre-norm decoder on ``streams`` parallel residual streams (hyper-connections: a sublayer reads a weighted sum of the streams and
writes back into all of them through a learned mixing matrix), all streams starting as the token embedding, their sum normed and
read out at the end.  A mixer's normed input first passes ``h + conv(h)``, a causal depthwise convolution.  A layer's mixer is one of
three, in an order the configuration lists:

* ``"attention"``: differential attention (two softmax maps over the same values, the second subtracted ``lambda`` times, each head
  RMS-normed without a weight) over all earlier positions, no rotation, queries growing with the logarithm of their position, one
  sigmoid gate per head;
* ``"attention_2"``: grouped attention under a sliding window, q, k and v convolved over time after their projections, rotary
  positions on neighbouring channels of part of q and k with frequencies slowed down for long contexts; with ``kv_from`` it has no
  keys and values of its own and reads the named layer's;
* ``"hgrn2"``: linear attention whose decay is a forget gate with a lower bound per channel, and whose keys are what that gate leaves free.

The feed-forward is dense (``W_down poly(W_up h)`` with biases, ``poly`` a polynomial of normalised powers), a mixture of gated silu
experts (softmax scores, the best groups of neighbours by their largest score, the chosen scores over their sum), or absent.

``config.json``: ``vocab``, ``width``, ``streams``, ``norm.eps``, ``canon.taps`` and ``layers``, one entry per layer: ``type``, ``mixer``
(``attention``: ``heads, kv_heads, dim, vdim, scale, diff, q_temp.{coef, every}``; ``attention_2``: ``heads, kv_heads, dim, vdim, scale, conv,
mask.size, rot.{dims, base, scaling.{factor, low, high, original}}, kv_from``; ``hgrn2``: ``heads, dim, vdim``) and ``mlp`` (``null``,
``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "expert.ff", "router.{experts, top, groups.{count, keep}}"}``).

Checkpoint names: ``embed``, ``final.norm``, ``head`` and per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.canon1``, ``l<i>.hc1.{in,mix,out}``,
``l<i>.hc2.{in,mix,out}``, ``l<i>.mix.*`` and ``l<i>.mlp.*`` (see the tables below).
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .errors import ConfigError
from .plan import (
    AttentionSpec,
    DenseMLPSpec,
    DifferentialSpec,
    EmbeddingSpec,
    HeadSpec,
    HyperBlockSpec,
    InputConvSpec,
    LinearAttentionSpec,
    LlamaScaling,
    ModelPlan,
    QueryTemperature,
    RMSNormSpec,
    RopeSpec,
    RoutedMLPSpec,
    ScheduleEntry,
    StreamConnectionSpec,
)

__all__ = ["MozetarConfig"]

LAYER_TYPES = ("attention", "attention_2", "hgrn2")


def _find(raw: Mapping[str, Any], path: str) -> Any:
    value: Any = raw
    for key in path.split("."):
        if not isinstance(value, Mapping) or value.get(key) is None:
            return None
        value = value[key]
    return value


def _get(raw: Mapping[str, Any], path: str, kind: type | tuple[type, ...], where: str) -> Any:
    value = _find(raw, path)
    if value is None:
        raise ConfigError(f"{where}.{path}", "is required but missing")
    if isinstance(value, bool) or not isinstance(value, kind):
        raise ConfigError(f"{where}.{path}", f"has the wrong type: {value!r}")
    return value


def _positive(raw: Mapping[str, Any], path: str, where: str) -> int:
    value = _get(raw, path, int, where)
    if value < 1:
        raise ConfigError(f"{where}.{path}", f"must be positive, got {value}")
    return value


def _number(raw: Mapping[str, Any], path: str, where: str) -> float:
    return float(_get(raw, path, (int, float), where))


def _positive_number(raw: Mapping[str, Any], path: str, where: str) -> float:
    value = _number(raw, path, where)
    if value <= 0.0:
        raise ConfigError(f"{where}.{path}", f"must be positive, got {value}")
    return value


def _heads(mixer: Mapping[str, Any], at: str) -> tuple[int, int]:
    heads, groups = _positive(mixer, "heads", at), _positive(mixer, "kv_heads", at)
    if heads % groups:
        raise ConfigError(f"{at}.kv_heads", f"{groups} does not divide heads={heads}")
    return heads, groups


@dataclass(frozen=True)
class MozetarConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: tuple[HyperBlockSpec, ...]
    kv_from: tuple[int | None, ...]  # per layer: the layer whose keys and values it reads
    raw: dict

    architecture = "Mozetar"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "MozetarConfig":
        name = raw.get("architecture")
        if name is not None and name != "Mozetar":
            raise ConfigError("architecture", f"expected 'Mozetar', got {name!r}")
        vocab, width, streams = (_positive(raw, key, "config") for key in ("vocab", "width", "streams"))
        eps = _number(raw, "norm.eps", "config")
        taps = _positive(raw, "canon.taps", "config")
        layer_list = raw.get("layers")
        if not isinstance(layer_list, list) or not layer_list:
            raise ConfigError("layers", "must be a non-empty list")
        layers: list[HyperBlockSpec] = []
        sources: list[int | None] = []
        for index, entry in enumerate(layer_list):
            spec, source = cls._layer(entry, index, width, streams, eps, taps)
            if source is not None:
                cls._check_source(layers, sources, spec.mixer, source, index)
            layers.append(spec)
            sources.append(source)
        return cls(vocab=vocab, width=width, streams=streams, norm_eps=eps, layers=tuple(layers), kv_from=tuple(sources), raw=copy.deepcopy(dict(raw)))

    @staticmethod
    def _check_source(layers: list[HyperBlockSpec], sources: list[int | None], borrower: AttentionSpec, source: int, index: int) -> None:
        where = f"layers[{index}].mixer.kv_from"
        if not 0 <= source < index:
            raise ConfigError(where, f"must name an earlier layer, got {source}")
        owner = layers[source].mixer
        if not isinstance(owner, AttentionSpec) or owner.differential is not None or sources[source] is not None:
            raise ConfigError(where, f"layer {source} has no keys and values to share")
        if (owner.num_groups, owner.head_dim, owner.value_dim, owner.position) != (borrower.num_groups, borrower.head_dim, borrower.value_dim, borrower.position):
            raise ConfigError(where, f"layer {source}'s key/value heads or rotation differ from this layer's")

    @staticmethod
    def _attention(mixer: Mapping[str, Any], at: str, width: int, eps: float) -> AttentionSpec:
        heads, groups = _heads(mixer, at)
        temperature = None
        if _find(mixer, "q_temp") is not None:
            temperature = QueryTemperature(_number(mixer, "q_temp.coef", at), _positive(mixer, "q_temp.every", at))
        return AttentionSpec(
            model_dim=width,
            num_heads=heads,
            num_groups=groups,
            head_dim=_positive(mixer, "dim", at),
            value_dim=_positive(mixer, "vdim", at),
            scale=_positive_number(mixer, "scale", at),
            differential=DifferentialSpec(offset=_number(mixer, "diff", at), norm_eps=eps, head_gate=True),
            query_temperature=temperature,
        )

    @staticmethod
    def _window_attention(mixer: Mapping[str, Any], at: str, width: int) -> tuple[AttentionSpec, int | None]:
        heads, groups = _heads(mixer, at)
        dim = _positive(mixer, "dim", at)
        dims = _get(mixer, "rot.dims", int, at) if _find(mixer, "rot.dims") is not None else 0
        if dims < 0 or dims % 2 or dims > dim:
            raise ConfigError(f"{at}.rot.dims", f"must be even and at most dim={dim}, got {dims}")
        position = None
        if dims:
            scaling = None
            if _find(mixer, "rot.scaling") is not None:
                scaling = LlamaScaling(*(_positive_number(mixer, f"rot.scaling.{key}", at) for key in ("factor", "low", "high", "original")))
            position = RopeSpec(rotary_dim=dims, theta=_positive_number(mixer, "rot.base", at), pairing="interleaved", scaling=scaling)
        source = _get(mixer, "kv_from", int, at) if _find(mixer, "kv_from") is not None else None
        spec = AttentionSpec(
            model_dim=width,
            num_heads=heads,
            num_groups=groups,
            head_dim=dim,
            value_dim=_positive(mixer, "vdim", at),
            position=position,
            window=_positive(mixer, "mask.size", at) if _find(mixer, "mask.size") is not None else None,
            scale=_positive_number(mixer, "scale", at),
            conv_taps=_positive(mixer, "conv", at) if _find(mixer, "conv") is not None else 0,
            borrows_kv=source is not None,
        )
        return spec, source

    @staticmethod
    def _hgrn2(mixer: Mapping[str, Any], at: str, width: int, eps: float) -> LinearAttentionSpec:
        return LinearAttentionSpec(
            model_dim=width,
            num_heads=_positive(mixer, "heads", at),
            key_dim=_positive(mixer, "dim", at),
            value_dim=_positive(mixer, "vdim", at),
            decay="forget",
            scaled="none",
            norm_weight=True,
            norm_eps=eps,
            gate_activation="none",
            query_activation="silu",
        )

    @staticmethod
    def _feed_forward(mlp: Any, at: str, width: int, eps: float) -> DenseMLPSpec | RoutedMLPSpec:
        if not isinstance(mlp, Mapping):
            raise ConfigError(at, "must be an object or null")
        if mlp.get("kind") == "dense":
            return DenseMLPSpec(model_dim=width, hidden_dim=_positive(mlp, "ff", at), activation="poly_norm", has_bias=True, norm_eps=eps)
        if mlp.get("kind") != "moe":
            raise ConfigError(f"{at}.kind", f"unknown feed-forward kind {mlp.get('kind')!r}; known: ['dense', 'moe']")
        experts, top = _positive(mlp, "router.experts", at), _positive(mlp, "router.top", at)
        count, keep = 1, 1
        if _find(mlp, "router.groups") is not None:
            count, keep = _positive(mlp, "router.groups.count", at), _positive(mlp, "router.groups.keep", at)
        if experts % count or keep > count:
            raise ConfigError(f"{at}.router.groups", f"{experts} experts do not form {count} equal groups of which {keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"{at}.router.top", f"{top} experts a token, but the kept groups hold {keep * (experts // count)}")
        return RoutedMLPSpec(
            model_dim=width,
            hidden_dim=_positive(mlp, "expert.ff", at),
            num_experts=experts,
            top=top,
            group_count=count,
            group_keep=keep,
            group_score="largest",
            score="softmax",
            renormalize=True,
            activation="silu",
        )

    @classmethod
    def _layer(cls, entry: Any, index: int, width: int, streams: int, eps: float, taps: int) -> tuple[HyperBlockSpec, int | None]:
        where = f"layers[{index}]"
        if not isinstance(entry, Mapping):
            raise ConfigError(where, "must be an object")
        kind = entry.get("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}.type", f"unknown layer type {kind!r}; known: {list(LAYER_TYPES)}")
        mixer, at = _get(entry, "mixer", Mapping, where), where + ".mixer"
        source: int | None = None
        if kind == "attention":
            mixer_spec: Any = cls._attention(mixer, at, width, eps)
        elif kind == "attention_2":
            mixer_spec, source = cls._window_attention(mixer, at, width)
        else:
            mixer_spec = cls._hgrn2(mixer, at, width, eps)
        norm = RMSNormSpec(dim=width, eps=eps, exact=True)
        connection = StreamConnectionSpec(streams=streams)
        mlp = entry.get("mlp")
        second: dict[str, Any] = {}
        if mlp is not None:
            second = dict(pre_ffn_norm=norm, ffn=cls._feed_forward(mlp, where + ".mlp", width, eps), ffn_connection=connection)
        return HyperBlockSpec(pre_mixer_norm=norm, mixer=mixer_spec, mixer_connection=connection, input_conv=InputConvSpec(width, taps), **second), source

    # --------------------------------------------------------------------- plan
    def to_plan(self) -> ModelPlan:
        return ModelPlan(
            vocab_size=self.vocab,
            model_dim=self.width,
            layers=self.layers,
            final_norm=RMSNormSpec(dim=self.width, eps=self.norm_eps, exact=True),
            tie_embeddings=False,
            embedding=EmbeddingSpec(self.vocab, self.width, 1.0),
            head=HeadSpec(self.vocab, self.width, tied=False),
            schedule=tuple(ScheduleEntry(index, cache_from=source) for index, source in enumerate(self.kv_from)),
            streams=self.streams,
        )

    # ---------------------------------------------------------- checkpoint names
    _ATTENTION = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "out_proj": "o", "head_gate": "g", "lambda_q1": "lq1", "lambda_k1": "lk1", "lambda_q2": "lq2",
                  "lambda_k2": "lk2", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}
    _LINEAR = {"q_proj": "q", "v_proj": "v", "forget_proj": "f", "forget_bias": "f.b", "lower": "lower", "out_norm": "norm", "out_proj": "o"}
    _MLP = {"up_proj": "up", "up_bias": "up.b", "down_proj": "down", "down_bias": "down.b", "coefficients": "act", "router": "router"}
    _CONNECTION = {"read": "in", "mix": "mix", "write": "out"}
    _NORMS = {"pre_mixer_norm": "norm1", "pre_ffn_norm": "norm2"}

    def checkpoint_names(self, path: tuple, local: str) -> list[str]:
        ends = {("embedding",): ("weight", "embed"), ("lm_head",): ("weight", "head"), ("final_norm",): ("scale", "final.norm")}
        if path in ends and ends[path][0] == local:
            return [ends[path][1]]
        if path[0] == "layers":
            index, role = path[1], path[2]
            root = f"l{index}"
            if role in self._NORMS and local == "scale":
                return [f"{root}.{self._NORMS[role]}"]
            if role == "input_conv" and local == "weight":
                return [f"{root}.canon1"]
            if role in ("mixer_connection", "ffn_connection") and local in self._CONNECTION:
                return [f"{root}.{'hc1' if role == 'mixer_connection' else 'hc2'}.{self._CONNECTION[local]}"]
            if role == "mixer":
                table = self._LINEAR if isinstance(self.layers[index].mixer, LinearAttentionSpec) else self._ATTENTION
                if local in table:
                    return [f"{root}.mix.{table[local]}"]
            if role == "ffn":
                if local in self._MLP:
                    return [f"{root}.mlp.{self._MLP[local]}"]
                parts = local.split(".")
                if len(parts) == 3 and parts[0] == "experts" and parts[2] in ("gate_proj", "up_proj", "down_proj"):
                    return [f"{root}.mlp.e{parts[1]}.{parts[2][:-5]}"]
        raise KeyError(f"Mozetar has no tensor {local!r} at {path!r}")

    def to_json_dict(self) -> dict[str, Any]:
        raw = copy.deepcopy(self.raw)
        raw["architecture"] = "Mozetar"
        return raw
