"""Typed configuration of the Zevetar architecture (``"architecture": "Zevetar"`` in ``config.json``).

A decoder of parallel blocks, ``h = norm1(x); x <- x + ls1 * mixer(h) + ls2 * ff(h)``: one RMS norm per layer, both sublayers read it, and
each one's output is multiplied by a learned vector.  A layer's mixer is one of two, in an order the configuration lists:

* ``"latent_attention"``: queries through a normed latent of their own, keys and values made from one normed latent vector per token
  plus one key part shared by all heads and rotated in pairs of neighbouring channels with stretched frequencies, a sliding window, a
  sigmoid gate on the heads' outputs; with ``kv_from`` it leaves nothing behind and reads the named layer's latents and key parts;
* ``"retention"``: linear attention with one fixed decay per head, q and k rotated in halves on part of each head, keys scaled by
  ``dim ** -0.5``, each head's read-out divided by its root mean square, a silu gate.

The feed-forward is gated (silu), a mixture of such experts (sigmoid scores, the largest chosen, a chosen score multiplying its expert's
input), optionally with a shared expert times ``sigmoid(w_sg . h)``, or absent.  The embedding is scaled; the read-out is the embedding
table itself, times ``logit_scale``, soft-capped.

``config.json``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``logit_scale``, ``logit_softcap`` and ``layers``, one entry per layer:
``type``, ``mixer`` (``latent_attention``: ``heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask.size, rot.{dims, base, scaling.{factor,
original, fast, slow}}, kv_from``; ``retention``: ``heads, dim, vdim, decay`` (a list, one per head), ``rot.{dims, base}``) and ``mlp`` (``null``,
``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "expert.ff", "router.{experts, top}", "shared.ff"}``).

Checkpoint names: ``embed``, ``final.norm`` and per layer ``l<i>.norm1``, ``l<i>.ls1``, ``l<i>.ls2``,
``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}`` or ``l<i>.mix.{q,k,v,g,o}``, and ``l<i>.mlp.{gate,up,down}`` or
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.shared.{gate,up,down,sg}``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .errors import ConfigError
from .plan import (
    EmbeddingSpec,
    GatedMLPSpec,
    HeadSpec,
    LatentAttentionSpec,
    LayerScaleSpec,
    LinearAttentionSpec,
    ModelPlan,
    ParallelBlockSpec,
    RMSNormSpec,
    RopeSpec,
    RoutedMLPSpec,
    ScheduleEntry,
    YarnScaling,
)

__all__ = ["ZevetarConfig"]

LAYER_TYPES = ("latent_attention", "retention")


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


def _rotation(mixer: Mapping[str, Any], at: str, most: int, pairing: str) -> RopeSpec | None:
    dims = _get(mixer, "rot.dims", int, at) if _find(mixer, "rot.dims") is not None else 0
    if dims < 0 or dims % 2 or dims > most:
        raise ConfigError(f"{at}.rot.dims", f"must be even and at most {most}, got {dims}")
    if dims == 0:
        return None
    base = _number(mixer, "rot.base", at)
    if base <= 1.0:
        raise ConfigError(f"{at}.rot.base", f"must exceed 1, got {base}")
    scaling = None
    if _find(mixer, "rot.scaling") is not None:
        scaling = YarnScaling(**{key: _number(mixer, f"rot.scaling.{key}", at) for key in ("factor", "original", "fast", "slow")})
        if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0.0:
            raise ConfigError(f"{at}.rot.scaling", "factor, original, fast and slow must be positive")
    return RopeSpec(rotary_dim=dims, theta=base, pairing=pairing, scaling=scaling, exact=True)


@dataclass(frozen=True)
class ZevetarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float  # 0: the logits are not capped
    layers: tuple[ParallelBlockSpec, ...]
    kv_from: tuple[int | None, ...]  # per layer: the layer whose latents it reads
    raw: dict

    architecture = "Zevetar"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "ZevetarConfig":
        name = raw.get("architecture")
        if name is not None and name != "Zevetar":
            raise ConfigError("architecture", f"expected 'Zevetar', got {name!r}")
        vocab, width = _positive(raw, "vocab", "config"), _positive(raw, "width", "config")
        eps = _number(raw, "norm.eps", "config")
        softcap = _number(raw, "logit_softcap", "config") if raw.get("logit_softcap") is not None else 0.0
        if softcap < 0.0:
            raise ConfigError("logit_softcap", f"must not be negative, got {softcap}")
        layer_list = raw.get("layers")
        if not isinstance(layer_list, list) or not layer_list:
            raise ConfigError("layers", "must be a non-empty list")
        layers: list[ParallelBlockSpec] = []
        sources: list[int | None] = []
        for index, entry in enumerate(layer_list):
            spec, source = cls._layer(entry, index, width, eps)
            if source is not None:
                cls._check_source(layers, sources, spec.mixer, source, index)
            layers.append(spec)
            sources.append(source)
        return cls(
            vocab=vocab,
            width=width,
            norm_eps=eps,
            embedding_scale=_number(raw, "embedding.scale", "config") if _find(raw, "embedding.scale") is not None else 1.0,
            logit_scale=_number(raw, "logit_scale", "config") if raw.get("logit_scale") is not None else 1.0,
            logit_softcap=softcap,
            layers=tuple(layers),
            kv_from=tuple(sources),
            raw=copy.deepcopy(dict(raw)),
        )

    @staticmethod
    def _check_source(layers: list[ParallelBlockSpec], sources: list[int | None], borrower: LatentAttentionSpec, source: int, index: int) -> None:
        where = f"layers[{index}].mixer.kv_from"
        if not 0 <= source < index:
            raise ConfigError(where, f"must name an earlier layer, got {source}")
        owner = layers[source].mixer
        if not isinstance(owner, LatentAttentionSpec) or sources[source] is not None:
            raise ConfigError(where, f"layer {source} has no latents to share")
        if (owner.latent_dim, owner.rope_dim, owner.position) != (borrower.latent_dim, borrower.rope_dim, borrower.position):
            raise ConfigError(where, f"layer {source}'s latent size or rotation differs from this layer's")

    @staticmethod
    def _latent_attention(mixer: Mapping[str, Any], at: str, width: int, eps: float) -> tuple[LatentAttentionSpec, int | None]:
        rot_dim = _positive(mixer, "rot_dim", at)
        position = _rotation(mixer, at, rot_dim, "interleaved")
        if position is None or position.rotary_dim != rot_dim:
            raise ConfigError(f"{at}.rot.dims", f"the rotated part has rot_dim={rot_dim} channels, got {_find(mixer, 'rot.dims')!r}")
        rank, query_rank = _positive(mixer, "kv_rank", at), _positive(mixer, "q_rank", at)
        source = _get(mixer, "kv_from", int, at) if _find(mixer, "kv_from") is not None else None
        spec = LatentAttentionSpec(
            model_dim=width,
            num_heads=_positive(mixer, "heads", at),
            head_dim=_positive(mixer, "dim", at),
            rope_dim=rot_dim,
            value_dim=_positive(mixer, "vdim", at),
            latent_dim=rank,
            latent_norm=RMSNormSpec(dim=rank, eps=eps, exact=True),
            position=position,
            window=_positive(mixer, "mask.size", at) if _find(mixer, "mask.size") is not None else None,
            scale=_number(mixer, "scale", at),
            gated=True,
            query_rank=query_rank,
            query_norm=RMSNormSpec(dim=query_rank, eps=eps, exact=True),
            borrows_kv=source is not None,
        )
        return spec, source

    @staticmethod
    def _retention(mixer: Mapping[str, Any], at: str, width: int, eps: float) -> LinearAttentionSpec:
        heads, dim = _positive(mixer, "heads", at), _positive(mixer, "dim", at)
        decay = _get(mixer, "decay", list, at)
        if len(decay) != heads or any(isinstance(value, bool) or not isinstance(value, (int, float)) for value in decay):
            raise ConfigError(f"{at}.decay", f"must list one number per head ({heads}), got {decay!r}")
        return LinearAttentionSpec(
            model_dim=width,
            num_heads=heads,
            key_dim=dim,
            value_dim=_positive(mixer, "vdim", at),
            decay="fixed",
            decay_values=tuple(float(value) for value in decay),
            scaled="key",
            norm_weight=False,
            norm_eps=eps,
            gate_activation="silu",
            position=_rotation(mixer, at, dim, "half"),
        )

    @staticmethod
    def _feed_forward(mlp: Any, at: str, width: int) -> GatedMLPSpec | RoutedMLPSpec:
        if not isinstance(mlp, Mapping):
            raise ConfigError(at, "must be an object or null")
        if mlp.get("kind") == "dense":
            return GatedMLPSpec(model_dim=width, hidden_dim=_positive(mlp, "ff", at), activation="silu")
        if mlp.get("kind") != "moe":
            raise ConfigError(f"{at}.kind", f"unknown feed-forward kind {mlp.get('kind')!r}; known: ['dense', 'moe']")
        experts, top = _positive(mlp, "router.experts", at), _positive(mlp, "router.top", at)
        if top > experts:
            raise ConfigError(f"{at}.router.top", f"{top} experts a token of {experts}")
        shared = None
        if _find(mlp, "shared") is not None:
            shared = GatedMLPSpec(model_dim=width, hidden_dim=_positive(mlp, "shared.ff", at), activation="silu")
        return RoutedMLPSpec(
            model_dim=width,
            hidden_dim=_positive(mlp, "expert.ff", at),
            num_experts=experts,
            top=top,
            score="sigmoid",
            renormalize=False,
            activation="silu",
            weigh_input=True,
            shared=shared,
            shared_gate=shared is not None,
        )

    @classmethod
    def _layer(cls, entry: Any, index: int, width: int, eps: float) -> tuple[ParallelBlockSpec, int | None]:
        where = f"layers[{index}]"
        if not isinstance(entry, Mapping):
            raise ConfigError(where, "must be an object")
        kind = entry.get("type")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"{where}.type", f"unknown layer type {kind!r}; known: {list(LAYER_TYPES)}")
        mixer, at = _get(entry, "mixer", Mapping, where), where + ".mixer"
        source: int | None = None
        if kind == "latent_attention":
            mixer_spec: Any
            mixer_spec, source = cls._latent_attention(mixer, at, width, eps)
        else:
            mixer_spec = cls._retention(mixer, at, width, eps)
        norm, scale, mlp = RMSNormSpec(dim=width, eps=eps, exact=True), LayerScaleSpec(dim=width), entry.get("mlp")
        if mlp is None:
            return ParallelBlockSpec(norm=norm, mixer=mixer_spec, mixer_scale=scale), source
        return ParallelBlockSpec(norm=norm, mixer=mixer_spec, ffn=cls._feed_forward(mlp, where + ".mlp", width), mixer_scale=scale, ffn_scale=scale), source

    # --------------------------------------------------------------------- plan
    def to_plan(self) -> ModelPlan:
        return ModelPlan(
            vocab_size=self.vocab,
            model_dim=self.width,
            layers=self.layers,
            final_norm=RMSNormSpec(dim=self.width, eps=self.norm_eps, exact=True),
            tie_embeddings=True,
            embedding=EmbeddingSpec(self.vocab, self.width, self.embedding_scale),
            head=HeadSpec(self.vocab, self.width, tied=True, scale=self.logit_scale, softcap=self.logit_softcap),
            schedule=tuple(ScheduleEntry(index, cache_from=source) for index, source in enumerate(self.kv_from)),
        )

    # ---------------------------------------------------------- checkpoint names
    _LATENT = {"q_down_proj": "dq", "q_norm": "dq.norm", "q_up_proj": "uq", "down_proj": "dkv", "latent_norm": "dkv.norm", "key_up_proj": "uk",
               "value_up_proj": "uv", "gate_proj": "g", "out_proj": "o"}
    _RETENTION = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "gate_proj": "g", "out_proj": "o"}
    _MLP = {"gate_proj": "gate", "up_proj": "up", "down_proj": "down", "router": "router", "shared.gate_proj": "shared.gate", "shared.up_proj": "shared.up",
            "shared.down_proj": "shared.down", "shared_gate": "shared.sg"}
    _VECTORS = {("norm", "scale"): "norm1", ("mixer_scale", "scale"): "ls1", ("ffn_scale", "scale"): "ls2"}

    def checkpoint_names(self, path: tuple, local: str) -> list[str]:
        ends = {("embedding",): ("weight", "embed"), ("final_norm",): ("scale", "final.norm")}
        if path in ends and ends[path][0] == local:
            return [ends[path][1]]
        if path[0] == "layers":
            index, role = path[1], path[2]
            root = f"l{index}"
            if (role, local) in self._VECTORS:
                return [f"{root}.{self._VECTORS[role, local]}"]
            if role == "mixer":
                table = self._LATENT if isinstance(self.layers[index].mixer, LatentAttentionSpec) else self._RETENTION
                if local in table:
                    return [f"{root}.mix.{table[local]}"]
            if role == "ffn":
                if local in self._MLP:
                    return [f"{root}.mlp.{self._MLP[local]}"]
                parts = local.split(".")
                if len(parts) == 3 and parts[0] == "experts" and parts[2] in ("gate_proj", "up_proj", "down_proj"):
                    return [f"{root}.mlp.e{parts[1]}.{parts[2][:-5]}"]
        raise KeyError(f"Zevetar has no tensor {local!r} at {path!r}")

    def unused_names(self) -> set[str]:
        """A layer without a feed-forward may still carry its scale."""
        return {f"l{index}.ls2" for index, layer in enumerate(self.layers) if layer.ffn is None}

    def to_json_dict(self) -> dict[str, Any]:
        raw = copy.deepcopy(self.raw)
        raw["architecture"] = "Zevetar"
        return raw
