"""Grouped-query causal attention over a paged cache
(``lalamo/modules/token_mixers/attention.py:511-620``): fused q/k/v projection, per-head RMS
norm of queries and keys, position encoding, keys and values written to the request's pages,
softmax attention in 32-bit over the visible keys, out-projection.

Differential attention (two maps over the same values, subtracted) is the same kernels with more heads: a K/V head's cache row holds
both maps' keys side by side, which is also the layout of twice as many key heads; its query heads are ordered first map, then second
map (the projection's rows are reordered once), and consecutive key heads share a value head.  Tokens that attend alone read such a row
once for both maps; in tiles each map is a key head of its own.  The maps' outputs stay 32-bit until they are combined."""

from __future__ import annotations

import math
import os

from typing import Mapping

import numpy as np
import torch

from .. import ops
from ..config.plan import AttentionSpec, RMSNormSpec, RopeSpec
from .base import REPLAY_MAX_TOKENS, BorrowedKVNeed, CacheNeed, CompositeNeed, CompositeView, HostSegments, Mixer, PagedKVNeed, PagedKVView, Runtime, SlotStateNeed, SlotStateView, StepInputs, TensorDecl, build_part, register_part

__all__ = ["ALONE_LIMIT", "TILE_TOKENS", "Attention", "shared_tile_keys"]

# How the attention kernels divide a step: tokens of portions of at most ALONE_LIMIT tokens attend
# alone (split over the keys); longer portions are cut into tiles of at most TILE_TOKENS consecutive tokens.
ALONE_LIMIT = 16
TILE_TOKENS = ops.PREFILL_TILE
EARLY_ATTENTION = os.environ.get("LALAMO_B200_EARLY_ATTENTION", "1") != "0"  # the split-key attention starts under the q/k/v rewrite
SHARED_TILE_KEYS = 512  # where tiles are shared, a tile that sees at least this many keys is worked on by two CTAs
LONG_TILE_KEYS = 3072  # a launch's tiles count as long if they see this many keys on average


def _slot_use(ctas: int, slots: int) -> float:
    """The share of the resident-CTA slots that ``ctas`` CTAs keep busy over the rounds they need."""
    return ctas / (-(-ctas // slots) * slots)


def shared_tile_keys(num_tiles: int, num_heads: int, num_groups: int, sms: int, tokens: int, lengths: tuple[int, ...] = (),
                     contexts: tuple[int, ...] = ()) -> int:
    """From how many visible keys on a tile of the tcgen05 prefill attention is worked on by two CTAs (each half of
    the keys, merged at the end); 0: never, the launch has one CTA per tile.  Two CTAs per tile pay where that
    fills the SMs better: with fewer CTAs than SMs; or, in steps that are never replayed (so that the answer may
    depend on the contexts), where tiles mostly see thousands of keys and their CTAs fill the resident slots
    (three per SM) badly, as 512 CTAs fill 444.  Launching as clusters costs 12 to 25 % by itself, so whole
    prompts from position 0, whose early tiles are short, stay unpaired."""
    per_group = num_heads // num_groups
    parts = -(-TILE_TOKENS // max(1, min(TILE_TOKENS, 128 // per_group)))
    ctas = num_tiles * num_groups * parts
    if ctas <= sms:
        return SHARED_TILE_KEYS
    if tokens > REPLAY_MAX_TOKENS and contexts:
        keys = sum(length * (context + length / 2) for length, context in zip(lengths, contexts))
        if keys / max(1, sum(lengths)) >= LONG_TILE_KEYS and _slot_use(2 * ctas, 3 * sms) > _slot_use(ctas, 3 * sms) + 0.1:
            return SHARED_TILE_KEYS
    return 0


def _interleaved_to_half(head_dim: int, rotary_dim: int) -> torch.Tensor:
    """The order of a head's channels that turns pairs (2i, 2i + 1) of its first ``rotary_dim`` channels into pairs
    (i, i + rotary_dim / 2): the even ones, the odd ones, then the channels that are not rotated."""
    return torch.cat([torch.arange(0, rotary_dim, 2), torch.arange(1, rotary_dim, 2), torch.arange(rotary_dim, head_dim)])


def _reorder_heads(rows: torch.Tensor, heads: int, order: torch.Tensor) -> torch.Tensor:
    """``rows`` ([heads * head_dim, ...]) with every head's rows taken in ``order``."""
    per_head = rows.reshape(heads, order.numel(), *rows.shape[1:])
    return per_head[:, order].reshape(rows.shape).contiguous()


@register_part(AttentionSpec)
class Attention(Mixer):
    graph_safe = True
    def __init__(self, spec: AttentionSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().__init__(spec, tensors, runtime)
        if spec.num_heads % spec.num_groups:
            raise ValueError(f"num_heads={spec.num_heads} is not a multiple of num_groups={spec.num_groups}")
        if spec.window is not None and spec.window < 1:
            raise ValueError(f"window must be positive, got {spec.window}")
        if spec.keep_first < 0:
            raise ValueError(f"keep_first must not be negative, got {spec.keep_first}")
        self.value_dim = spec.value_dim or spec.head_dim
        self.keep_first = spec.keep_first if spec.window is not None else 0
        differential = spec.differential
        self.maps = 2 if differential is not None else 1
        # heads as the kernels count them: with two maps every query head and every key head is two
        self.kernel_heads, self.kernel_groups = self.maps * spec.num_heads, self.maps * spec.num_groups
        if differential is not None and (spec.gated or spec.has_bias or spec.qk_norm is not None):
            raise ValueError("differential attention with biases, a norm of q and k or a gate per channel is not supported")
        if spec.borrows_kv and (spec.has_bias or spec.qk_norm is not None):
            raise ValueError("borrowed keys and values with biases or a norm of q and k are not supported")
        if spec.conv_taps < 0 or spec.conv_taps > ops.CONV_MAX_TAPS or (spec.conv_taps and spec.has_bias):
            raise ValueError(f"a convolution of q, k and v has up to {ops.CONV_MAX_TAPS} taps, and their projections no biases")
        q_proj = tensors["q_proj"]
        k_proj, v_proj = (q_proj[:0], q_proj[:0]) if spec.borrows_kv else (tensors["k_proj"], tensors["v_proj"])
        q_conv = k_conv = v_conv = None
        if spec.conv_taps:
            q_conv = tensors["q_conv"]
            k_conv, v_conv = (q_conv[:0], q_conv[:0]) if spec.borrows_kv else (tensors["k_conv"], tensors["v_conv"])
        q_bias, k_bias = (tensors["q_bias"], tensors["k_bias"]) if spec.has_bias else (None, None)
        if isinstance(spec.position, RopeSpec) and spec.position.pairing == "interleaved":
            # The kernels rotate channel i with i + rotary_dim / 2.  Scores are sums over a head's channels, so the same
            # reordering of the channels of q and k changes none of them: the even channels of the rotated part first,
            # then the odd ones, and pair (2i, 2i + 1) becomes pair (i, i + rotary_dim / 2) with its angle.
            if spec.qk_norm is not None:
                raise ValueError("interleaved rotation with a norm of q and k is not supported (the norm's weight would have to be reordered too)")
            order = _interleaved_to_half(spec.head_dim, spec.position.rotary_dim)
            q_proj = _reorder_heads(q_proj, self.kernel_heads, order)
            k_proj = _reorder_heads(k_proj, self.kernel_groups, order) if k_proj.shape[0] else k_proj
            if spec.conv_taps:
                q_conv = _reorder_heads(q_conv, self.kernel_heads, order)
                k_conv = _reorder_heads(k_conv, self.kernel_groups, order) if k_conv.shape[0] else k_conv
            if spec.has_bias:
                q_bias, k_bias = _reorder_heads(q_bias, spec.num_heads, order), _reorder_heads(k_bias, spec.num_groups, order)
        elif isinstance(spec.position, RopeSpec) and spec.position.pairing != "half":
            raise ValueError(f"unknown rotary pairing {spec.position.pairing!r}; known: 'half', 'interleaved'")
        if differential is not None:
            # [K/V head, its query heads, map] -> [K/V head, map, its query heads]
            def maps_first(rows: torch.Tensor) -> torch.Tensor:
                split = rows.reshape(spec.num_groups, spec.num_heads // spec.num_groups, 2, spec.head_dim, *rows.shape[1:])
                return split.transpose(1, 2).reshape(rows.shape).contiguous()

            q_proj = maps_first(q_proj)
            q_conv = maps_first(q_conv) if q_conv is not None else None
        # One product for everything that reads the mixer's input: queries, keys, values and, behind them, the gate's logits.
        self.qkv_width = q_proj.shape[0] + k_proj.shape[0] + v_proj.shape[0]
        rows = [q_proj, k_proj, v_proj] + ([tensors["gate_proj"]] if spec.gated else [])
        self.gate_start = self.qkv_width
        if differential is not None and differential.head_gate:
            self.gate_start = -(-self.qkv_width // 8) * 8   # one row per head behind the values, the whole padded to multiples of 8 rows
            end = -(-(self.gate_start + spec.num_heads) // 8) * 8
            rows += [q_proj.new_zeros(self.gate_start - self.qkv_width, spec.model_dim), tensors["head_gate"],
                     q_proj.new_zeros(end - self.gate_start - spec.num_heads, spec.model_dim)]
        self.qkv = runtime.matrix(torch.cat(rows, dim=0))
        self.conv_weight = runtime.vector(torch.cat([q_conv, k_conv, v_conv], dim=0).reshape(self.qkv_width, spec.conv_taps)) if spec.conv_taps else None
        self.lam = 0.0
        if differential is not None:
            first, second = (math.exp(float((tensors[f"lambda_q{m}"].double() * tensors[f"lambda_k{m}"].double()).sum())) for m in (1, 2))
            self.lam = first - second + differential.offset
        self.out_proj = runtime.matrix(tensors["out_proj"])
        # Biases are 32-bit vectors: those of q, k and v are added where the product's rows are split into heads,
        # the output's by whoever consumes the output (`output_bias`), or here.
        self.qkv_bias = runtime.vector(torch.cat([q_bias, k_bias, tensors["v_bias"]], dim=0)) if spec.has_bias else None
        self.output_bias = runtime.vector(tensors["out_bias"]) if spec.has_bias else None
        self.q_norm = self.k_norm = None
        self.norm_eps, self.norm_offset = 0.0, 0.0
        if spec.qk_norm is not None:
            if not isinstance(spec.qk_norm, RMSNormSpec) or spec.qk_norm.dim != spec.head_dim:
                raise ValueError("the per-head norm must be an RMS norm over head_dim")
            if spec.qk_norm_whole and spec.has_bias:
                raise ValueError("a norm over the whole projection with biases on q and k is not supported")
            self.q_norm = runtime.vector(tensors["q_norm"])
            self.k_norm = runtime.vector(tensors["k_norm"])
            self.norm_eps, self.norm_offset = spec.qk_norm.eps, spec.qk_norm.scale_offset
        self.position = None
        if spec.position is not None:
            if not isinstance(spec.position, RopeSpec):
                raise ValueError(f"attention applies rotary position encodings, not {type(spec.position).__name__}")
            self.position = build_part(spec.position, {}, runtime)
        self.scale = spec.scale if spec.scale is not None else spec.head_dim**-0.5

    @classmethod
    def tensor_decls(cls, spec: AttentionSpec) -> dict[str, TensorDecl]:
        decls = {
            "q_proj": TensorDecl((spec.num_heads * (2 if spec.differential else 1) * spec.head_dim, spec.model_dim)),
            "k_proj": TensorDecl((spec.num_groups * (2 if spec.differential else 1) * spec.head_dim, spec.model_dim)),
            "v_proj": TensorDecl((spec.num_groups * (spec.value_dim or spec.head_dim), spec.model_dim)),
            "out_proj": TensorDecl((spec.model_dim, spec.num_heads * (spec.value_dim or spec.head_dim))),
        }
        if spec.conv_taps:
            for part in ("q", "k", "v"):
                decls[f"{part}_conv"] = TensorDecl((decls[f"{part}_proj"].shape[0], spec.conv_taps), role="vector")
        if spec.borrows_kv:
            for local in ("k_proj", "v_proj", "k_conv", "v_conv"):
                decls.pop(local, None)
        if spec.differential is not None:
            for local in ("lambda_q1", "lambda_k1", "lambda_q2", "lambda_k2"):
                decls[local] = TensorDecl((spec.head_dim,), role="vector")
            if spec.differential.head_gate:
                decls["head_gate"] = TensorDecl((spec.num_heads, spec.model_dim))
        if spec.has_bias:
            decls["q_bias"] = TensorDecl((spec.num_heads * spec.head_dim,), role="vector")
            decls["k_bias"] = TensorDecl((spec.num_groups * spec.head_dim,), role="vector")
            decls["v_bias"] = TensorDecl((spec.num_groups * (spec.value_dim or spec.head_dim),), role="vector")
            decls["out_bias"] = TensorDecl((spec.model_dim,), role="vector")
        if spec.qk_norm is not None:
            # per head, or one element per row of the projection where the norm runs over the whole of it
            decls["q_norm"] = TensorDecl((spec.head_dim * (spec.num_heads if spec.qk_norm_whole else 1),), role="vector", init="ones")
            decls["k_norm"] = TensorDecl((spec.head_dim * (spec.num_groups if spec.qk_norm_whole else 1),), role="vector", init="ones")
        if spec.gated:
            decls["gate_proj"] = TensorDecl((spec.num_heads * (spec.value_dim or spec.head_dim), spec.model_dim))
        return decls

    def cache_need(self) -> CacheNeed | None:
        spec = self.spec
        if spec.borrows_kv:
            paged: CacheNeed = BorrowedKVNeed(window=spec.window, keep_first=self.keep_first)
        else:
            # a row of the cache holds both maps' keys of a K/V head side by side
            paged = PagedKVNeed(num_groups=spec.num_groups, head_dim=spec.head_dim * (2 if spec.differential is not None else 1), window=spec.window,
                                value_dim=spec.value_dim if spec.differential is None else self.value_dim, keep_first=self.keep_first)
        if spec.conv_taps > 1:
            return CompositeNeed((paged, SlotStateNeed(shape=(spec.conv_taps - 1, self.qkv_width))))
        return paged

    # The kernels' work lists depend on where the portions start and how long they are, not on what
    # the cache holds, and they are the same for every attention layer.
    step_plan_uses_context = False

    def step_plan_key(self) -> object:
        return ("attention", ALONE_LIMIT, TILE_TOKENS)

    def plan_step(self, segments: HostSegments) -> dict[str, np.ndarray]:
        """``alone``: the rows that attend alone; ``tiles``: ``(first row, count)`` of each tile."""
        alone: list[int] = []
        tiles: list[tuple[int, int]] = []
        for start, length in zip(segments.start, segments.length):
            if length <= ALONE_LIMIT:
                alone.extend(range(start, start + length))
            else:
                tiles.extend((first, min(TILE_TOKENS, start + length - first)) for first in range(start, start + length, TILE_TOKENS))
        return {"alone": np.asarray(alone, dtype=np.int32), "tiles": np.asarray(tiles, dtype=np.int32).reshape(-1)}

    can_accumulate = True
    can_defer = True

    def _project_out(self, mixed: torch.Tensor, residual: torch.Tensor | None, add_output_bias: bool = True, gate: torch.Tensor | None = None,
                     defer: bool = False) -> "torch.Tensor | ops.SlicedSum | None":
        spec = self.spec
        if spec.differential is not None:
            combined = self.runtime.empty(mixed.shape[0], spec.num_heads * self.value_dim)
            ops.combine_maps(mixed, gate, combined, num_heads=spec.num_heads, num_groups=spec.num_groups, value_dim=self.value_dim, lam=self.lam,
                             eps=spec.differential.norm_eps, factor=1.0 - spec.differential.offset)
            mixed = combined
        elif gate is not None:
            # the concatenated heads times sigmoid(gate), the gate's logits being the last columns of the in-projection
            gated = self.runtime.empty(*mixed.shape)
            ops.gate_heads(mixed.view(1, *mixed.shape), gate, gated)
            mixed = gated
        if self.output_bias is not None:
            out = ops.linear(mixed, self.out_proj, status=self.runtime.status)
            if isinstance(out, ops.SlicedSum):
                out = out.sum()
            if add_output_bias:
                ops.add_bias(out, self.output_bias)
            return out
        if defer:
            return ops.linear_pending(mixed, self.out_proj, status=self.runtime.status)
        if residual is not None:
            return ops.linear_accumulate(mixed, self.out_proj, residual, status=self.runtime.status)
        return ops.linear(mixed, self.out_proj, status=self.runtime.status)

    def forward(self, x: torch.Tensor, step: StepInputs, cache: "PagedKVView | CompositeView", residual: torch.Tensor | None = None,  # type: ignore[override]
                add_output_bias: bool = True, defer: bool = False) -> "torch.Tensor | ops.SlicedSum | None":
        """``add_output_bias=False``: the caller adds :attr:`output_bias` to what this returns."""
        spec = self.spec
        conv_view: SlotStateView | None = None
        if isinstance(cache, CompositeView):
            cache, conv_view = cache.views
        projected = ops.linear(x, self.qkv, status=self.runtime.status)
        gate = None
        if spec.gated:
            gate = projected[:, self.qkv_width :]
        elif spec.differential is not None and spec.differential.head_gate:
            gate = projected[:, self.gate_start : self.gate_start + spec.num_heads]
        qkv = projected[:, : self.qkv_width] if projected.shape[1] != self.qkv_width else projected
        if self.conv_weight is not None:
            qkv = ops.causal_conv(qkv, conv_view.state if conv_view is not None else None, self.conv_weight, segment_start=step.segment_start,
                                  segment_length=step.segment_length, segment_slot=step.segment_slot, segments=step.segments,
                                  max_length=step.max_segment_length, status=self.runtime.status)
        queries = self.runtime.empty(step.tokens, self.kernel_heads * spec.head_dim)
        page_size = cache.k_pages.shape[1]
        # the cache's keys as the kernels' key heads: the two maps of a K/V head are two
        keys = cache.k_pages if self.maps == 1 else cache.k_pages.view(-1, page_size, self.kernel_groups, spec.head_dim)
        temperature = spec.query_temperature
        ops.qk_norm_rope_write(
            qkv,
            queries,
            keys,
            cache.v_pages,
            q_weight=self.q_norm,
            k_weight=self.k_norm,
            eps=self.norm_eps,
            scale_offset=self.norm_offset,
            inv_freq=self.position.inv_freq if self.position is not None else None,
            rotary_dim=self.position.rotary_dim if self.position is not None else 0,
            positions=step.positions,
            token_segment=step.token_segment,
            block_table=cache.block_table,
            num_heads=self.kernel_heads,
            num_groups=self.kernel_groups,
            head_dim=spec.head_dim,
            write_kv=cache.owns,
            status=self.runtime.status,
            value_dim=self.value_dim,
            bias=self.qkv_bias,
            whole_norm=spec.qk_norm_whole and spec.qk_norm is not None,
            turn_scale=self.position.magnitude if self.position is not None else 1.0,
            value_groups=spec.num_groups,
            temperature=temperature.coefficient if temperature is not None else 0.0,
            temperature_every=temperature.every if temperature is not None else 0,
        )
        # The maps' outputs are combined in 32-bit.
        mixed = self.runtime.empty(step.tokens, self.kernel_heads * self.value_dim, dtype=torch.float32 if self.maps > 1 else None)
        common = dict(
            positions=step.positions,
            token_segment=step.token_segment,
            block_table=cache.block_table,
            num_heads=self.kernel_heads,
            num_groups=self.kernel_groups,
            head_dim=spec.head_dim,
            scale=self.scale,
            window=spec.window,
            keep_first=self.keep_first,
            status=self.runtime.status,
            value_dim=self.value_dim,
            value_groups=spec.num_groups,
        )
        # Keys and values of one size, one map: every tensor-core kernel.  Other sizes and two maps: the split-key kernel and the tcgen05 one.
        plain_shape = self.value_dim == spec.head_dim and self.maps == 1
        alone_common, alone_keys = common, keys
        if self.maps > 1 and ops.decode_attention_supported(self.runtime.dtype, self.maps * spec.head_dim, page_size, self.value_dim):
            # a token that attends alone reads a row of the cache once for both maps
            alone_common = dict(common, num_groups=spec.num_groups, head_dim=self.maps * spec.head_dim, two_maps=True)
            alone_keys = cache.k_pages
        alone_ok = ops.decode_attention_supported(self.runtime.dtype, alone_common["head_dim"], page_size, self.value_dim)
        if plain_shape:
            tiles_ok = ops.prefill_attention_supported(self.runtime.dtype, spec.num_heads, spec.num_groups, spec.head_dim, page_size)
        else:
            tiles_ok = ops.wide_prefill_attention_supported(self.runtime.dtype, self.kernel_heads, self.kernel_groups, spec.head_dim, self.value_dim, page_size)
        if alone_ok:
            lists, host_lists = step.plan_of(self)
            num_alone, num_tiles = host_lists["alone"].size, host_lists["tiles"].size // 2
        if alone_ok and (tiles_ok or num_tiles == 0):
            # Tokens of short portions attend alone (split over the keys); long portions run in tiles.
            if num_alone:
                everything = num_alone == step.tokens
                # The rewrite of q, k and v just above is the kernel before this one and writes, for any token that
                # attends alone, no more than the newest ALONE_LIMIT positions it sees (its own portion's).
                ops.attention_decode(queries, alone_keys, cache.v_pages, mixed, max_context=step.max_context,
                                     token_list=None if everything else lists["alone"], num_listed=num_alone,
                                     fresh_keys=ALONE_LIMIT if cache.owns and EARLY_ATTENTION else None, **alone_common)
            if num_tiles:
                split_tiles = 0
                if plain_shape and spec.head_dim == 64 and ops.USE_TCGEN05_ATTENTION:
                    split_tiles = shared_tile_keys(num_tiles, spec.num_heads, spec.num_groups, ops.sm_count(), step.tokens,
                                                   step.host_segment_length, step.host_segment_context) // 64
                ops.attention_prefill(queries, keys, cache.v_pages, mixed, tiles=lists["tiles"], num_tiles=num_tiles, split_tiles=split_tiles, **common)
            return self._project_out(mixed, residual, add_output_bias, gate, defer)
        ops.paged_attention_plain(queries, keys, cache.v_pages, mixed, **common)
        return self._project_out(mixed, residual, add_output_bias, gate, defer)
