"""Latent attention over a paged cache: a token leaves one row ``[latent | rope]`` behind (its normed latent vector and
one rotated key part shared by all heads), from which every head's keys and values are made.

The heads' key and value projections are not applied to the cached rows.  A query head's unrotated part is taken into
the latent's space instead (``W_uk_h^T q_h``), so that the score against a cached row is one dot product over
``latent + rope`` channels; the attention sums the rows' latent parts, and the head's value projection is applied to
that sum.  Both are exact rearrangements of ``(q . W_uk c)`` and ``sum_j p_j W_uv c_j``.

Queries may go through a normed latent of their own; its norm and the token's row are then one kernel (``ops.latent_down``) between the
down-projections, which are one product, and the queries' up-projection.  A layer may leave no rows behind and read another's."""

from __future__ import annotations

from typing import Mapping

import numpy as np
import torch

from .. import ops
from ..config.plan import LatentAttentionSpec, RMSNormSpec, RopeSpec
from .base import BorrowedKVNeed, CacheNeed, HostSegments, Mixer, PagedKVNeed, PagedKVView, Runtime, StepInputs, TensorDecl, build_part, register_part

__all__ = ["LatentAttention"]


@register_part(LatentAttentionSpec)
class LatentAttention(Mixer):
    graph_safe = True

    def __init__(self, spec: LatentAttentionSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().__init__(spec, tensors, runtime)
        if spec.window is not None and spec.window < 1:
            raise ValueError(f"window must be positive, got {spec.window}")
        if not isinstance(spec.latent_norm, RMSNormSpec) or spec.latent_norm.dim != spec.latent_dim:
            raise ValueError("the latent vector's norm must be an RMS norm over latent_dim")
        if not isinstance(spec.position, RopeSpec) or spec.position.rotary_dim != spec.rope_dim or spec.position.pairing not in ("half", "interleaved"):
            raise ValueError("latent attention rotates all rope_dim channels of the rotated parts, in halves or in pairs of neighbours")
        heads, dim, rope = spec.num_heads, spec.head_dim, spec.rope_dim
        q_proj = tensors["q_up_proj" if spec.query_rank else "q_proj"]
        down_proj = None if spec.borrows_kv else tensors["down_proj"]
        if spec.query_rank and (not isinstance(spec.query_norm, RMSNormSpec) or spec.query_norm.dim != spec.query_rank or spec.query_norm.scale_offset != 0.0):
            raise ValueError("the query latent's norm must be an RMS norm over query_rank with a plain weight")
        if spec.position.pairing == "interleaved":
            # The kernels rotate channel i with i + rope / 2.  A score sums over the rotated channels of the query and of the
            # shared key part, so taking both in the same other order (even channels first, then the odd ones) changes no
            # score, and pair (2i, 2i + 1) becomes pair (i, i + rope / 2) with its angle.
            order = torch.cat([torch.arange(0, rope, 2), torch.arange(1, rope, 2)])
            per_head = q_proj.reshape(heads, dim + rope, -1)
            q_proj = torch.cat([per_head[:, :dim], per_head[:, dim:][:, order]], dim=1).reshape(q_proj.shape)
            if down_proj is not None:
                down_proj = torch.cat([down_proj[: spec.latent_dim], down_proj[spec.latent_dim :][order]], dim=0)
        # One product for everything that reads the mixer's input: queries (or their latent's down-projection), the gate, the latent's
        # down-projection; each part starts at a multiple of 8 rows.
        parts = [tensors["q_down_proj"] if spec.query_rank else q_proj] + ([tensors["gate_proj"]] if spec.gated else []) + ([down_proj] if down_proj is not None else [])
        starts = [0]
        for part in parts:
            starts.append(-(-(starts[-1] + part.shape[0]) // 8) * 8)
        rows = torch.zeros(starts[-1], spec.model_dim, dtype=q_proj.dtype)
        for start, part in zip(starts, parts):
            rows[start : start + part.shape[0]] = part
        self.in_proj = runtime.matrix(rows)
        self.gate_start, self.down_start = starts[1], starts[2 if spec.gated else 1]
        self.q_width = heads * (dim + rope)
        self.gate_width = heads * spec.value_dim if spec.gated else 0
        self.query_up = self.query_norm = None
        if spec.query_rank:
            # columns of zeros behind the query latent's, for a product of whole 32-column blocks
            up = torch.zeros(self.q_width, -(-spec.query_rank // 32) * 32, dtype=q_proj.dtype)
            up[:, : spec.query_rank] = q_proj
            self.query_up = runtime.matrix(up)
            self.query_norm = runtime.vector(tensors["q_norm"])
        self.key_up = runtime.matrix(tensors["key_up_proj"].reshape(heads, dim, spec.latent_dim))        # [head][channel][latent]
        self.value_up = runtime.matrix(tensors["value_up_proj"].reshape(heads, spec.value_dim, spec.latent_dim))
        self.out_proj = runtime.matrix(tensors["out_proj"])
        self.latent_norm = None if spec.borrows_kv else runtime.vector(tensors["latent_norm"])
        self.sink = runtime.vector(tensors["sink"]) if spec.sink else None
        self.position = build_part(spec.position, {}, runtime)
        self.scale = spec.scale if spec.scale is not None else (dim + rope) ** -0.5

    @classmethod
    def tensor_decls(cls, spec: LatentAttentionSpec) -> dict[str, TensorDecl]:
        heads = spec.num_heads
        decls = {
            "key_up_proj": TensorDecl((heads * spec.head_dim, spec.latent_dim)),
            "value_up_proj": TensorDecl((heads * spec.value_dim, spec.latent_dim)),
            "out_proj": TensorDecl((spec.model_dim, heads * spec.value_dim)),
        }
        if spec.query_rank:
            decls["q_down_proj"] = TensorDecl((spec.query_rank, spec.model_dim))
            decls["q_norm"] = TensorDecl((spec.query_rank,), role="vector", init="ones")
            decls["q_up_proj"] = TensorDecl((heads * (spec.head_dim + spec.rope_dim), spec.query_rank))
        else:
            decls["q_proj"] = TensorDecl((heads * (spec.head_dim + spec.rope_dim), spec.model_dim))
        if not spec.borrows_kv:
            decls["down_proj"] = TensorDecl((spec.latent_dim + spec.rope_dim, spec.model_dim))
            decls["latent_norm"] = TensorDecl((spec.latent_dim,), role="vector", init="ones")
        if spec.gated:
            decls["gate_proj"] = TensorDecl((heads * spec.value_dim, spec.model_dim))
        if spec.sink:
            decls["sink"] = TensorDecl((heads,), role="vector")
        return decls

    def cache_need(self) -> CacheNeed | None:
        spec = self.spec
        if spec.borrows_kv:
            return BorrowedKVNeed(window=spec.window)
        return PagedKVNeed(num_groups=1, head_dim=spec.latent_dim + spec.rope_dim, window=spec.window, value_dim=spec.latent_dim, values_in_keys=True)

    # The tensor-core kernel's items depend on where the portions start and how long they are, not on what the cache
    # holds, and they are the same for every latent layer with as many heads.
    step_plan_uses_context = False

    def step_plan_key(self) -> object:
        return ("latent_attention", ops.latent_attention_tiling(self.spec.num_heads))

    def plan_step(self, segments: HostSegments) -> dict[str, np.ndarray]:
        """``items``: ``(first row, count)`` of every run of consecutive tokens that one CTA takes."""
        _, run = ops.latent_attention_tiling(self.spec.num_heads)
        items = [(first, min(run, start + length - first)) for start, length in zip(segments.start, segments.length) for first in range(start, start + length, run)]
        return {"items": np.asarray(items, dtype=np.int32).reshape(-1)}

    can_accumulate = True
    can_defer = True
    can_fork = True

    def forward(self, x: torch.Tensor, step: StepInputs, cache: PagedKVView, residual: torch.Tensor | None = None,  # type: ignore[override]
                defer: bool = False) -> "torch.Tensor | ops.SlicedSum | None":
        spec, runtime = self.spec, self.runtime
        heads, dim, rope, latent = spec.num_heads, spec.head_dim, spec.rope_dim, spec.latent_dim
        tokens = step.tokens
        projected = ops.linear(x, self.in_proj, status=runtime.status)
        gate = projected[:, self.gate_start : self.gate_start + self.gate_width] if spec.gated else None
        down = projected[:, self.down_start : self.down_start + latent + rope] if not spec.borrows_kv else None
        rotation = dict(inv_freq=self.position.inv_freq, turn_scale=self.position.magnitude)
        writes_row = cache.owns and down is not None
        if spec.query_rank:
            q_latent = runtime.empty(tokens, self.query_up.shape[1])
            ops.latent_down(projected[:, : spec.query_rank], down if writes_row else None, q_latent, cache.k_pages, q_norm_weight=self.query_norm,
                            q_eps=spec.query_norm.eps, norm_weight=self.latent_norm, eps=spec.latent_norm.eps, scale_offset=spec.latent_norm.scale_offset,
                            positions=step.positions, token_segment=step.token_segment, block_table=cache.block_table, latent=latent, rope=rope,
                            status=runtime.status, **rotation)
            q = ops.linear(q_latent, self.query_up, status=runtime.status)
            writes_row = False   # done
        else:
            q = projected[:, : self.q_width]
        queries = runtime.empty(tokens, heads, latent + rope)
        per_head = q.view(tokens, heads, dim + rope)
        # the heads' unrotated query parts into the latent's space: the framework's own kernel writes them where the attention
        # reads them; sizes it does not take (and the 32-bit path) go through a batched library product, [head][token][latent]
        own_products = ops.heads_product_supported(runtime.dtype, dim, latent) and ops.heads_product_supported(runtime.dtype, latent, spec.value_dim) \
            and q.stride(0) % 8 == 0 and (dim + rope) % 8 == 0
        q_latent = None
        if own_products:
            ops.heads_product(per_head[:, :, :dim], self.key_up, queries[:, :, :latent], weight_is_kn=True)
        else:
            q_latent = ops.heads_linear(per_head[:, :, :dim].transpose(0, 1), self.key_up)
        ops.latent_prepare(q, q_latent, down, queries, cache.k_pages, norm_weight=self.latent_norm, eps=spec.latent_norm.eps,
                           scale_offset=spec.latent_norm.scale_offset, positions=step.positions,
                           token_segment=step.token_segment, block_table=cache.block_table, num_heads=heads, head_dim=dim, latent=latent, rope=rope,
                           write_kv=writes_row, status=runtime.status, **rotation)
        summed = runtime.empty(tokens, heads, latent)
        common = dict(positions=step.positions, token_segment=step.token_segment, block_table=cache.block_table, num_heads=heads, latent=latent, rope=rope,
                      scale=self.scale, window=spec.window, status=runtime.status, sink=self.sink)
        if ops.latent_attention_supported(runtime.dtype, latent, rope, cache.k_pages.shape[1]):
            lists, host_lists = step.plan_of(self)
            num_items = host_lists["items"].size // 2
            splits = ops.latent_attention_splits(num_items, heads, latent, spec.window, step.max_context)
            ops.latent_attention(queries, cache.k_pages, summed, items=lists["items"], num_items=num_items, splits=splits, **common)
        else:
            ops.latent_attention_plain(queries, cache.k_pages, summed, **common)
        mixed = runtime.empty(tokens, heads * spec.value_dim)
        if own_products:
            # the heads' value projections applied to the sums, times the gate, laid out for the out-projection
            ops.heads_product(summed, self.value_up, mixed.view(tokens, heads, spec.value_dim), weight_is_kn=False,
                              gate=gate.view(tokens, heads, spec.value_dim) if gate is not None else None)
        else:
            values = ops.heads_linear(summed.transpose(0, 1), self.value_up, transpose_weight=True)   # [head][token][vdim]
            ops.gate_heads(values, gate, mixed)
        if residual is not None:
            return ops.linear_accumulate(mixed, self.out_proj, residual, status=runtime.status)
        if defer:
            return ops.linear_pending(mixed, self.out_proj, status=runtime.status)
        return ops.linear(mixed, self.out_proj, status=runtime.status)
