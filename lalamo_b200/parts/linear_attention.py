"""Linear attention with a decaying matrix state per head: ``S_t = diag(a_t) S_(t-1) + k_t v_t^T; o_t = S_t^T q_t``, no softmax
and no denominator.  The decay is one fixed number per head (retention) or one number per head and key channel made from
the token through a bottleneck, ``a = sigmoid(W_a2 (W_a1 h) + b) ** (1 / tau)`` (gated linear attention), or it is a forget gate
with a lower bound, ``a = l + (1 - l) sigmoid(W_f h + b)``, that also says what is written, ``k = 1 - a`` (HGRN2).  The read-out is
RMS-normed per head, multiplied by an activated gate (if there is one) and projected out.

One product gives q, k, v and the gate's logits (rows padded to a multiple of 8); the decay's logits come from two small
products (the bottleneck padded with zeros to a multiple of 32 columns), those of a forget gate from rows of the first.  A kernel lays the recurrence's inputs out in 32-bit
with the scale on q or k and the decays; the recurrence is the scan the gated delta rule uses, without that rule's correction;
the read-out kernel is shared with it too.  A rotation of q and k is part of the first of these kernels.  Per request the mixer holds the matrix state in 32-bit."""

from __future__ import annotations

from typing import Mapping

import numpy as np
import torch

from .. import ops
from ..config.plan import LinearAttentionSpec, RopeSpec
from .base import CacheNeed, HostSegments, Mixer, Runtime, SlotStateNeed, SlotStateView, StepInputs, TensorDecl, build_part, register_part

__all__ = ["LinearAttention"]


def _round_up(value: int, multiple: int) -> int:
    return -(-value // multiple) * multiple


@register_part(LinearAttentionSpec)
class LinearAttention(Mixer):
    graph_safe = True

    def __init__(self, spec: LinearAttentionSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().__init__(spec, tensors, runtime)
        heads, dk, dv = spec.num_heads, spec.key_dim, spec.value_dim
        if spec.decay not in ("fixed", "channel", "forget"):
            raise ValueError(f"unknown decay {spec.decay!r}; known: 'fixed', 'channel', 'forget'")
        if spec.scaled not in ("query", "key", "none"):
            raise ValueError(f"unknown place of the scale {spec.scaled!r}; known: 'query', 'key', 'none'")
        if spec.gate_activation not in ("sigmoid", "silu", "none"):
            raise ValueError(f"unknown gate activation {spec.gate_activation!r}; known: 'sigmoid', 'silu', 'none'")
        if spec.query_activation not in ("identity", "silu"):
            raise ValueError(f"unknown query activation {spec.query_activation!r}; known: 'identity', 'silu'")
        # [q ; (k) ; v | gate | forget gate], each part of the product starting at a multiple of 8 rows
        names = ["q_proj", "v_proj"] if spec.decay == "forget" else ["q_proj", "k_proj", "v_proj"]
        parts = [torch.cat([tensors[name] for name in names], dim=0)]
        end = _round_up(parts[0].shape[0], 8)
        self.gate_offset = self.forget_offset = None
        if spec.gate_activation != "none":
            self.gate_offset, end = end, _round_up(end + heads * dv, 8)
            parts.append(tensors["gate_proj"])
        if spec.decay == "forget":
            self.forget_offset, end = end, _round_up(end + heads * dk, 8)
            parts.append(tensors["forget_proj"])
        padded = torch.zeros(end, spec.model_dim, dtype=parts[0].dtype)
        offset = 0
        for part in parts:
            padded[offset : offset + part.shape[0]] = part
            offset = _round_up(offset + part.shape[0], 8)
        self.in_proj = runtime.matrix(padded)
        self.fixed_decay = self.decay_down = self.decay_up = self.decay_bias = self.lower = None
        if spec.decay == "forget":
            self.decay_bias = runtime.vector(tensors["forget_bias"])
            self.lower = runtime.vector(tensors["lower"])
        elif spec.decay == "fixed":
            if len(spec.decay_values) != heads:
                raise ValueError(f"{len(spec.decay_values)} fixed decays for {heads} heads")
            self.fixed_decay = runtime.vector(torch.tensor(spec.decay_values, dtype=torch.float64))
        else:
            if spec.decay_rank < 1 or spec.tau <= 0.0:
                raise ValueError("a decay made from the token needs a bottleneck of positive rank and a positive tau")
            rank = _round_up(spec.decay_rank, 32)
            down = torch.zeros(rank, spec.model_dim, dtype=padded.dtype)
            down[: spec.decay_rank] = tensors["decay_down"]
            up = torch.zeros(_round_up(heads * dk, 8), rank, dtype=padded.dtype)
            up[: heads * dk, : spec.decay_rank] = tensors["decay_up"]
            self.decay_down, self.decay_up = runtime.matrix(down), runtime.matrix(up)
            self.decay_bias = runtime.vector(tensors["decay_bias"])
        self.norm_weight = runtime.vector(tensors["out_norm"] if spec.norm_weight else torch.ones(dv))
        self.out_proj = runtime.matrix(tensors["out_proj"])
        self.position = None
        if spec.position is not None:
            if not isinstance(spec.position, RopeSpec) or spec.position.pairing != "half" or spec.position.rotary_dim > dk:
                raise ValueError("linear attention rotates up to key_dim channels of q and k, in halves")
            if spec.decay == "forget" or spec.query_activation != "identity":
                raise ValueError("a rotation with keys made from the forget gate or an activation on q is not supported")
            self.position = build_part(spec.position, {}, runtime)
        scale = dk ** -0.5
        self.query_scale = scale if spec.scaled == "query" else 1.0
        self.key_scale = scale if spec.scaled == "key" else 1.0

    @classmethod
    def tensor_decls(cls, spec: LinearAttentionSpec) -> dict[str, TensorDecl]:
        heads, dk, dv = spec.num_heads, spec.key_dim, spec.value_dim
        decls = {
            "q_proj": TensorDecl((heads * dk, spec.model_dim)),
            "v_proj": TensorDecl((heads * dv, spec.model_dim)),
            "out_proj": TensorDecl((spec.model_dim, heads * dv)),
        }
        if spec.decay == "forget":
            decls["forget_proj"] = TensorDecl((heads * dk, spec.model_dim))
            decls["forget_bias"] = TensorDecl((heads * dk,), role="vector")
            decls["lower"] = TensorDecl((heads * dk,), role="vector", init="zeros")
        else:
            decls["k_proj"] = TensorDecl((heads * dk, spec.model_dim))
        if spec.gate_activation != "none":
            decls["gate_proj"] = TensorDecl((heads * dv, spec.model_dim))
        if spec.decay == "channel":
            decls["decay_down"] = TensorDecl((spec.decay_rank, spec.model_dim))
            decls["decay_up"] = TensorDecl((heads * dk, spec.decay_rank))
            decls["decay_bias"] = TensorDecl((heads * dk,), role="vector")
        if spec.norm_weight:
            decls["out_norm"] = TensorDecl((dv,), role="vector", init="ones")
        return decls

    def cache_need(self) -> CacheNeed | None:
        spec = self.spec
        return SlotStateNeed(shape=(spec.num_heads, spec.key_dim, spec.value_dim), dtype=torch.float32)

    # Long portions run in chunks side by side (the plan the gated delta rule's layers make, shared with them; one of shorter chunks where
    # the decay is one fixed number per head): which rows belong to which chunk depends on the portions' lengths only.
    step_plan_uses_context = False

    def step_plan_key(self) -> object:
        return ("gated_delta", *self._chunking())

    def _chunking(self) -> tuple[int, int]:
        """``(tokens a chunk, tokens from which on a portion is cut into chunks)``."""
        if self.spec.decay == "fixed":
            return ops.RETENTION_CHUNK_TOKENS, ops.RETENTION_LONG_PORTION
        return ops.GDR_CHUNK_TOKENS, ops.GDR_LONG_PORTION

    def plan_step(self, segments: HostSegments) -> dict[str, np.ndarray]:
        return ops.gated_delta_chunk_plan(segments.start, segments.length, *self._chunking())

    can_accumulate = True
    can_defer = True
    can_fork = True

    def forward(self, x: torch.Tensor, step: StepInputs, cache: SlotStateView, residual: torch.Tensor | None = None,  # type: ignore[override]
                defer: bool = False) -> "torch.Tensor | ops.SlicedSum | None":
        spec = self.spec
        if not cache.owns:
            raise ValueError("a linear-attention layer cannot read another layer's state")
        status = self.runtime.status
        lists, host_lists = step.plan_of(self)
        chunk_plan = dict(lists, num_chunks=host_lists["chunk_start"].size, num_long=host_lists["long_table"].size // 3, num_direct=host_lists["direct"].size,
                          chunk_tokens=self._chunking()[0])
        proj = ops.linear(x, self.in_proj, status=status)
        logits = proj[:, self.forget_offset :] if self.forget_offset is not None else None
        if self.decay_down is not None:
            logits = ops.linear(ops.linear(x, self.decay_down, status=status), self.decay_up, status=status)
        read_out = ops.linear_attention(
            proj,
            cache.state,
            num_heads=spec.num_heads,
            key_dim=spec.key_dim,
            value_dim=spec.value_dim,
            decay_logits=logits,
            decay_bias=self.decay_bias,
            fixed_decay=self.fixed_decay,
            tau=spec.tau,
            query_scale=self.query_scale,
            key_scale=self.key_scale,
            norm_weight=self.norm_weight,
            norm_eps=spec.norm_eps,
            gate_offset=self.gate_offset,
            gate_activation=spec.gate_activation if self.gate_offset is not None else "silu",
            lower=self.lower,
            query_silu=spec.query_activation == "silu",
            segment_start=step.segment_start,
            segment_length=step.segment_length,
            segment_slot=cache.segment_slot,
            segments=step.segments,
            status=status,
            chunk_plan=chunk_plan,
            inv_freq=self.position.inv_freq if self.position is not None else None,
            positions=step.positions,
            turn_scale=self.position.magnitude if self.position is not None else 1.0,
        )
        if residual is not None:
            return ops.linear_accumulate(read_out, self.out_proj, residual, status=status)
        if defer:
            return ops.linear_pending(read_out, self.out_proj, status=status)
        return ops.linear(read_out, self.out_proj, status=status)
