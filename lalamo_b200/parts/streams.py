"""What a block on parallel residual streams is made of besides its mixer and feed-forward: the connection through which a
sublayer reads the streams and writes back into them (hyper-connections), and the causal convolution that a sublayer's
input may pass first.  The reading, the writing and the norm in between are one kernel (``ops.stream_step``); for steps of
single tokens it runs the input convolution as well."""

from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from ..config.plan import InputConvSpec, StreamConnectionSpec
from .base import CacheNeed, Part, Runtime, SlotStateNeed, SlotStateView, StepInputs, TensorDecl, register_part

__all__ = ["InputConv", "StreamConnection"]


@register_part(StreamConnectionSpec)
class StreamConnection(Part):
    """``read [streams]``, ``mix [from, to]`` and ``write [streams]`` in 32-bit."""

    def __init__(self, spec: StreamConnectionSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().__init__(spec, tensors, runtime)
        if not 1 <= spec.streams <= ops.MAX_STREAMS:
            raise ValueError(f"1 to {ops.MAX_STREAMS} residual streams are supported, not {spec.streams}")
        self.read = runtime.vector(tensors["read"])
        self.mix = runtime.vector(tensors["mix"])
        self.write = runtime.vector(tensors["write"])

    @classmethod
    def tensor_decls(cls, spec: StreamConnectionSpec) -> dict[str, TensorDecl]:
        return {
            "read": TensorDecl((spec.streams,), role="vector", init="ones"),
            "mix": TensorDecl((spec.streams, spec.streams), role="vector", init="identity"),
            "write": TensorDecl((spec.streams,), role="vector", init="ones"),
        }


@register_part(InputConvSpec)
class InputConv(Part):
    """``h + conv(h)`` with the last ``taps - 1`` inputs of every request kept in a slot (in the activation type)."""

    def __init__(self, spec: InputConvSpec, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().__init__(spec, tensors, runtime)
        if not 1 <= spec.taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"a convolution has 1 to {ops.CONV_MAX_TAPS} taps, not {spec.taps}")
        self.weight = runtime.vector(tensors["weight"].reshape(spec.model_dim, spec.taps))

    @classmethod
    def tensor_decls(cls, spec: InputConvSpec) -> dict[str, TensorDecl]:
        return {"weight": TensorDecl((spec.model_dim, spec.taps), role="vector")}

    def cache_need(self) -> CacheNeed | None:
        return SlotStateNeed(shape=(self.spec.taps - 1, self.spec.model_dim)) if self.spec.taps > 1 else None

    def fused(self, step: StepInputs, cache: SlotStateView | None) -> dict | None:
        """The convolution as an argument of ``ops.stream_step``, which runs it where every portion is one token."""
        if step.segments != step.tokens:
            return None
        return dict(weight=self.weight, state=cache.state if cache is not None else None, token_segment=step.token_segment,
                    segment_slot=step.segment_slot, status=self.runtime.status)

    def forward(self, h: torch.Tensor, step: StepInputs, cache: SlotStateView | None) -> torch.Tensor:
        return ops.causal_conv(h, cache.state if cache is not None else None, self.weight, add_input=True, segment_start=step.segment_start,
                               segment_length=step.segment_length, segment_slot=step.segment_slot, segments=step.segments, max_length=step.max_segment_length,
                               status=self.runtime.status)
