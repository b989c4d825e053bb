"""The decoder: embedding, the scheduled blocks, final norm and LM head
(``lalamo/modules/decoder.py:220-317``, ``lalamo/modules/transformer.py:95-263``).

It runs the tokens of one :class:`~lalamo_b200.parts.base.StepInputs` and returns 32-bit logits
at the wanted rows only.
"""

from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from ..config.plan import ModelPlan
from .base import BorrowedKVNeed, CacheNeed, CacheView, CompositeNeed, Norm, Part, Runtime, StepInputs, TensorDecl, build_part, part_type
from .embedding import Embedding, Head
from .block import Block, block_tensor_decls, build_block

__all__ = ["DecoderModel", "plan_tensor_decls"]

TensorKey = tuple[tuple, str]


def plan_tensor_decls(plan: ModelPlan) -> dict[TensorKey, TensorDecl]:
    """Every tensor of the model: ``(path of the part, local name) -> declaration``."""
    decls: dict[TensorKey, TensorDecl] = {}
    for local, decl in part_type(plan.embedding).tensor_decls(plan.embedding).items():
        decls[(("embedding",), local)] = decl
    for index, layer in enumerate(plan.layers):
        for (role, local), decl in block_tensor_decls(layer).items():
            decls[(("layers", index, role), local)] = decl
    if plan.stream_mix is not None:
        for local, decl in part_type(plan.stream_mix).tensor_decls(plan.stream_mix).items():
            decls[(("stream_mix",), local)] = decl
    for local, decl in part_type(plan.final_norm).tensor_decls(plan.final_norm).items():
        decls[(("final_norm",), local)] = decl
    for local, decl in part_type(plan.head).tensor_decls(plan.head).items():
        decls[(("lm_head",), local)] = decl
    return decls


def _borrows(need: CacheNeed | None) -> bool:
    """Whether some part of the need is read from another schedule entry's cache."""
    if isinstance(need, CompositeNeed):
        return any(_borrows(part) for part in need.needs)
    return isinstance(need, BorrowedKVNeed)


class DecoderModel:
    def __init__(self, plan: ModelPlan, tensors: Mapping[TensorKey, torch.Tensor], runtime: Runtime) -> None:
        self.plan = plan
        self.runtime = runtime
        embedding_tensors = {local: tensor for (path, local), tensor in tensors.items() if path == ("embedding",)}
        self.embedding: Embedding = build_part(plan.embedding, embedding_tensors, runtime)  # type: ignore[assignment]
        head_tensors = {local: tensor for (path, local), tensor in tensors.items() if path == ("lm_head",)}
        if getattr(plan.head, "tied", False):
            head_tensors = {**head_tensors, "weight": self.embedding.weight}
        self.head: Head = build_part(plan.head, head_tensors, runtime)  # type: ignore[assignment]
        self.blocks: list[Block] = []
        for index, layer in enumerate(plan.layers):
            block_tensors = {
                (path[2], local): tensor
                for (path, local), tensor in tensors.items()
                if len(path) == 3 and path[0] == "layers" and path[1] == index
            }
            self.blocks.append(build_block(layer, block_tensors, runtime))
        self.stream_mix = None
        if plan.stream_mix is not None:
            mix_tensors = {local: tensor for (path, local), tensor in tensors.items() if path == ("stream_mix",)}
            self.stream_mix = build_part(plan.stream_mix, mix_tensors, runtime)
        final_tensors = {local: tensor for (path, local), tensor in tensors.items() if path == ("final_norm",)}
        self.final_norm: Norm = build_part(plan.final_norm, final_tensors, runtime)  # type: ignore[assignment]
        self.sum_of_streams = runtime.vector(torch.ones(plan.streams)) if plan.streams > 0 else None

    def cache_needs(self) -> list[CacheNeed | None]:
        """For each schedule entry the cache it needs (``None``: none of its own; an entry that borrows only keys and values says so
        inside its need)."""
        needs: list[CacheNeed | None] = []
        for entry in self.plan.schedule:
            need = self.blocks[entry.layer].cache_need()
            needs.append(need if entry.cache_from is None or _borrows(need) else None)
        return needs

    def step_planners(self) -> list[Part]:
        """The parts that plan work on the host for every step (one per plan key)."""
        planners: dict[object, Part] = {}
        for entry in self.plan.schedule:
            block = self.blocks[entry.layer]
            parts = list(block.parts())
            while parts:
                part = parts.pop(0)
                parts.extend(getattr(part, "sub_parts", list)())   # a part made of parts (mixers side by side)
                if type(part).plan_step is not Part.plan_step:
                    planners.setdefault(part.step_plan_key(), part)
        return list(planners.values())

    def weight_bytes(self) -> int:
        """Bytes of every weight a step reads once: all parts' tensors and the LM head (of the
        embedding table a step reads only its tokens' rows).  For roofline arithmetic."""
        seen: dict[int, int] = {}

        def visit(obj: object, depth: int = 0) -> None:
            for value in vars(obj).values():
                if isinstance(value, torch.Tensor):
                    if value.is_cuda and value.data_ptr() != self.runtime.status.data_ptr():
                        seen[value.data_ptr()] = value.numel() * value.element_size()
                elif isinstance(value, (Part, Block)) and depth < 4:
                    visit(value, depth + 1)
                elif isinstance(value, list) and depth < 4:
                    for item in value:
                        if isinstance(item, Part):
                            visit(item, depth + 1)

        for entry in self.plan.schedule:
            visit(self.blocks[entry.layer])
        visit(self.final_norm)
        visit(self.head)
        if self.stream_mix is not None:
            visit(self.stream_mix)
        return sum(seen.values())

    def forward(self, step: StepInputs, caches: list[CacheView | None]) -> torch.Tensor:
        runtime = self.runtime
        residual = self.embedding.forward(step.token_ids, step.tokens, step.positions)
        if self.plan.streams > 0:
            residual = ops.ResidualStreams(residual, self.plan.streams)   # all streams equal: one copy is enough until something is written
        pending: torch.Tensor | None = None
        for position, entry in enumerate(self.plan.schedule):
            if entry.add_embedding:
                if pending is not None:
                    ops.residual_add(residual, pending)
                    pending = None
                step.carry.clear()   # what a block left for its successor described the stream before this sum
                self.embedding.add_to(residual, step.token_ids)
            if entry.mix_embedding:
                if pending is not None:
                    ops.residual_add(residual, pending)
                    pending = None
                step.carry.clear()   # as above: the stream is another one from here on
                residual = self.stream_mix.forward(residual, self.embedding, step.token_ids)
            # the norm the next block begins with, for a block that can compute it on its way out
            following = self.plan.schedule[position + 1] if position + 1 < len(self.plan.schedule) else None
            step.carry["next_norm"] = None if following is None or following.add_embedding or following.mix_embedding else getattr(self.blocks[following.layer], "first_norm", None)
            pending = self.blocks[entry.layer].forward(residual, pending, step, caches[position])
        if step.wanted == 0:
            return runtime.empty(0, self.plan.vocab_size, dtype=torch.float32)
        if self.sum_of_streams is not None:
            normed = self.final_norm.streams_forward(residual, pending, self.sum_of_streams, keep=False, rows=step.want_rows, num_rows=step.wanted)
        else:
            normed = self.final_norm.residual_forward(residual, pending, step.want_rows, step.wanted)
        return self.head.forward(normed)
