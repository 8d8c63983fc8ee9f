"""Token embedding (a row gather with no scaling, upstream src/tinyserve/model.py:192) and
the output head (``logits = float32(x W^T)`` with ``W`` the embedding table when tied,
src/tinyserve/model.py:129-130,208).
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..kernels import ops
from .base import (EMBEDDINGS, EVERY_STEP, HEADS, STREAM_INPUTS, Part, ResidualStream, StepContext, StreamInput,
                   TensorSpec)


class TokenEmbedding(Part):
    recordable = EVERY_STEP

    def __init__(self, name: str, vocab_size: int, hidden_size: int, scale: float = 1.0) -> None:
        # scale: the gathered row is multiplied by it on its way into the 32-bit stream
        self.name, self.vocab_size, self.hidden_size = name, int(vocab_size), int(hidden_size)
        self.scale = float(scale)
        self.table: torch.Tensor | None = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        return [TensorSpec(prefix + self.name, (self.vocab_size, self.hidden_size))]

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.table = tensors[prefix + self.name]

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """The 32-bit residual stream ``[T, hidden]`` of this step's tokens."""
        out = ctx.arena.take((ctx.num_tokens, self.hidden_size), torch.float32)
        ops.embed(ctx.tokens, self.table, out, self.scale)
        return out


class PositionedEmbedding(Part):
    """Token embedding plus a learned position row, optionally followed by an RMS norm with a plain
    weight: ``x = table[token] * scale + positions[p]``, then ``x / sqrt(mean(x^2) + eps) * w``. One
    kernel writes the result into the 32-bit stream. Positions count from 0 in each request; a
    position beyond the table gives a row of NaN."""

    recordable = EVERY_STEP

    def __init__(self, name: str, vocab_size: int, hidden_size: int, position_name: str, max_positions: int,
                 norm_name: str | None = None, eps: float = 1e-6, scale: float = 1.0) -> None:
        self.name, self.vocab_size, self.hidden_size = name, int(vocab_size), int(hidden_size)
        self.position_name, self.max_positions = position_name, int(max_positions)
        self.norm_name, self.eps, self.scale = norm_name, float(eps), float(scale)
        self.table = self.positions = self.norm_w = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        specs = [TensorSpec(prefix + self.name, (self.vocab_size, self.hidden_size)),
                 TensorSpec(prefix + self.position_name, (self.max_positions, self.hidden_size))]
        if self.norm_name is not None:
            specs.append(TensorSpec(prefix + self.norm_name, (self.hidden_size,), init="one_plus_normal"))
        return specs

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.table, self.positions = tensors[prefix + self.name], tensors[prefix + self.position_name]
        self.norm_w = None if self.norm_name is None else tensors[prefix + self.norm_name]

    def forward(self, ctx: StepContext) -> torch.Tensor:
        out = ctx.arena.take((ctx.num_tokens, self.hidden_size), torch.float32)
        ops.embed_pos_norm(ctx.tokens, ctx.positions, self.table, self.positions, self.norm_w, self.eps, out, self.scale)
        return out


class SinusoidalEmbedding(Part):
    """Token embedding plus a fixed vector of the position: ``x = table[token] * scale``, to which column ``2 i`` adds
    ``sin(p * base^(-2 i / hidden))`` and column ``2 i + 1`` the cosine of the same angle. Positions count from 0 in each
    request. Angles are formed in 64-bit and reduced before they are rounded; one kernel writes the 32-bit stream."""

    recordable = EVERY_STEP

    def __init__(self, name: str, vocab_size: int, hidden_size: int, scale: float = 1.0, base: float = 10000.0) -> None:
        if not base > 0:
            raise ValueError(f"base={base} must be positive")
        self.name, self.vocab_size, self.hidden_size = name, int(vocab_size), int(hidden_size)
        self.scale, self.base = float(scale), float(base)
        self.table = self.freq = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        return [TensorSpec(prefix + self.name, (self.vocab_size, self.hidden_size))]

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.table = tensors[prefix + self.name]
        pairs = torch.arange((self.hidden_size + 1) // 2, dtype=torch.float64)
        self.freq = (self.base ** (-2.0 * pairs / self.hidden_size)).to(self.table.device)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        out = ctx.arena.take((ctx.num_tokens, self.hidden_size), torch.float32)
        ops.embed_pos_norm(ctx.tokens, ctx.positions, self.table, None, None, 0.0, out, self.scale, freq=self.freq)
        return out


class LMHead(Part):
    recordable = EVERY_STEP

    def __init__(self, name: str, tied: bool, vocab_size: int, hidden_size: int,
                 ignored_when_tied: str | None = None, softcap: float | None = None) -> None:
        # softcap: logits <- softcap * tanh(logits / softcap) after the product (None: no cap)
        if softcap is not None and not softcap > 0:
            raise ValueError(f"softcap must be positive or None, got {softcap}")
        self.softcap = None if softcap is None else float(softcap)
        self.name, self.tied = name, bool(tied)
        self.vocab_size, self.hidden_size = int(vocab_size), int(hidden_size)
        self.ignored_when_tied = ignored_when_tied
        self.weight: torch.Tensor | None = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        # When tied this names the embedding table, which the embedding declares as well;
        # equal declarations are one tensor.
        return [TensorSpec(prefix + self.name, (self.vocab_size, self.hidden_size))]

    def ignorable_tensors(self, prefix: str) -> set[str]:
        # A tied checkpoint may still ship a copy of the table under the head's name.
        return {prefix + self.ignored_when_tied} if self.tied and self.ignored_when_tied else set()

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[prefix + self.name]

    def forward(self, x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        """``x [R, hidden]`` in the model dtype -> ``out [R, vocab]`` float32."""
        ops.gemm(x, self.weight, out)
        if self.softcap is not None:
            ops.softcap(out, self.softcap)
        return out


class PassVector(StreamInput):
    """In front of pass ``index`` of layers that run ``count`` times: row ``index`` of the learned table
    ``name [count, hidden]`` is added to the stream, and with ``add_origin`` the embedding output once more.
    Both are left pending: the pass's first norm adds them in 32-bit in the pass it makes anyway."""

    recordable = EVERY_STEP

    def __init__(self, name: str, hidden_size: int, index: int, count: int, add_origin: bool = False) -> None:
        if not 0 <= index < count:
            raise ValueError(f"pass {index} of {count}")
        self.name, self.hidden_size, self.index, self.count = name, int(hidden_size), int(index), int(count)
        self.needs_origin = bool(add_origin)
        self.vector: torch.Tensor | None = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        return [TensorSpec(prefix + self.name, (self.count, self.hidden_size))]

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.vector = tensors[prefix + self.name][self.index]

    def forward(self, stream: ResidualStream, ctx: StepContext) -> None:
        if stream.extra is not None:
            raise RuntimeError("something is already waiting to be added to the stream")
        stream.extra = (stream.origin if self.needs_origin else None, self.vector)


class PassProjection(StreamInput):
    """In front of a pass of layers that run several times: the stream is replaced by a product of itself beside the
    embedding output, ``x <- W [x; x0]`` (tensor ``name [hidden, 2 * hidden]``, the same for every pass). What is pending on
    the stream is added in 32-bit first; the product's sums are the new 32-bit stream."""

    recordable = EVERY_STEP
    needs_origin = True
    replaces = True

    def __init__(self, name: str, hidden_size: int) -> None:
        self.name, self.hidden_size = name, int(hidden_size)
        self.weight: torch.Tensor | None = None

    def tensor_specs(self, prefix: str) -> list[TensorSpec]:
        return [TensorSpec(prefix + self.name, (self.hidden_size, 2 * self.hidden_size))]

    def bind(self, prefix: str, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[prefix + self.name]

    def forward(self, stream: ResidualStream, ctx: StepContext) -> None:
        if stream.post is not None or stream.second is not None or stream.extra is not None or stream.lanes is not None:
            raise NotImplementedError("a product of the stream behind anything but one plain pending output")
        beside = ctx.arena.take((ctx.num_tokens, 2 * self.hidden_size), ctx.dtype)
        ops.stream_beside(stream.resid, stream.delta, stream.origin, beside)
        ops.gemm(beside, self.weight, stream.resid)
        stream.delta = stream.sumsq = None


STREAM_INPUTS.register("pass_projection", PassProjection)
STREAM_INPUTS.register("pass_vector", PassVector)
EMBEDDINGS.register("token_embedding", TokenEmbedding)
EMBEDDINGS.register("positioned_embedding", PositionedEmbedding)
EMBEDDINGS.register("sinusoidal_embedding", SinusoidalEmbedding)
HEADS.register("lm_head", LMHead)
