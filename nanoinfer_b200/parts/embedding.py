"""Token embedding: x[t] = table[token_t] * scale, written to the 32-bit residual stream; a position
encoding that is a plain table is added in the same kernel
(reference: crates/core/src/stages/blocks.rs:19-27)."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .base import INIT_ONE_PLUS_NORMAL, TABLE, VECTOR, Embedding, ParamSpec, PositionEncoding, StepContext, register_embedding


@register_embedding("token_embedding")
class TokenEmbedding(Embedding):
    def __init__(self, vocab_size: int, width: int, scale: float = 1.0):
        self.vocab_size, self.width, self.scale = int(vocab_size), int(width), float(scale)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("table", (self.vocab_size, self.width), TABLE)]

    def forward(self, ctx: StepContext, x: torch.Tensor, position: Optional[PositionEncoding]) -> None:
        table = position.additive_table() if position is not None else None
        ops.embed(ctx.tokens[:ctx.n_rows], self.params["table"], x, table,
                  ctx.positions if table is not None else None, feedback=ctx.token_feedback, scale=self.scale)
        if position is not None and table is None:
            position.on_embedding(x, ctx)


@register_embedding("normed_token_embedding")
class NormedTokenEmbedding(TokenEmbedding):
    """A token embedding with a norm behind it (an RMS norm in ``groups`` parts, one group being the plain one), in one
    kernel: x[t] = norm(table[token_t] * scale), 32-bit.  A position encoding is added behind the norm."""

    def __init__(self, vocab_size: int, width: int, eps: float, groups: int = 1, scale: float = 1.0):
        super().__init__(vocab_size, width, scale)
        if groups <= 0 or width % groups:
            raise ValueError(f"normed_token_embedding: {groups} groups do not divide a width of {width}")
        self.eps, self.groups = float(eps), int(groups)

    def param_specs(self) -> List[ParamSpec]:
        return super().param_specs() + [ParamSpec("norm", (self.width,), VECTOR, INIT_ONE_PLUS_NORMAL)]

    def forward(self, ctx: StepContext, x: torch.Tensor, position: Optional[PositionEncoding]) -> None:
        if position is not None and position.additive_table() is not None:
            raise ValueError("normed_token_embedding: a position table behind the norm is not built")
        ops.embed_group_norm(ctx.tokens[:ctx.n_rows], self.params["table"], x, self.params["norm"], self.groups, self.eps,
                             feedback=ctx.token_feedback, scale=self.scale)
        if position is not None:
            position.on_embedding(x, ctx)
