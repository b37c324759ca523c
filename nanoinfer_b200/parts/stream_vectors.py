"""Vectors added to the residual stream ahead of runs of a schedule: a looped stack of layers is told by such a vector
which of its passes it is in."""
from __future__ import annotations

from typing import List

import torch

from .base import INIT_NORMAL, VECTOR, ParamSpec, StreamVectors, register_stream_vectors


@register_stream_vectors("stream_vector_table")
class StreamVectorTable(StreamVectors):
    """``count`` learned vectors of the model's width, 32-bit."""

    def __init__(self, count: int, width: int):
        if count <= 0 or width <= 0:
            raise ValueError("stream_vector_table: sizes must be positive")
        self.count, self.width = int(count), int(width)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("table", (self.count, self.width), VECTOR, INIT_NORMAL)]

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        # (the kernel that adds one reads 16 bytes at a time: every vector starts on its own boundary)
        self.vectors = [self.params["table"][i].clone() for i in range(self.count)]

    def vector(self, i: int) -> torch.Tensor:
        return self.vectors[i]
