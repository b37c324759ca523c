"""The minimal gated recurrent unit: a gated recurrence whose gate and candidate read the current token only, so that
every channel of its state is a linear recurrence of its own.

z = sigmoid(W_z h + b_z), u = W_x h + b_x, both of size ``inner``; the candidate c is u + 1/2 where u >= 0 and sigmoid(u)
where u < 0; element by element S <- (1 - z) S + z c, and the mixer's result is W_o (S * silu(W_g h)).

What a request keeps is S, one 32-bit float a channel, in its state slot.  Gates, candidates, the recurrence and the
product with the output gate are 32-bit: the fused projection [z | u | g] leaves 32-bit floats.  The recurrence runs cut
in time (``csrc/min_gru.cu``); the device's work is shaped by the step's shape alone, so steps are captured in graphs."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .base import (MATRIX, VECTOR, KVCacheView, Mixer, ParamSpec, StateSpec, StepContext, StepLimits, TwoProducts, Workspace,
                   register_mixer)


@register_mixer("min_gru")
class MinGRU(TwoProducts, Mixer):
    capture_safe = True

    def __init__(self, width: int, inner: int):
        if width <= 0 or inner <= 0:
            raise ValueError("min_gru: sizes must be positive")
        self.width, self.n_inner = int(width), int(inner)
        self.offsets = (0, self.n_inner, 2 * self.n_inner)
        self.n_in = -(-3 * self.n_inner // 8) * 8

    def param_specs(self) -> List[ParamSpec]:
        n, c = self.n_inner, self.width
        return [ParamSpec("z_weight", (n, c), MATRIX), ParamSpec("z_bias", (n,), VECTOR), ParamSpec("x_weight", (n, c), MATRIX),
                ParamSpec("x_bias", (n,), VECTOR), ParamSpec("g_weight", (n, c), MATRIX), ParamSpec("out_weight", (c, n), MATRIX)]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.n_inner,), torch.float32)

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        self.stack_input(tuple(zip(("z", "x", "g"), self.offsets)), self.width)
        self.w_out = self.params["out_weight"]

    def reserve(self, workspace: Workspace, limits: StepLimits) -> None:
        self.reserve_products(workspace, limits)

    def forward(self, xn: torch.Tensor, x: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView],
                state: Optional[torch.Tensor], writes_cache: bool = True) -> None:
        self.run_alone(xn, x, ctx, cache, state, writes_cache, names=("scan_in", "scan_proj"))

    def inner(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView] = None,
              state: Optional[torch.Tensor] = None, writes_cache: bool = True) -> None:
        if state is None:
            raise ValueError("min_gru needs a state slot tensor")
        ops.min_gru(proj, self.offsets, self.n_inner, state, ctx, out)
