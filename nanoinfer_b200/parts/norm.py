"""LayerNorm: mean and biased variance in two passes, rstd = 1/sqrt(var + eps), then
scale and shift (reference: crates/core/src/kernels/reference.rs:42-51).  The eps is a
parameter; the reference has it as a constant (crates/core/src/config.rs:20-21)."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .base import INIT_NORMAL, INIT_ONE_PLUS_NORMAL, VECTOR, Norm, ParamSpec, register_norm


@register_norm("layernorm")
class LayerNorm(Norm):
    def __init__(self, width: int, eps: float):
        self.width, self.eps = int(width), float(eps)

    def param_specs(self) -> List[ParamSpec]:
        return [
            ParamSpec("weight", (self.width,), VECTOR, INIT_ONE_PLUS_NORMAL),
            ParamSpec("bias", (self.width,), VECTOR, INIT_NORMAL),
        ]

    def reserve(self, workspace, limits) -> None:
        # where a product cannot fold the norm into its own kernel it normalises into this buffer
        workspace.reserve("norm.fallback", limits.max_rows * self.width, limits.dtype)

    def as_input(self, x: torch.Tensor, ctx, dtype: torch.dtype, rows: Optional[torch.Tensor] = None):
        """This norm applied to the residual stream, in the form a matrix product can take as its
        activations (the product then normalises the rows itself where it can)."""
        return ops.NormInput(x, self.params["weight"], self.params["bias"], self.eps, ctx.workspace, dtype,
                             rows=rows, max_rows=0 if rows is not None else ctx.max_rows)

    def forward(self, x: torch.Tensor, out: torch.Tensor, n_rows: int,
                rows: Optional[torch.Tensor] = None) -> None:
        ops.layernorm(x, self.params["weight"], self.params["bias"], self.eps, out, n_rows, rows)


@register_norm("rmsnorm")
class RMSNorm(Norm):
    """x / sqrt(mean(x^2) + eps) * weight, the eps inside the root; statistics in 32-bit.  ``one_plus``: the
    checkpoint stores the weight around zero and the norm multiplies by 1 + w; the one is added once, after
    loading, in 32-bit, so that every kernel sees a plain weight."""

    def __init__(self, width: int, eps: float, one_plus: bool = False):
        self.width, self.eps, self.one_plus = int(width), float(eps), bool(one_plus)
        self._shifted = False

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("weight", (self.width,), VECTOR, INIT_NORMAL if self.one_plus else INIT_ONE_PLUS_NORMAL)]

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        if self.one_plus and not self._shifted:
            self.params["weight"] = self.params["weight"] + 1.0
            self._shifted = True

    def forward(self, x: torch.Tensor, out: torch.Tensor, n_rows: int,
                rows: Optional[torch.Tensor] = None) -> None:
        ops.rmsnorm(x, self.params["weight"], self.eps, out, n_rows, rows)


@register_norm("scalar_rmsnorm")
class ScalarRMSNorm(RMSNorm):
    """An RMS norm whose weight is ONE number for all coordinates: x / sqrt(mean(x^2) + eps) * g.  The checkpoint's
    tensor is a scalar; after loading it is spread over the width, so that every kernel that takes an RMS norm's
    weight takes this one too."""

    def __init__(self, width: int, eps: float):
        super().__init__(width, eps, one_plus=False)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("weight", (), VECTOR, INIT_ONE_PLUS_NORMAL)]

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        w = self.params["weight"]
        if w.numel() == 1:
            self.scalar = w.reshape(())
            self.params["weight"] = w.reshape(1).expand(self.width).contiguous()


@register_norm("grouped_rmsnorm")
class GroupedRMSNorm(Norm):
    """An RMS norm in groups: the vector is cut into ``groups`` equal consecutive parts, each part is divided by its own
    sqrt(mean(part^2) + eps), and the whole is multiplied by one weight of the vector's size; statistics in 32-bit.  One
    group is the plain RMS norm.  ``add`` (a 32-bit vector) and ``add_rows`` (a 32-bit row for each) are added to the stream
    first, in the same kernel.  ``one_plus``: as in ``rmsnorm``."""

    takes_vector = True

    def __init__(self, width: int, eps: float, groups: int = 1, one_plus: bool = False):
        if groups <= 0 or width % groups:
            raise ValueError(f"grouped_rmsnorm: {groups} groups do not divide a width of {width}")
        self.width, self.eps, self.groups, self.one_plus = int(width), float(eps), int(groups), bool(one_plus)
        self._shifted = False

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec("weight", (self.width,), VECTOR, INIT_NORMAL if self.one_plus else INIT_ONE_PLUS_NORMAL)]

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        if self.one_plus and not self._shifted:
            self.params["weight"] = self.params["weight"] + 1.0
            self._shifted = True

    def reserve(self, workspace, limits) -> None:
        if self.groups == 1:      # (what ``as_input`` falls back to)
            workspace.reserve("norm.fallback", limits.max_rows * self.width, limits.dtype)

    def as_input(self, x: torch.Tensor, ctx, dtype: torch.dtype, rows: Optional[torch.Tensor] = None):
        """One group: this norm in the form a matrix product can take as its activations."""
        if self.groups != 1:
            return None
        return ops.NormInput(x, self.params["weight"], None, self.eps, ctx.workspace, dtype, rows=rows,
                             max_rows=0 if rows is not None else ctx.max_rows)

    def forward(self, x: torch.Tensor, out: torch.Tensor, n_rows: int, rows: Optional[torch.Tensor] = None,
                add: Optional[torch.Tensor] = None, add_rows: Optional[torch.Tensor] = None) -> None:
        ops.group_norm(x, self.params["weight"], self.groups, self.eps, out, n_rows, rows, add, add_rows)
