"""Differential attention: every head has two attention maps over the same values, and the second is subtracted.

q = W_q h, k = W_k h, v = W_v h (with biases where ``bias``); q is laid out head by head [map 1: dim | map 2: dim], k
likewise for its ``n_kv_head`` heads, v has ``n_kv_head`` heads of ``v_dim``; query head h uses key/value head
h // (n_head / n_kv_head).  With ``qk_norm`` every (head, map) of q and of k is divided by its root mean square over
``dim`` (``eps`` inside the root) and multiplied by a weight of ``dim`` values shared by all heads and maps; then the
rotation (``position``: a ``rotary_halves`` part, on the first dims of every map).  Map t of head h is an attention of
its own: s = (q_t . k_t) * scale, with ``softcap`` > 0 s <- softcap * tanh(s / softcap), softmax over the last ``window``
positions (0: all), a_t = the weighted sum of values.  With
    lambda = exp(sum(lq1 lk1)) - exp(sum(lq2 lk2)) + diff
(one number a layer) the head's output is o = a_1 - lambda a_2, divided by its root mean square over ``v_dim`` (no weight)
and times (1 - diff); then W_o.

The cache knows one key row and one value row a head and position, of max(2 dim, v_dim) values rounded up to 16: a row of
keys holds both maps' side by side, so values are stored and read once.  A query of map t is laid into a row of that size
with zeros in the other map's place, which makes two query heads of it that the attention kernels take as they take any
(2 n_head query heads on n_kv_head key/value heads).  Their results stay 32-bit until the second map is subtracted
(``csrc/differential.cu``).  Scores, softmax, lambda, the subtraction and all norms are 32-bit."""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from ..kernels import ops
from .attention import AttentionPlan, _round_up
from .base import (INIT_ONE_PLUS_NORMAL, MATRIX, VECTOR, KVCacheSpec, KVCacheView, Mixer, ParamSpec, PositionEncoding, StepContext,
                   StepLimits, TwoProducts, Workspace, register_mixer)

MAPS = 2


@register_mixer("differential_attention")
class DifferentialAttention(TwoProducts, Mixer):
    def __init__(self, width: int, n_head: int, n_kv_head: int, head_dim: int, v_dim: int, scale: float, eps: float,
                 diff: float, window: int = 0, softcap: float = 0.0, bias: bool = True, qk_norm: bool = True,
                 position: Optional[PositionEncoding] = None):
        if n_head <= 0 or n_kv_head <= 0 or n_head % n_kv_head:
            raise ValueError(f"n_head {n_head} must be a positive multiple of n_kv_head {n_kv_head}")
        if head_dim <= 0 or v_dim <= 0 or window < 0 or softcap < 0.0:
            raise ValueError("differential_attention: sizes must be positive, window and softcap not negative")
        self.cache_dim = _round_up(max(MAPS * head_dim, v_dim), 16)
        if self.cache_dim > 256:
            raise ValueError(f"differential_attention: two maps of {head_dim} values, or {v_dim} values of a head, do not fit "
                             "a cached row of 256")
        self.width, self.n_head, self.n_kv_head, self.head_dim, self.v_dim = int(width), int(n_head), int(n_kv_head), \
            int(head_dim), int(v_dim)
        self.scale, self.eps, self.diff, self.window, self.softcap = float(scale), float(eps), float(diff), int(window), float(softcap)
        self.bias, self.qk_norm, self.position = bool(bias), bool(qk_norm), position
        rot = getattr(position, "dims", 0)
        if position is not None and (getattr(position, "layout", None) != "halves" or rot > self.head_dim):
            raise ValueError("differential_attention: the position encoding must be rotary_halves with dims <= head_dim")
        self.n_q, self.n_k = self.n_head * MAPS * self.head_dim, self.n_kv_head * MAPS * self.head_dim
        self.n_v, self.n_inner = self.n_kv_head * self.v_dim, self.n_head * self.v_dim
        self.offsets = (0, self.n_q, self.n_q + self.n_k)
        self.n_in = _round_up(self.n_q + self.n_k + self.n_v, 8)
        self.q_dim = self.n_head * MAPS * self.cache_dim

    def param_specs(self) -> List[ParamSpec]:
        c, d = self.width, self.head_dim
        specs = [ParamSpec("q_weight", (self.n_q, c), MATRIX), ParamSpec("k_weight", (self.n_k, c), MATRIX),
                 ParamSpec("v_weight", (self.n_v, c), MATRIX), ParamSpec("out_weight", (c, self.n_inner), MATRIX)]
        specs += [ParamSpec(key, (d,), VECTOR) for key in ("lq1", "lk1", "lq2", "lk2")]
        if self.bias:
            specs += [ParamSpec("q_bias", (self.n_q,), VECTOR), ParamSpec("k_bias", (self.n_k,), VECTOR),
                      ParamSpec("v_bias", (self.n_v,), VECTOR)]
        if self.qk_norm:
            specs += [ParamSpec("q_norm", (d,), VECTOR, INIT_ONE_PLUS_NORMAL), ParamSpec("k_norm", (d,), VECTOR, INIT_ONE_PLUS_NORMAL)]
        return specs

    def kv_spec(self) -> Optional[KVCacheSpec]:
        return KVCacheSpec(self.n_kv_head, self.cache_dim, self.window)

    def step_planner(self):
        return "causal_attention", AttentionPlan

    def flops_per_key(self) -> float:
        return 2.0 * self.n_head * MAPS * (self.head_dim + self.v_dim)

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        p = self.params
        self.stack_input((("q", self.offsets[0]), ("k", self.offsets[1]), ("v", self.offsets[2])), self.width)
        self.w_out = p["out_weight"]
        dot = lambda a, b: float((p[a].double() * p[b].double()).sum())
        self.lam = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.diff

    def reserve(self, workspace: Workspace, limits: StepLimits) -> None:
        self.reserve_products(workspace, limits)
        workspace.reserve("attention.q", limits.max_rows * self.q_dim, self.dtype)
        workspace.reserve("attention.maps", limits.max_rows * self.q_dim, torch.float32)
        ops.attention_decode_reserve(workspace, self.n_head * MAPS, self.cache_dim)

    def forward(self, xn: torch.Tensor, x: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView],
                state: Optional[torch.Tensor], writes_cache: bool = True) -> None:
        self.run_alone(xn, x, ctx, cache, state, writes_cache, names=("qkv", "attn_proj"))

    def inner(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView] = None,
              state: Optional[torch.Tensor] = None, writes_cache: bool = True) -> None:
        if cache is None or not writes_cache:
            raise ValueError("differential_attention needs a paged cache of its own")
        p, ws, pos, H = self.params, ctx.workspace, self.position, self.n_head
        q = ws.get("attention.q", (ctx.max_rows, self.q_dim), self.dtype)
        ops.norm_rope_maps_append(proj, self.offsets, H, self.n_kv_head, MAPS, self.head_dim, self.v_dim, p.get("q_norm"),
                                  p.get("k_norm"), self.eps, pos.dims if pos is not None else 0,
                                  pos.freqs if pos is not None else None, pos.amplitude if pos is not None else 1.0, ctx, q,
                                  cache.layer, cache.block_table)
        maps = ws.get("attention.maps", (ctx.max_rows, self.q_dim), torch.float32)
        plan = ctx.plans.get("causal_attention")
        if plan is None:
            plan = ctx.plans["causal_attention"] = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0,
                                                                 device=proj.device)
        ops.differential_attention(q, cache.layer, maps, out, cache.block_table, ctx, H, self.head_dim, self.v_dim, self.scale,
                                   self.window, self.softcap, self.lam, self.eps, 1.0 - self.diff, plan)
