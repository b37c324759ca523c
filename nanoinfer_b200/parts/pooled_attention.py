"""Attention over a window of tokens and, behind it, over one pooled key and value for every block of tokens.

q = W_q h, k = W_k h (with biases where ``bias``), a short causal convolution over time on every channel of both (``taps`` >
0), and then, with ``qk_norm``, every head over its root mean square (no weight).  There is no value projection: a key head as
it leaves the convolution, ahead of the norm, is the value head.  No rotation.

Position i sees the last ``window`` positions (0: all), and with ``pool`` = P > 0 one key and one value for each block of
positions bP .. bP + P - 1 that lies wholly behind the window (bP + P - 1 <= i - window): the means of the block's keys and
values as the cache holds them.  Positions that have left the window and whose block has not are not seen.  All scores
(q . k) * ``scale`` share one softmax, which with ``learned_sink`` has one more term exp(sink_h) in its denominator.  With
``element_gate`` the heads' outputs are multiplied element by element with sigmoid(W_g h) ahead of W_o.

A pooled row is written by the row that ends its block, from the keys of the step and of the cache, into pages of its own
(``KVCacheSpec.pool``), so the pages of positions go back behind the window like any window's.  One product makes
[q | k | gate] as 32-bit floats; one kernel the convolution, the norms, the cast, the cache write and the pooled rows
(csrc/conv_pool_append.cu); then the attention kernels with pooled blocks, sinks and gate as options."""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .attention import AttentionPlan, _round_up
from .base import (MATRIX, VECTOR, KVCacheSpec, KVCacheView, Mixer, ParamSpec, StateSpec, StepContext, StepLimits, TwoProducts,
                   Workspace, register_mixer)


@register_mixer("pooled_attention")
class PooledAttention(TwoProducts, Mixer):
    capture_safe = True

    def __init__(self, width: int, n_head: int, n_kv_head: int, head_dim: int, scale: float, eps: float, window: int = 0,
                 pool: int = 0, taps: int = 0, bias: bool = True, qk_norm: bool = True, learned_sink: bool = True,
                 element_gate: bool = True):
        if n_head <= 0 or n_kv_head <= 0 or n_head % n_kv_head:
            raise ValueError(f"n_head {n_head} must be a positive multiple of n_kv_head {n_kv_head}")
        if head_dim <= 0 or window < 0 or pool < 0 or taps < 0:
            raise ValueError("pooled_attention: sizes must be positive, window, pool and taps not negative")
        if pool > 0 and window <= 0:
            raise ValueError("pooled_attention: pooled blocks lie behind a window")
        self.cache_dim = _round_up(head_dim, 16)
        if self.cache_dim > 256:
            raise ValueError(f"pooled_attention: heads of {head_dim} values do not fit a cached row of 256")
        self.width, self.n_head, self.n_kv_head, self.head_dim = int(width), int(n_head), int(n_kv_head), int(head_dim)
        self.scale, self.eps, self.window, self.pool = float(scale), float(eps), int(window), int(pool)
        #: (no convolution is a convolution of one tap with weight 1)
        self.taps, self.conv = max(int(taps), 1), taps > 0
        self.bias, self.qk_norm = bool(bias), bool(qk_norm)
        self.learned_sink, self.element_gate = bool(learned_sink), bool(element_gate)
        self.n_q, self.n_k = self.n_head * self.head_dim, self.n_kv_head * self.head_dim
        self.channels = self.n_q + self.n_k
        self.gate_off = _round_up(self.channels, 8)
        self.n_in = self.gate_off + (_round_up(self.n_q, 8) if self.element_gate else 0)
        self.n_inner = self.n_head * self.cache_dim
        self.state_floats = _round_up((self.taps - 1) * self.channels, 4)

    def param_specs(self) -> List[ParamSpec]:
        c = self.width
        specs = [ParamSpec("q_weight", (self.n_q, c), MATRIX), ParamSpec("k_weight", (self.n_k, c), MATRIX),
                 ParamSpec("out_weight", (c, self.n_q), MATRIX)]
        if self.bias:
            specs += [ParamSpec("q_bias", (self.n_q,), VECTOR), ParamSpec("k_bias", (self.n_k,), VECTOR),
                      ParamSpec("out_bias", (c,), VECTOR)]
        if self.conv:
            specs += [ParamSpec("q_conv", (self.n_q, self.taps), VECTOR), ParamSpec("k_conv", (self.n_k, self.taps), VECTOR)]
        if self.learned_sink:
            specs.append(ParamSpec("sink", (self.n_head,), VECTOR))
        if self.element_gate:
            specs.append(ParamSpec("gate_weight", (self.n_q, c), MATRIX))
        return specs

    def kv_spec(self) -> Optional[KVCacheSpec]:
        return KVCacheSpec(self.n_kv_head, self.cache_dim, self.window, pool=self.pool)

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.state_floats,), torch.float32) if self.state_floats else None

    def step_planner(self):
        return "causal_attention", AttentionPlan

    def flops_per_key(self) -> float:
        return 4.0 * self.n_q

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        p = self.params
        self.stack_input([("q", 0), ("k", self.n_q)] + ([("gate", self.gate_off)] if self.element_gate else []), self.width)
        w = p["out_weight"]
        if self.cache_dim == self.head_dim:
            self.w_out = w
        else:                       # heads of the cache's size: zero columns where a head is shorter
            wo = torch.zeros(self.width, self.n_head, self.cache_dim, dtype=w.dtype, device=w.device)
            wo[:, :, :self.head_dim] = w.view(self.width, self.n_head, self.head_dim)
            self.w_out = wo.view(self.width, self.n_inner)
            p["out_weight"] = wo[:, :, :self.head_dim]
        self.b_out = p.get("out_bias")
        # by tap, so that neighbouring channels lie side by side
        self.conv_w = torch.cat([p["q_conv"], p["k_conv"]], 0).t().contiguous() if self.conv else \
            torch.ones(1, self.channels, dtype=torch.float32, device=w.device)

    def rebase(self, w_in, b_in, w_out) -> None:
        super().rebase(w_in, b_in, w_out)
        self.params["out_weight"] = self.w_out.unflatten(1, (self.n_head, self.cache_dim))[:, :, :self.head_dim]

    def reserve(self, workspace: Workspace, limits: StepLimits) -> None:
        self.reserve_products(workspace, limits)
        workspace.reserve("attention.q", limits.max_rows * self.n_inner, self.dtype)
        ops.attention_decode_reserve(workspace, self.n_head, self.cache_dim)

    def forward(self, xn: torch.Tensor, x: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView],
                state: Optional[torch.Tensor], writes_cache: bool = True) -> None:
        self.run_alone(xn, x, ctx, cache, state, writes_cache, names=("qkv", "attn_proj"))

    def inner(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView] = None,
              state: Optional[torch.Tensor] = None, writes_cache: bool = True) -> None:
        if cache is None or not writes_cache:
            raise ValueError("pooled_attention needs a paged cache of its own")
        if self.state_floats and state is None:
            raise ValueError("pooled_attention: the convolution needs a state slot tensor")
        ws = ctx.workspace
        q = ws.get("attention.q", (ctx.max_rows, self.n_inner), self.dtype)
        ops.conv_pool_append(proj, self.taps, self.conv_w, state, self.n_head, self.n_kv_head, self.head_dim, self.qk_norm,
                             self.eps, self.pool, ctx, q, cache.layer, cache.block_table, cache.pool_table)
        plan = ctx.plans.get("causal_attention")
        if plan is None:
            plan = ctx.plans["causal_attention"] = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0,
                                                                 device=proj.device)
        extras = ops.AttnExtras(
            sinks=self.params.get("sink"), gate=proj[:, self.gate_off:self.gate_off + self.n_q] if self.element_gate else None,
            gate_dim=self.head_dim if self.element_gate else 0, pool=self.pool, pool_table=cache.pool_table)
        ops.pooled_attention(q, cache.layer, out, cache.block_table, ctx, self.n_head, self.head_dim, self.scale, self.window,
                             plan, extras)
