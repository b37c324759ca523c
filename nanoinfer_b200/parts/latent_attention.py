"""Attention through a low-rank latent shared by all heads.

Queries go through a latent of their own: c_q = rmsnorm(W_dq h) * w, q = W_uq c_q, head by head
[nope_dim unrotated | rot_dim rotated].  Keys and values come from ONE latent per token:
W_dkv h = [c raw (kv_rank) | k_rot raw (rot_dim)], c = rmsnorm(c raw) * w, k_rot rotated by the token's
position and shared by all heads; a head's unrotated key is W_uk[h] c and its value W_uv[h] c.  The cache
holds c and k_rot only (one row of kv_rank + rot_dim per token, one plane, one head).

Scores never build the keys: (q_nope . W_uk[h] c) = (W_uk[h]^T q_nope) . c, so each head's query is
carried into the latent space, every head attends over the same cached rows, and W_uv[h] is applied to
the weighted sum of latents (csrc/latent_attention.cu, csrc/linear_heads.cu).  A layer built with
``own_kv=False`` has no W_dkv and reads the cache of the layer the schedule names, with its own W_uk,
W_uv, queries and window.  Rotation: interleaved pairs (2i, 2i+1) of the first ``rot_dims`` values of the
rotated part or, with ``rot_layout`` "halves", value i with value i + rot_dims / 2; angle = position *
rot_base^(-2i / rot_dims).  ``head_gate``: head h's output is multiplied by sigmoid(W_g h)_h, one number per row
and head; its logits are rows of the down-projections' product (32-bit), and the gate is applied to the head's
weighted sum of latents.  ``element_gate`` instead: W_g has a row for every element of the heads' values, and the heads'
outputs are multiplied by its sigmoid in the product with W_uv.  ``learned_sink``: a number per head whose exponential joins
the softmax's denominator (a key without a value, not scaled).
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .attention import AttentionPlan
from .base import (INIT_ONE_PLUS_NORMAL, MATRIX, VECTOR, KVCacheSpec, KVCacheView, Mixer, ParamSpec, StepContext,
                   StepLimits, TwoProducts, Workspace, register_mixer)


@register_mixer("latent_attention")
class LatentAttention(TwoProducts, Mixer):
    def __init__(self, width: int, n_head: int, nope_dim: int, rot_dim: int, v_dim: int, q_rank: int,
                 kv_rank: int, scale: float, eps: float, window: int = 0, rot_base: float = 10000.0,
                 rot_dims: Optional[int] = None, own_kv: bool = True, rot_layout: str = "pairs", head_gate: bool = False,
                 element_gate: bool = False, learned_sink: bool = False):
        rot_dims = rot_dim if rot_dims is None else rot_dims
        for name, v in (("width", width), ("n_head", n_head), ("v_dim", v_dim), ("q_rank", q_rank),
                        ("kv_rank", kv_rank)):
            if int(v) <= 0:
                raise ValueError(f"latent_attention: {name} must be positive, got {v}")
        if nope_dim < 0 or rot_dim < 0 or nope_dim + rot_dim == 0:
            raise ValueError("latent_attention: a head needs unrotated or rotated query dimensions")
        if rot_dims < 0 or rot_dims > rot_dim or rot_dims % 2:
            raise ValueError(f"latent_attention: rot_dims {rot_dims} must be even and at most rot_dim {rot_dim}")
        if kv_rank > 1024 or window < 0:
            raise ValueError("latent_attention: kv_rank at most 1024, window >= 0")
        self.width, self.n_head, self.nope_dim, self.rot_dim, self.v_dim = int(width), int(n_head), int(nope_dim), int(rot_dim), int(v_dim)
        self.q_rank, self.kv_rank, self.scale, self.eps = int(q_rank), int(kv_rank), float(scale), float(eps)
        self.window, self.rot_base, self.rot_dims, self.own_kv = int(window), float(rot_base), int(rot_dims), bool(own_kv)
        self.qk_dim = self.nope_dim + self.rot_dim
        self.latent_dim = self.kv_rank + self.rot_dim
        if rot_layout not in ("pairs", "halves"):
            raise ValueError(f"latent_attention: rot_layout {rot_layout!r} is not 'pairs' or 'halves'")
        if head_gate and element_gate:
            raise ValueError("latent_attention: a gate per head or per element, not both")
        self.halves, self.head_gate = rot_layout == "halves", bool(head_gate)
        self.element_gate, self.learned_sink = bool(element_gate), bool(learned_sink)
        self.n_gate = self.n_head if self.head_gate else self.n_head * self.v_dim if self.element_gate else 0
        #: columns of the down-projections' product: the query latent, the key/value latent and the rotated part (not
        #: in a layer on another's cache), the gate's logits
        self.gate_off = self.q_rank + (self.latent_dim if self.own_kv else 0)
        self.n_in = self.gate_off + self.n_gate
        self.n_inner = self.n_head * self.v_dim

    def param_specs(self) -> List[ParamSpec]:
        H = self.n_head
        specs = [ParamSpec("q_down", (self.q_rank, self.width), MATRIX),
                 ParamSpec("q_norm", (self.q_rank,), VECTOR, INIT_ONE_PLUS_NORMAL),
                 ParamSpec("q_up", (H * self.qk_dim, self.q_rank), MATRIX)]
        if self.own_kv:
            specs += [ParamSpec("kv_down", (self.latent_dim, self.width), MATRIX),
                      ParamSpec("kv_norm", (self.kv_rank,), VECTOR, INIT_ONE_PLUS_NORMAL)]
        specs += [ParamSpec("k_up", (H * self.nope_dim, self.kv_rank), MATRIX),
                  ParamSpec("v_up", (H * self.v_dim, self.kv_rank), MATRIX),
                  ParamSpec("out_weight", (self.width, H * self.v_dim), MATRIX)]
        if self.n_gate:
            specs.append(ParamSpec("gate_weight", (self.n_gate, self.width), MATRIX))
        if self.learned_sink:
            specs.append(ParamSpec("sink", (H,), VECTOR))
        return specs

    def kv_spec(self) -> Optional[KVCacheSpec]:
        return KVCacheSpec(1, self.latent_dim, self.window, planes=1)

    def step_planner(self):
        return "causal_attention", AttentionPlan

    def flops_per_key(self) -> float:
        return 2.0 * self.n_head * (self.latent_dim + self.kv_rank)

    def prepare(self, dtype, device) -> None:
        super().prepare(dtype, device)
        p, H = self.params, self.n_head
        # the down-projections and the gate read the same rows: one product
        keys = ["q_down"] + (["kv_down"] if self.own_kv else []) + (["gate_weight"] if self.n_gate else [])
        self.w_in = torch.cat([p[k] for k in keys], 0).contiguous()
        self.w_out, at = p["out_weight"], 0
        for k in keys:
            n = p[k].shape[0]
            p[k] = self.w_in[at:at + n]
            at += n
        # W_uk per head, transposed: the map from a head's unrotated query into the latent space
        self.k_up_t = p["k_up"].view(H, self.nope_dim, self.kv_rank).transpose(1, 2).contiguous()
        self.v_up = p["v_up"].view(H, self.v_dim, self.kv_rank)
        i = torch.arange(self.rot_dims // 2, dtype=torch.float64)
        self.freqs = (self.rot_base ** (-2.0 * i / max(self.rot_dims, 1))).to(device)

    def reserve(self, workspace: Workspace, limits: StepLimits) -> None:
        n, H = limits.max_rows, self.n_head
        self.reserve_products(workspace, limits)
        workspace.reserve("latent.cq", n * self.q_rank, self.dtype)
        workspace.reserve("latent.q", n * H * self.qk_dim, self.dtype)
        workspace.reserve("latent.q_full", n * H * self.latent_dim, self.dtype)
        workspace.reserve("latent.out", n * H * self.kv_rank, self.dtype)
        ops.latent_attention_reserve(workspace, H, self.kv_rank)

    def forward(self, xn: torch.Tensor, x: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView],
                state: Optional[torch.Tensor], writes_cache: bool = True) -> None:
        self.run_alone(xn, x, ctx, cache, state, writes_cache, names=("latent_down", "attn_proj"))

    def inner(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext, cache: Optional[KVCacheView] = None,
              state: Optional[torch.Tensor] = None, writes_cache: bool = True) -> None:
        if cache is None:
            raise ValueError("latent_attention needs a paged latent cache")
        if writes_cache != self.own_kv:
            raise ValueError("latent_attention: a layer without W_dkv must read another layer's cache, and only it")
        T, p, H, ws, n = ctx.n_rows, self.params, self.n_head, ctx.workspace, ctx.max_rows
        D = self.latent_dim
        cq = ws.get("latent.cq", (n, self.q_rank), self.dtype)
        ops.latent_prep(proj, self.q_rank, self.kv_rank, self.rot_dim, self.rot_dims, self.freqs, p["q_norm"],
                        p.get("kv_norm"), self.eps, cq, cache.layer if self.own_kv else None,
                        cache.block_table if self.own_kv else None, ctx.row_entry, ctx.positions, T, ctx.status,
                        halves=self.halves)
        q = ws.get("latent.q", (n, H * self.qk_dim), self.dtype)
        ops.trace_scope(ctx.layer, "q_up")
        ops.linear(cq, p["q_up"], None, q, T)
        # the queries over the latent, [absorbed | rotated] a head, in the engine's dtype
        qf = ws.get("latent.q_full", (n, H, D), self.dtype)
        if self.nope_dim:
            ops.trace_scope(ctx.layer, "q_absorb")
            ops.linear_heads(q, self.qk_dim, self.k_up_t, qf.view(n, H * D), D, T,
                             rot=(ctx.positions, self.freqs, self.rot_dim, self.rot_dims, self.halves) if self.rot_dim else None)
        else:
            qf[:T, :, :self.kv_rank].zero_()
            ops.rope_heads(q, self.nope_dim, self.rot_dim, self.rot_dims, self.freqs, ctx.positions, qf, self.kv_rank, H, T,
                           halves=self.halves)
        plan = ctx.plans.get("causal_attention")
        if plan is None:
            plan = ctx.plans["causal_attention"] = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0,
                                                                 device=proj.device)
        lat = ws.get("latent.out", (n, H * self.kv_rank), self.dtype)
        ops.latent_attention(qf, cache.layer, lat, cache.block_table, ctx, H, self.kv_rank, self.scale, self.window,
                             gate=proj[:, self.gate_off:self.gate_off + H] if self.head_gate else None, plan=plan,
                             sinks=p.get("sink"))
        ops.trace_scope(ctx.layer, "v_up")
        ops.linear_heads(lat, self.kv_rank, self.v_up, out, self.v_dim, T,
                         gate=proj[:, self.gate_off:self.gate_off + self.n_gate] if self.element_gate else None)
