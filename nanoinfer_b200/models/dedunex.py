"""Dedunex as a ModelSpec: a token embedding with a norm behind it; layers in which a mixer and a gated feed-forward
(GELU in the tanh form) read the same norm and are summed together; a stretch of layers that runs several times in a row
with the same weights, a learned vector added to the stream ahead of each pass; every norm of the model an RMS norm in
groups; a final norm and a head of its own.

Mixers: ``attention`` (differential attention: two maps a head, the second subtracted; grouped key/value heads, biases,
a norm on every map's query and key, rotary halves with YaRN's scaling, capped scores, a window), ``latent_attention``
(queries and keys/values through latents, a rotated key part shared by the heads, a sigmoid gate per head) and ``mingru``
(a gated recurrence whose gates read the current token only).

Tensor names: ``embed``, ``embed.norm``, ``loop.step``, ``final.norm``, ``head``, ``l<i>.norm1``; attention
``l<i>.mix.{q, k, v}`` with ``.b``, ``l<i>.mix.{q.norm, k.norm, lq1, lk1, lq2, lk2, o}``; latent attention
``l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o}``; mingru ``l<i>.mix.{z, z.b, x, x.b, g, o}``; feed-forward
``l<i>.mlp.{gate, up, down}``.  Matrices are stored [out, in].
"""
from __future__ import annotations

from ..config.dedunex import DedunexConfig
from ..parts.base import TensorRef
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _refs(prefix: str, names: dict) -> dict:
    return {key: TensorRef(prefix + name) for key, name in names.items()}


def build_dedunex_spec(cfg: DedunexConfig) -> ModelSpec:
    c, eps, groups = cfg.width, cfg.eps, cfg.groups

    def norm(name: str) -> PartSpec:
        return PartSpec("grouped_rmsnorm", dict(width=c, eps=eps, groups=groups), {"weight": TensorRef(name)})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        parts, position = {"norm_1": norm(p + "norm1")}, None
        rot = m.get("rot") or {}
        if layer["type"] == "attention":
            if rot.get("dims"):
                position = PartSpec("rotary_halves", dict(base=float(rot["base"]), dims=int(rot["dims"]),
                                                          scaling=rot.get("scaling")))
            parts["mixer"] = PartSpec("differential_attention", dict(
                width=c, n_head=m["heads"], n_kv_head=m.get("kv_heads") or m["heads"], head_dim=m["dim"], v_dim=m["vdim"],
                scale=float(m["scale"]), eps=eps, diff=float(m["diff"]), window=int((m.get("mask") or {}).get("size") or 0),
                softcap=float(m.get("softcap") or 0.0), bias=True, qk_norm=True),
                _refs(p, {"q_weight": "mix.q", "q_bias": "mix.q.b", "k_weight": "mix.k", "k_bias": "mix.k.b",
                          "v_weight": "mix.v", "v_bias": "mix.v.b", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm",
                          "lq1": "mix.lq1", "lk1": "mix.lk1", "lq2": "mix.lq2", "lk2": "mix.lk2", "out_weight": "mix.o"}))
        elif layer["type"] == "latent_attention":
            parts["mixer"] = PartSpec("latent_attention", dict(
                width=c, n_head=m["heads"], nope_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], q_rank=m["q_rank"],
                kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=eps, window=0, rot_base=float(rot.get("base") or 10000.0),
                rot_dims=int(rot.get("dims") or 0), rot_layout="halves", head_gate=True),
                _refs(p, {"q_down": "mix.dq", "q_norm": "mix.dq.norm", "q_up": "mix.uq", "kv_down": "mix.dkv",
                          "kv_norm": "mix.dkv.norm", "k_up": "mix.uk", "v_up": "mix.uv", "gate_weight": "mix.g",
                          "out_weight": "mix.o"}))
        else:
            parts["mixer"] = PartSpec("min_gru", dict(width=c, inner=m["width"]),
                                      _refs(p, {"z_weight": "mix.z", "z_bias": "mix.z.b", "x_weight": "mix.x",
                                                "x_bias": "mix.x.b", "g_weight": "mix.g", "out_weight": "mix.o"}))
        if layer.get("mlp") is not None:
            parts["feed_forward"] = PartSpec("gated_mlp", dict(width=c, inner=layer["mlp"]["ff"], activation="tanh"),
                                             _refs(p, {"gate_weight": "mlp.gate", "up_weight": "mlp.up",
                                                       "down_weight": "mlp.down"}))
        layers.append(LayerSpec("parallel_norm", parts, mixer_position=position))
    return ModelSpec(
        width=c,
        embedding=PartSpec("normed_token_embedding", dict(vocab_size=cfg.vocab, width=c, eps=eps, groups=groups),
                           {"table": TensorRef("embed"), "norm": TensorRef("embed.norm")}),
        position=None,
        layers=layers,
        # every run of a looped layer has keys and values, or a state, of its own
        schedule=[ScheduleEntry(i, add_vector=t) for i, t in cfg.run_order()],
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab, width=c), {"weight": TensorRef("head")}),
        max_positions=None,
        stream_vectors=None if cfg.loop is None else PartSpec(
            "stream_vector_table", dict(count=int(cfg.loop["times"]), width=c), {"table": TensorRef("loop.step")}),
    )
