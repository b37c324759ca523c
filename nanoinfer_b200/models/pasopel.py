"""Pasopel as a ModelSpec: a token embedding; pre-norm layers of a mixer and an optional feed-forward; a stretch of layers that
runs several times in a row with the same weights, ahead of each pass but the first the embedding's output added to the stream
again, and ahead of every pass a learned vector; a final norm, a head tied to the embedding table and a soft cap on the logits.
The norms across the width are RMS norms whose weight is stored around zero.

Mixers: ``attention`` (a window of tokens and, behind it, one pooled key and value a block; a short convolution on queries and
keys, a norm per head, the keys as values, no rotation) and ``latent_attention`` (queries and keys/values through latents, a
rotated key part shared by the heads, a window); both with a learned sink per head and a sigmoid gate per element of the heads'
outputs.  Feed-forwards: dense (square of relu) or routed gated experts (silu; biased router logits, a softmax over the chosen
ones) beside a shared one.

Tensor names: ``embed``, ``loop.step``, ``final.norm``, ``l<i>.norm1``, ``l<i>.norm2``; attention ``l<i>.mix.{q, k, o}`` with
``.b``, ``l<i>.mix.{q.conv, k.conv, sink, g}``; latent attention ``l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, g,
o}``; dense ``l<i>.mlp.{up, down}``; experts ``l<i>.mlp.{router, router.b}``, ``l<i>.mlp.e<j>.{gate, up, down}`` and
``l<i>.mlp.shared.{gate, up, down}``.  Matrices are stored [out, in].
"""
from __future__ import annotations

from ..config.pasopel import PasopelConfig
from ..parts.base import TensorRef
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _refs(prefix: str, names: dict) -> dict:
    return {key: TensorRef(prefix + name) for key, name in names.items()}


def _mixer(c: int, eps: float, kind: str, m: dict, p: str) -> PartSpec:
    mask = m.get("mask") or {}
    window = int(mask.get("size") or 0)
    if kind == "attention":
        names = {"q_weight": "mix.q", "q_bias": "mix.q.b", "k_weight": "mix.k", "k_bias": "mix.k.b", "out_weight": "mix.o",
                 "out_bias": "mix.o.b", "sink": "mix.sink", "gate_weight": "mix.g"}
        if m.get("conv"):
            names.update({"q_conv": "mix.q.conv", "k_conv": "mix.k.conv"})
        return PartSpec("pooled_attention", dict(
            width=c, n_head=m["heads"], n_kv_head=m.get("kv_heads") or m["heads"], head_dim=m["dim"], scale=float(m["scale"]),
            eps=eps, window=window, pool=int(mask.get("pool") or 0), taps=int(m.get("conv") or 0), bias=True, qk_norm=True,
            learned_sink=True, element_gate=True), _refs(p, names))
    rot = m.get("rot") or {}
    return PartSpec("latent_attention", dict(
        width=c, n_head=m["heads"], nope_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], q_rank=m["q_rank"],
        kv_rank=m["kv_rank"], scale=float(m["scale"]), eps=eps, window=window, rot_base=float(rot.get("base") or 10000.0),
        rot_dims=int(rot.get("dims") or 0), rot_layout="pairs", element_gate=True, learned_sink=True),
        _refs(p, {"q_down": "mix.dq", "q_norm": "mix.dq.norm", "q_up": "mix.uq", "kv_down": "mix.dkv",
                  "kv_norm": "mix.dkv.norm", "k_up": "mix.uk", "v_up": "mix.uv", "sink": "mix.sink", "gate_weight": "mix.g",
                  "out_weight": "mix.o"}))


def _feed_forward(c: int, mlp: dict, p: str) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("dense_mlp", dict(width=c, inner=mlp["ff"], activation="relu2", bias=False),
                        _refs(p, {"fc_weight": "mlp.up", "proj_weight": "mlp.down"}))
    n, shared = int(mlp["router"]["experts"]), mlp.get("shared")
    names = {"router": "mlp.router", "router_bias": "mlp.router.b"}
    for e in range(n):
        names.update({f"expert{e}_{k}": f"mlp.e{e}.{k}" for k in ("gate", "up", "down")})
    if shared:
        names.update({f"shared_{k}": f"mlp.shared.{k}" for k in ("gate", "up", "down")})
    # (a softmax over all logits, divided by the chosen ones' sum, is the softmax over the chosen logits)
    return PartSpec("routed_experts", dict(
        width=c, n_expert=n, top=mlp["router"]["top"], inner=mlp["expert"]["ff"], activation="silu", renorm=True, gated=True,
        shared_inner=shared["ff"] if shared else 0, shared_activation="silu", router_bias=True), _refs(p, names))


def build_pasopel_spec(cfg: PasopelConfig) -> ModelSpec:
    c, eps = cfg.width, cfg.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("grouped_rmsnorm", dict(width=c, eps=eps, groups=1, one_plus=True), {"weight": TensorRef(name)})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"norm_1": norm(p + "norm1"), "mixer": _mixer(c, eps, layer["type"], layer["mixer"], p)}
        if layer.get("mlp") is not None:
            parts["norm_2"], parts["feed_forward"] = norm(p + "norm2"), _feed_forward(c, layer["mlp"], p)
        layers.append(LayerSpec("pre_norm", parts))
    return ModelSpec(
        width=c,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, width=c), {"table": TensorRef("embed")}),
        position=None,
        layers=layers,
        # every run of a looped layer has keys and values, and a state, of its own
        schedule=[ScheduleEntry(i, add_vector=t, add_embedding=t is not None and t > 0) for i, t in cfg.run_order()],
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab, width=c, softcap=float(cfg.logit_softcap or 0.0)),
                      {"weight": TensorRef("embed")}),
        max_positions=None,
        stream_vectors=None if cfg.loop is None else PartSpec(
            "stream_vector_table", dict(count=int(cfg.loop["times"]), width=c), {"table": TensorRef("loop.step")}),
    )
