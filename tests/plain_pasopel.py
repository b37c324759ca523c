"""A plain, slow Pasopel for the tests: whole sequences, no cache, one function a mechanism.

It shares no code with ``nanoinfer_b200``: it takes a configuration (the dictionary of config.json) and a dictionary
of tensors by their checkpoint names, and computes in float64 torch.  Linear weights are [out, in] and applied as
W x.

Notation: h is a sublayer's input [n, width]; positions count from 0; rms(x) = x / sqrt(mean(x^2) + eps).
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Sequence

import torch

Tensors = Dict[str, torch.Tensor]


# --------------------------------------------------------------------------- small pieces
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_zero(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal convolution over time per channel: x [n, channels], w [channels, taps]; the last tap is the current
    token's and what lies before the sequence is zero."""
    n, taps = x.shape[0], w.shape[1]
    xx = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x], 0)
    out = torch.zeros_like(x)
    for j in range(taps):
        out += w[:, j] * xx[j:j + n]
    return out


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [n, heads, dim]: of the first ``dims`` values of every head (2i, 2i + 1) turn by position * base^(-2i/dims)."""
    if not rot or not rot.get("dims"):
        return x
    dims = rot["dims"]
    i = torch.arange(dims // 2, dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * float(rot["base"]) ** (-2.0 * i / dims)
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def softmax_with_sink(s: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)) over the keys that are seen."""
    s = s.masked_fill(~seen, -math.inf)
    top = torch.maximum(s.max(dim=1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=1, keepdim=True) + torch.exp(sink - top))


def pooled(x: torch.Tensor, P: int) -> torch.Tensor:
    """x [n, ...] -> the means of the whole blocks of P rows, [n // P, ...]."""
    nb = x.shape[0] // P
    return x[:nb * P].reshape(nb, P, *x.shape[1:]).mean(dim=1)


# --------------------------------------------------------------------------- mixers
def pooled_window_attention(h: torch.Tensor, w: Tensors, p: str, m: dict, eps: float) -> torch.Tensor:
    """Tokens of a window, and a mean key and value for every block of ``pool`` tokens wholly behind it, in one softmax
    with a learned sink; the keys as they leave a short convolution are the values; a gate per element of the output."""
    n, H, G, d = h.shape[0], m["heads"], m.get("kv_heads") or m["heads"], m["dim"]
    q, k = h @ w[p + "q"].T + w[p + "q.b"], h @ w[p + "k"].T + w[p + "k.b"]
    if m.get("conv"):
        q, k = short_conv(q, w[p + "q.conv"]), short_conv(k, w[p + "k.conv"])
    v = k.view(n, G, d)
    q, k = rms(q.view(n, H, d), eps), rms(k.view(n, G, d), eps)
    mask = m.get("mask") or {}
    size, P = mask.get("size") or 0, mask.get("pool") or 0
    pos = torch.arange(n)
    i, j = pos[:, None], pos[None, :]
    seen = j <= i
    if size:
        seen = seen & (i - j < size)
    keys, values = k, v
    if size and P:
        b = torch.arange(n // P)[None, :]
        seen = torch.cat([seen, b * P + P - 1 <= i - size], dim=1)
        keys, values = torch.cat([k, pooled(k, P)], 0), torch.cat([v, pooled(v, P)], 0)
    out = torch.zeros(n, H, d, dtype=torch.float64)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ keys[:, g].T) * m["scale"]
        out[:, a] = softmax_with_sink(s, seen, w[p + "sink"][a]) @ values[:, g]
    gated = out.reshape(n, H * d) * torch.sigmoid(h @ w[p + "g"].T)
    return gated @ w[p + "o"].T + w[p + "o.b"]


def latent_attention(h: torch.Tensor, w: Tensors, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values from one latent a token, a rotated key part shared by the heads, a window, a learned sink, a gate
    per element of the output."""
    n, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(n)
    q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    q = q.view(n, H, d + r)
    kv = h @ w[p + "dkv"].T
    c = rms(kv[:, :R], eps) * w[p + "dkv.norm"]
    qr = rotate_pairs(q[..., d:], pos, m.get("rot"))
    kr = rotate_pairs(kv[:, None, R:], pos, m.get("rot"))[:, 0]
    ku, v = (c @ w[p + "uk"].T).view(n, H, d), (c @ w[p + "uv"].T).view(n, H, dv)
    i, j = pos[:, None], pos[None, :]
    seen = j <= i
    size = (m.get("mask") or {}).get("size") or 0
    if size:
        seen = seen & (i - j < size)
    out = torch.zeros(n, H, dv, dtype=torch.float64)
    for a in range(H):
        s = (q[:, a, :d] @ ku[:, a].T + qr[:, a] @ kr.T) * m["scale"]
        out[:, a] = softmax_with_sink(s, seen, w[p + "sink"][a]) @ v[:, a]
    return (out.reshape(n, H * dv) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forward
def dense_feed_forward(h: torch.Tensor, w: Tensors, p: str) -> torch.Tensor:
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def expert(h: torch.Tensor, w: Tensors, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_choice(h: torch.Tensor, w: Tensors, p: str, top: int):
    """(the chosen experts [n, top], their weights): the largest logits, softmax over the chosen ones only."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best = torch.topk(z, top, dim=1)
    return best.indices, torch.softmax(best.values, dim=1)


def router_margin(h: torch.Tensor, w: Tensors, p: str, top: int) -> torch.Tensor:
    """How far the last chosen expert's logit lies above the first one left out, per row (a large number: none is)."""
    z = (h @ w[p + "router"].T + w[p + "router.b"]).sort(dim=1, descending=True).values
    return z[:, top - 1] - z[:, top] if z.shape[1] > top else torch.full((h.shape[0],), math.inf, dtype=torch.float64)


def routed_feed_forward(h: torch.Tensor, w: Tensors, p: str, m: dict) -> torch.Tensor:
    ids, s = router_choice(h, w, p, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        weight = (s * (ids == e)).sum(dim=1, keepdim=True)
        rows = weight[:, 0] > 0
        if rows.any():
            out[rows] += weight[rows] * expert(h[rows], w, f"{p}e{e}.")
    if m.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


# --------------------------------------------------------------------------- the model
def run_order(cfg: dict) -> List[tuple]:
    """(layer, pass or None) in the order of the runs: layers start .. stop - 1 ``times`` times in a row; the pass is
    named at the first layer of each pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def forward(cfg: dict, w: Tensors, tokens: Sequence[int], layers_out: Optional[list] = None,
            margins_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of a whole sequence.  ``layers_out`` receives the stream after every layer run, ``margins_out``
    every router's margin per position."""
    w = {k: v.to(torch.float64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    start = x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = (x + start if t > 0 else x) + w["loop.step"][t]
        h = norm_around_zero(x, w[p + "norm1"], eps)
        mixer = pooled_window_attention if layer["type"] == "attention" else latent_attention
        x = x + mixer(h, w, p + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = norm_around_zero(x, w[p + "norm2"], eps)
            if margins_out is not None and mlp["kind"] == "moe":
                margins_out.append(router_margin(h, w, p + "mlp.", mlp["router"]["top"]))
            x = x + (dense_feed_forward(h, w, p + "mlp.") if mlp["kind"] == "dense"
                     else routed_feed_forward(h, w, p + "mlp.", mlp))
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = norm_around_zero(x, w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap") or 0.0
    return cap * torch.tanh(logits / cap) if cap else logits


def load_folder(model_dir: str):
    """(config, tensors) of a model folder, read with the ``safetensors`` package."""
    from safetensors import safe_open

    with open(os.path.join(model_dir, "config.json")) as fh:
        cfg = json.load(fh)
    w = {}
    with safe_open(os.path.join(model_dir, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            w[name] = f.get_tensor(name)
    return cfg, w


class PlainPasopel:
    """The plain model of a folder: ``logits(tokens)`` float64 [n, vocab] of a whole sequence."""

    def __init__(self, model_dir: str):
        self.cfg, self.w = load_folder(model_dir)

    def logits(self, tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
        return forward(self.cfg, self.w, tokens, layers_out)

    def margins(self, tokens: Sequence[int]) -> torch.Tensor:
        """The smallest margin of any router, per position (infinite in a model without routers)."""
        out: List[torch.Tensor] = []
        forward(self.cfg, self.w, tokens, None, out)
        return torch.stack(out).min(dim=0).values if out else torch.full((len(tokens),), math.inf, dtype=torch.float64)

    def greedy(self, prompt: Sequence[int], n: int) -> List[int]:
        """The ``n`` tokens that greedy decoding appends to ``prompt`` (ties to the lower index)."""
        seq, out = list(prompt), []
        for _ in range(n):
            out.append(int(torch.argmax(self.logits(seq)[-1])))
            seq.append(out[-1])
        return out
