"""A plain, slow Dedunex for the tests: whole sequences, no cache, one function a mechanism.

It shares no code with ``nanoinfer_b200``: it takes a configuration (the dictionary of config.json) and a dictionary
of tensors by their checkpoint names, and computes in float64 torch.  Linear weights are [out, in] and applied as
W x.

Notation: h is a layer's normed input [n, width]; positions count from 0; rms(x) = x / sqrt(mean(x^2) + eps).
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


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """``groups`` equal consecutive parts of the vector, each over its own root mean square; the whole times w."""
    n, c = x.shape
    return rms(x.view(n, groups, c // groups), eps).reshape(n, c) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotary_frequencies(rot: dict):
    """(frequencies [dims / 2], factor on cosine and sine) of a configuration's ``rot``: base^(-2i/dims), and with
    ``scaling`` the low frequencies divided by ``factor``, the high ones kept, a ramp over the indices in between."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return torch.tensor(f, dtype=torch.float64), 1.0

    def index_of(turns: float) -> float:      # the (real) index whose wave turns so many times in `original` tokens
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(sc["fast"])), 0), min(math.ceil(index_of(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [n, heads, dim]: of every head the first ``dims`` values turn, value i paired with value i + dims/2; the
    other values pass."""
    if not rot or not rot.get("dims"):
        return x
    dims = rot["dims"]
    half = dims // 2
    f, amp = rotary_frequencies(rot)
    ang = positions.to(torch.float64)[:, None] * f                                # [n, half]
    c, s = (torch.cos(ang) * amp)[:, None, :], (torch.sin(ang) * amp)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def softmax_over(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    s = s.masked_fill(~seen, -math.inf)
    e = torch.exp(s - s.max(dim=1, keepdim=True).values)
    return e / e.sum(dim=1, keepdim=True)


# --------------------------------------------------------------------------- mixers
def differential_lambda(w: Tensors, p: str, diff: float) -> torch.Tensor:
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_attention(h: torch.Tensor, w: Tensors, p: str, m: dict, eps: float) -> torch.Tensor:
    """Two attention maps a head over the same values, the second subtracted; behind a window, with capped scores."""
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    pos = torch.arange(n)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(n, H * 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(n, G * 2, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(n, G, dv)
    q = rotate_halves(rms(q, eps) * w[p + "q.norm"], pos, m.get("rot"))
    k = rotate_halves(rms(k, eps) * w[p + "k.norm"], pos, m.get("rot"))
    i, j = pos[:, None], pos[None, :]
    seen = j <= i
    size = (m.get("mask") or {}).get("size") or 0
    if size:
        seen = seen & (i - j < size)
    lam = differential_lambda(w, p, m["diff"])
    cap = m.get("softcap") or 0.0
    out = torch.zeros(n, H, dv, dtype=torch.float64)
    for a in range(H):
        g = a // (H // G)
        maps = []
        for t in (0, 1):
            s = (q[:, 2 * a + t] @ k[:, 2 * g + t].T) * m["scale"]
            if cap:
                s = cap * torch.tanh(s / cap)
            maps.append(softmax_over(s, seen) @ v[:, g])
        out[:, a] = rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"])
    return out.reshape(n, H * dv) @ w[p + "o"].T


def latent_attention(h: torch.Tensor, w: Tensors, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values from one latent a token, a rotated key part shared by the heads, a gate per head."""
    n, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(n)
    q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    q = q.view(n, H, d + r)
    kv = h @ w[p + "dkv"].T
    c = rms(kv[:, :R], eps) * w[p + "dkv.norm"]
    qr = rotate_halves(q[..., d:], pos, m.get("rot"))
    kr = rotate_halves(kv[:, None, R:], pos, m.get("rot"))[:, 0]
    ku, v = (c @ w[p + "uk"].T).view(n, H, d), (c @ w[p + "uv"].T).view(n, H, dv)
    seen = pos[None, :] <= pos[:, None]
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = torch.zeros(n, H, dv, dtype=torch.float64)
    for a in range(H):
        s = (q[:, a, :d] @ ku[:, a].T + qr[:, a] @ kr.T) * m["scale"]
        out[:, a] = (softmax_over(s, seen) @ v[:, a]) * gate[:, a:a + 1]
    return out.reshape(n, H * dv) @ w[p + "o"].T


def min_gru(h: torch.Tensor, w: Tensors, p: str) -> torch.Tensor:
    """A gated recurrence, element by element, whose gate and candidate see the current token only."""
    z = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros(z.shape[1], dtype=torch.float64)
    y = torch.zeros_like(z)
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        y[t] = S
    return (y * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forward
def gated_feed_forward(h: torch.Tensor, w: Tensors, p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


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


def forward(cfg: dict, w: Tensors, tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of a whole sequence.  ``layers_out`` receives the stream after every layer run."""
    w = {k: v.to(torch.float64) for k, v in w.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups") or 1
    x = grouped_norm(w["embed"][torch.tensor(list(tokens), dtype=torch.long)], w["embed.norm"], groups, eps)
    for i, t in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        h = grouped_norm(x, w[p + "norm1"], groups, eps)
        kind = layer["type"]
        if kind == "attention":
            y = differential_attention(h, w, p + "mix.", layer["mixer"], eps)
        elif kind == "latent_attention":
            y = latent_attention(h, w, p + "mix.", layer["mixer"], eps)
        else:
            y = min_gru(h, w, p + "mix.")
        if layer.get("mlp") is not None:
            y = y + gated_feed_forward(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return grouped_norm(x, w["final.norm"], groups, eps) @ w["head"].T


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


class PlainDedunex:
    """The plain model of a folder: ``logits(tokens)`` float64 [n, vocab] of a whole sequence."""

    def __init__(self, model_dir: str):
        self.cfg, self.w = load_folder(model_dir)

    def logits(self, tokens: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
        return forward(self.cfg, self.w, tokens, layers_out)

    def greedy(self, prompt: Sequence[int], n: int) -> List[int]:
        """The ``n`` tokens that greedy decoding appends to ``prompt`` (ties to the lower index)."""
        seq, out = list(prompt), []
        for _ in range(n):
            out.append(int(torch.argmax(self.logits(seq)[-1])))
            seq.append(out[-1])
        return out
