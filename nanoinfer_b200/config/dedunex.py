"""Dedunex's configuration: a list of layers, each with a mixer of one of three kinds (differential attention behind a
window, attention through a latent, the minimal gated recurrent unit) beside an optional gated feed-forward, and a
stretch of layers that runs several times in a row, read from the nested keys of its config.json:

    {"architecture": "Dedunex", "vocab": V, "width": C, "norm": {"eps": e, "groups": g},
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": v, "scale": s, "softcap": c, "diff": l,
                           "mask": {"size": w},
                           "rot": {"dims": r, "base": b,
                                   "scaling": {"factor": f, "original": n, "fast": x, "slow": y}}},
                 "mlp": {"kind": "dense", "ff": F}},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": v, "q_rank": q, "kv_rank": k, "scale": s,
                           "rot": {"dims": r, "base": b}}, "mlp": ...},
                {"type": "mingru", "mixer": {"width": W}, "mlp": null}]}

Every size and constant comes from the file.  Left out (or null), ``norm.groups`` is 1, ``loop`` means that every layer
runs once, ``kv_heads`` is ``heads``, ``softcap`` no cap, ``mask`` all keys, ``rot`` no rotation, ``rot.scaling`` none.
"""
from __future__ import annotations

import dataclasses
from typing import ClassVar, List, Optional, Tuple

from .base import ConfigError, ModelConfig, field
from .mulavik import _positive
from .vadonex import _get

MIXER_KINDS = ("attention", "latent_attention", "mingru")


def _rotation(m: dict, bad: List[str], w: str, limit, scaled: bool) -> None:
    if m.get("rot") is None:
        return
    dims = _get(m, "rot.dims", int, bad, w)
    base = _positive(m, "rot.base", float, bad, w)
    if isinstance(dims, int) and (dims < 0 or dims % 2 or (isinstance(limit, int) and dims > limit)):
        bad.append(f"{w}.rot.dims {dims} must be even, not negative and at most {limit}")
    if isinstance(m["rot"], dict) and m["rot"].get("scaling") is not None:
        if not scaled:
            bad.append(f"{w}.rot.scaling: this kind of layer has no scaled rotation")
            return
        for key in ("factor", "original", "fast", "slow"):
            _positive(m, f"rot.scaling.{key}", float, bad, w)
        if base == 1.0:
            bad.append(f"{w}.rot.base must not be 1 with a scaling")


@dataclasses.dataclass
class DedunexConfig(ModelConfig):
    architecture_names: ClassVar[Tuple[str, ...]] = ("Dedunex",)

    vocab: int = field()
    width: int = field()
    layers: list = field()
    norm: dict = field()
    loop: Optional[dict] = field(default=None)

    def validate(self) -> None:
        bad: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            bad.append("vocab and width must be positive")
        _positive(self.norm, "eps", float, bad, "norm")
        groups = _positive(self.norm, "groups", int, bad, "norm", default=1)
        if isinstance(groups, int) and groups > 0 and self.width > 0 and self.width % groups:
            bad.append(f"norm.groups {groups} must divide width {self.width}")
        if not self.layers:
            bad.append("layers: at least one layer is needed")
        if self.loop is not None:
            if not isinstance(self.loop, dict):
                bad.append("loop: expected an object with 'start', 'stop' and 'times'")
            else:
                a = _get(self.loop, "start", int, bad, "loop")
                b = _get(self.loop, "stop", int, bad, "loop")
                _positive(self.loop, "times", int, bad, "loop")
                if isinstance(a, int) and isinstance(b, int) and not 0 <= a < b <= len(self.layers):
                    bad.append(f"loop: start {a} and stop {b} must satisfy 0 <= start < stop <= {len(self.layers)}")
        for i, layer in enumerate(self.layers):
            w = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                bad.append(f"{w}: expected an object with 'type', 'mixer' and 'mlp'")
                continue
            kind, m, wm = layer.get("type"), layer["mixer"], f"{w}.mixer"
            if kind not in MIXER_KINDS:
                bad.append(f"{w}.type {kind!r} is not one of {MIXER_KINDS}")
                continue
            if kind == "mingru":
                _positive(m, "width", int, bad, wm)
            else:
                heads = _positive(m, "heads", int, bad, wm)
                dim = _positive(m, "dim", int, bad, wm)
                vdim = _positive(m, "vdim", int, bad, wm)
                _get(m, "scale", float, bad, wm)
                if kind == "attention":
                    g = _positive(m, "kv_heads", int, bad, wm, default=heads)
                    if isinstance(heads, int) and isinstance(g, int) and g > 0 and heads % g:
                        bad.append(f"{wm}.heads {heads} must be a multiple of kv_heads {g}")
                    if isinstance(dim, int) and dim > 128:
                        bad.append(f"{wm}.dim {dim} is larger than 128")
                    if isinstance(vdim, int) and vdim > 256:
                        bad.append(f"{wm}.vdim {vdim} is larger than 256")
                    _get(m, "diff", float, bad, wm)
                    _positive(m, "softcap", float, bad, wm, default=None)
                    if m.get("mask") is not None:
                        _positive(m, "mask.size", int, bad, wm)
                    _rotation(m, bad, wm, dim, scaled=True)
                else:
                    r = _get(m, "rot_dim", int, bad, wm)
                    if isinstance(r, int) and r < 0:
                        bad.append(f"{wm}.rot_dim must not be negative")
                    _positive(m, "q_rank", int, bad, wm)
                    k = _positive(m, "kv_rank", int, bad, wm)
                    if isinstance(k, int) and k > 1024:
                        bad.append(f"{wm}.kv_rank {k} is larger than 1024")
                    _rotation(m, bad, wm, r, scaled=False)
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                bad.append(f"{w}.mlp.kind must be 'dense' (or mlp null)")
                continue
            _positive(mlp, "ff", int, bad, f"{w}.mlp")
        if bad:
            raise ConfigError("config.json: " + "; ".join(bad))

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def groups(self) -> int:
        return int(self.norm.get("groups") or 1)

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    def run_order(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, the number of the pass that begins with this run or None) for every run, in order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        a, b = int(self.loop["start"]), int(self.loop["stop"])
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for t in range(int(self.loop["times"])):
            runs += [(i, t if i == a else None) for i in range(a, b)]
        return runs + [(i, None) for i in range(b, n)]

    def to_dict(self):
        out = {"architecture": self.architecture_names[0], "vocab": self.vocab, "width": self.width,
               "norm": dict(self.norm), "layers": self.layers}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        return out
