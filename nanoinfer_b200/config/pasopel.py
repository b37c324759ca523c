"""Pasopel's configuration: a list of layers, each with one of two mixers (attention over a window with pooled blocks behind
it, or attention through a latent) and an optional feed-forward (dense, or a mixture of experts with a shared one), and a
stretch of layers that runs several times in a row, read from the nested keys of its config.json:

    {"architecture": "Pasopel", "vocab": V, "width": C, "norm": {"eps": e}, "logit_softcap": c,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "conv": t, "scale": s,
                           "mask": {"size": w, "pool": P}},
                 "mlp": {"kind": "dense", "ff": F}},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": v, "q_rank": q, "kv_rank": k, "scale": s,
                           "mask": {"size": w}, "rot": {"dims": r, "base": b}},
                 "mlp": {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F}, "shared": {"ff": S}}},
                {"type": ..., "mixer": ..., "mlp": null}]}

Every size and constant comes from the file.  Left out (or null), ``logit_softcap`` is no cap, ``loop`` means that every layer
runs once, ``kv_heads`` is ``heads``, ``vdim`` of an attention layer (whose values are its keys) is ``dim``, ``conv`` no
convolution, ``mask`` all keys, ``mask.pool`` no pooled blocks, ``rot`` no rotation, ``shared`` no shared expert.
"""
from __future__ import annotations

import dataclasses
from typing import ClassVar, List, Optional, Tuple

from .base import ConfigError, ModelConfig, field
from .dedunex import _rotation
from .mulavik import _positive
from .vadonex import _get

MIXER_KINDS = ("attention", "latent_attention")


@dataclasses.dataclass
class PasopelConfig(ModelConfig):
    architecture_names: ClassVar[Tuple[str, ...]] = ("Pasopel",)

    vocab: int = field()
    width: int = field()
    layers: list = field()
    norm: dict = field()
    loop: Optional[dict] = field(default=None)
    logit_softcap: Optional[float] = field(default=None)

    def validate(self) -> None:
        bad: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            bad.append("vocab and width must be positive")
        _positive(self.norm, "eps", float, bad, "norm")
        if self.logit_softcap is not None and not self.logit_softcap > 0.0:
            bad.append(f"logit_softcap must be positive, got {self.logit_softcap}")
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
            if layer.get("type") not in MIXER_KINDS:
                bad.append(f"{w}.type {layer.get('type')!r} is not one of {MIXER_KINDS}")
                continue
            self._check_mixer(layer["type"], layer["mixer"], bad, f"{w}.mixer")
            self._check_mlp(layer.get("mlp"), bad, f"{w}.mlp")
        if bad:
            raise ConfigError("config.json: " + "; ".join(bad))

    @staticmethod
    def _check_mixer(kind: str, m: dict, bad: List[str], w: str) -> None:
        heads = _positive(m, "heads", int, bad, w)
        dim = _positive(m, "dim", int, bad, w)
        _get(m, "scale", float, bad, w)
        if m.get("mask") is not None:
            _positive(m, "mask.size", int, bad, w)
        if kind == "attention":
            g = _positive(m, "kv_heads", int, bad, w, default=heads)
            if isinstance(heads, int) and isinstance(g, int) and g > 0 and heads % g:
                bad.append(f"{w}.heads {heads} must be a multiple of kv_heads {g}")
            v = _positive(m, "vdim", int, bad, w, default=dim)
            if isinstance(dim, int) and isinstance(v, int) and v != dim:
                bad.append(f"{w}.vdim {v} must be dim {dim}: the values are the keys")
            if isinstance(dim, int) and dim > 256:
                bad.append(f"{w}.dim {dim} is larger than 256")
            taps = _positive(m, "conv", int, bad, w, default=None)
            if isinstance(taps, int) and taps > 64:
                bad.append(f"{w}.conv {taps} is larger than 64")
            if isinstance(m.get("mask"), dict):
                _positive(m, "mask.pool", int, bad, w, default=None)
            return
        _positive(m, "vdim", int, bad, w)
        r = _get(m, "rot_dim", int, bad, w)
        if isinstance(r, int) and r < 0:
            bad.append(f"{w}.rot_dim must not be negative")
        _positive(m, "q_rank", int, bad, w)
        k = _positive(m, "kv_rank", int, bad, w)
        if isinstance(k, int) and k > 1024:
            bad.append(f"{w}.kv_rank {k} is larger than 1024")
        _rotation(m, bad, w, r, scaled=False)

    @staticmethod
    def _check_mlp(mlp, bad: List[str], w: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            bad.append(f"{w}.kind must be 'dense' or 'moe' (or mlp null)")
            return
        if mlp["kind"] == "dense":
            _positive(mlp, "ff", int, bad, w)
            return
        n = _positive(mlp, "router.experts", int, bad, w)
        top = _positive(mlp, "router.top", int, bad, w)
        if isinstance(n, int) and isinstance(top, int) and top > n:
            bad.append(f"{w}.router.top {top} is larger than the number of experts {n}")
        _positive(mlp, "expert.ff", int, bad, w)
        if mlp.get("shared") is not None:
            _positive(mlp, "shared.ff", int, bad, w)

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

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
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out
