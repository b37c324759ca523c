"""Helpers of the Pasopel tests: small configurations, model folders with seeded weights made so that faults show,
and the error measure."""
import json
import os

import torch

from mulavik_util import TOL, assert_close, moe, rel_err, row_errs  # noqa: F401  (the same measure and bounds)


def dense(ff=48):
    return dict(kind="dense", ff=ff)


def pooled_layer(heads=4, kv_heads=2, dim=16, conv=3, scale=None, window=24, pool=8, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale if scale is not None else dim ** -0.5)
    if conv:
        m["conv"] = conv
    if window:
        m["mask"] = dict(size=window)
        if pool:
            m["mask"]["pool"] = pool
    return dict(type="attention", mixer=m, mlp=mlp)


def latent_layer(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=32, scale=None, base=900.0, window=20, mlp=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
             scale=scale if scale is not None else (dim + rot_dim) ** -0.5)
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
    if window:
        m["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def config(layers, vocab=200, width=64, eps=1e-5, loop=None, cap=20.0):
    """``loop``: (start, stop, times) or None."""
    out = dict(architecture="Pasopel", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap:
        out["logit_softcap"] = cap
    return out


def write_model(cfg_dict, out_dir, dtype=torch.float32, seed=1, sharpen=3.0):
    """A model folder from the product's random-weights rule, then reshaped so that faults show: the scores' scale (the
    normed queries and keys leave no other handle) and the latents' up-projections raised so that the softmax leans on single
    keys, blocks or the sink; convolution taps of like size; norm weights and the loop's vectors far from their neutral value;
    biases of ordinary size; half-open gates; a decisive router whose bias matters."""
    from nanoinfer_b200.config import PasopelConfig
    from nanoinfer_b200.models.model import Model
    from nanoinfer_b200.registry import get_architecture
    from nanoinfer_b200.weights import random_tensors, write_safetensors

    cfg_dict = json.loads(json.dumps(cfg_dict))
    for layer in cfg_dict["layers"]:
        if layer["type"] == "attention":
            layer["mixer"]["scale"] *= sharpen ** 0.5
    cfg = PasopelConfig.from_dict(cfg_dict)
    model = Model(get_architecture(cfg.architecture).build_spec(cfg), cfg)
    tensors = random_tensors(model, seed, 0.02, torch.float32)
    g = torch.Generator().manual_seed(seed + 99)
    rn = lambda t, s=1.0: torch.randn(t.shape, generator=g) * s
    ru = lambda t: torch.rand(t.shape, generator=g)
    for name, t in tensors.items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if name == "embed":
            t.copy_(rn(t, 0.5))
        elif name == "loop.step":
            t.copy_(rn(t, 0.3))
        elif name == "final.norm":
            t.copy_(rn(t) - 1.0)      # (signs of its own: the tied table does not give every token back at once)
        elif leaf in ("norm1", "norm2"):
            t.copy_(1.2 * ru(t) - 0.6)
        elif leaf in ("mix.dq.norm", "mix.dkv.norm"):
            t.copy_(0.5 + ru(t))
        elif leaf.endswith(".conv"):
            t.copy_(rn(t, 0.7))
        elif leaf == "mix.sink":
            t.copy_(rn(t, 1.5))
        elif leaf.endswith(".b"):
            t.copy_(rn(t, 0.5))
        elif leaf in ("mix.uq", "mix.uk"):
            t.copy_(rn(t, (sharpen / max(1, t.shape[1])) ** 0.5))
        elif leaf in ("mix.q", "mix.k", "mlp.router"):
            t.copy_(rn(t, t.shape[1] ** -0.5))
        elif leaf == "mix.g":
            t.copy_(rn(t, 1.5 * t.shape[1] ** -0.5))
        else:
            t *= 6.0
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as fh:
        json.dump(cfg.to_dict(), fh)
    write_safetensors(os.path.join(out_dir, "model.safetensors"), {k: v.to(dtype) for k, v in tensors.items()})
    return out_dir


#: a router whose choice hangs on less than this (of logits of size one) may choose otherwise in bfloat16
CLOSE_CALL = 0.05


def assert_close_where_routing_is_clear(errs, margins, dtype, what=""):
    """``assert_close``; in bfloat16 over the positions at which no router's choice is a close call."""
    if dtype != "float32":
        clear = margins >= CLOSE_CALL
        assert int(clear.sum()) * 4 >= len(clear), f"{what}: too few positions with a clear choice to say anything"
        errs = errs[clear.to(errs.device)]
    assert_close(errs, dtype, what)
