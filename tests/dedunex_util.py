"""Helpers of the Dedunex tests: small configurations, model folders with seeded weights made so that faults show,
and the error measure."""
import json
import os

import torch

from mulavik_util import TOL, assert_close, rel_err, row_errs  # noqa: F401  (the same measure and bounds)


def dense(ff=48):
    return dict(kind="dense", ff=ff)


def diff_layer(heads=4, kv_heads=2, dim=16, vdim=40, scale=None, softcap=9.0, diff=0.4, window=24, rot=8, base=5000.0,
               scaling=(3.0, 100, 8.0, 0.5), mlp=None):
    """``scaling``: (factor, original, fast, slow) or None."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else dim ** -0.5, diff=diff)
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = dict(size=window)
    if rot:
        m["rot"] = dict(dims=rot, base=base)
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(type="attention", mixer=m, mlp=mlp)


def latent_layer(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=32, scale=None, base=900.0, mlp=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
             scale=scale if scale is not None else (dim + rot_dim) ** -0.5)
    if rot_dim:
        m["rot"] = dict(dims=rot_dim, base=base)
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def gru_layer(width=40, mlp=None):
    return dict(type="mingru", mixer=dict(width=width), mlp=mlp)


def config(layers, vocab=200, width=64, groups=2, eps=1e-5, loop=None):
    """``loop``: (start, stop, times) or None."""
    out = dict(architecture="Dedunex", vocab=vocab, width=width, norm=dict(eps=eps, groups=groups), layers=layers)
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def write_model(cfg_dict, out_dir, dtype=torch.float32, seed=1, sharpen=3.0, long_memory=False):
    """A model folder from the product's random-weights rule, then reshaped so that faults show: the weights of the query
    and key norms (and the latents' up-projections of queries and keys) scaled so that the softmax leans on single keys;
    norm weights and the loop's vectors far from 1 and from one another; biases of ordinary size; the numbers behind lambda
    large enough that it differs from the configuration's constant; gates that are half open; the recurrent unit's update
    gates spread so that some channels forget within a few tokens and others remember for hundreds (``long_memory``: all
    remember)."""
    from nanoinfer_b200.config import DedunexConfig
    from nanoinfer_b200.models.model import Model
    from nanoinfer_b200.registry import get_architecture
    from nanoinfer_b200.weights import random_tensors, write_safetensors

    cfg = DedunexConfig.from_dict(json.loads(json.dumps(cfg_dict)))
    model = Model(get_architecture(cfg.architecture).build_spec(cfg), cfg)
    tensors = random_tensors(model, seed, 0.02, torch.float32)
    g = torch.Generator().manual_seed(seed + 99)
    rn = lambda t, s=1.0: torch.randn(t.shape, generator=g) * s
    ru = lambda t: torch.rand(t.shape, generator=g)
    for name, t in tensors.items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        if name == "embed":
            t *= 50.0
        elif name == "head":
            t *= 5.0
        elif name == "loop.step":
            t.copy_(rn(t, 0.7))
        elif leaf in ("norm1", "embed.norm", "final.norm"):
            t.copy_(0.4 + 1.2 * ru(t))
        elif leaf.endswith((".q.norm", ".k.norm")):
            t.copy_((1.0 + 0.3 * rn(t)) * sharpen ** 0.5)
        elif leaf in ("mix.dq.norm", "mix.dkv.norm"):
            t.copy_(0.5 + ru(t))
        elif leaf.endswith(("lq1", "lk1", "lq2", "lk2")):
            t.copy_(rn(t, 0.25))
        elif leaf == "mix.z.b":
            t.copy_(ru(t) * 7.0 - 6.0 if not long_memory else ru(t) - 7.0)
        elif leaf.endswith(".b"):
            t.copy_(rn(t, 0.5))
        elif leaf in ("mix.uq", "mix.uk"):
            t.copy_(rn(t, (sharpen / max(1, t.shape[1])) ** 0.5))
        elif leaf in ("mix.g",):
            t *= 12.0
        elif leaf.startswith("mix.") or leaf.startswith("mlp."):
            t *= 6.0
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as fh:
        json.dump(cfg.to_dict(), fh)
    write_safetensors(os.path.join(out_dir, "model.safetensors"), {k: v.to(dtype) for k, v in tensors.items()})
    return out_dir
