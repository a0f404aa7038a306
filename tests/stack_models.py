"""Small random declared stacks for the tests: configurations, weights and a checkpoint writer."""
import copy
import json
import os

import torch
from safetensors.torch import save_file


def delta(heads=4, kv_heads=2, dim=24, vdim=16, conv=4, ff=80, **kw):
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def latent(heads=3, dim=40, rot_dim=8, vdim=24, kv_rank=48, window=20, scale=0.17, base=5000.0, factor=3.0, original=32, fast=8.0, slow=1.0, ff=96,
           scaled=True, **kw):
    rot = dict(base=base, dims=rot_dim)
    if scaled:
        rot["scaling"] = dict(factor=factor, original=original, fast=fast, slow=slow)
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                                                    mask=dict(size=window), rot=rot), mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def stack(layers, vocab=90, width=72, eps=3e-5):
    return dict(architecture="Luzatar", layers=copy.deepcopy(layers), norm=dict(eps=eps), vocab=vocab, width=width)


def chunked(heads=4, kv_heads=2, dim=24, vdim=16, chunk=20, scale=0.4, dims=16, base=3000.0, factor=5.0, original=60, low=1.0, high=4.0, ff=80, scaled=True,
            experts=0, top=2, limit=0.7, **kw):
    """A chunked-attention layer; experts > 0: routed experts of width ff instead of a dense feed-forward."""
    rot = dict(base=base, dims=dims)
    if scaled:
        rot["scaling"] = dict(factor=factor, original=original, low=low, high=high)
    mlp = dict(kind="dense", ff=ff) if ff else None
    if experts:
        mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=chunk), rot=rot), mlp=mlp, **kw)


def output_normed_stack(layers, vocab=90, width=72, eps=3e-5, residual_mult=0.6, embed_scale=1.7):
    return dict(architecture="Zevopel", layers=copy.deepcopy(layers), norm=dict(eps=eps), vocab=vocab, width=width, residual_mult=residual_mult,
                embedding=dict(scale=embed_scale))


def weights(cfg, seed=0, dtype=torch.bfloat16, gain=1.0, clear_routes=False):
    """Random weights of useful magnitude (projections near unit gain, decays between slow and fast).  clear_routes: a router reads one
    column of the stream per expert, these columns hold well separated values in every embedding row, and no sub-layer writes them."""
    from onnxruntime_genai_b200.models.arch import from_stack_config, stack_weight_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in stack_weight_shapes(from_stack_config(cfg)).items():
        x = torch.randn(shape, generator=g)
        if cfg["architecture"] == "Zevopel" and (name == "final.norm" or name.endswith(("norm1", "norm2"))):
            x = 0.2 * x                                   # stored around zero
        elif name.endswith(("norm", "norm1", "ls1", "ls2")):
            x = 1.0 + 0.2 * x
        elif name.endswith("router"):
            x = 2.0 * x / shape[1] ** 0.5
        elif name.endswith("sink"):
            x = x + 0.5
        elif name.endswith(".b") and len(shape) == 1 or name.endswith("dt_bias"):
            x = 0.3 * x
        elif name.endswith("A_log"):
            x = 0.7 * x - 1.0
        elif name.endswith(".conv"):
            x = 0.6 * x
        elif name == "embed":
            pass
        else:
            x = gain * x / shape[1] ** 0.5
        out[name] = x.to(dtype)
    most = max([e["mlp"]["router"]["experts"] for e in cfg["layers"] if (e.get("mlp") or {}).get("kind") == "moe"], default=0)
    if clear_routes and most:
        assert most < cfg["width"]
        for v in range(cfg["vocab"]):
            out["embed"][v, :most] = (torch.randperm(most, generator=g).float() / most * 3 - 1.5).to(dtype)
        for i, e in enumerate(cfg["layers"]):
            for n in ("norm1", "norm2"):
                if f"l{i}.{n}" in out:
                    out[f"l{i}.{n}"][:most] = -1.0
            if (e.get("mlp") or {}).get("kind") == "moe":
                out[f"l{i}.mlp.router"].zero_()[:, :most].fill_diagonal_(1.0)
    return out


def write(cfg, w, path):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return str(path)
