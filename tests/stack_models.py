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


def experts(ff=40, n=6, top=2, limit=0.8, shared_ff=None, shared_limit=None):
    """Routed experts; shared_ff: width of a shared expert (None: as wide as the others, 0: none)."""
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=n, top=top))
    if shared_ff != 0:
        mlp["shared"] = dict(ff=shared_ff or ff, limit=shared_limit or limit)
    return mlp


def capped(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.3, softcap=6.0, dims=16, base=3000.0, mlp=experts()):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap, rot=dict(base=base, dims=dims)),
                mlp=mlp)


def differential(heads=4, kv_heads=2, dim=16, vdim=24, window=20, scale=0.35, diff=0.4, dims=12, base=900.0, factor=3.0, mlp=experts()):
    return dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, mask=dict(size=window),
                                               rot=dict(base=base, dims=dims, scaling=dict(factor=factor))), mlp=mlp)


def compressed_latent(heads=3, dim=40, rot_dim=8, vdim=24, kv_rank=48, q_rank=56, window=25, scale=0.17, base=5000.0, mlp=experts()):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
                                                    mask=dict(size=window) if window else None, rot=dict(base=base, dims=rot_dim)), mlp=mlp)


def looped_stack(layers, vocab=90, width=72, eps=3e-5, embed_scale=1.7, buckets=53, mul_prev=31, mul_cur=7, loop=(0, None, 2)):
    cfg = dict(architecture="Sugelix", layers=copy.deepcopy(layers), norm=dict(eps=eps), vocab=vocab, width=width,
               embedding=dict(scale=embed_scale, bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)))
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=len(layers) if loop[1] is None else loop[1], times=loop[2])
    return cfg


def grouped(ff=40, n=6, top=2, groups=2, keep=1, scale=1.5):
    """Experts without gates, chosen among the best groups."""
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=n, top=top, groups=dict(count=groups, keep=keep), scale=scale))


def plain(ff=80):
    return dict(kind="dense", ff=ff)


def side_by_side(heads=4, kv_heads=2, dim=24, vdim=16, window=20, scale=0.3, dims=16, base=3000.0, factor=5.0, width=40, scales=(0.7, 0.45), mlp=plain()):
    """Attention with mixed heads beside a gated average of `width` columns."""
    rot = dict(base=base, dims=dims, **(dict(scaling=dict(factor=factor)) if factor else {})) if dims else None
    left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window) if window else None, rot=rot)
    return dict(type="parallel", mixer=dict(left=left, right=dict(width=width), left_scale=scales[0], right_scale=scales[1]), mlp=mlp)


def memories(heads=3, dim=16, vdim=24, gate_cap=9.0, mlp=plain()):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap), mlp=mlp)


def two_norm_stack(layers, vocab=90, width=72, eps=3e-5, embed_scale=1.7, loop=(0, None, 2)):
    cfg = dict(architecture="Tevilix", layers=copy.deepcopy(layers), norm=dict(eps=eps), vocab=vocab, width=width, embedding=dict(scale=embed_scale))
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=len(layers) if loop[1] is None else loop[1], times=loop[2])
    return cfg


def weights(cfg, seed=0, dtype=torch.bfloat16, gain=1.0, clear_routes=False):
    """Random weights of useful magnitude (projections near unit gain, decays between slow and fast).  clear_routes: a router reads one
    column of the stream per expert, these columns hold well separated values in every embedding row, and no sub-layer writes them."""
    from onnxruntime_genai_b200.models.arch import from_stack_config, stack_weight_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in stack_weight_shapes(from_stack_config(cfg)).items():
        x = torch.randn(shape, generator=g)
        if name.endswith("alpha"):
            x = 0.35 + 0.1 * torch.rand((), generator=g)
        elif name == "bigram" or name == "loop.step":
            x = 0.7 * x
        elif name.endswith(("lq1", "lk1", "lq2", "lk2")):
            x = x / shape[0] ** 0.5                       # a factor well away from its starting value
        elif cfg["architecture"] == "Zevopel" and (name == "final.norm" or name.endswith(("norm1", "norm2"))):
            x = 0.2 * x                                   # stored around zero
        elif name.endswith(("norm", "norm1", "norm2", "ls1", "ls2")):
            x = 1.0 + 0.2 * x
        elif name.endswith("router"):
            x = 2.0 * x / shape[1] ** 0.5
        elif name.endswith("sink"):
            x = x + 0.5
        elif name.endswith("talk"):
            x = torch.eye(shape[0]) + 0.5 * x             # every head's scores show in the others'
        elif name.endswith("correction"):
            x = 0.4 * x
        elif name.endswith(".f.b"):
            x = 2.0 + 1.5 * x                             # memories of a few and of many tokens
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
    if clear_routes and most and cfg["architecture"] == "Tevilix":
        assert most < cfg["width"]
        for v in range(cfg["vocab"]):
            out["embed"][v, :most] = (torch.randperm(most, generator=g).float() / most * 4 - 2).to(dtype)
        for name, x in out.items():
            if name.endswith((".o", ".o.b", ".down")):
                x[:most] = 0
            elif name.endswith("norm2"):
                x[:most] = 1
            elif name.endswith("router"):
                x.zero_()[:, :most].fill_diagonal_(4.0)
            elif name.endswith("correction"):             # groups far apart: their choice is constant
                r = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
                x.copy_((3 * torch.randperm(r["groups"]["count"], generator=g)).repeat_interleave(r["experts"] // r["groups"]["count"]))
    elif clear_routes and most and cfg["architecture"] == "Sugelix":
        assert most < cfg["width"]
        turns = (cfg.get("loop") or dict(times=1))["times"]
        for v in range(cfg["vocab"]):
            out["embed"][v, :most] = ((torch.randperm(most, generator=g).float() / most * 3 - 1.5) / turns / cfg["embedding"]["scale"]).to(dtype)
        out["bigram"][:, :most] = 0
        if "loop.step" in out:
            out["loop.step"][:, :most] = 0
        for name, x in out.items():
            if name.endswith(("mix.o", ".down")):
                x[:most] = 0
            elif name.endswith("norm2"):
                x[:most] = 1
            elif name.endswith("norm2.b"):
                x[:most] = 0
            elif name.endswith("router"):
                x.zero_()[:, :most].fill_diagonal_(3.0)
    elif clear_routes and most:
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
