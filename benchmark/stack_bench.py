"""Prefill and decode throughput of a declared stack beside the closest other model of the framework at equal size.  Luzatar: the
gated-delta-net + full-attention hybrid (Qwen3.5 style) with the same width, feed-forward, layer count, delta layers and attention heads.
Zevopel: Qwen3-style dense layers (normed query and key heads), and gpt-oss-style layers with bf16 experts (sinks, clamped experts), each
with the same width, heads and feed-forwards; the chunks are as long as the context, so both attend to the same keys.  Sugelix: gpt-oss-style
layers again, as many as the design runs, with the same width, head count, key and value sizes and as many experts per token (one of the
design's is the shared one); soft-capped scores on both sides where the design's layers have them.  Tevilix: the Qwen3.5-style hybrid again, its
delta layers in the places of the matrix memories (as many states of the same size), its attention in those of the pairs of attention and gated
average, with the same heads and the same feed-forward (dense, or as many experts of the same width); windows as long as the context.  Random weights drawn
on the device; CUDA events around whole decoder forwards (decode steps replay a CUDA graph); the weights and caches of a step are larger
than L2.  Reached through `python bench.py --design luzatar | zevopel | sugelix | tevilix`."""
import json
import os
import shutil
import tempfile

import numpy as np
import torch

SIZES = {
    # name: width, ff, layers (alternating delta / attention), attention heads, kv heads of the hybrid, delta key heads, delta value heads
    "2k": dict(width=2048, ff=6144, layers=16, heads=16, kv=4, dk=8, dv=16, vocab=65536),
    "4k": dict(width=4096, ff=12288, layers=8, heads=32, kv=8, dk=16, dv=32, vocab=65536),
}
ZEVOPEL_SIZES = {
    # name: width, feed-forward (of one expert where there are experts), layers, heads, kv heads, head size
    "2k dense": dict(width=2048, ff=6144, layers=16, heads=16, kv=4, dim=128, vocab=65536),
    "4k dense": dict(width=4096, ff=12288, layers=8, heads=32, kv=8, dim=128, vocab=65536),
    "2.9k experts": dict(width=2880, ff=2880, layers=8, heads=64, kv=8, dim=64, vocab=65536, experts=32, top=4),
}
SUGELIX_SIZES = {
    # name: the layers' mixers ("a" soft-capped, "d" differential, "l" latent), how often the stack runs, width, one expert's feed-forward, heads,
    # kv heads, head size (of both maps together where there are two), experts (one more is shared), experts per token with the shared one
    "2.9k capped": dict(mixers="aaaaaaaa", times=1, width=2880, ff=2880, heads=32, kv=8, dim=128, vocab=65536, experts=32, top=4, softcap=50.0),
    "2.9k differential": dict(mixers="dddddddd", times=1, width=2880, ff=2880, heads=32, kv=8, dim=128, vocab=65536, experts=32, top=4),
    "2.9k latent": dict(mixers="llllllll", times=1, width=2880, ff=2880, heads=32, kv=8, dim=128, vocab=65536, experts=32, top=4),
    "2k mixed, twice": dict(mixers="adal", times=2, width=2048, ff=1024, heads=16, kv=4, dim=128, vocab=65536, experts=64, top=6, softcap=50.0),
}
TEVILIX_SIZES = {
    # name: width, feed-forward (of one expert where there are experts), layers (alternating memories / attention beside a gated average), attention heads,
    # kv heads, head size, columns of the gated average, heads of the memories (128 x 128 each; dk, dv: the hybrid's key and value heads)
    "2k dense": dict(width=2048, ff=6144, layers=16, heads=16, kv=4, dim=128, gru=1024, dk=8, dv=16, vocab=65536),
    "4k dense": dict(width=4096, ff=12288, layers=8, heads=32, kv=4, dim=128, gru=2048, dk=16, dv=32, vocab=65536),
    "2k experts": dict(width=2048, ff=1024, layers=16, heads=16, kv=2, dim=128, gru=1024, dk=8, dv=16, vocab=65536, experts=64, top=6, groups=8, keep=4),
}
PREFILL = [(1, 4096), (8, 1024)]
DECODE = [(1, 2048), (16, 2048), (64, 2048), (256, 1024)]
BLOCK = 16


def luzatar_dir(z, path):
    delta = dict(type="delta", mixer=dict(heads=z["dv"], kv_heads=z["dk"], dim=128, vdim=128, conv=4), mlp=dict(kind="dense", ff=z["ff"]))
    lat = dict(type="latent_attention", mixer=dict(heads=z["heads"], dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, mask=dict(size=8192),
                                                   rot=dict(base=1e6, dims=64)), mlp=dict(kind="dense", ff=z["ff"]))
    cfg = dict(architecture="Luzatar", layers=[delta, lat] * (z["layers"] // 2), norm=dict(eps=1e-6), vocab=z["vocab"], width=z["width"])
    os.makedirs(os.path.join(path, "src"), exist_ok=True)
    with open(os.path.join(path, "src", "config.json"), "w") as f:
        json.dump(cfg, f)
    from onnxruntime_genai_b200.models.builder import create_model
    return create_model(os.path.join(path, "src"), os.path.join(path, "model"), "bf16", "cuda", {"synthetic_weights": 1, "context_length": 8192})


def tevilix_dir(z, path):
    mlp = dict(kind="dense", ff=z["ff"])
    if z.get("experts"):
        mlp = dict(kind="moe", expert=dict(ff=z["ff"]), router=dict(experts=z["experts"], top=z["top"], groups=dict(count=z["groups"], keep=z["keep"]), scale=1.0))
    d = z["dim"]
    pair = dict(left=dict(heads=z["heads"], kv_heads=z["kv"], dim=d, vdim=d, scale=d ** -0.5, mask=dict(size=8192),
                          rot=dict(base=5e5, dims=d, scaling=dict(factor=4.0))), right=dict(width=z["gru"]), left_scale=0.7, right_scale=0.5)
    layers = [dict(type="mlstm", mixer=dict(heads=z["dv"], dim=128, vdim=128, gate_cap=15.0), mlp=mlp), dict(type="parallel", mixer=pair, mlp=mlp)] * (z["layers"] // 2)
    cfg = dict(architecture="Tevilix", layers=layers, norm=dict(eps=1e-6), vocab=z["vocab"], width=z["width"], embedding=dict(scale=1.0))
    os.makedirs(os.path.join(path, "src"), exist_ok=True)
    with open(os.path.join(path, "src", "config.json"), "w") as f:
        json.dump(cfg, f)
    from onnxruntime_genai_b200.models.builder import create_model
    return create_model(os.path.join(path, "src"), os.path.join(path, "model"), "bf16", "cuda", {"synthetic_weights": 1, "context_length": 8192})


def hybrid_dir(z, path):
    from onnxruntime_genai_b200.models.arch import ArchConfig
    from onnxruntime_genai_b200.models.builder import export_model
    a = ArchConfig(model_type="qwen3_next", vocab_size=z["vocab"], hidden_size=z["width"], num_layers=z["layers"], num_heads=z["heads"],
                   num_kv_heads=z["kv"], head_dim=128, intermediate_size=z["ff"], context_length=8192, bos_token_id=0, eos_token_id=1, pad_token_id=0,
                   layer_types=["linear_attention", "full_attention"] * (z["layers"] // 2), linear_num_key_heads=z["dk"], linear_num_value_heads=z["dv"],
                   linear_key_head_dim=128, linear_value_head_dim=128, linear_conv_kernel_dim=4)
    if z.get("experts"):
        a.moe_style, a.num_experts, a.experts_per_token = "standard", z["experts"], z["top"]
    return export_model(a, path, precision="bf16", execution_provider="cuda", paged=True, block_size=BLOCK, synthetic_weights=True)


def zevopel_dir(z, path):
    mlp = dict(kind="dense", ff=z["ff"])
    if z.get("experts"):
        mlp = dict(kind="moe", expert=dict(ff=z["ff"], limit=7.0), router=dict(experts=z["experts"], top=z["top"]))
    layer = dict(type="attention", mlp=mlp, mixer=dict(heads=z["heads"], kv_heads=z["kv"], dim=z["dim"], vdim=z["dim"], scale=z["dim"] ** -0.5,
                                                       mask=dict(size=8192), rot=dict(base=5e5, dims=z["dim"])))
    cfg = dict(architecture="Zevopel", layers=[layer] * z["layers"], norm=dict(eps=1e-6), vocab=z["vocab"], width=z["width"], residual_mult=0.3,
               embedding=dict(scale=1.0))
    os.makedirs(os.path.join(path, "src"), exist_ok=True)
    with open(os.path.join(path, "src", "config.json"), "w") as f:
        json.dump(cfg, f)
    from onnxruntime_genai_b200.models.builder import create_model
    return create_model(os.path.join(path, "src"), os.path.join(path, "model"), "bf16", "cuda", {"synthetic_weights": 1, "context_length": 8192})


def closest_to_zevopel_dir(z, path):
    from onnxruntime_genai_b200.models.arch import ArchConfig
    from onnxruntime_genai_b200.models.builder import export_model
    a = ArchConfig(model_type="qwen3", vocab_size=z["vocab"], hidden_size=z["width"], num_layers=z["layers"], num_heads=z["heads"], num_kv_heads=z["kv"],
                   head_dim=z["dim"], intermediate_size=z["ff"], context_length=8192, qk_norm=True, rope_theta=5e5, bos_token_id=0, eos_token_id=1,
                   pad_token_id=0)
    if z.get("experts"):
        a.model_type, a.qk_norm, a.attn_bias, a.o_bias, a.mlp_bias, a.attn_sinks = "gptoss", False, True, True, True, True
        a.num_experts, a.experts_per_token = z["experts"], z["top"]
    return export_model(a, path, precision="bf16", execution_provider="cuda", paged=True, block_size=BLOCK, synthetic_weights=True)


def sugelix_dir(z, path):
    d, mlp = z["dim"], dict(kind="moe", expert=dict(ff=z["ff"], limit=7.0), shared=dict(ff=z["ff"], limit=7.0), router=dict(experts=z["experts"], top=z["top"] - 1))
    kinds = {"a": ("attention", dict(heads=z["heads"], kv_heads=z["kv"], dim=d, vdim=d, scale=d ** -0.5, softcap=z.get("softcap"), rot=dict(base=5e5, dims=d))),
             "d": ("attention_2", dict(heads=z["heads"], kv_heads=z["kv"], dim=d // 2, vdim=d, scale=(d // 2) ** -0.5, diff=0.5, mask=dict(size=8192),
                                       rot=dict(base=5e5, dims=d // 2, scaling=dict(factor=8.0)))),
             "l": ("latent_attention", dict(heads=z["heads"], dim=d, rot_dim=64, vdim=d, kv_rank=512, q_rank=1024, scale=(d + 64) ** -0.5, mask=dict(size=8192),
                                            rot=dict(base=5e5, dims=64)))}
    cfg = dict(architecture="Sugelix", layers=[dict(type=kinds[m][0], mixer=kinds[m][1], mlp=mlp) for m in z["mixers"]], norm=dict(eps=1e-6), vocab=z["vocab"],
               width=z["width"], embedding=dict(scale=z["width"] ** 0.5, bigram=dict(buckets=50021, mul_prev=31, mul_cur=17)))
    if z["times"] > 1:
        cfg["loop"] = dict(start=0, stop=len(z["mixers"]), times=z["times"])
    os.makedirs(os.path.join(path, "src"), exist_ok=True)
    with open(os.path.join(path, "src", "config.json"), "w") as f:
        json.dump(cfg, f)
    from onnxruntime_genai_b200.models.builder import create_model
    return create_model(os.path.join(path, "src"), os.path.join(path, "model"), "bf16", "cuda", {"synthetic_weights": 1, "context_length": 8192})


def closest_to_sugelix_dir(z, path):
    from onnxruntime_genai_b200.models.arch import ArchConfig
    from onnxruntime_genai_b200.models.builder import export_model
    a = ArchConfig(model_type="gptoss", vocab_size=z["vocab"], hidden_size=z["width"], num_layers=len(z["mixers"]) * z["times"], num_heads=z["heads"],
                   num_kv_heads=z["kv"], head_dim=z["dim"], intermediate_size=z["ff"], context_length=8192, rope_theta=5e5, attn_bias=True, o_bias=True,
                   mlp_bias=True, num_experts=z["experts"] + 1, experts_per_token=z["top"], bos_token_id=0, eos_token_id=1, pad_token_id=0)
    if z.get("softcap"):
        a.softcap = z["softcap"]
    else:
        a.attn_sinks = True
    return export_model(a, path, precision="bf16", execution_provider="cuda", paged=True, block_size=BLOCK, synthetic_weights=True)


DESIGNS = {"tevilix": (TEVILIX_SIZES, tevilix_dir, "hybrid", hybrid_dir), "sugelix": (SUGELIX_SIZES, sugelix_dir, "closest", closest_to_sugelix_dir), "luzatar": (SIZES, luzatar_dir, "hybrid", hybrid_dir), "zevopel": (ZEVOPEL_SIZES, zevopel_dir, "closest", closest_to_zevopel_dir)}


def _step(model, lens):
    """(StepInputs, cache) of a step with the given (past, new) lengths over fresh zero caches."""
    from onnxruntime_genai_b200.models.decoder import PagedKVCache, StepInputs
    dec = model.decoder
    nb = [(p + n + BLOCK - 1) // BLOCK for p, n in lens]
    kv = PagedKVCache(dec.arch, sum(nb), BLOCK, "cuda", dec.dtype, kv_heads=dec.kv_heads_local, conv_channels=dec.conv_channels_local)
    kv.ensure_state_slots(len(lens))
    for pool in (kv.full, kv.conv, kv.latent, kv.state, *(p for pools in kv.spec_kv.values() for p in pools)):
        if pool is not None and pool.numel():
            pool.normal_(0, 0.1)
    table = np.zeros((len(lens), max(nb)), dtype=np.int32)
    at, pos, slots = 0, [], []
    for b, (p, n) in enumerate(lens):
        table[b, :nb[b]] = np.arange(at, at + nb[b])
        q = np.arange(p, p + n)
        pos.append(q)
        slots.append(at * BLOCK + q)
        at += nb[b]
    t = lambda x: torch.from_numpy(np.asarray(x, dtype=np.int32)).cuda()
    cu = np.cumsum([0] + [n for _, n in lens])
    ids = np.random.RandomState(1).randint(0, dec.arch.vocab_size, int(cu[-1]))
    s = StepInputs(input_ids=t(ids), positions=t(np.concatenate(pos)), slot_mapping=t(np.concatenate(slots)), cu_seqlens=t(cu),
                   past_lens=t([p for p, _ in lens]), block_table=t(table), logits_rows=t(cu[1:] - 1), max_q_len=max(n for _, n in lens),
                   max_kv_len=max(p + n for p, n in lens), min_q_len=min(n for _, n in lens), host_lens=list(lens),
                   state_slots=t(np.arange(len(lens))))
    return s, kv


def _time(fn, iters, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


def measure(model, steps, warmup):
    from onnxruntime_genai_b200 import ops
    from onnxruntime_genai_b200.ops import _lib
    out = {}
    with torch.no_grad():
        for n, length in PREFILL:
            s, kv = _step(model, [(0, length)] * n)
            ms = _time(lambda: model.decoder.forward(s, kv), max(3, steps // 10), warmup)
            out[f"prefill {n}x{length}"] = {"ms": round(ms, 3), "tokens_per_s": round(n * length / ms * 1e3)}
            del s, kv
        for n, past in DECODE:
            s, kv = _step(model, [(past, 1)] * n)
            model.decoder.forward(s, kv)
            torch.cuda.synchronize()
            before = _lib.LAUNCH_COUNT
            g = torch.cuda.CUDAGraph()
            with ops.graph_capture(g):
                model.decoder.forward(s, kv)
            launches = _lib.LAUNCH_COUNT - before
            ms = _time(g.replay, steps, warmup)
            out[f"decode {n} at {past}"] = {"ms": round(ms, 4), "tokens_per_s": round(n / ms * 1e3), "launches": launches}
            del g, s, kv
    ops.check_kernel_status()
    torch.cuda.empty_cache()
    return out


def run(sampler, steps=50, warmup=3, sizes=None, design="luzatar"):
    import onnxruntime_genai_b200 as og
    table, make_design, other, make_other = DESIGNS[design]
    result = {}
    for name in sizes or table:
        z = table[name]
        result[name] = {"shape": z}
        for label, make in ((design, make_design), (other, make_other)):
            d = tempfile.mkdtemp(prefix="ogb_stack_")
            try:
                model = og.Model(make(z, d))
                sampler.start()
                result[name][label] = measure(model, steps, warmup)
                result[name][label]["clocks"] = sampler.stop()
                result[name][label]["weight_gb"] = round(model.decoder.weight_bytes() / 1e9, 2)
                del model
            finally:
                shutil.rmtree(d, ignore_errors=True)
            torch.cuda.empty_cache()
        mine, theirs = result[name][design], result[name][other]
        pairs = [k for k in mine if isinstance(mine[k], dict) and "ms" in mine[k]]
        result[name][f"time ratio {design} / {other}"] = {k: round(mine[k]["ms"] / theirs[k]["ms"], 3) for k in pairs}
    return result
