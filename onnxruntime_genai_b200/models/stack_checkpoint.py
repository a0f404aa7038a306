"""Checkpoints of declared stacks: a directory with `config.json` (the layers one by one, see arch.from_stack_config) and
`model.safetensors` (weights [out, in] under the names of arch.stack_weight_shapes).

Such a directory is a model directory as it is: `Model(path)` reads it without an export step, with the genai_config.json that the
builder would have written made in memory (`genai_config_of`).  A directory exported by the builder holds the same two files beside
its genai_config.json.  A weights file named `*.synthetic.json` ({"seed", "std"}) stands for random weights drawn on the device."""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

import torch

from .arch import ArchConfig, from_stack_config, is_stack_config, rotary_tables, stack_weight_shapes
from .decoder import DecoderModel, LayerWeights

WEIGHTS = "model.safetensors"


def read_stack_config(model_dir: str) -> Optional[dict]:
    """config.json of the directory when it describes a declared stack, else None."""
    path = os.path.join(model_dir, "config.json")
    if not os.path.isfile(path):
        return None
    with open(path) as f:
        cfg = json.load(f)
    return cfg if is_stack_config(cfg) else None


def genai_config_of(cfg: dict, execution_provider: str = "cuda", precision: str = "bf16", filename: str = WEIGHTS, block_size: int = 16,
                    max_batch_size: int = 64, context_length: Optional[int] = None) -> dict:
    """The genai_config.json document of a declared stack."""
    from .builder import make_genai_config
    arch = from_stack_config(cfg)
    if context_length:
        arch.context_length = int(context_length)
    doc = make_genai_config(arch, precision, execution_provider, True, block_size, max_batch_size, filename=filename)
    if execution_provider == "cuda":
        doc["model"]["decoder"]["session_options"]["provider_options"] = [{"cuda": {"compute_dtype": "float32" if precision == "fp32" else "bfloat16"}}]
    return doc


def _file_tensors(path: str) -> Callable[[str], torch.Tensor]:
    from safetensors import safe_open
    f = safe_open(path, framework="pt", device="cpu")
    names = set(f.keys())

    def get(name):
        if name not in names:
            raise ValueError(f"{path}: tensor '{name}' is missing")
        return f.get_tensor(name)
    return get


def _synthetic_tensors(path: str, shapes: Dict[str, tuple], device, norm_offset: float = 0.0) -> Callable[[str], torch.Tensor]:
    from .builder import random_tensor
    with open(path) as f:
        meta = json.load(f)

    def get(name):
        t = random_tensor(name, shapes[name], int(meta.get("seed", 0)), float(meta.get("std", 0.02)), device=device)
        around_one = name.endswith((".norm", "norm1", "norm2")) and (norm_offset == 0 or ".mix." in name) or name.endswith(("ls1", "ls2"))
        return t + 1.0 if around_one else t
    return get


def load_stack_decoder(model_dir: str, filename: str, context_length: int, device, dtype, tp=None) -> DecoderModel:
    if tp is not None and getattr(tp, "size", 1) > 1:
        raise NotImplementedError("declared stacks are not sharded: run these models on one GPU")
    cfg = read_stack_config(model_dir)
    if cfg is None:
        raise ValueError(f"{model_dir}: config.json does not describe a declared stack")
    arch = from_stack_config(cfg)
    arch.context_length = context_length
    path = os.path.join(model_dir, filename)
    shapes = stack_weight_shapes(arch)
    get = _synthetic_tensors(path, shapes, device, arch.norm_offset) if filename.endswith(".synthetic.json") else _file_tensors(path)
    return build_stack_decoder(arch, get, device, dtype)


def build_stack_decoder(arch: ArchConfig, get: Callable[[str], torch.Tensor], device, dtype) -> DecoderModel:
    """DecoderModel from a tensor source: input projections stacked per layer, the key map transposed per head, the output projections
    of both sub-layers of a parallel block joined side by side, the factors on a sub-layer's normed output multiplied into one vector,
    experts stacked, heads and feed-forwards filled up with zeros where a kernel wants whole tiles, small vectors and recurrence constants
    in fp32."""
    shapes = stack_weight_shapes(arch)
    model = DecoderModel(arch, device, dtype)
    cuda = torch.device(device).type == "cuda"

    def raw(name):
        t = get(name)
        if tuple(t.shape) != tuple(shapes[name]):
            raise ValueError(f"tensor '{name}' has shape {tuple(t.shape)}, the configuration asks for {tuple(shapes[name])}")
        return t.to(device)

    def mat(*names):
        return torch.cat([raw(n) for n in names], 0).to(dtype).contiguous()

    def vec(name):
        return raw(name).float().contiguous()

    tables: Dict[tuple, tuple] = {}

    def rotary(spec):
        if spec is None:
            return None, None
        if spec.key() not in tables:
            tables[spec.key()] = tuple(torch.from_numpy(t).to(device) for t in rotary_tables(spec, arch.context_length))
        return tables[spec.key()]

    up8 = lambda n: (n + 7) // 8 * 8      # columns of the joined input start on 16-byte boundaries
    tiled = cuda and dtype == torch.bfloat16

    def head_rows(name, heads, size, row):
        """[heads * size, K] -> [heads * row, K]: every head filled up with zero rows."""
        w = raw(name).to(dtype)
        return w if size == row else torch.nn.functional.pad(w.view(heads, size, -1), (0, 0, 0, row - size)).reshape(heads * row, -1)

    def attention_weights(lw, sp, m):
        lw.qkv_w = torch.cat([head_rows(m + "q", sp.heads, sp.dim, sp.key_row), head_rows(m + "k", sp.kv_heads, sp.dim, sp.key_row),
                              head_rows(m + "v", sp.kv_heads, sp.vdim, sp.value_row)] + ([raw(m + "g").to(dtype)] if sp.head_gate else []), 0).contiguous()
        if sp.qk_norm:
            lw.q_norm_w, lw.k_norm_w = vec(m + "q.norm"), vec(m + "k.norm")
        if sp.sinks:
            lw.sinks = vec(m + "sink")
        lw.rope_cos, lw.rope_sin = rotary(sp.rotary)

    def output_map(name, sp):
        """The mixer's output map over its heads as they leave the mixer."""
        w = raw(name).to(dtype)
        if sp.kind != "attention" or sp.vdim == sp.value_row:
            return w.contiguous()
        return torch.nn.functional.pad(w.view(-1, sp.heads, sp.vdim), (0, sp.value_row - sp.vdim)).reshape(w.shape[0], -1).contiguous()

    def output_factor(p, n):
        """What multiplies a sub-layer's normalised output: norm weight, layer scale and residual multiplier."""
        w = (vec(f"{p}norm{n}") + arch.norm_offset) * arch.residual_multiplier
        return w * vec(f"{p}ls{n}") if arch.layer_scale else w

    def feed_forward(lw, sp, p):
        from ..ops import interleave_gate_up
        lw.gate_up_w, lw.down_w = mat(p + "gate", p + "up"), mat(p + "down")
        if tiled:      # whole blocks of 64 features (zero gates and zero ups give zero)
            fill = (-sp.ff) % 64
            w = torch.nn.functional.pad(lw.gate_up_w.view(2, sp.ff, -1), (0, 0, 0, fill)).reshape(2 * (sp.ff + fill), -1)
            lw.gate_up_w, lw.gate_up_interleaved = interleave_gate_up(w), True
            lw.down_w = torch.nn.functional.pad(lw.down_w, (0, fill)).contiguous()

    def expert_weights(lw, sp, p):
        from ..ops import interleave_experts_gate_up
        E, W = sp.moe.experts, arch.hidden_size
        lw.moe, lw.router_w, lw.exp_hi = sp.moe, mat(p + "router"), E
        lw.exp_blocked = tiled and W % 8 == 0
        F = (sp.ff + 63) // 64 * 64 if lw.exp_blocked else sp.ff      # (an expert's zero gates give zero, whatever its ups are)
        gate_up = torch.zeros(E, 2, F, W, dtype=dtype, device=device)
        lw.exp_down_w = torch.zeros(E, W, F, dtype=dtype, device=device)
        for e in range(E):
            gate_up[e, 0, :sp.ff], gate_up[e, 1, :sp.ff] = raw(f"{p}e{e}.gate").to(dtype), raw(f"{p}e{e}.up").to(dtype)
            lw.exp_down_w[e, :, :sp.ff] = raw(f"{p}e{e}.down").to(dtype)
        if lw.exp_blocked:
            lw.exp_gate_up_w = interleave_experts_gate_up(gate_up.view(E, 2 * F, W), fused_interleaved=False)
        else:
            lw.exp_gate_up_w = gate_up.transpose(1, 2).reshape(E, 2 * F, W).contiguous()

    def layer(i) -> LayerWeights:
        sp, p, m = arch.layer_specs[i], f"l{i}.", f"l{i}.mix."
        lw = LayerWeights(ln1_w=None, qkv_w=None, o_w=None, ln2_w=None)
        lw.mix_cols = sp.heads * (sp.value_row or sp.vdim)
        if sp.kind == "linear_attention":
            lw.lin_in_w = mat(m + "q", m + "k", m + "v", m + "g", m + "b", m + "a")
            lw.lin_conv_w = mat(m + "q.conv", m + "k.conv", m + "v.conv")
            lw.lin_neg_exp_a = -torch.exp(vec(m + "A_log"))
            lw.lin_dt_bias, lw.lin_norm_w = vec(m + "dt_bias"), vec(m + "norm")
        elif sp.kind == "attention":
            attention_weights(lw, sp, m)
        else:
            lw.lat_in_w = mat(m + "q", m + "dkv")
            lw.lat_norm_w = vec(m + "dkv.norm")
            lw.lat_uk_t = mat(m + "uk").view(sp.heads, sp.dim, sp.kv_rank).transpose(1, 2).reshape(sp.heads * sp.kv_rank, sp.dim).contiguous()
            lw.lat_ukv = mat(m + "uk", m + "uv")
            lw.lat_uv = lw.lat_ukv[sp.heads * sp.dim:]
            lw.rope_cos, lw.rope_sin = rotary(sp.rotary)
        if not arch.parallel_block:
            lw.o_w, lw.post_attn_norm_w = output_map(m + "o", sp), output_factor(p, 1)
            if sp.ff:
                (feed_forward if sp.moe is None else expert_weights)(lw, sp, p + "mlp.")
                lw.post_ffn_norm_w = output_factor(p, 2)
            return lw
        lw.ln1_w, lw.ln1_b = vec(p + "norm1"), vec(p + "norm1.b") if arch.layernorm else None
        lw.mlp_col = up8(lw.mix_cols)
        lw.join_w = torch.zeros(arch.hidden_size, lw.mlp_col + up8(sp.ff), dtype=dtype, device=device)
        lw.join_w[:, :lw.mix_cols] = output_map(m + "o", sp)
        if sp.ff:
            lw.join_w[:, lw.mlp_col:lw.mlp_col + sp.ff] = raw(p + "mlp.down").to(dtype)
            lw.gate_up_w = mat(p + "mlp.gate", p + "mlp.up")
            if tiled and sp.ff % 64 == 0:
                from ..ops import interleave_gate_up
                lw.gate_up_w, lw.gate_up_interleaved = interleave_gate_up(lw.gate_up_w), True
        return lw

    model.embed, model.lm_head_w = mat("embed"), mat("head")
    model.final_norm_w = vec("final.norm") + arch.norm_offset
    model.final_norm_b = vec("final.norm.b") if arch.layernorm else None
    own = {i: layer(i) for i, sp in enumerate(arch.layer_specs) if sp.weights_of is None}
    model.layers = [own[i if sp.weights_of is None else sp.weights_of] for i, sp in enumerate(arch.layer_specs)]
    return model
