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
        if name.endswith("alpha"):
            return torch.full_like(t, 0.5)
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
    experts stacked, two mixers' input projections joined where they stand side by side, heads and feed-forwards filled up with zeros where a
    kernel wants whole tiles, small vectors and recurrence constants in fp32."""
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

    def padded(w, heads, size, row):
        """[heads * size, ...] -> [heads * row, ...]: every head filled up with zero rows."""
        if size == row:
            return w
        v = w.reshape(heads, size, -1)
        return torch.nn.functional.pad(v, (0, 0, 0, row - size)).reshape(heads * row, *w.shape[1:])

    def attention_weights(lw, sp, m):
        # neighbours that rotate as pairs are brought to the places of the two halves: the same permutation of queries and keys
        def halves(t):
            n = sp.rotary.dims if sp.rotary and sp.rotary.neighbours else 0
            if not n:
                return t
            t = t.view(-1, sp.dim, *t.shape[1:])
            return torch.cat([t[:, 0:n:2], t[:, 1:n:2], t[:, n:]], 1).flatten(0, 1)

        def rows(name, heads, size, row, place=lambda t: t):
            return padded(place(raw(name).to(dtype)), heads, size, row)
        sizes = [("q", sp.heads * sp.maps, sp.dim, sp.map_row, halves), ("k", sp.kv_heads * sp.maps, sp.dim, sp.map_row, halves),
                 ("v", sp.kv_heads, sp.vdim, sp.value_row, lambda t: t)]
        parts = [rows(m + n, *z) for n, *z in sizes]
        gates = []
        if sp.head_gate:
            gates = [raw(m + "g").to(dtype)]
        elif sp.out_gate:
            gates = [rows(m + "g", sp.heads, sp.vdim, sp.value_row)]
        lw.qkv_w = torch.cat(parts + gates, 0).contiguous()
        if sp.qkv_bias:
            b = torch.cat([rows(f"{m}{n}.b", *z) for n, *z in sizes])
            lw.qkv_b = torch.nn.functional.pad(b, (0, lw.qkv_w.shape[0] - b.numel())).contiguous()
        if sp.qk_norm:
            lw.q_norm_w, lw.k_norm_w = halves(vec(m + "q.norm")).contiguous(), halves(vec(m + "k.norm")).contiguous()
        if sp.maps == 2:
            lam = [torch.exp((vec(f"{m}lq{i}") * vec(f"{m}lk{i}")).sum()) for i in (1, 2)]
            lw.diff_lambda = float(lam[0] - lam[1]) + sp.diff
        if sp.sinks:
            lw.sinks = vec(m + "sink")
        if sp.talk:
            lw.talk = vec(m + "talk")
        lw.rope_cos, lw.rope_sin = rotary(sp.rotary)

    def add_beside(lw, sp, m):
        """The projections [update gate | candidate | output gate] of a gated average, each filled up to whole 16-byte pieces, behind the projection of
        the mixer it stands beside."""
        W = lw.qkv_w.shape[1]
        fill = (0, (-sp.vdim) % 8)
        parts = [torch.nn.functional.pad(raw(m + n).to(dtype), (0, 0) + fill) for n in ("z", "x", "g")]
        bias = [torch.nn.functional.pad(raw(m + n).to(dtype), fill) for n in ("z.b", "x.b")]
        lw.beside_in = up8(lw.qkv_w.shape[0])
        gap = lw.beside_in - lw.qkv_w.shape[0]
        first = lw.qkv_b if lw.qkv_b is not None else lw.qkv_w.new_zeros(lw.qkv_w.shape[0])
        lw.qkv_w = torch.cat([lw.qkv_w, lw.qkv_w.new_zeros(gap, W)] + parts, 0).contiguous()
        lw.qkv_b = torch.cat([first, first.new_zeros(gap)] + bias + [torch.zeros_like(bias[0])]).contiguous()

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
        if sp.moe.weights == "sigmoid":
            lw.router_b = vec(p + "correction")
        names = [f"{p}e{e}." for e in range(E)]
        if not sp.moe.gated:
            F = up8(sp.ff) if lw.exp_blocked else sp.ff
            lw.exp_gate_up_w = torch.zeros(E, F, W, dtype=dtype, device=device)
            lw.exp_down_w = torch.zeros(E, W, F, dtype=dtype, device=device)
            for e, n in enumerate(names):
                lw.exp_gate_up_w[e, :sp.ff], lw.exp_down_w[e, :, :sp.ff] = raw(n + "up").to(dtype), raw(n + "down").to(dtype)
            return
        # a shared expert of the same width and limit is one more expert that every token takes
        ff2 = sp.moe.shared_ff
        lw.exp_shared = ff2 == sp.ff and sp.moe.shared_limit == sp.moe.limit and E < 1024 and sp.moe.top < 32
        if lw.exp_shared:
            names.append(p + "shared.")
        elif ff2:
            gate, up = raw(p + "shared.gate").to(dtype), raw(p + "shared.up").to(dtype)
            fill = (-ff2) % 8                                          # rows of whole 16-byte pieces
            lw.shared_gate_up_w = torch.nn.functional.pad(torch.stack([gate, up], 1), (0, 0, 0, 0, 0, fill)).reshape(2 * (ff2 + fill), W).contiguous()
            lw.shared_down_w = torch.nn.functional.pad(raw(p + "shared.down").to(dtype), (0, fill)).contiguous()
        E = len(names)
        gate_up = torch.zeros(E, 2, F, W, dtype=dtype, device=device)
        lw.exp_down_w = torch.zeros(E, W, F, dtype=dtype, device=device)
        for e, n in enumerate(names):
            gate_up[e, 0, :sp.ff], gate_up[e, 1, :sp.ff] = raw(n + "gate").to(dtype), raw(n + "up").to(dtype)
            lw.exp_down_w[e, :, :sp.ff] = raw(n + "down").to(dtype)
        if lw.exp_blocked:
            lw.exp_gate_up_w = interleave_experts_gate_up(gate_up.view(E, 2 * F, W), fused_interleaved=False)
        else:
            lw.exp_gate_up_w = gate_up.transpose(1, 2).reshape(E, 2 * F, W).contiguous()

    def tanh_norm(name):
        from ..ops import TanhNorm
        return TanhNorm(vec(name), vec(name + ".b"), float(raw(name + ".alpha")))

    def latent_input(lw, sp, m):
        """Input projection of a latent-attention layer: [queries or their latent | latent and shared rotary key | gate logits], the parts
        starting on 16-byte boundaries where there are more than the first two."""
        parts = [raw(m + ("dq" if sp.q_rank else "q")).to(dtype), raw(m + "dkv").to(dtype)] + ([raw(m + "g").to(dtype)] if sp.out_gate else [])
        starts, at, rows = [], 0, []
        for t in parts:
            if sp.q_rank or sp.out_gate:
                rows.append(t.new_zeros(up8(at) - at, t.shape[1]))
                at = up8(at)
            starts.append(at)
            rows.append(t)
            at += t.shape[0]
        lw.lat_in_w, lw.lat_down_col = torch.cat(rows, 0).contiguous(), starts[1]
        if sp.out_gate:
            lw.lat_gate_col = starts[2]
        if sp.q_rank:
            lw.lat_q_norm_w, lw.lat_uq_w = vec(m + "dq.norm"), mat(m + "uq")

    def layer(i) -> LayerWeights:
        sp = arch.layer_specs[i]
        p = f"l{i if sp.source is None else sp.source}."
        m = p + "mix."
        lw = LayerWeights(ln1_w=None, qkv_w=None, o_w=None, ln2_w=None)
        lw.mix_cols = sp.heads * (sp.value_row or sp.vdim)
        if sp.kind == "linear_attention":
            lw.lin_in_w = mat(m + "q", m + "k", m + "v", m + "g", m + "b", m + "a")
            lw.lin_conv_w = mat(m + "q.conv", m + "k.conv", m + "v.conv")
            lw.lin_neg_exp_a = -torch.exp(vec(m + "A_log"))
            lw.lin_dt_bias, lw.lin_norm_w = vec(m + "dt_bias"), vec(m + "norm")
        elif sp.kind == "attention":
            attention_weights(lw, sp, m + sp.prefix)
            if sp.beside:
                add_beside(lw, sp.beside, m + sp.beside.prefix)
        elif sp.kind == "mlstm":
            lw.mem_in_w, lw.mem_gate_w = mat(m + "q", m + "k", m + "v", m + "g"), mat(m + "i", m + "f")
            lw.mem_gate_b, lw.mem_norm_w = torch.cat([vec(m + "i.b"), vec(m + "f.b")]), vec(m + "norm")
        else:
            latent_input(lw, sp, m)
            if sp.sinks:
                lw.sinks = vec(m + "sink")
            lw.lat_norm_w = vec(m + "dkv.norm")
            lw.lat_uk_t = mat(m + "uk").view(sp.heads, sp.dim, sp.kv_rank).transpose(1, 2).reshape(sp.heads * sp.kv_rank, sp.dim).contiguous()
            lw.lat_ukv = mat(m + "uk", m + "uv")
            lw.lat_uv = lw.lat_ukv[sp.heads * sp.dim:]
            lw.rope_cos, lw.rope_sin = rotary(sp.rotary)
        if arch.tanh_norm:
            lw.o_w, lw.norm1 = output_map(m + "o", sp), tanh_norm(p + "norm1")
            if sp.ff:
                expert_weights(lw, sp, p + "mlp.")
                lw.norm2 = tanh_norm(p + "norm2")
            return lw
        if not arch.parallel_block:
            lw.o_w, lw.post_attn_norm_w = output_map(m + "o", sp), output_factor(p, 1)
            if sp.ff:
                (feed_forward if sp.moe is None else expert_weights)(lw, sp, p + "mlp.")
                lw.post_ffn_norm_w = output_factor(p, 2)
            return lw
        lw.ln1_w, lw.ln1_b = vec(p + "norm1"), vec(p + "norm1.b") if arch.layernorm and arch.norm_bias else None
        if sp.ff and arch.sublayer_norms:
            lw.ln2_w = vec(p + "norm2")
        ff, side = sp.ff if sp.moe is None else 0, sp.beside.vdim if sp.beside else 0
        lw.beside_col = up8(lw.mix_cols)
        lw.mlp_col = lw.beside_col + up8(side)
        lw.join_cols = lw.mix_cols + side + ff
        lw.join_w = torch.zeros(arch.hidden_size, lw.mlp_col + up8(ff), dtype=dtype, device=device)
        lw.join_w[:, :lw.mix_cols] = output_map(m + sp.prefix + "o", sp)
        if side:
            lw.join_w[:, lw.beside_col:lw.beside_col + side] = raw(m + sp.beside.prefix + "o").to(dtype)
        if sp.o_bias:
            lw.join_b = (vec(m + sp.prefix + "o.b") * sp.mix_scale).to(dtype)
        if sp.moe is not None:
            expert_weights(lw, sp, p + "mlp.")
        elif sp.ff and not arch.mlp_gated:
            lw.fc1_w = mat(p + "mlp.up")
            lw.join_w[:, lw.mlp_col:lw.mlp_col + sp.ff] = raw(p + "mlp.down").to(dtype)
        elif sp.ff:
            lw.join_w[:, lw.mlp_col:lw.mlp_col + sp.ff] = raw(p + "mlp.down").to(dtype)
            lw.gate_up_w = mat(p + "mlp.gate", p + "mlp.up")
            if tiled and sp.ff % 64 == 0:
                from ..ops import interleave_gate_up
                lw.gate_up_w, lw.gate_up_interleaved = interleave_gate_up(lw.gate_up_w), True
        return lw

    model.embed, model.lm_head_w = mat("embed"), mat("head")
    if arch.tanh_norm:
        model.final_norm = tanh_norm("final.norm")
    else:
        model.final_norm_w = vec("final.norm") + arch.norm_offset
        model.final_norm_b = vec("final.norm.b") if arch.layernorm and arch.norm_bias else None
    if arch.bigram:
        model.bigram = mat("bigram")
    if arch.passes and arch.tanh_norm:
        model.loop_step = vec("loop.step")
    own = {i: layer(i) for i, sp in enumerate(arch.layer_specs) if sp.weights_of is None}
    model.layers = [own[i if sp.weights_of is None else sp.weights_of] for i, sp in enumerate(arch.layer_specs)]
    return model
