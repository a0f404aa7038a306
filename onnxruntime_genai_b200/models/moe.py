"""Mixture-of-experts MLP: router -> top-k -> routing weights -> per-expert gated MLP -> weighted sum.
Two styles: gpt-oss (biases, softmax over the selected logits, clamped SwiGLU(alpha, limit)) and standard (Mixtral, Qwen-MoE,
PhiMoE, GraniteMoE: no biases, silu(gate) * up, softmax over all experts with or without renormalisation).  Declared stacks describe
the experts of each layer by themselves (`LayerWeights.moe`, an arch.MoeSpec), with any mix of these rules, and may have a shared expert:
of the same width and limit it is one more expert of the grouped products that every token is routed to with weight 1, else it runs
beside them and the add + norm that follows folds it.  Experts without a gate matrix keep their up matrix in `exp_gate_up_w`.

Semantics follow the MoE / QMoE contrib op the reference's builder emits
(src/python/py/models/builders/base.py:4176-4408, builders/gptoss.py:653-847): `k` experts per token,
`normalize_routing_weights` (softmax over the k selected router logits), `swiglu_fusion = 1`
(gate and up interleaved along the output dimension: even = gate, odd = up), activation
gate * sigmoid(alpha * gate) * (up + 1) with gate clamped to <= limit and up to [-limit, limit].

CUDA path (everything on the device, no counts read back, so it replays inside a CUDA graph):
router GEMM (fp32 out) -> `moe_topk` -> `moe_sort` (rows grouped by expert + tile list) -> row gather ->
grouped tcgen05 GEMM gate/up with the clamped SwiGLU in its epilogue -> grouped GEMM down -> `moe_combine`.

Expert parallelism: attention is tensor parallel, so after its all-reduce every rank already holds every
token; a rank therefore needs no dispatch — it routes all tokens, runs only the experts it owns
(`lw.exp_lo .. lw.exp_hi`), and the partial outputs are summed by the same all-reduce a dense row-parallel
MLP uses.  The combine of the all-to-all formulation is that all-reduce.
"""
from __future__ import annotations

import os

import torch

from .. import ops
from .arch import MoeSpec


# OGB_MOE_ROW_MAP=0: the token rows of packed experts are gathered into a copy instead of being read through the row map
_ROW_MAP = os.environ.get("OGB_MOE_ROW_MAP", "1") != "0"


def swiglu_interleaved(gu: torch.Tensor, alpha: float, limit: float) -> torch.Tensor:
    g, u = gu[..., 0::2].float(), gu[..., 1::2].float()
    if limit > 0:
        g = g.clamp(max=limit)
        u = u.clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(alpha * g) * (u + 1.0)).to(gu.dtype)


def spec_of(model, lw) -> MoeSpec:
    """The routing rule and the activation of a layer: its own, or the model's."""
    return lw.moe if lw.moe is not None else model.arch.moe_spec


_TOPK_MODES = {"selected": 0, "all": 1, "renormed": 2}      # softmax over the selected logits / over all / over all, then over the selected


def route(model, lw, x):
    """Routing weights and expert ids [T, k].  Softmax over the selected logits equals softmax over all experts renormalised
    over the selected; the standard style without renormalisation keeps the probabilities of the full softmax."""
    sp = spec_of(model, lw)
    if sp.weights == "sigmoid":
        return corrected_choice(ops.linear(x, lw.router_w, out_fp32=True), lw.router_b, sp)
    logits = ops.linear(x, lw.router_w, lw.router_b).float()
    if sp.weights == "sparse_mixer":
        return sparse_mixer(logits, sp.jitter_eps)
    top_v, top_i = torch.topk(logits, sp.top, dim=-1)
    if sp.weights == "all":
        return torch.softmax(logits, dim=-1).gather(-1, top_i), top_i
    return torch.softmax(top_v, dim=-1), top_i


def corrected_choice(logits: torch.Tensor, correction: torch.Tensor, sp: MoeSpec):
    """Sigmoid scores; the choice goes by score + correction, among the `keep` groups of neighbours with the largest sums of two."""
    s = torch.sigmoid(logits.float())
    c = s + correction
    if sp.groups > 1:
        g = c.view(c.shape[0], sp.groups, -1)
        best = g.topk(min(2, g.shape[-1]), dim=-1).values.sum(-1).topk(sp.keep, dim=-1).indices
        open_ = torch.zeros(g.shape[:2], dtype=torch.bool, device=c.device).scatter_(1, best, True)
        c = g.masked_fill(~open_[:, :, None], float("-inf")).reshape(c.shape)
    ids = torch.topk(c, sp.top, dim=-1).indices
    w = s.gather(-1, ids)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * sp.scale, ids


def sparse_mixer(logits: torch.Tensor, eps: float):
    """PhiMoE's inference-time routing (reference: the MoE contrib op's use_sparse_mixer attribute,
    src/python/py/models/builders/phi.py:542-547): the best expert, then the best of the rest; each weight is that
    expert's probability in a softmax over the logits that lie within a relative margin of 2 * eps below the current
    maximum.  Pure tensor ops (no host synchronisation), so the step still captures into a CUDA graph."""
    s = logits.float()
    neg = torch.finfo(torch.float32).min

    def pick(scores):
        top, idx = scores.max(dim=-1, keepdim=True)
        factor = s.abs().clamp(min=top)
        keep = ((top - s) / factor) <= 2.0 * eps
        gates = torch.softmax(torch.where(keep, scores, torch.full_like(scores, neg)), dim=-1)
        return gates.gather(-1, idx), idx

    w1, i1 = pick(s)
    w2, i2 = pick(s.scatter(-1, i1, neg))
    return torch.cat([w1, w2], dim=-1), torch.cat([i1, i2], dim=-1)


def silu_mul_interleaved(gu: torch.Tensor) -> torch.Tensor:
    g, u = gu[..., 0::2].float(), gu[..., 1::2].float()
    return (torch.nn.functional.silu(g) * u).to(gu.dtype)


def _unblock(t: torch.Tensor) -> torch.Tensor:
    """[.., 2I, ..] in blocks of 64 gate + 64 up rows -> even/odd interleaved rows."""
    two_i = t.shape[0]
    v = t.reshape(two_i // 128, 2, 64, *t.shape[1:])
    return torch.stack([v[:, 0], v[:, 1]], dim=2).reshape(t.shape)


def expert_mlp(model, lw, e: int, xs: torch.Tensor) -> torch.Tensor:
    """One expert (index into this rank's slice) over its rows: the unfused path (CPU, odd shapes)."""
    sp = spec_of(model, lw)
    packed = isinstance(lw.exp_gate_up_w, ops.Fp4Experts)   # MXFP4 experts: expand this one expert
    w = lw.exp_gate_up_w.dequantize(e).to(xs) if packed else lw.exp_gate_up_w[e]
    b = lw.exp_gate_up_b[e] if lw.exp_gate_up_b is not None else None
    if not sp.gated:
        return ops.linear(ops.linear_act(xs, w, sp.act), lw.exp_down_w[e])
    if lw.exp_blocked:
        w, b = _unblock(w).contiguous(), _unblock(b).contiguous() if b is not None else None
    gu = ops.linear(xs, w, b)
    act = silu_mul_interleaved(gu) if sp.act == "silu" else swiglu_interleaved(gu, sp.alpha, sp.limit)
    wd = lw.exp_down_w.dequantize(e).to(xs) if packed else lw.exp_down_w[e]
    return ops.linear(act.contiguous(), wd, lw.exp_down_b[e] if lw.exp_down_b is not None else None)


def shared_expert(lw, x: torch.Tensor, sp: MoeSpec) -> torch.Tensor:
    """The expert every token takes, where it stands beside the routed ones (sizes or limits of its own)."""
    gu = ops.linear(x, lw.shared_gate_up_w)
    h = ops.expert_act(gu, "clamped", sp.alpha, sp.shared_limit) if x.is_cuda else swiglu_interleaved(gu, sp.alpha, sp.shared_limit)
    return ops.linear(h, lw.shared_down_w)


def _forward_loop(model, lw, x):
    sp = spec_of(model, lw)
    lo, hi = lw.exp_lo, lw.exp_hi or sp.experts
    weights, experts = route(model, lw, x)
    out = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
    flat_e = experts.reshape(-1)
    order = torch.argsort(flat_e, stable=True)
    counts = torch.bincount(flat_e, minlength=sp.experts).tolist()
    tok = order // sp.top
    w_sorted = weights.reshape(-1)[order]
    start = 0
    for e, n in enumerate(counts):
        if n and lo <= e < hi:
            idx = tok[start:start + n]
            y = expert_mlp(model, lw, e - lo, x[idx].contiguous()).float()
            out.index_add_(0, idx, y * w_sorted[start:start + n, None])
        start += n
    if lw.exp_shared:
        out += expert_mlp(model, lw, sp.experts, x).float()
    elif lw.shared_gate_up_w is not None:
        out += shared_expert(lw, x, sp).float()
    return out.to(x.dtype)


def _plan(model, lw, x, sp, token_tile=0):
    """Routing of the tokens, on the device."""
    lo, hi = lw.exp_lo, lw.exp_hi or sp.experts
    if sp.weights == "sigmoid":
        return ops.moe_route(ops.linear(x, lw.router_w, out_fp32=True), sp.top, 3, (lo, hi), token_tile, correction=lw.router_b, groups=sp.groups, keep=sp.keep,
                             scale=sp.scale)
    logits = ops.linear(x, lw.router_w, lw.router_b, out_fp32=True)
    if lw.exp_shared:
        return ops.moe_route(logits, sp.top, _TOPK_MODES[sp.weights], None, token_tile, shared=True)
    if sp.weights == "sparse_mixer":
        tw, ti = sparse_mixer(logits, sp.jitter_eps)
        return ops.moe_route(logits, 2, 0, (lo, hi), token_tile, topk=(ti.to(torch.int32).contiguous(), tw.contiguous()))
    return ops.moe_route(logits, sp.top, _TOPK_MODES[sp.weights], (lo, hi), token_tile)


def _forward_device(model, lw, x, defer=False):
    sp = spec_of(model, lw)
    plan = _plan(model, lw, x, sp)
    beside = shared_expert(lw, x, sp) if lw.shared_gate_up_w is not None else None
    if beside is not None and not defer:
        raise RuntimeError("a shared expert beside the routed ones needs the add + norm that folds it")
    half = isinstance(lw.exp_gate_up_w, ops.Fp4Experts) and lw.exp_gate_up_w.half and lw.exp_down_w.half
    if half:
        # packed MXFP4 experts in their fp16 form: fp16 rows in, fp16 between the two grouped GEMMs, bf16 out; the streaming
        # kernel of decode-sized steps reads the token rows through the plan's row map instead of a gathered copy
        mapped = _ROW_MAP and ops.moe_fp4_reads_rows(lw.exp_gate_up_w, plan) and x.dtype == torch.bfloat16 and x.stride(0) % 8 == 0
        xs = x if mapped else ops.gather_rows(x, plan.sorted_token, f16=True)
        h = ops.moe_gemm(xs, lw.exp_gate_up_w, plan, lw.exp_gate_up_b, act_kind=2, alpha=sp.alpha, limit=sp.limit,
                         out_dtype=torch.float16, row_map=mapped)
        y = ops.moe_gemm(h, lw.exp_down_w, plan, lw.exp_down_b)
        return ops.PendingCombine(y, plan) if defer else ops.moe_combine(y, plan)
    xs = ops.gather_rows(x, plan.sorted_token)
    if not sp.gated:
        h = ops.moe_gemm(xs, lw.exp_gate_up_w, plan, None, act_kind=ops.MOE_ACTS[sp.act], pair=False)
    elif sp.act == "silu":
        h = ops.moe_gemm(xs, lw.exp_gate_up_w, plan, None, act_kind=1)
    else:
        h = ops.moe_gemm(xs, lw.exp_gate_up_w, plan, lw.exp_gate_up_b, act_kind=2, alpha=sp.alpha, limit=sp.limit)
    y = ops.moe_gemm(h, lw.exp_down_w, plan, lw.exp_down_b)
    return ops.PendingCombine(y, plan, beside) if defer else ops.moe_combine(y, plan)


def _forward_simt(model, lw, x):
    """32-bit models and sizes the tensor-core kernels cannot address: the same steps in plain arithmetic, experts' rows read through the
    routing plan.  The result is pending: the caller's norm folds the weighted sum."""
    sp = spec_of(model, lw)
    plan = _plan(model, lw, x, sp, token_tile=64)
    gu = ops.moe_gemm_simt(x, lw.exp_gate_up_w, plan, mapped=True)
    h = ops.expert_act(gu, sp.act, sp.alpha, sp.limit)
    return ops.PendingCombine(ops.moe_gemm_simt(h, lw.exp_down_w, plan), plan, shared_expert(lw, x, sp) if lw.shared_gate_up_w is not None else None)


def moe_forward(model, lw, x: torch.Tensor, defer: bool = False):
    """defer: the caller folds the combine step into the residual add + norm that follows (`ops.norm_moe_combine`); the
    result is then an `ops.PendingCombine` when the layer ran on the device path of a single rank."""
    a, sp = model.arch, spec_of(model, lw)
    fast = x.is_cuda and lw.exp_blocked and a.hidden_size % 8 == 0 and sp.experts + lw.exp_shared <= 1024 and sp.top + lw.exp_shared <= 32
    if model.tp.size > 1 and getattr(model.tp, "ep_mode", "replicated") == "all_to_all":
        # token-sharded expert parallelism: dispatch / combine all-to-all, the output is complete on every rank
        from ..parallel.ep import moe_all_to_all
        return moe_all_to_all(model, lw, x)
    if fast:
        return _forward_device(model, lw, x, defer and model.tp.size == 1) if model.tp.size == 1 else model.tp.reduce(_forward_device(model, lw, x))
    if x.is_cuda and lw.moe is not None and defer and model.tp.size == 1:
        return _forward_simt(model, lw, x)
    out = _forward_loop(model, lw, x)
    return model.tp.reduce(out) if model.tp.size > 1 else out
