"""ctypes binding of libogb200_kernels.so (the sm_100a kernel library).

The library is built in-tree by `onnxruntime_genai_b200.build_native`.  On a machine with a CUDA
device the library MUST load: ops on CUDA tensors never fall back to PyTorch silently.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_void_p

_PKG = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIB_PATH = os.path.join(_PKG, "libogb200_kernels.so")

_lib = None
_initialised_devices = set()

_P = c_void_p


class GemmFused(ctypes.Structure):
    """OgbGemmFused of csrc/kernels.h: the decode-step fusions of ogb_gemm_bf16_fused."""
    _fields_ = [("norm_eps", c_float), ("positions", _P), ("slots", _P), ("cos", _P), ("sin", _P), ("k_cache", _P), ("v_cache", _P),
                ("Hq", c_int), ("Hkv", c_int), ("D", c_int), ("rot", c_int), ("max_pos", c_int)]


class LatentShape(ctypes.Structure):
    """OgbLatentShape of csrc/kernels.h: sizes of a latent-attention layer."""
    _fields_ = [(n, c_int) for n in ("H", "dim", "rot", "vdim", "R", "rot_dims")]


class AttnLayer(ctypes.Structure):
    """OgbAttnLayer of csrc/kernels.h: an attention layer with sizes and a mask of its own."""
    _fields_ = ([(n, c_int) for n in ("Hq", "Hkv", "dk", "dv", "window", "chunk", "gate_stride")] + [("scale", c_float), ("sinks", _P), ("gate", _P)] +
                [(n, c_int) for n in ("gate_wide", "maps", "raw")] + [("softcap", c_float), ("joint", c_int), ("out_scale", c_float)])


class NormStream(ctypes.Structure):
    """OgbNormStream of csrc/kernels.h: norms of rows of the fp32 residual stream."""
    _fields_ = ([(n, _P) for n in ("x", "rows", "w", "b", "w2", "out", "out2", "y", "inv_pos", "topk_w")] +
                [(n, c_int) for n in ("ldy", "k", "n_rows", "H", "layernorm", "fp32")] + [("eps", c_float)])


class Mlstm(ctypes.Structure):
    """OgbMlstm of csrc/kernels.h: matrix memories."""
    _fields_ = ([(n, _P) for n in ("q", "k", "v", "g", "gates", "gate_b", "norm_w", "out", "state", "slots", "cu_seqlens", "past_lens")] +
                [("slot_stride", c_longlong)] + [(n, c_int) for n in ("ld", "ldg", "ldo", "B", "H", "d", "dv", "T", "max_q_len", "fp32", "long_tokens", "all_long")] +
                [("cap", c_float), ("eps", c_float), ("scratch", _P), ("scratch_bytes", c_longlong)])


class TanhNorm(ctypes.Structure):
    """OgbTanhNorm of csrc/kernels.h: a sum into the residual stream and the tanh norm of the result."""
    _fields_ = ([(n, _P) for n in ("h_in", "h_out", "y", "y2", "inv_pos", "topk_w", "first", "step", "w", "b", "x", "rows")] +
                [(n, c_int) for n in ("ldy", "ldy2", "k", "n_rows", "H", "fp32")] + [("alpha", c_float)])


class Bigram(ctypes.Structure):
    """OgbBigram of csrc/kernels.h: token embedding with rows hashed from (previous token, token)."""
    _fields_ = ([(n, _P) for n in ("ids", "slots", "positions", "cu_seqlens", "block_table", "tokens")] +
                [(n, c_int) for n in ("table_cols", "block_size", "B", "T", "H", "vocab", "buckets", "fp32")] +
                [("mul_prev", c_longlong), ("mul_cur", c_longlong), ("scale", c_float)])


_LS = ctypes.POINTER(LatentShape)
_AL = ctypes.POINTER(AttnLayer)

_SIGS = {
    "ogb_runtime_init": (c_int, [c_int]),
    "ogb_status_device_ptr": (_P, [c_int]),
    "ogb_status_read_and_clear": (c_int, [c_int]),
    "ogb_sm_count": (c_int, [c_int]),
    "ogb_last_cuda_error": (ctypes.c_char_p, []),
    "ogb_gemm_token_tile": (c_int, [c_int, c_int]),
    "ogb_gemm_auto_splits": (c_int, [c_int, c_int, c_int, c_int, c_int]),
    "ogb_gemm_max_active_clusters": (c_int, [c_int, c_int]),
    "ogb_gemm_bf16": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, c_int, c_int, _P, c_int, _P]),
    "ogb_gemm_bf16_fused": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, c_int, c_int, _P, c_int, _P, _P]),
    "ogb_comm_register": (c_int, [c_int, c_int, c_int, _P, _P, c_longlong]),
    "ogb_comm_register_nvls": (c_int, [c_int, _P, _P, _P, _P, _P, _P, _P, c_longlong]),
    "ogb_comm_has_nvls": (c_int, [c_int]),
    "ogb_comm_set_options": (c_int, [c_int, c_longlong, c_int]),
    "ogb_comm_capacity": (c_longlong, [c_int]),
    "ogb_w4_packed_bytes": (c_longlong, [c_int, c_int]),
    "ogb_gemm_w4": (c_int, [_P, c_int, _P, _P, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, c_int, _P, c_int, _P]),
    "ogb_moe_gemm": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float, c_float, _P, _P, _P,
                             _P, c_int, c_int, _P, _P]),
    "ogb_fp4_packed_bytes": (c_longlong, [c_int, c_int, c_int]),
    "ogb_moe_gemm_fp4": (c_int, [_P, c_int, _P, _P, c_int, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float, c_float, _P, _P, _P,
                                 _P, c_int, c_int, c_int, _P, _P, _P]),
    "ogb_moe_fp4_reads_row_map": (c_int, [c_int, c_int, c_int]),
    "ogb_collective": (c_int, [c_int, _P, _P, _P, c_longlong, c_int, _P, c_int, _P]),
    "ogb_moe_topk": (c_int, [_P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P]),
    "ogb_moe_max_tiles": (c_int, [c_int, c_int, c_int]),
    "ogb_moe_sort": (c_int, [_P, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, c_int, _P]),
    "ogb_moe_combine": (c_int, [_P, c_int, _P, _P, c_int, c_int, c_int, _P, c_int, _P, c_int, _P]),
    "ogb_embedding": (c_int, [_P, _P, _P, c_int, c_int, c_int, c_float, _P]),
    "ogb_norm": (c_int, [_P, _P, _P, _P, _P, _P, c_int, c_int, c_float, c_int, _P]),
    "ogb_norm_moe_combine": (c_int, [_P, c_int, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_float, c_int, _P]),
    "ogb_rope_kv_append": (c_int, [_P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, c_int, c_int, c_int,
                                   c_int, _P]),
    "ogb_rope_kv_append_bits": (c_int, [_P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_float, c_int, c_int, c_int, c_int, c_int, c_int,
                                        c_int, c_int, _P, c_int, c_int, _P]),
    "ogb_embedding_q4": (c_int, [_P, _P, _P, _P, _P, c_int, c_int, c_int, c_float, _P]),
    "ogb_act_mul": (c_int, [_P, _P, c_int, c_int, c_int, _P]),
    "ogb_act": (c_int, [_P, _P, c_longlong, c_int, _P]),
    "ogb_causal_conv": (c_int, [_P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_causal_conv_rows": (c_int, [_P, c_int, _P, _P, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_gemm_bf16_batched": (c_int, [_P, c_int, c_int, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P, _P]),
    "ogb_gemm_simt": (c_int, [_P, c_int, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_int, _P, c_int, c_int, c_int, _P]),
    "ogb_moe_gemm_simt": (c_int, [_P, c_int, _P, _P, c_int, c_int, c_int, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P]),
    "ogb_embedding_stream": (c_int, [_P, _P, c_int, _P, _P, c_int, c_int, c_int, c_float, _P]),
    "ogb_add_normed": (c_int, [_P, _P, c_int, c_int, _P, c_float, _P, _P, _P, c_int, c_int, c_int, _P]),
    "ogb_qkv_prep": (c_int, [_P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, _P, c_float, _P, _P, _P, c_int, c_int, _P, _P, _P, c_int, _P, _P, c_int, _P]),
    "ogb_expert_act": (c_int, [_P, _P, c_longlong, c_int, c_int, c_float, c_float, c_int, _P]),
    "ogb_attention_mixed_supported": (c_int, [c_int, c_int]),
    "ogb_attention_mixed": (c_int, [_AL, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_longlong, _P, _P,
                                    _P, c_int]),
    "ogb_attention_joint_supported": (c_int, [c_int, c_int]),
    "ogb_attention_joint": (c_int, [_AL, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, _P, c_longlong, _P, _P, _P, c_int]),
    "ogb_attention_tc_joint_supported": (c_int, [c_int, c_int, c_int, c_int]),
    "ogb_attention_tc_mixed_supported": (c_int, [c_int, c_int, c_int, c_int]),
    "ogb_attention_tc_mixed": (c_int, [_AL, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P,
                                       c_longlong, _P, _P]),
    "ogb_attention_simt": (c_int, [_AL, _P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, _P, c_longlong, c_int, _P]),
    "ogb_attention_diff_merge": (c_int, [_P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_float, c_float, _P, c_int, _P, c_int, c_int, _P]),
    "ogb_add_tanh_norm": (c_int, [ctypes.POINTER(TanhNorm), _P]),
    "ogb_embedding_bigram": (c_int, [ctypes.POINTER(Bigram), _P, _P, _P, _P]),
    "ogb_norm_stream": (c_int, [ctypes.POINTER(NormStream), _P]),
    "ogb_min_gru": (c_int, [_P, _P, _P, c_int, _P, c_longlong, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_float, c_int, _P, c_longlong, c_int, _P]),
    "ogb_min_gru_scratch_bytes": (c_longlong, [c_int, c_int, c_int]),
    "ogb_mlstm_scratch_bytes": (c_longlong, [c_int, c_int, c_int, c_int, c_int]),
    "ogb_mlstm": (c_int, [ctypes.POINTER(Mlstm), _P]),
    "ogb_moe_topk_grouped": (c_int, [_P, c_int, c_int, c_int, c_int, _P, c_int, c_int, c_float, _P, _P, _P]),
    "ogb_act_mul_rows": (c_int, [_P, c_int, _P, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_latent_prep": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, _P, _LS, _P, c_float, _P, _P, _P, c_int, _P, _P, c_int, c_int, c_int, _P]),
    "ogb_gate_rows": (c_int, [_P, c_int, _P, c_int, c_int, c_int, c_int, _P]),
    "ogb_latent_mma_supported": (c_int, [_LS]),
    "ogb_latent_rows_per_tile": (c_int, [c_int, c_int]),
    "ogb_latent_scratch_bytes": (c_longlong, [c_int, c_int, c_int]),
    "ogb_latent_attention": (c_int, [_P, _P, c_int, _LS, _P, c_int, _P, _P, _P, c_int, c_int, _P, c_float, c_int, _P, c_int, c_int, c_int, c_int, c_int,
                                     _P, c_longlong, _P, _P, _P]),
    "ogb_latent_attention_simt": (c_int, [_P, _P, c_int, _LS, _P, c_int, _P, _P, _P, c_int, c_int, _P, c_float, c_int, _P, c_int, c_int, c_int, c_int, _P]),
    "ogb_latent_gather": (c_int, [_P, c_int, _P, c_int, c_int, _P, _P, _P, _P, c_int, c_int, c_int, _P, c_int, _P]),
    "ogb_attention_tc_latent_supported": (c_int, [c_int, c_int, c_int]),
    "ogb_attention_tc_latent": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, _P, _P, _P, _P, _P, c_int, c_float, c_int, _P, _P, c_int, c_int, c_int, c_int,
                                        c_int, c_int, c_int, _P, _P]),
    "ogb_short_conv": (c_int, [_P, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, c_int, c_int, c_int, _P]),
    "ogb_decode_advance": (c_int, [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P]),
    "ogb_logits_edit": (c_int, [_P, c_int, _P, _P, _P, _P, c_int, _P]),
    "ogb_logits_bitmask": (c_int, [_P, c_int, c_int, _P, _P, _P]),
    "ogb_bf16_to_f32": (c_int, [_P, _P, c_longlong, _P]),
    "ogb_gather_rows": (c_int, [_P, _P, _P, c_int, c_int, _P]),
    "ogb_gather_rows_f16": (c_int, [_P, _P, _P, c_int, c_int, _P]),
    "ogb_attention_scratch_bytes": (c_longlong, [c_int, c_int, c_int, c_int]),
    "ogb_paged_attention": (c_int, [_P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P, c_float, c_float, c_int, c_int,
                                    c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_longlong, c_int, _P, _P, _P]),
    "ogb_paged_attention_skip": (c_int, [_P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P, c_float, c_float, c_int, c_int,
                                         c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_longlong, c_int, _P, _P, _P, c_int]),
    "ogb_attention_tc_supported": (c_int, [c_int, c_int, c_int, c_int]),
    "ogb_attention_tc": (c_int, [_P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P, c_float, c_float, c_int, c_int, c_int,
                                 c_int, c_int, c_int, c_int, c_int, _P, _P]),
    "ogb_paged_attention_kv8": (c_int, [_P, c_int, _P, _P, _P, _P, _P, c_int, c_int, _P, c_int, _P, c_float, c_float, c_int, c_int,
                                    c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P, c_longlong, c_int, _P, _P, _P]),
    "ogb_gated_delta_fused": (c_int, [_P, c_longlong, c_longlong, c_longlong, c_longlong, _P, c_longlong, c_longlong, c_longlong, _P, _P, c_float,
                                      c_float, _P, c_longlong, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_gdn_gate_norm": (c_int, [_P, _P, c_longlong, _P, c_float, _P, c_longlong, c_int, c_int, c_int, c_int, _P]),
    "ogb_gated_delta": (c_int, [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_mamba2_scan_fused": (c_int, [_P, c_longlong, _P, c_longlong, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_mamba_gate_norm": (c_int, [_P, _P, c_longlong, _P, c_float, _P, c_int, c_int, _P]),
    "ogb_mamba2_scan": (c_int, [_P, _P, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P]),
    "ogb_copy_state_slots": (c_int, [_P, _P, c_int, c_int, c_longlong, _P, _P, c_int, _P]),
    "ogb_sample": (c_int, [_P, c_longlong, c_int, c_int, _P, _P, _P, _P, _P, _P, _P]),
    "ogb_argmax": (c_int, [_P, c_longlong, c_int, c_int, _P, _P]),
    "ogb_topk": (c_int, [_P, c_longlong, c_int, c_int, c_int, c_int, _P, _P, _P, _P]),
    "ogb_beam_merge": (c_int, [_P, _P, c_int, c_int, c_int, _P, _P, _P, _P]),
    "ogb_beam_scorer_step": (c_int, [_P, _P, _P, _P, _P, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_float,
                                     _P, c_int, _P]),
    "ogb_beam_scorer_finalize": (c_int, [_P, _P, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_float, _P,
                                         c_int, _P]),
    "ogb_verify_sampled": (c_int, [_P, c_longlong, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, _P, _P, _P, _P, _P, _P]),
    "ogb_verify_greedy": (c_int, [_P, _P, c_int, _P, _P, _P]),
}

_OPTIONAL = set()


def lib():
    """Returns the loaded kernel library, building it first when the sources are newer."""
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(LIB_PATH):
        from ..build_native import build_kernels
        build_kernels()
    handle = ctypes.CDLL(LIB_PATH)
    for name, (res, args) in _SIGS.items():
        try:
            fn = getattr(handle, name)
        except AttributeError:
            if name in _OPTIONAL:
                continue
            raise RuntimeError(f"{LIB_PATH} is stale (missing {name}); rebuild with python -m onnxruntime_genai_b200.build_native")
        fn.restype = res
        fn.argtypes = args
    _lib = handle
    return _lib


def bind(name: str, restype, argtypes):
    """Registers the signature of an extra entry point (used by optional kernel files)."""
    fn = getattr(lib(), name)
    fn.restype = restype
    fn.argtypes = argtypes
    return fn


def init_device(index: int) -> None:
    if index in _initialised_devices:
        return
    rc = lib().ogb_runtime_init(index)
    if rc != 0:
        raise RuntimeError(f"ogb_runtime_init({index}) failed with {rc}")
    _initialised_devices.add(index)


STATUS_NAMES = {0: "ok", 1: "TMA pipeline wait ran out", 2: "accumulator wait ran out", 3: "peer wait ran out", 4: "bad argument"}


def check_status(index: int) -> None:
    """Synchronises the device and raises if a kernel reported a bounded wait that ran out."""
    code = lib().ogb_status_read_and_clear(index)
    if code != 0:
        raise RuntimeError(f"sm_100a kernel reported status {code}: {STATUS_NAMES.get(code, 'unknown')}")


LAUNCH_COUNT = 0  # launcher calls so far (one kernel each; split-KV attention adds its combine kernel)


def check(rc: int, what: str) -> None:
    global LAUNCH_COUNT
    LAUNCH_COUNT += 1
    if rc != 0:
        why = ""
        if rc == -4:     # a launch (or the configuration call before it) was refused by the CUDA runtime
            try:
                why = ": " + lib().ogb_last_cuda_error().decode()
            except Exception:
                pass
        raise RuntimeError(f"{what} failed with code {rc}{why}")
