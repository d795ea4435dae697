"""ctypes bindings of libglorcq_b200.so (the C ABI declared in include/glorcq_b200.h) and of
libglorcq_b200_dense.so (include/glorcq_b200_dense.h, the unquantized decoders; built at first use).

There is no fallback: if the library is missing, or a call returns a non-zero status, a
RuntimeError is raised -- the same exception type the reference's native modules raise through
TORCH_CHECK (inference/kernels/turbo_matmul.cu:250-283).
"""

from __future__ import annotations

import ctypes as C
import os

HERE = os.path.dirname(os.path.abspath(__file__))
# GLQ_LIB selects another build of the same ABI (e.g. one compiled with -DGLQ_CHECKED)
LIB_PATH = os.environ.get("GLQ_LIB") or os.path.join(HERE, "libglorcq_b200.so")

FMT_Q2, FMT_Q4, FMT_T2, FMT_F16 = 0, 1, 2, 3
EPI_LINEAR, EPI_SWIGLU = 0, 1

vp = C.c_void_p


class Weight(C.Structure):
    """glq_weight_t"""
    _fields_ = [("codes", vp), ("reserved0", vp), ("norms", vp), ("centroids", vp), ("sv", vp), ("bias", vp),
                ("N", C.c_int32), ("K", C.c_int32), ("rank", C.c_int32), ("reserved", C.c_int32)]


class MMArgs(C.Structure):
    """glq_mm_args_t"""
    _fields_ = [("fmt", C.c_int32), ("group_size", C.c_int32), ("epilogue", C.c_int32), ("n_problems", C.c_int32),
                ("max_rows", C.c_int32), ("rows_stride", C.c_int32), ("N", C.c_int32), ("K", C.c_int32),
                ("rank", C.c_int32), ("total_rows", C.c_int32),
                ("w", Weight), ("w_table", vp),
                ("slot_index", vp), ("n_slots", vp), ("slot_count", vp), ("slot_offset", vp), ("entry_row", vp),
                ("entry_scale", vp),
                ("x", vp), ("ldx", C.c_int64), ("a0", vp), ("a1", vp), ("lda", C.c_int64),
                ("y", vp), ("ldy", C.c_int64), ("workspace", vp), ("workspace_bytes", C.c_size_t),
                ("counters", vp), ("n_counters", C.c_size_t), ("flags", C.c_int32), ("reserved", C.c_int32)]


class MoeDesc(C.Structure):
    """glq_moe_desc_t"""
    _fields_ = [("H", C.c_int32), ("I", C.c_int32), ("E", C.c_int32), ("top_k", C.c_int32),
                ("I_shared", C.c_int32), ("rank", C.c_int32), ("fmt", C.c_int32), ("group_size", C.c_int32),
                ("norm_topk_prob", C.c_int32), ("router_rows", C.c_int32), ("slot_order_max_tokens", C.c_int32),
                ("reserved", C.c_int32),
                ("router_t", vp), ("gate_up", vp), ("down", vp), ("ut_gate_up", vp), ("ut_down", vp),
                ("dense0_rows", C.c_int32), ("sh_a_row", C.c_int32),
                ("sh_gate_up", Weight), ("sh_down", Weight),
                ("sh_ut_gate", vp), ("sh_ut_up", vp), ("sh_ut_down", vp),
                ("rot_in", vp), ("rot_mid", vp), ("sh_rot_mid", vp),
                ("rht_in", vp), ("rht_mid", vp), ("sh_rht_mid", vp),
                ("router_rm", vp), ("ut_rm_gate_up", vp), ("ut_rm_down", vp), ("sh_ut_rm_down", vp)]


class EpPeers(C.Structure):
    """glq_ep_peers_t"""
    _fields_ = [("entry_bufs", vp), ("flags", vp), ("epoch", vp), ("error", vp), ("half_elems", C.c_size_t),
                ("wait_limit_ns", C.c_uint64)]


class MoeEp(C.Structure):
    """glq_moe_ep_t"""
    _fields_ = [("rank", C.c_int32), ("world", C.c_int32), ("phase", C.c_int32), ("flags", C.c_int32),
                ("entry_out", vp), ("sel_in", vp), ("weight_in", vp),
                ("residual", vp), ("norm_weight", vp), ("normed_out", vp), ("norm_eps", C.c_float), ("reserved2", C.c_int32),
                ("peers", C.POINTER(EpPeers))]


MOE_PHASE_ALL, MOE_PHASE_EXPERTS, MOE_PHASE_COMBINE, MOE_PHASE_EXCHANGE = 0, 1, 2, 3
MOE_EP_NO_ZERO_FILL = 1

_SIGS = {
    "glq_version": (C.c_int, []),
    "glq_status_string": (C.c_char_p, [C.c_int]),
    "glq_last_cuda_error": (C.c_int, []),
    "glq_turbo_dequant_matmul": (C.c_int, [vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, vp]),
    "glq_static_scratch_bytes": (C.c_size_t, []),
    "glq_static_scratch_needed": (C.c_size_t, [C.c_int, C.c_int, C.c_int]),
    "glq_turbo_dequant_matmul_static": (C.c_int, [vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, vp]),
    "glq_turbo_dequant_grouped_gemv": (C.c_int, [vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, vp]),
    "glq_gptq_dequant_matmul": (C.c_int, [vp, vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int,
                                          C.c_int, vp]),
    "glq_tiled_bytes": (C.c_size_t, [C.c_int, C.c_int, C.c_int, C.c_int]),
    "glq_sv_bytes": (C.c_size_t, [C.c_int, C.c_int, C.c_int]),
    "glq_rows_f32_count": (C.c_size_t, [C.c_int, C.c_int]),
    "glq_tiled_f16_bytes": (C.c_size_t, [C.c_int, C.c_int]),
    "glq_pack_gptq": (C.c_int, [vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, vp, C.c_int, C.c_int, vp]),
    "glq_pack_turbo": (C.c_int, [vp, C.c_int, C.c_int, vp, C.c_int, C.c_int, vp]),
    "glq_pack_rows_f32": (C.c_int, [vp, C.c_int, vp, C.c_int, C.c_int, vp]),
    "glq_pack_sv": (C.c_int, [vp, C.c_int, C.c_int, vp, C.c_int, C.c_int, vp]),
    "glq_pack_f16": (C.c_int, [vp, C.c_long, C.c_long, C.c_int, C.c_int, vp, vp]),
    "glq_dequant_tiled": (C.c_int, [C.c_int, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, vp, vp]),
    "glq_debug_error": (C.c_int, [vp, C.c_int]),
    "glq_add_rmsnorm": (C.c_int, [vp, vp, vp, C.c_float, C.c_int, C.c_int, vp, vp, vp]),
    "glq_attn_decode_workspace_bytes": (C.c_size_t, [C.c_int, C.c_int, C.c_int, C.c_int]),
    "glq_rope_prefill": (C.c_int, [vp, vp, vp, vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, vp, vp,
                         C.c_float, vp]),
    "glq_attn_prefill": (C.c_int, [vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, vp]),
    "glq_attn_decode": (C.c_int, [vp, vp, vp, vp, vp, vp, vp, vp, vp, C.c_int, C.c_int, C.c_int, C.c_int, C.c_int, vp, vp,
                                  C.c_float, vp, C.c_size_t, vp, C.c_size_t, vp]),
    "glq_lm_head_workspace_bytes": (C.c_size_t, []),
    "glq_lm_head": (C.c_int, [vp, C.c_int64, vp, C.c_int, C.c_int, C.c_int, vp, C.c_int64, vp, vp, C.c_size_t, vp, vp]),
    "glq_rht_forward": (C.c_int, [vp, C.c_int, C.c_int64, vp, C.c_int, C.c_int, C.c_float, vp, C.c_int, C.c_int64, vp]),
    "glq_mm_workspace_bytes": (C.c_size_t, [C.POINTER(MMArgs)]),
    "glq_mm_counters": (C.c_size_t, [C.POINTER(MMArgs)]),
    "glq_grouped_matmul": (C.c_int, [C.POINTER(MMArgs), vp]),
    "glq_linear_counters": (C.c_size_t, [C.c_int, C.c_int, C.POINTER(Weight), C.c_int]),
    "glq_linear_workspace_bytes": (C.c_size_t, [C.c_int, C.c_int, C.POINTER(Weight), C.c_int]),
    "glq_linear_forward": (C.c_int, [C.c_int, C.c_int, C.POINTER(Weight), vp, vp, C.c_int64, vp, vp, C.c_int64,
                                     C.c_int, vp, C.c_size_t, vp, C.c_size_t, vp]),
    "glq_moe_fused_trace": (C.c_int, [vp, C.c_int]),
    "glq_moe_uses_fused_kernel": (C.c_int, [C.POINTER(MoeDesc), C.c_int]),
    "glq_moe_workspace_bytes": (C.c_size_t, [C.POINTER(MoeDesc), C.c_int]),
    "glq_moe_counters": (C.c_size_t, [C.POINTER(MoeDesc), C.c_int]),
    "glq_moe_forward": (C.c_int, [C.POINTER(MoeDesc), vp, C.c_int, vp, vp, vp, vp, vp, C.c_size_t, vp, C.c_size_t, vp,
                                  vp, vp, vp]),
    "glq_moe_forward_ep": (C.c_int, [C.POINTER(MoeDesc), vp, C.c_int, vp, vp, vp, vp, vp, C.c_size_t, vp, C.c_size_t,
                                     vp, vp, vp, vp, C.POINTER(MoeEp)]),
}


# ---- unquantized decoders -----------------------------------------------------------------------------
DT_BF16, DT_F32 = 0, 1
ACT_NONE, ACT_RELU2, ACT_GELU_ERF, ACT_GELU_TANH, ACT_SILU_GLU = range(5)
GATE_SIGMOID, GATE_SILU = 0, 1


class DenseMM(C.Structure):
    """glq_dense_mm_t"""
    _fields_ = [(f, C.c_int32) for f in ("dtype", "act", "N", "K", "rows", "n_matrices", "max_slots", "max_slot_rows", "split")] + \
               [("alpha", C.c_float)] + [(f, vp) for f in ("slot_index", "n_slots", "slot_count", "slot_offset", "entry_row", "x")] + \
               [("ldx", C.c_int64), ("W", vp), ("ldw", C.c_int64), ("y", vp), ("ldy", C.c_int64), ("y32", vp), ("ldy32", C.c_int64), ("gather", vp),
                ("hn_o", vp), ("hn_g", vp), ("hn_ldg", C.c_int64), ("hn_w", vp), ("hn_heads", C.c_int32), ("hn_eps", C.c_float),
                ("mul", vp), ("ldmul", C.c_int64), ("mul_row", vp),
                ("mul_rows", C.c_int32), ("residual", C.c_int32)]


class MLstm(C.Structure):
    """glq_mlstm_t"""
    _fields_ = [(f, C.c_int32) for f in ("dtype", "B", "T", "H", "D", "V", "state_idle")] + \
               [("gate_cap", C.c_float), ("eps", C.c_float), ("qkvg", vp), ("ldp", C.c_int64), ("gates", vp), ("ldg", C.c_int64)] + \
               [(f, vp) for f in ("bias_i", "bias_f", "norm_w", "S", "n", "m", "o", "out", "workspace")] + \
               [("workspace_bytes", C.c_size_t)]


class Decay(C.Structure):
    """glq_decay_t"""
    _fields_ = [(f, C.c_int32) for f in ("dtype", "B", "T", "H", "D", "V", "rank", "rot_dims", "rot_pairs", "max_len", "norm_stride", "gate",
                                         "state_idle")] + [(f, C.c_float) for f in ("q_scale", "k_scale", "eps", "tau")] + \
               [(f, vp) for f in ("q", "k", "v", "g")] + [("ldp", C.c_int64), ("decay", vp), ("a", vp), ("lda", C.c_int64)] + \
               [(f, vp) for f in ("a2", "a2b", "start", "cos_t", "sin_t", "norm_w", "S", "o", "out", "workspace")] + \
               [("workspace_bytes", C.c_size_t)]


class Gqa(C.Structure):
    """glq_gqa_t"""
    _fields_ = [(f, C.c_int32) for f in ("dtype", "B", "T", "H", "G", "D", "V", "rot_dims", "rot_pairs", "qk_norm", "max_len", "S",
                                         "state_idle")] + [("scale", C.c_float), ("eps", C.c_float)] + \
               [(f, vp) for f in ("start", "q", "k", "v")] + [("ldp", C.c_int64)] + \
               [(f, vp) for f in ("cos_t", "sin_t", "kc", "vc", "out", "workspace")] + [("workspace_bytes", C.c_size_t)]


class Latent(C.Structure):
    """glq_latent_t"""
    _fields_ = [(f, C.c_int32) for f in ("dtype", "B", "T", "H", "D", "R", "V", "K", "rot_dims", "max_len")] + \
               [("scale", C.c_float), ("eps", C.c_float), ("start", vp), ("q", vp), ("ldq", C.c_int64), ("ckr", vp),
                ("ldk", C.c_int64)] + [(f, vp) for f in ("gate", "norm_w", "cos_t", "sin_t", "cache")] + \
               [("ldc", C.c_int64)] + [(f, vp) for f in ("ukt", "uv", "out", "kv")] + \
               [("ldkv", C.c_int64), ("vt", vp), ("ldvt", C.c_int64), ("S", C.c_int32), ("max_splits", C.c_int32), ("workspace", vp), ("workspace_bytes", C.c_size_t)]


class Route(C.Structure):
    """glq_route_t"""
    _fields_ = [(f, C.c_int32) for f in ("n", "E", "identity", "top", "chunk", "reserved")] + [("logits", vp), ("ldl", C.c_int64)] + \
               [(f, vp) for f in ("correction", "sel", "wts", "entry_scale", "tok_entries", "entry_row", "active", "slot_count",
                                  "slot_offset", "n_active")] + \
               [("max_slots", C.c_int32), ("reserved2", C.c_int32), ("block_counts", vp)]


_i, _f, _l, _z = C.c_int, C.c_float, C.c_int64, C.c_size_t
_DENSE_SIGS = {
    "glq_dense_status_string": (C.c_char_p, [_i]),
    "glq_dense_last_cuda_error": (_i, []),
    "glq_dense_debug_error": (_i, [vp, _i]),
    "glq_dense_matmul": (_i, [C.POINTER(DenseMM), vp]),
    "glq_dense_matmul_path": (_i, [C.POINTER(DenseMM)]),
    "glq_dense_embed": (_i, [_i, vp, vp, _i, _i, _i, vp, _f, vp, vp, vp]),
    "glq_dense_rms_add": (_i, [_i, vp, _l, vp, vp, _l, vp, _f, vp, _f, _i, _i, vp, vp, vp]),
    "glq_dense_add_norm": (_i, [_i, vp, vp, vp, _f, _i, _i, vp, vp, vp]),
    "glq_mlstm_slices": (_i, [_i]),
    "glq_mlstm_workspace_bytes": (_z, [C.POINTER(MLstm)]),
    "glq_mlstm_step": (_i, [C.POINTER(MLstm), vp]),
    "glq_mlstm_chunk": (_i, [C.POINTER(MLstm), vp]),
    "glq_decay_slices": (_i, [_i]),
    "glq_decay_workspace_bytes": (_z, [C.POINTER(Decay)]),
    "glq_decay_step": (_i, [C.POINTER(Decay), vp]),
    "glq_decay_chunk_supported": (_i, [C.POINTER(Decay)]),
    "glq_decay_chunk": (_i, [C.POINTER(Decay), vp]),
    "glq_gqa_form": (_i, [C.POINTER(Gqa)]),
    "glq_gqa_decode_workspace_bytes": (_z, [C.POINTER(Gqa)]),
    "glq_gqa": (_i, [C.POINTER(Gqa), vp]),
    "glq_latent_prep": (_i, [C.POINTER(Latent), vp]),
    "glq_latent_absorbed_workspace_bytes": (_z, [C.POINTER(Latent)]),
    "glq_latent_absorbed": (_i, [C.POINTER(Latent), vp]),
    "glq_latent_prefill_form": (_i, [C.POINTER(Latent)]),
    "glq_latent_prefill": (_i, [C.POINTER(Latent), vp]),
    "glq_route_max_slots": (_i, [_i, _i, _i, _i]),
    "glq_route": (_i, [C.POINTER(Route), vp]),
    "glq_dense_combine_norm": (_i, [_i, vp, _l, vp, vp, _i, vp, vp, _f, _i, _i, vp, vp, vp]),
    "glq_dense_head_workspace_bytes": (_z, []),
    "glq_dense_head": (_i, [vp, _l, vp, _i, _i, _i, _f, vp, _l, vp, vp, _z, vp, vp]),
}

_lib = None
_dense = None


def dense():
    """The library of the unquantized decoders, compiled first when it is missing or older than its sources."""
    global _dense
    if _dense is None:
        from . import _build
        L = C.CDLL(_build.build(lib=_build.DENSE_LIB))
        for name, (res, args) in _DENSE_SIGS.items():
            fn = getattr(L, name)
            fn.restype, fn.argtypes = res, args
        _dense = L
    return _dense


def dense_symbols():
    return list(_DENSE_SIGS.keys())


def check_dense(status: int, what: str):
    if status != 0:
        L = dense()
        extra = f" (cudaError {L.glq_dense_last_cuda_error()})" if status == -4 else ""
        raise RuntimeError(f"{what}: {L.glq_dense_status_string(status).decode()}{extra}")


def lib():
    """The loaded library; raises RuntimeError when it has not been built."""
    global _lib
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise RuntimeError(
                f"{LIB_PATH} is missing: build it with `python -m glorcq_b200._build` (nvcc, sm_100a). "
                "glorcq_b200 has no CPU or PyTorch fallback.")
        L = C.CDLL(LIB_PATH)
        for name, (res, args) in _SIGS.items():
            if not hasattr(L, name):
                continue
            fn = getattr(L, name)
            fn.restype = res
            fn.argtypes = args
        _lib = L
    return _lib


def exported_symbols():
    return list(_SIGS.keys())


def check(status: int, what: str = "glorcq_b200"):
    if status != 0:
        L = lib()
        msg = L.glq_status_string(status).decode()
        extra = f" (cudaError {L.glq_last_cuda_error()})" if status == -4 else ""
        raise RuntimeError(f"{what}: {msg}{extra}")
