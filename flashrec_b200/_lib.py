"""ctypes binding of ``libflashrec_b200.so`` (the C ABI in ``include/flashrec_b200.h``).

The library is the product path: there is no CPU or eager fallback. If the
shared object is missing, or a kernel reports a non-zero status, the caller
gets an exception.
"""

from __future__ import annotations

import ctypes
import os
from ctypes import c_char_p, c_float, c_int, c_int64, c_void_p, POINTER
from pathlib import Path
from typing import Optional

import torch

# FLASHREC_B200_LIB selects another build of the same library (e.g. to compare two builds in one process
# launch each); by default the library built in-tree next to this file is loaded.
_LIB_PATH = Path(os.environ.get("FLASHREC_B200_LIB") or Path(__file__).resolve().parent / "libflashrec_b200.so").resolve()
_lib: Optional[ctypes.CDLL] = None

FR_OK = 0
_STATUS_NAMES = {
    0: "FR_OK",
    -1: "FR_ERR_BAD_ARG",
    -2: "FR_ERR_UNSUPPORTED",
    -3: "FR_ERR_CUDA",
    -4: "FR_ERR_TIMEOUT",
}


class FlashRecKernelError(RuntimeError):
    """A C-ABI entry point returned a non-zero status."""

    def __init__(self, fn: str, status: int):
        self.fn = fn
        self.status = int(status)
        super().__init__(f"{fn} failed: {_STATUS_NAMES.get(int(status), status)}")


class FrTrie(ctypes.Structure):
    """Mirror of ``struct fr_trie`` (include/flashrec_b200.h)."""

    _fields_ = [
        ("kind", ctypes.c_int32),
        ("next_is_i32", ctypes.c_int32),
        ("allow", c_void_p),
        ("next", c_void_p),
        ("csr_keys", c_void_p),
        ("csr_child", c_void_p),
        ("n_edges", c_int64),
        ("bitmap", c_void_p),
        ("child_base", c_void_p),
        ("level_off", c_void_p),
        ("words_per_node", ctypes.c_int32),
        ("reserved_", ctypes.c_int32),
        ("n_rows", c_int64),
        ("vsz", c_int64),
        ("token_base", c_int64),
        ("invalid_node", c_int64),
    ]


class FrOutSegment(ctypes.Structure):
    """Mirror of ``struct fr_out_segment``."""

    _fields_ = [("kind", ctypes.c_int32), ("n0", ctypes.c_int32), ("n", ctypes.c_int32), ("pad_", ctypes.c_int32),
                ("out", c_void_p), ("ldo", c_int64), ("row_map", c_void_p), ("bias", c_void_p), ("limit", c_float),
                ("alpha", c_float), ("up_bias", c_float), ("pad2_", ctypes.c_int32), ("mul", c_void_p), ("ld_mul", c_int64),
                ("mul_map", c_void_p)]


class FrGatedPart(ctypes.Structure):
    """Mirror of ``struct fr_gated_part``."""

    _fields_ = [("a", c_void_p), ("w", c_void_p), ("gate", c_void_p), ("lda", c_int64), ("ldw", c_int64),
                ("ldg", c_int64), ("K", ctypes.c_int32), ("pad_", ctypes.c_int32)]


class FrConvOut(ctypes.Structure):
    """Mirror of ``struct fr_conv_out``."""

    _fields_ = [("out", c_void_p), ("ldo", c_int64), ("row_map", c_void_p), ("c0", ctypes.c_int32), ("c", ctypes.c_int32)]


class FrMixAttn(ctypes.Structure):
    """Mirror of ``struct fr_mix_attn``."""

    _fields_ = ([(n, ctypes.c_int32) for n in ("dtype", "mix", "mask", "mask_size", "keep_first", "heads", "kv_heads",
                                               "dim", "vdim", "vdim_true")]
                + [(n, c_float) for n in ("scale", "lambda_", "eps", "out_scale")]
                + [("coef", c_void_p), ("slopes", c_void_p), ("q", c_void_p), ("ldq", c_int64), ("k", c_void_p),
                   ("v", c_void_p), ("ldk", c_int64), ("ldv", c_int64), ("out", c_void_p), ("ldo", c_int64),
                   ("req_to_token", c_void_p), ("table_stride", c_int64), ("req_rows", c_void_p),
                   ("tok_req", c_void_p), ("pos", c_void_p), ("num_slots", c_int64), ("head_gate", c_void_p),
                   ("ld_gate", c_int64)])


class FrNormPart(ctypes.Structure):
    """Mirror of ``struct fr_norm_part``."""

    _fields_ = [("y", c_void_p), ("ldy", c_int64), ("weight", c_void_p), ("coef", c_float), ("n_splits", ctypes.c_int32)]


class FrNormUpdate(ctypes.Structure):
    """Mirror of ``struct fr_norm_update``."""

    _fields_ = ([(n, ctypes.c_int32) for n in ("dtype", "n_parts", "n_partials")] + [("eps", c_float), ("offset", c_float),
                ("pad_", ctypes.c_int32), ("x", c_void_p), ("ldx", c_int64), ("partials", c_void_p), ("partial_stride", c_int64),
                ("parts", FrNormPart * 2), ("add", c_void_p), ("row_idx", c_void_p), ("weight", c_void_p), ("out", c_void_p),
                ("ldo", c_int64)])


class FrGroupNorm(ctypes.Structure):
    """Mirror of ``struct fr_group_norm``."""

    _fields_ = ([(n, ctypes.c_int32) for n in ("dtype", "gate_mode", "groups", "size", "weight_per_group")] + [("eps", c_float),
                ("y", c_void_p), ("ldy", c_int64), ("gate", c_void_p), ("ldg", c_int64), ("weight", c_void_p), ("out", c_void_p),
                ("ldo", c_int64)])


class FrQkRope(ctypes.Structure):
    """Mirror of ``struct fr_qk_rope``."""

    _fields_ = ([(n, ctypes.c_int32) for n in ("dtype", "heads", "kv_heads", "dim", "dim_true", "rot_dims")] + [("eps", c_float),
                ("pad_", ctypes.c_int32), ("q", c_void_p), ("ldq", c_int64), ("k", c_void_p), ("ldk", c_int64),
                ("q_weight", c_void_p), ("k_weight", c_void_p), ("table", c_void_p), ("loc", c_void_p),
                ("k_cache", c_void_p), ("ldkc", c_int64)])


class FrLinearScan(ctypes.Structure):
    """Mirror of ``struct fr_linear_scan``."""

    _fields_ = ([(n, ctypes.c_int32) for n in ("dtype", "decay", "heads", "key_heads", "dim", "vdim", "rank")]
                + [("scale", c_float), ("inv_tau", c_float), ("pad_", ctypes.c_int32), ("q", c_void_p), ("ldq", c_int64),
                   ("k", c_void_p), ("ldk", c_int64), ("v", c_void_p), ("ldv", c_int64), ("out", c_void_p), ("ldo", c_int64),
                   ("step", c_void_p), ("ldstep", c_int64), ("step_bias", c_void_p), ("rate", c_void_p), ("up", c_void_p),
                   ("skip", c_void_p), ("state", c_void_p), ("state_slots", c_void_p), ("qo_indptr", c_void_p),
                   ("pos", c_void_p)])


FR_SEG_STORE, FR_SEG_SWIGLU, FR_SEG_SIGMOID, FR_SEG_STORE_F32, FR_SEG_GLU_CLAMP, FR_SEG_GELU_MUL = 0, 1, 2, 3, 4, 5
FR_MIX_DIFF, FR_MIX_TALK, FR_MIX_PLAIN = 0, 1, 2
FR_CONV_LINEAR, FR_CONV_SILU = 0, 1
FR_GATE_NONE, FR_GATE_BEFORE, FR_GATE_AFTER = 0, 1, 2
FR_DECAY_CHANNEL, FR_DECAY_HEAD = 0, 1
FR_MASK_WINDOW, FR_MASK_CHUNK = 0, 1

FR_TRIE_NONE, FR_TRIE_DENSE, FR_TRIE_CSR, FR_TRIE_BITMAP = 0, 1, 2, 3

P = c_void_p
_I = c_int
_L = c_int64
_F = c_float

# name -> argtypes (restype is always int unless listed in _RESTYPES)
_SIGNATURES = {
    "fr_version": [],
    "fr_device_status": [POINTER(c_int), POINTER(c_int)],
    "fr_rms_quant_fp8": [P, P, P, _F, P, P, _I, _I, P],
    "fr_rmsnorm_bf16": [P, P, P, _F, P, _I, _I, P],
    "fr_token_quant_fp8": [P, _I, P, P, _I, _I, P],
    "fr_silu_mul_quant_fp8": [P, P, P, _I, _I, P],
    "fr_silu_mul_bf16": [P, P, _I, _I, P],
    "fr_gemm_fp8_w8a8": [P, P, P, P, P, P, _I, _I, _I, _I, _L, _L, _L, _I, P],
    "fr_gemm_fp8_w8a8_add": [P, P, P, P, P, _I, _I, _I, _L, _L, _L, _I, P],
    "fr_gemm_fp8_qkv_rope": [P, P, P, P, P, _L, _I, _I, _I, _I, _I, _L, _L, P, P, P, P, _F, P, _I, P, P, _L, _L, _L, _L, _I,
                             P],
    "fr_gemm_fp8_silu_mul": [P, P, P, P, P, P, _I, _I, _I, _L, _L, _L, _I, P],
    "fr_quant_known_amax_fp8": [P, P, P, P, _I, _I, P],
    "fr_qk_norm_rope_kv_fp8": [P, P, P, _L, _L, _L, _L, _L, _L, P, P, P, P, _F, P, _I, P, P, _L, _L, _L, _L, _I,
                               _I, _I, _I, _I, P],
    "fr_rope_neox_inplace": [P, P, P, _L, _L, _L, _L, _L, _L, P, P, P, _I, P, P, _L, _L, _L, _L, _I, _I, _I, _I, _I, P],
    "fr_store_kv_fp8": [P, P, _L, _L, _L, _L, P, P, P, _L, _L, _L, _L, _I, _I, _I, _I, _I, P],
    "fr_gather_kv_indices": [P, _L, P, P, P, P, _I, _I, P],
    "fr_kv_table_step": [P, _L, _I, _I, P, P, _I, P, P, P, P, P, P, _I, _I, P],
    "fr_kv_table_fanout": [P, _L, _I, P, P, _I, _I, _I, P],
    "fr_embedding_bf16": [P, P, P, _I, _I, _I, P],
    "fr_decode_attn_plan": [P, P, P, _I, _I, P, P],
    "fr_decode_attn_scratch_bytes": [_I, _I, _I],
    "fr_trie_build_workspace_bytes": [_L],
    "fr_trie_build_csr": [P, _L, _I, P, P, P, _L, P, P, _L, P],
    "fr_trie_csr_to_bitmap": [P, P, _L, _I, P, P, P, P, P, _I, P],
    "fr_decode_attn_fp8": [P, _L, _L, P, P, _L, _L, _L, _L, P, P, P, P, P, _L, _I, _I, _I, _I, _I, _I, _I, _F, P, _L,
                           _I, P],
    "fr_prefill_attn_fp8": [P, _L, _L, P, P, _L, _L, _L, _L, P, P, P, P, _L, _I, _I, _I, _I, _I, _I, _I, _I, _F, P, _L,
                            P],
    "fr_decode_attn_reuse_fp8": [P, _L, _L, P, P, _L, _L, _L, _L, P, P, P, P, P, _L, _I, _I, _I, _I, _I, _I, _I, _F, P,
                                 _L, _I, P, P],
    "fr_logsumexp_rows": [P, _L, P, P, P, _L, _I, _I, P],
    "fr_topk_rows": [P, _L, P, P, P, P, _I, _I, _I, P],
    "fr_lse_combine_shards": [P, P, P, P, _I, _I, _L, P],
    "fr_trie_mask": [P, P, P, P, P, _F, _L, _L, P],
    "fr_trie_advance": [P, P, P, P, P, _I, _I, _I, P],
    "fr_beam_expand": [P, P, P, P, _I, _I, _I, _I, P],
    "fr_mask_topk_expand": [P] * 16 + [_I] * 8 + [P],
    "fr_mask_topk_expand_static": [P] * 15 + [_I] * 8 + [P],
    "fr_sid_beam_step": [P] * 7 + [_L] + [P] * 9 + [_L] * 3 + [_I] * 7 + [P],
    "fr_joint_select_workspace_bytes": [_I, _I],
    "fr_joint_select": [P] * 8 + [P, P, P, P, P, _I, P, _L, _I, _I, _I, _I, P],
    "fr_select_final_topk": [P] * 4 + [P, P, P, P, _I, _I, _I, _I, P],
    "fr_sid_head_topk_workspace_bytes": [_I, _I, _I, _I],
    "fr_sid_head_topk": [P] * 6 + [P, P, _L, P, P, _L, _I] + [P] * 8 + [_L] * 3 + [_I] * 8 + [P, P, P, _L, _I, P],
    "fr_topk_merge_shards": [P] * 16 + [_L] * 2 + [_I] * 7 + [P],
    "fr_dense_proj": [_I, P, _L, P, _L, _I, _I, _I, P, _I, _I, P],
    "fr_dense_proj_split": [_I, P, _L, P, _L, _I, _I, _I, P, _I, P, _I, P],
    "fr_dense_gated_add": [_I, P, _I, P, _L, _I, _I, P, _I, P, _L, _I, P],
    "fr_dense_gated_add_splits": [_I] * 5,
    "fr_lm_embed": [_I, P, _L, P, P, _L, _I, _I, _I, _F, P, _L, P, P, P, P],
    "fr_lm_norm": [_I, P, _L, P, _F, _F, P, _I, _L, P, P, _L, _I, _I, P],
    "fr_lm_update_norm": [P, _I, _I, P],
    "fr_lm_group_norm": [P, _I, P],
    "fr_lm_rotary_table": [P, _I, P, P, _I, P],
    "fr_lm_qk_norm_rope": [P, _I, P],
    "fr_linear_state_floats": [_I, _I],
    "fr_linear_scan_rows": [P, _I, _I, _I, P],
    "fr_linear_scan_chunks": [P, _I, _I, _I, _I, P, _L, P],
    "fr_linear_scan_chunks_scratch": [P, _I, _I, _I],
    "fr_linear_scan_chunks_fit": [P],
    "fr_short_conv": [_I, P, _L, P, P, _I, _I, _I, P, _I, P, P, P, P, P, _I, _I, _I, P],
    "fr_mix_attn_rows": [P, _I, _I, _I, _I, P, _L, P, P],
    "fr_mix_attn_rows_scratch": [_I] * 6,
    "fr_mix_attn_tc": [P, P, _I, _I, _I, P, _L, P],
    "fr_mix_attn_tc_scratch": [P, _I, _I, _L],
    "fr_mix_attn_tc_fits": [_I] * 5,
}
_RESTYPES = {"fr_version": c_char_p, "fr_decode_attn_scratch_bytes": c_int64,
             "fr_sid_head_topk_workspace_bytes": c_int64, "fr_joint_select_workspace_bytes": c_int64,
             "fr_trie_build_workspace_bytes": c_int64, "fr_mix_attn_rows_scratch": c_int64,
             "fr_mix_attn_tc_scratch": c_int64, "fr_linear_state_floats": c_int64, "fr_linear_scan_chunks_scratch": c_int64}


def lib_path() -> Path:
    return _LIB_PATH


def use_library(path) -> None:
    """Bind another build of the library (``flashrec_b200.build`` can compile a subset of the sources: the entry
    points a model family needs). Must come before the first ``load()``; symbols the build lacks stay unbound."""
    global _LIB_PATH
    path = Path(path).resolve()
    if _lib is not None and path != _LIB_PATH:
        raise RuntimeError("use_library: a library is loaded already")
    _LIB_PATH = path


def load() -> ctypes.CDLL:
    """Load the shared library (once). Raises if it has not been built."""
    global _lib
    if _lib is not None:
        return _lib
    if not _LIB_PATH.exists():
        raise FlashRecKernelError(
            f"load({_LIB_PATH}): not built; run `python -m flashrec_b200.build`", -3
        )
    lib = ctypes.CDLL(str(_LIB_PATH))
    for name, argtypes in _SIGNATURES.items():
        fn = getattr(lib, name, None)
        if fn is None:
            continue  # checked by tests against include/flashrec_b200.h
        fn.argtypes = argtypes
        fn.restype = _RESTYPES.get(name, c_int)
    _lib = lib
    return lib


def stream_ptr(device: Optional[torch.device] = None) -> int:
    """Raw cudaStream_t of torch's current stream."""
    return torch.cuda.current_stream(device).cuda_stream


def ptr(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def call(name: str, *args) -> None:
    """Call an int-status entry point; raise on non-zero status."""
    fn = getattr(load(), name)
    st = fn(*args)
    if st != FR_OK:
        raise FlashRecKernelError(name, st)


def device_status() -> tuple[int, int]:
    """Read-and-clear the device status word: (code, site). Synchronises."""
    code = c_int(0)
    site = c_int(0)
    call("fr_device_status", ctypes.byref(code), ctypes.byref(site))
    return code.value, site.value


def require_cuda(*tensors: Optional[torch.Tensor]) -> None:
    for t in tensors:
        if t is not None and not t.is_cuda:
            raise FlashRecKernelError("flashrec_b200 (tensor not on a CUDA device: no CPU path)", -1)
