"""ctypes binding of ``libnkipy_b200_kernels.so`` (C ABI in ``csrc/kernels/api.h``).

The library is built in-tree by ``nkipy_b200.ops._build.build()``.  Loading is
lazy; on a machine with a CUDA device a missing library is an error (the ops
never fall back to eager PyTorch on the GPU), on a CPU-only machine the ops use
their PyTorch reference implementations instead.
"""

from __future__ import annotations

import ctypes
import os
from ctypes import c_float, c_int, c_longlong, c_ulonglong, c_void_p
from pathlib import Path

LIB_PATH = Path(__file__).resolve().parent / "libnkipy_b200_kernels.so"

_lib = None
_initialised = False
_subset = False

_P = c_void_p


class ProjArg(ctypes.Structure):
    """One slice of a projection's result (csrc/kernels/proj_src.h)."""
    _fields_ = [("ptr", c_void_p), ("ld", c_longlong), ("split_stride", c_longlong), ("splits", c_int), ("bf16", c_int)]


class MapsArg(ctypes.Structure):
    """Sizes and constants of attention with several score maps (csrc/kernels/attn_maps.h)."""
    _fields_ = [(n, c_int) for n in ("maps", "heads", "kv_heads", "dim", "dim_p", "vdim", "vdim_p")] + \
               [(n, c_float) for n in ("scale", "softcap", "lam", "out_scale", "eps")] + \
               [("window", c_int), ("chunk", c_int), ("sinks", c_void_p)] + \
               [(n, c_longlong) for n in ("q_token", "q_head", "o_token", "o_head")] + \
               [("v_ld", c_int), ("keep_first", c_int), ("dist_a", c_void_p), ("dist_b", c_void_p)]


class ScoreModsArg(ctypes.Structure):
    """What plain attention does to a score beyond scaling it (csrc/kernels/attn_maps.h)."""
    _fields_ = [("softcap", c_float), ("keep_first", c_int), ("dist_a", c_void_p), ("dist_b", c_void_p)]


class LatentArg(ctypes.Structure):
    """Sizes and constants of latent attention (csrc/kernels/latent_attn.h)."""
    _fields_ = [(n, c_int) for n in ("heads", "dim", "rot", "rank", "q_rank", "row")] + \
               [("eps", c_float), ("scale", c_float), ("window", c_int), ("sinks", c_void_p)] + \
               [(n, c_longlong) for n in ("q_token", "q_head", "o_token", "o_head")]


class BranchArg(ctypes.Structure):
    """One addend of a residual update (csrc/kernels/proj_src.h)."""
    _fields_ = [("y", ProjArg), ("g", ProjArg), ("gbias", c_void_p), ("pair_pos", c_void_p), ("pair_w", c_void_p),
                ("norm_w", c_void_p), ("top_k", c_int), ("token_gate", c_int), ("scale", c_float)]


class LinAttnArg(ctypes.Structure):
    """Arguments of the linear-attention kernels (csrc/kernels/linear_attn.h)."""
    _fields_ = [(n, ProjArg) for n in ("q", "k", "v", "z", "g")] + \
               [(n, c_void_p) for n in ("w2", "z_bias", "bonus", "norm_w", "state", "slot_ids", "q_start", "q_lens",
                                        "context_lens", "heads_out", "out")] + [("out_ld", c_longlong)] + \
               [(n, c_int) for n in ("w2_bf16", "rank", "z_act", "decay", "norm_stride", "gate_act", "bf16", "batch",
                                     "tokens", "heads", "dim", "vdim")] + \
               [(n, c_float) for n in ("q_scale", "inv_tau", "out_scale", "eps")]


class HeadRecArg(ctypes.Structure):
    """Arguments of recurrences with one decay per head (csrc/kernels/head_recurrence.h)."""
    _fields_ = [(n, ProjArg) for n in ("x", "a", "b", "g")] + \
               [(n, c_void_p) for n in ("conv_w", "conv_b", "conv_state", "rate", "dt_bias", "skip", "norm_w", "state", "slot_ids",
                                        "q_start", "q_lens", "context_lens", "out")] + \
               [(n, c_int) for n in ("taps", "channels", "q_col", "k_col", "v_col", "gate_act", "bf16", "batch", "tokens", "heads",
                                     "groups", "dim", "vdim")] + [(n, c_float) for n in ("q_scale", "eps", "unit_eps")]


class TanhNormArg(ctypes.Structure):
    _fields_ = [("w", c_void_p), ("b", c_void_p), ("alpha", c_float), ("out", c_void_p)]


class PostBranchArg(ctypes.Structure):
    _fields_ = [("y", ProjArg), ("shift", c_void_p), ("norm_w", c_void_p), ("scale", c_float)]


class PostResidualArg(ctypes.Structure):
    """Arguments of a residual update through a norm (csrc/kernels/post_residual.h)."""
    _fields_ = [("x_in", c_void_p), ("ids", c_void_p), ("table", c_void_p), ("br", PostBranchArg * 2), ("post", TanhNormArg),
                ("norm", TanhNormArg * 2), ("history", c_void_p), ("coef", c_void_p), ("result", c_void_p), ("x_out", c_void_p),
                ("history_stride", c_longlong)] + \
               [(n, c_int) for n in ("vocab", "table_bf16", "branches", "norms", "past", "out_bf16", "rows", "width")] + \
               [("table_scale", c_float), ("eps", c_float)]


_PP = ctypes.POINTER(ProjArg)
_PM = ctypes.POINTER(MapsArg)
_PL = ctypes.POINTER(LatentArg)
_SIGNATURES = {
    "nkb_init": (c_int, []),
    "nkb_status": (c_int, [c_int]),
    "nkb_set_pdl": (None, [c_int]),
    "nkb_gemm_bf16": (
        c_int,
        [_P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, c_int, c_int, c_longlong,
         c_int, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_int, c_float, c_float, _P],
    ),
    "nkb_gemm_bf16_2cta": (c_int, [_P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, _P, _P, c_int,
                                   c_int, c_int, c_float, c_float, _P]),
    "nkb_gemm_simt": (c_int, [_P, c_int, _P, c_int, _P, c_int, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong,
                              _P]),
    "nkb_gemm_simt_grouped": (c_int, [_P, c_int, _P, c_int, _P, c_int, _P, _P, c_int, c_int, c_int, c_int, c_longlong,
                                      c_longlong, _P]),
    "nkb_linattn_scan": (c_int, [ctypes.POINTER(LinAttnArg), _P]),
    "nkb_linattn_step": (c_int, [ctypes.POINTER(LinAttnArg), _P]),
    "nkb_low_rank": (c_int, [_PP, c_int, _P, c_int, _P, c_int, c_int, c_int, _P]),
    "nkb_token_mix": (c_int, [_P, c_int, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, _P]),
    "nkb_gate_heads": (c_int, [_P, c_int, c_longlong, c_longlong, _PP, c_int, c_int, _P, c_int, c_float, c_float, _P, c_int,
                               c_longlong, c_int, c_int, c_int, _P]),
    "nkb_row_norm_append": (c_int, [_PM, _PP, _PP, _PP, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P]),
    "nkb_rope_norm_append": (c_int, [_PM, _PP, _PP, _PP, _P, _P, c_int, c_int, _P, _P, c_int, c_int, _P, _P, _P, c_int, c_int,
                                     c_int, _P]),
    "nkb_short_conv": (c_int, [_PP, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "nkb_head_rec_scan": (c_int, [ctypes.POINTER(HeadRecArg), _P]),
    "nkb_head_rec_step": (c_int, [ctypes.POINTER(HeadRecArg), _P]),
    "nkb_gated_group_norm": (c_int, [_P, c_int, _PP, c_int, _P, c_float, _P, c_int, c_int, c_int, c_int, _P]),
    "nkb_post_residual": (c_int, [ctypes.POINTER(PostResidualArg), _P]),
    "nkb_latent_append": (c_int, [_PL, _PP, _PP, _P, _P, _P, c_int, _P, _P, _P, _P, c_int, c_int, c_int, _P]),
    "nkb_latent_queries": (c_int, [_PL, _PP, _P, c_int, _P, _P, c_longlong, c_longlong, c_int, _P, c_longlong, c_longlong,
                                   c_int, c_int, c_int, _P]),
    "nkb_latent_gather": (c_int, [_P, _P, c_int, c_int, c_int, c_int, c_int, _P, _P, c_int, c_int, _P]),
    "nkb_latent_prefill": (c_int, [_P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                   c_longlong, c_longlong, c_int, c_int, c_float, c_int, _P, _P]),
    "nkb_latent_attn": (c_int, [_PL, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "nkb_gated_residual": (c_int, [_P, _P, _P, c_int, c_int, c_float, c_int, ctypes.POINTER(BranchArg), _P, _P, _P,
                                   c_int, c_int, ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P), c_int, c_int,
                                   c_int, c_int, c_float, _P]),
    "nkb_gated_act": (c_int, [_PP, _PP, _P, c_int, c_int, c_int, c_int, c_float, c_float, _P, c_int, _P]),
    "nkb_hgrn2_scan_scratch": (c_longlong, [c_int, c_int, c_int]),
    "nkb_hgrn2_scan": (c_int, [_PP, _PP, _PP, _P, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                               _P, c_float, _P]),
    "nkb_hgrn2_step": (c_int, [_PP, _PP, _PP, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P, c_float,
                               _P]),
    "nkb_maps_append": (c_int, [_PM, _PP, _PP, _PP, _P, c_int, c_int, _P, _P, _P, _P, _P, c_int, c_int, c_int, _P]),
    "nkb_maps_attn_simple": (c_int, [_PM, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P]),
    "nkb_maps_decode_scratch_floats": (c_longlong, [_PM, c_int, c_int]),
    "nkb_maps_attn_decode": (c_int, [_PM, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P]),
    "nkb_maps_attn_prefill": (c_int, [_PM, _P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                                      _P]),
    "nkb_gemm_bf16_grouped": (
        c_int,
        [_P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_longlong, c_longlong, c_int, c_int, _P, c_longlong,
         c_float, c_float, c_int, _P, _P, c_int, _P, ctypes.c_uint, _P],
    ),
    "nkb_moe_a2a_dispatch": (c_int, [_P, _P, c_int, c_int, c_int, c_int, c_int, c_int, ctypes.c_uint,
                                     ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P),
                                     ctypes.POINTER(_P), ctypes.POINTER(_P), _P, _P, _P, _P, c_int, c_int, _P, _P,
                                     c_int, _P, _P, _P, _P]),
    "nkb_moe_a2a_combine": (c_int, [_P, _P, c_int, c_int, c_int, c_int, c_int, ctypes.c_uint, ctypes.POINTER(_P),
                                    ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P), ctypes.POINTER(_P),
                                    ctypes.POINTER(_P), _P, _P]),
    "nkb_moe_dispatch": (c_int, [_P, c_int, c_int, c_int, c_int, _P, c_int, c_int, _P, _P, _P, _P, _P, _P, _P, c_int, _P, _P,
                                 c_int, _P, _P, _P]),
    "nkb_moe_combine": (c_int, [_P, _P, _P, c_int, c_int, c_int, _P, _P]),
    "nkb_gemm_effective_splits": (c_int, [c_int, c_int]),
    "nkb_decode_gemm_splits": (c_int, [c_int, c_int, c_int]),
    "nkb_decode_gemm": (c_int, [_P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, c_int,
                                c_int, _P, _P, c_float, c_float, c_int, c_int, _P]),
    "nkb_decode_gemm_push": (c_int, [_P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, _P, c_int,
                                     ctypes.POINTER(_P), ctypes.POINTER(_P), c_int, c_int, _P, _P, _P, _P]),
    "nkb_decode_gemm_rope": (c_int, [_P, _P, c_int, c_int, c_longlong, c_longlong, c_int, _P, _P, _P, _P, _P, _P,
                                     c_float, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, _P]),
    "nkb_noalloc_status": (c_int, [c_int]),
    "nkb_gemm_fix_scratch_floats": (c_longlong, [c_int, c_int, c_int, c_int]),
    "nkb_gemm_fix_store": (c_int, [_P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, _P, _P,
                                   _P, _P, c_int, _P]),
    "nkb_gemm_fix_swiglu": (c_int, [_P, _P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_longlong, c_int, _P,
                                    c_float, c_float, _P, _P, c_int, _P]),
    "nkb_gemm_fix_rope": (c_int, [_P, _P, c_int, c_int, c_longlong, c_longlong, c_int, _P, _P, _P, _P, _P, _P, c_float,
                                  _P, _P, _P, c_int, c_int, c_int, c_int, c_int, _P, _P, c_int, _P]),
    "nkb_gemm_fix_push": (c_int, [_P, _P, c_int, c_int, c_int, c_longlong, c_longlong, c_int, _P, ctypes.POINTER(_P),
                                  ctypes.POINTER(_P), c_int, c_int, _P, _P, _P, _P, _P, c_int, _P]),
    "nkb_rmsnorm": (c_int, [_P, _P, _P, c_int, c_int, c_float, _P]),
    "nkb_add_rmsnorm": (c_int, [_P, c_int, c_longlong, _P, _P, _P, _P, _P, _P, c_int, c_int, c_float, _P]),
    "nkb_silu_mul": (c_int, [_P, _P, c_int, c_int, c_float, c_float, _P]),
    "nkb_silu_mul_partials": (c_int, [_P, c_int, c_longlong, _P, _P, c_int, c_int, c_float, c_float, _P]),
    "nkb_embedding": (c_int, [_P, _P, _P, c_int, c_int, c_int, _P]),
    "nkb_rope_kv_append": (
        c_int,
        [_P, _P, c_int, c_longlong, _P, _P, _P, _P, _P, _P, c_float, _P, _P, _P, c_int, c_int, c_int, c_int, c_int,
         c_int, _P],
    ),
    "nkb_decode_advance": (c_int, [_P, _P, _P, _P, c_int, c_int, c_int, c_int, _P]),
    "nkb_argmax": (c_int, [_P, c_int, _P, _P, c_int, c_int, c_longlong, _P]),
    "nkb_sample": (c_int, [_P, c_int, _P, c_int, c_int, c_longlong, c_float, c_int, c_float, c_ulonglong,
                           c_ulonglong, _P]),
    "nkb_softcap": (c_int, [_P, c_longlong, c_float, _P]),
    "nkb_router_topk": (c_int, [_P, c_int, c_int, c_longlong, c_longlong, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int,
                                c_float, _P]),
    "nkb_paged_attn_decode": (
        c_int,
        [_P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_int,
         _P, ctypes.POINTER(ScoreModsArg), c_int, _P],
    ),
    "nkb_paged_attn_decode_fused": (
        c_int,
        [_P, c_int, c_longlong, _P, _P, _P, _P, _P, _P, c_float, c_int, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int,
         c_int, c_int, c_int, c_int, c_float, c_int, _P, c_int, _P],
    ),
    "nkb_paged_attn_decode_scratch_floats": (c_longlong, [c_int, c_int, c_int, c_int, c_int]),
    "nkb_flash_attn_prefill": (
        c_int,
        [_P, _P, _P, _P, _P, _P, _P, _P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float,
         c_int, c_int, c_int, _P, ctypes.POINTER(ScoreModsArg), _P],
    ),
}


class KernelLibraryError(RuntimeError):
    """The native kernel library is missing, failed to load, or a launch failed."""


def available() -> bool:
    return LIB_PATH.exists()


def use_serving_subset() -> None:
    """For a process that only serves a single-GPU decoder: when the library has to be built first, build and load
    only the kernels such a model launches (`_build.SERVING_SOURCES`).  A library that is up to date is used as is."""
    global _subset
    _subset = True


def lib():
    """Load the shared library (once) and declare its signatures."""
    global _lib
    if _lib is not None:
        return _lib
    from . import _build

    if _subset and _build.is_stale():
        try:
            return _declare(_build.build_subset())
        except RuntimeError as e:
            raise KernelLibraryError(f"the serving kernels could not be built: {e}")

    # The signatures below are declared from the sources in the tree, so the binary must have been built
    # from exactly those sources: a stale library would be handed shifted arguments.
    if _build.is_stale():
        if os.environ.get("NKIPY_B200_AUTOBUILD", "1") == "1":
            try:
                _build.build()          # takes an inter-process lock; other ranks wait and then find it fresh
            except RuntimeError as e:
                raise KernelLibraryError(f"the kernel library is missing or stale and could not be rebuilt: {e}")
        if _build.is_stale():
            raise KernelLibraryError(
                f"{LIB_PATH} is missing or was built from other sources than csrc/kernels: "
                "run `python -m nkipy_b200.ops._build` (needs nvcc) first"
            )
    return _declare(LIB_PATH)


def _declare(path):
    global _lib
    handle = ctypes.CDLL(str(path))
    for name, (res, args) in _SIGNATURES.items():
        try:
            fn = getattr(handle, name)
        except AttributeError:
            continue  # optional entry points are checked at their call site
        fn.restype = res
        fn.argtypes = args
    _lib = handle
    return _lib


def ensure_init():
    """Create the device status word and resolve the TMA encoder (needs a GPU)."""
    global _initialised
    if not _initialised:
        rc = lib().nkb_init()
        if rc != 0:
            raise KernelLibraryError(f"nkb_init failed with code {rc}")
        _initialised = True


def check(rc: int, what: str):
    if rc != 0:
        raise KernelLibraryError(f"{what} failed with code {rc}")


_ERRORS = {
    1: "TMA producer timed out waiting for a free shared-memory stage",
    2: "MMA warp timed out waiting for TMA data",
    3: "MMA warp timed out waiting for the epilogue to free TMEM",
    4: "epilogue timed out waiting for the MMA result",
    5: "a peer or producer flag never arrived",
    6: "bad argument detected on the device",
    7: "MMA warp timed out waiting for the softmax warps",
}


def device_status(reset: bool = True) -> int:
    """Read the device status word (synchronises).  0 means no bounded wait gave up."""
    return int(lib().nkb_status(1 if reset else 0))


def raise_on_device_error():
    code = device_status(reset=True)
    if code:
        raise KernelLibraryError(
            f"device kernel reported status {code & 0xFF} ({_ERRORS.get(code & 0xFF, 'unknown')}) "
            f"from CTA {code >> 8}"
        )
