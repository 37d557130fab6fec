"""ctypes binding of the native sm_100a library.

The library is plain C entry points over raw device pointers and a CUDA stream, so the
binding needs no torch headers; tensors are passed as ``tensor.data_ptr()`` and kernels
run on ``torch.cuda.current_stream()`` (which is what makes them capturable in CUDA graphs
together with the surrounding torch code).

On a machine with a GPU the library is mandatory: ``lib()`` raises if it cannot be loaded,
so a missing build can never turn into a silent PyTorch fallback.
"""
from __future__ import annotations

import ctypes as C
from functools import lru_cache

import torch

from . import build as _build


class GemmParams(C.Structure):
    """Mirror of ``E2hGemmParams`` (csrc/gemm_umma.cuh)."""

    _fields_ = [
        ("F", C.c_int), ("T", C.c_int), ("K", C.c_int),
        ("splitk", C.c_int), ("epi", C.c_int), ("stages", C.c_int),
        ("a_mn_major", C.c_int), ("b_mn_major", C.c_int),
        ("bn", C.c_int), ("dual", C.c_int), ("accumulate", C.c_int), ("pdl", C.c_int),
        ("lda", C.c_longlong), ("lda2", C.c_longlong), ("ldb", C.c_longlong),
        ("a", C.c_void_p), ("a2", C.c_void_p), ("b", C.c_void_p),
        ("out", C.c_void_p), ("ldo", C.c_longlong),
        ("out2", C.c_void_p), ("ldo2", C.c_longlong),
        ("aux", C.c_void_p), ("scale", C.c_void_p),
        ("freqs", C.c_void_p), ("pos_base", C.c_void_p),
        ("sq", C.c_int), ("n_head", C.c_int), ("n_kv", C.c_int), ("head_dim", C.c_int),
        ("smax", C.c_int),
        ("kcache", C.c_void_p), ("vcache", C.c_void_p),
        ("status", C.c_void_p),
        ("tf", C.c_int),
        ("th", C.c_int),
        ("stage_epi", C.c_int),
        ("kps", C.c_int),
        ("n_signal", C.c_int),
        ("signal", C.c_void_p * 8),
        ("ticket", C.c_void_p),
        ("a_tiled", C.c_int),
        ("groupsize", C.c_int), ("qsz", C.c_void_p), ("qsz2", C.c_void_p),
        ("phase_clock", C.c_void_p),
        ("bias", C.c_void_p), ("act", C.c_int), ("act_from", C.c_int), ("tail_from", C.c_int),
        ("ldt", C.c_longlong), ("tail", C.c_void_p),
        ("n_groups", C.c_int), ("group_tmax", C.c_int), ("group_off", C.c_void_p),
        ("out_scale", C.c_float), ("softcap", C.c_float),
        ("n_batch", C.c_int), ("batch_k", C.c_int), ("batch_out", C.c_int),
    ]


class StreamNormParams(C.Structure):
    """Mirror of ``StreamNormParams`` (csrc/stream_norm.cu)."""

    _fields_ = [
        ("x", C.c_void_p), ("tokens", C.c_void_p), ("emb", C.c_void_p), ("lde", C.c_longlong),
        ("vocab", C.c_int), ("emb_scale", C.c_float), ("y", C.c_void_p), ("ldy", C.c_longlong),
        ("place", C.c_void_p), ("ew", C.c_void_p), ("top", C.c_int), ("y_rows", C.c_int),
        ("rows", C.c_void_p), ("x_rows", C.c_int), ("weight", C.c_void_p), ("offset", C.c_float),
        ("eps", C.c_float), ("out", C.c_void_p), ("ldo", C.c_longlong), ("W", C.c_int),
        ("col", C.c_void_p), ("left_pad", C.c_void_p), ("pos_out", C.c_void_p),
        ("status", C.c_void_p),
    ]


class AttnWindowParams(C.Structure):
    """Mirror of ``AttnWindowParams`` (csrc/attn_window.cu)."""

    _fields_ = [
        ("act", C.c_void_p), ("ld", C.c_longlong), ("off_q", C.c_int), ("off_k", C.c_int),
        ("off_v", C.c_int), ("off_g", C.c_int), ("kc", C.c_void_p), ("vc", C.c_void_p),
        ("pos", C.c_void_p), ("slot", C.c_void_p), ("n", C.c_int), ("slots", C.c_int),
        ("smax", C.c_int), ("H", C.c_int), ("G", C.c_int), ("dim", C.c_int), ("vdim", C.c_int),
        ("dimp", C.c_int), ("vdimp", C.c_int), ("rot", C.c_int), ("rot_table", C.c_void_p),
        ("scale", C.c_float), ("window", C.c_int), ("keep", C.c_int), ("qn", C.c_void_p),
        ("kn", C.c_void_p), ("eps", C.c_float), ("splits", C.c_int), ("status", C.c_void_p),
    ]


class LatentParams(C.Structure):
    """Mirror of ``LatentParams`` (csrc/latent_attn.cu)."""

    _fields_ = [
        ("act", C.c_void_p), ("ld", C.c_longlong), ("off_q", C.c_int), ("off_c", C.c_int),
        ("ql", C.c_void_p), ("ol", C.c_void_p), ("cache", C.c_void_p), ("pos", C.c_void_p),
        ("slot", C.c_void_p), ("n", C.c_int), ("slots", C.c_int), ("smax", C.c_int),
        ("H", C.c_int), ("dim", C.c_int), ("rank", C.c_int), ("rot", C.c_int),
        ("rank_n", C.c_int), ("rot_table", C.c_void_p), ("norm", C.c_void_p), ("eps", C.c_float),
        ("scale", C.c_float), ("window", C.c_int), ("splits", C.c_int), ("ctx", C.c_void_p),
        ("ctx_src", C.c_void_p), ("ctx_pos", C.c_void_p), ("ctx_slot", C.c_void_p),
        ("n_ctx", C.c_int), ("n_long", C.c_int), ("status", C.c_void_p),
    ]


class FlashWindowArgs(C.Structure):
    """Mirror of ``FlashWindowArgs`` (csrc/flash_window.cu)."""

    _fields_ = [
        ("act", C.c_void_p), ("ld", C.c_longlong), ("off_q", C.c_int), ("q_head", C.c_int),
        ("off_g", C.c_int), ("k", C.c_void_p), ("ld_k", C.c_longlong), ("k_head", C.c_longlong),
        ("k_slot", C.c_longlong), ("v", C.c_void_p), ("ld_v", C.c_longlong),
        ("v_head", C.c_longlong), ("v_slot", C.c_longlong), ("k2", C.c_void_p),
        ("ld_k2", C.c_longlong), ("rows", C.c_int), ("slots", C.c_int), ("smax", C.c_int),
        ("shift", C.c_void_p), ("seg", C.c_void_p), ("n_seg", C.c_int), ("seg_max", C.c_int),
        ("pos", C.c_void_p), ("slot", C.c_void_p), ("n", C.c_int), ("H", C.c_int), ("G", C.c_int),
        ("dim", C.c_int), ("dim2", C.c_int), ("vdim", C.c_int), ("scale", C.c_float),
        ("window", C.c_int), ("keep", C.c_int), ("status", C.c_void_p),
    ]


class GlaParams(C.Structure):
    """Mirror of ``E2hGlaParams`` (csrc/gla.cuh)."""

    _fields_ = [
        ("act", C.c_void_p), ("ld", C.c_longlong), ("off_q", C.c_int), ("off_k", C.c_int),
        ("off_v", C.c_int), ("off_g", C.c_int), ("a", C.c_void_p), ("lda", C.c_longlong),
        ("r", C.c_int), ("w2", C.c_void_p), ("ldw", C.c_longlong), ("b2", C.c_void_p),
        ("inv_tau", C.c_float), ("qscale", C.c_float), ("eps", C.c_float), ("norm", C.c_void_p),
        ("state", C.c_void_p), ("slots", C.c_int), ("H", C.c_int), ("dim", C.c_int),
        ("vdim", C.c_int), ("vp", C.c_int), ("pos", C.c_void_p), ("slot", C.c_void_p),
        ("n", C.c_int), ("splits", C.c_int), ("seg", C.c_void_p), ("n_seg", C.c_int),
        ("seg_max", C.c_int), ("logdec", C.c_void_p), ("o", C.c_void_p), ("chunks", C.c_int),
        ("cq", C.c_void_p), ("ck", C.c_void_p), ("ca", C.c_void_p), ("cg", C.c_void_p),
        ("status", C.c_void_p),
    ]


EPI_STORE_BF16 = 0
EPI_STORE_F32 = 1
EPI_SWIGLU = 2
EPI_ROPE_KV = 3
EPI_RESIDUAL = 4
EPI_ROWMAJOR_F32_ACC = 5
EPI_ROWMAJOR_BF16 = 6
EPI_DUAL_STORE = 7
EPI_RESIDUAL_F32 = 8
EPI_GATE = 9

_vp, _i, _ll, _f, _ull = C.c_void_p, C.c_int, C.c_longlong, C.c_float, C.c_ulonglong

_SIGNATURES = {
    "e2h_gemm_umma": [C.POINTER(GemmParams), _vp],
    "e2h_gemm_persistent": [C.POINTER(GemmParams), _vp],
    "e2h_gemm_w8": [C.POINTER(GemmParams), _vp],
    "e2h_gemm_w4": [C.POINTER(GemmParams), _vp],
    "e2h_gemm_f32": [C.POINTER(GemmParams), _vp],
    "e2h_stream_norm": [C.POINTER(StreamNormParams), _i, _i, _vp],
    "e2h_attn_prep": [C.POINTER(AttnWindowParams), _i, _vp],
    "e2h_attn_window": [C.POINTER(AttnWindowParams), _i, _i, _vp],
    "e2h_gla_chunk": [C.POINTER(GlaParams), _vp],
    "e2h_flash_window": [C.POINTER(FlashWindowArgs), _vp],
    "e2h_latent_prep": [C.POINTER(LatentParams), _i, _vp],
    "e2h_latent_attn": [C.POINTER(LatentParams), _i, _i, _vp],
    "e2h_gla_step": [C.POINTER(GlaParams), _i, _vp],
    "e2h_gla_decay": [C.POINTER(GlaParams), _i, _vp],
    "e2h_gla_scan": [C.POINTER(GlaParams), _i, _vp],
    "e2h_gla_out": [C.POINTER(GlaParams), _i, _vp],
    "e2h_moe_route": [_vp, _ll, _i, _i, _i, _i, _i, _vp, _ll, _i, _vp, _ll, _vp, _vp, _vp, _vp, _i,
                      _vp],
    "e2h_rmsnorm_fwd": [_vp, _vp, _vp, _i, C.POINTER(C.c_void_p), _i, _vp, _vp, _vp, _vp, _i, _i, _f,
                        _vp, _vp, _vp, _vp, _vp],
    "e2h_reduce_residual_norm_bf16": [_vp, C.POINTER(C.c_void_p), _i, _vp, _vp, _vp, _i, _i, _f,
                                      _vp, _vp, _vp, _vp, _vp],
    "e2h_rmsnorm_bwd": [_vp, _vp, _vp, _vp, _vp, _i, _i, _f, _vp],
    "e2h_embedding": [_vp, _vp, _i, _vp, _i, _i, _vp, _vp],
    "e2h_swiglu_fwd": [_vp, _vp, _vp, _ll, _vp],
    "e2h_swiglu_bwd": [_vp, _vp, _vp, _vp, _vp, _ll, _vp],
    "e2h_rope": [_vp, _vp, _vp, _vp, _i, _i, _i, _ll, _i, _vp],
    "e2h_attn_decode": [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _f, _i, _vp, _vp,
                        _vp],
    "e2h_adamw": [_vp, _vp, _vp, _vp, _ll, _i, _i, _i, _f, _f, _f, _f, _f, _f, _f, _vp, _vp, _vp],
    "e2h_sqnorm": [_vp, _ll, _i, _vp, _vp],
    "e2h_clip_coef": [_vp, _f, _vp, _vp, _vp],
    "e2h_reward_head": [_vp, _ll, _vp, _vp, _ll, _i, _i, _i, _f, _vp, _i, _ll, _vp, _vp, _i, _vp, _vp,
                        _vp, _vp],
    "e2h_gae": [_vp, _vp, _vp, _vp, _i, _i, _f, _f, _vp],
    "e2h_flash_fwd": [_vp, _ll, _ll, _ll, _vp, _vp, _ll, _ll, _ll, _vp, _ll, _ll, _ll, _vp, _vp,
                      _i, _i, _i, _i, _i, _i, _f, _vp, _vp],
    "e2h_signal_peers": [C.POINTER(C.c_void_p), _i, _vp],
    "e2h_reduce_scatter_accum": [C.POINTER(C.c_void_p), _i, _vp, _ll, _f, _i, _vp, _vp, _vp, _i,
                                 _vp, _vp],
    "e2h_wait_flags": [_vp, _i, _vp, _i, _i, _vp, _vp],
    "e2h_p2p_all_gather": [C.POINTER(C.c_void_p), _i, _vp, _ll, _vp, _vp, _vp, _i, _vp, _vp],
    "e2h_p2p_reduce_bf16": [C.POINTER(C.c_void_p), _i, _vp, _ll, _f, _vp, _vp, _vp, _i, _vp, _vp],
    "e2h_tp_reduce_norm": [_vp, _vp, _vp, C.POINTER(C.c_void_p), C.POINTER(C.c_void_p),
                           C.POINTER(C.c_void_p), _vp, _vp, _vp, _vp, _i, _i, _i, _i, _f, _i, _i,
                           _i, _i, _vp, _vp],
    "e2h_tp_rows": [_i, _vp, _vp, _vp, C.POINTER(C.c_void_p), C.POINTER(C.c_void_p),
                    C.POINTER(C.c_void_p), C.POINTER(C.c_void_p), _vp, _vp, _vp, _vp, _i, _i, _i,
                    _i, _f, _i, _i, _i, _vp, _vp],
    "e2h_tp_embed_partial": [_vp, _vp, _i, _i, _vp, _i, _i, C.POINTER(C.c_void_p), _i, _vp, _vp],
    "e2h_tp_gather_logits": [C.POINTER(C.c_void_p), _i, _i, _i, _vp, _ll, _vp, _vp, _vp, _i, _vp,
                             _vp],
    "e2h_relayout_pull": [C.POINTER(C.c_void_p), _i, _ll, _ll, _ll, _ll, _ll, _ll, _ll, _ll, _vp,
                          _vp],
    "e2h_set_pdl": [_i],
    "e2h_set_flag_wait_ms": [_i],
    "e2h_flash_bwd": [_vp, _ll, _ll, _ll, _vp, _vp, _ll, _ll, _ll, _vp, _ll, _ll, _ll, _vp, _ll,
                      _ll, _ll, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _f, _vp,
                      _vp],
    "e2h_ce_stats": [_vp, _ll, _i, _i, _vp, _i, _f, _vp, _vp],
    "e2h_ce_grad": [_vp, _ll, _i, _i, _vp, _i, _f, _vp, _vp, _vp, _vp, _vp, _ll, _vp],
    "e2h_sample": [_vp, _ll, _i, _i, _f, _i, _ull, _vp, _i, _vp, _vp, _ll, _i, _i, _vp, _vp,
                   _vp, _vp, _vp],
}


class NativeLibraryError(RuntimeError):
    pass


_only = None


def build_only(names) -> None:
    """For programs that run a few kernels: unless the whole library is built already, ``lib()``
    builds and loads one of these sources (stems of csrc/*.cu) alone."""
    global _only
    _only = tuple(names)


@lru_cache(maxsize=1)
def lib() -> C.CDLL:
    """Load (building first if the sources changed and nvcc is present) the native library."""
    path = _build.lib_path()
    try:
        if _build.needs_build():
            path = _build.build(only=_only)
    except Exception as e:  # no nvcc on this machine: use the shipped binary if there is one
        if not path.exists():
            raise NativeLibraryError(f"native library missing and cannot be built: {e}") from e
    try:
        cdll = C.CDLL(str(path))
    except OSError as e:
        raise NativeLibraryError(f"cannot load {path}: {e}") from e
    for name, argtypes in _SIGNATURES.items():
        try:
            fn = getattr(cdll, name)
        except AttributeError:
            continue  # optional entry point of a newer / older build
        fn.argtypes = argtypes
        fn.restype = C.c_int
    return cdll


def available() -> bool:
    """True when CUDA kernels can run here (a GPU is visible and the library loads)."""
    if not torch.cuda.is_available():
        return False
    lib()  # raises loudly on a GPU machine without the library
    return True


def ptr(t) -> int | None:
    if t is None:
        return None
    return t.data_ptr()


def stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def check(rc: int, what: str) -> None:
    if rc != 0:
        raise NativeLibraryError(f"{what} failed with code {rc}")


_status_words: dict = {}


def status_word(device=None) -> torch.Tensor:
    """Per-device int32 status word that kernels write a code to when a bounded wait expires."""
    dev = torch.device(device if device is not None else torch.cuda.current_device())
    if dev.type != "cuda":
        dev = torch.device("cuda", torch.cuda.current_device())
    if dev.index is None:
        dev = torch.device("cuda", torch.cuda.current_device())
    w = _status_words.get(dev.index)
    if w is None:
        w = torch.zeros(1, dtype=torch.int32, device=dev)
        _status_words[dev.index] = w
    return w


def read_status(device=None, reset: bool = True) -> int:
    w = status_word(device)
    v = int(w.item())
    if reset and v != 0:
        w.zero_()
    return v
