"""ctypes binding of the sm_100a kernel library (``_lib/libb200_kernels.so``).

The library is built in-tree by ``mojo_linuxperiments_b200._build``.  On a machine with a GPU a missing
library is an error (there is no PyTorch fallback for the hot ops); on a CPU-only machine importing this
module works and ``lib()`` raises only when a kernel is actually requested.
"""
from __future__ import annotations

import ctypes
from ctypes import c_int, c_void_p, c_size_t, c_float, c_longlong, c_uint64
from functools import lru_cache
from pathlib import Path

import torch

import os


def _variant() -> str:
    """Which build of the kernel library this process loads: B200RT_KERNELS=trace (in-kernel time stamps), debug
    (range-checked peer / scratch accesses) or dense (only the kernels of the unquantised models); B200RT_DEBUG=1 also
    selects the debug build.  Default: production."""
    v = os.environ.get("B200RT_KERNELS", "").strip().lower()
    if v in ("trace", "debug", "dense"):
        return v
    return "debug" if os.environ.get("B200RT_DEBUG", "0") not in ("", "0") else ""


def _lib_path() -> Path:
    v = _variant()
    return Path(__file__).resolve().parent.parent / "_lib" / ("libb200_kernels.so" if not v else f"libb200_kernels_{v}.so")


class KernelError(RuntimeError):
    pass


@lru_cache(maxsize=None)
def lib() -> ctypes.CDLL:
    path = _lib_path()
    if not path.exists():
        raise KernelError(
            f"{path} is missing: run `python -m mojo_linuxperiments_b200._build --all` (needs nvcc, no GPU)")
    L = ctypes.CDLL(str(path))
    subset = _variant() == "dense"          # a part of the library: what it does not have is an error where it is called
    for name in dir(_Sig):
        if name.startswith("b200_"):
            restype, argtypes = getattr(_Sig, name)
            try:
                fn = getattr(L, name)
            except AttributeError as e:  # stale library
                if subset:
                    continue
                raise KernelError(f"{name} not found in {path}; rebuild the kernel library") from e
            fn.restype = restype
            fn.argtypes = argtypes
    return L


P = c_void_p
I = c_int
LL = c_longlong
F = c_float


class _Sig:
    b200_w8a8_gemm_ws_bytes = (c_size_t, [I, I, I, I])
    b200_w8a8_gemm = (I, [P, P, P, P, P, P, I, I, I, I, I, P, c_size_t, P, I, P, I, I, P])
    b200_w8a8_gemm_decode = (I, [P, P, P, P, P, P, I, I, I, I, I, P, I, I, P])
    b200_w8a8_gemm_decode_resident_clusters = (I, [I, I])
    b200_w8a8_gemm_decode_p = (I, [P, P, P, P, P, I, I, I, I, I, P, I, P])
    b200_w8a8_gemm_decode_ar_p = (I, [P, P, P, P, P, I, I, I, I, P, I, P, P, P, I, I, c_size_t, c_size_t, P, I, I, c_size_t, c_size_t, c_size_t, I, c_size_t, c_size_t, c_size_t, P])
    b200_peer_allreduce = (I, [P, P, P, I, I, c_size_t, c_size_t, P, P, c_size_t, I, I, P, P, I, I, I, P])
    b200_peer_argmax = (I, [P, P, I, I, c_size_t, P, P, I, I, P, P, P, I, P])
    b200_w8a8_gemm_ag = (I, [P, P, P, P, P, I, I, I, I, I, P, P, I, I, c_size_t, c_size_t, c_size_t, c_size_t, c_size_t, c_size_t, I, I, P, P, I, I, P, I, I, P])
    b200_w8a8_gemm_rs = (I, [P, P, P, P, P, P, I, I, I, I, I, I, P, I, I, c_size_t, c_size_t, c_size_t, I, P, I, P, I, I, P])
    b200_ep_dispatch = (I, [P, P, P, P, I, I, I, I, I, P, I, I] + [c_size_t] * 10 + [I, P, P, P, I, P])
    b200_ep_wait = (I, [P, I, I] + [c_size_t] * 5 + [I, I, I, I, P, P, P, P, I, P])
    b200_ep_gather = (I, [P] + [c_size_t] * 4 + [P, I, P, P, I, P, P, P])
    b200_ep_combine_scatter = (I, [P, LL, P, P, I, I, I, I, P, I, I, c_size_t, c_size_t, c_size_t, I, P, P, I, P, I, P])
    b200_ep_combine_reduce = (I, [P, I, I, I, I, I, P, I, I, c_size_t, c_size_t, c_size_t, I, P, P, LL, P, I, I, P])
    b200_ag_sync = (I, [P, I, I, c_size_t, c_size_t, I, I, I, P, I, I, P, I, P])
    b200_w8a8_gemm_decode_ar = (I, [P, P, P, P, P, P, I, I, I, I, P, I, P, P, P, I, I, c_size_t, c_size_t, P, I, I, c_size_t, c_size_t, c_size_t, I, c_size_t, c_size_t, c_size_t, P])
    b200_where_am_i = (I, [P, I, I, P])
    b200_debug_compiled = (I, [])
    b200_debug_set_heap_extent = (I, [c_size_t])
    b200_trace_compiled = (I, [])
    b200_trace_set = (I, [P, ctypes.c_uint])
    b200_fill_uniform_reduce = (I, [P, c_uint64, c_uint64, c_uint64, P, I, P, P, P])
    b200_w8a8_gemm_decode_grouped = (I, [P, P, P, P, P, I, I, I, I, I, I, P, P, P, I, P])
    b200_w8a8_gemm_grouped = (I, [P, P, P, P, P, I, I, I, I, I, P, P, I, P, I, P])
    b200_router_topk = (I, [P, LL, I, I, I, I, P, P, P])
    b200_moe_align = (I, [P, I, I, I, I, P, P, P, P, P, P, P])
    b200_moe_gather = (I, [P, P, I, P, P, I, P, P, P])
    b200_moe_combine = (I, [P, LL, P, P, I, I, I, P, LL, P])
    b200_act_quant = (I, [P, LL, P, LL, P, F, P, LL, P, P, LL, I, I, I, P])
    b200_rope_kv_write = (I, [P, LL, P, P, P, P, P, P, F, P, P, P, P, P, I, I, I, I, I, I, I, P, P])
    b200_embed_gather = (I, [P, P, P, I, I, I, P])
    b200_argmax_rows = (I, [P, LL, I, I, I, I, P, P, P])
    b200_argmax_rows_f32 = (I, [P, LL, I, I, I, I, P, P, P])
    b200_bf16_gemm = (I, [P, LL, P, LL, I, I, I, P, P, I, I, P])
    b200_bf16_gemm_decode = (I, [P, LL, P, LL, I, I, I, P, P, I, I, P])
    b200_f32_gemm = (I, [P, LL, P, LL, I, I, I, P, P])
    b200_bf16_gemm_grouped = (I, [P, LL, P, LL, I, I, I, P, P, P, I, I, P])
    b200_bf16_gemm_decode_grouped = (I, [P, LL, P, LL, I, I, I, I, P, P, P, I, I, P])
    b200_f32_gemm_grouped = (I, [P, LL, P, LL, I, I, I, P, P, P])
    b200_stream_rows_launch = (I, [P, I, I, I, P])
    b200_route_grouped = (I, [P, LL, P, I, I, I, I, I, F, P, P, P])
    b200_moe_gather_rows = (I, [P, LL, P, P, I, P, P])
    b200_mingru_scratch_floats = (I, [I, I, I])
    b200_mingru = (I, [P, LL, P, P, I, I, P, LL, I, P, P, P, P, I, I, P, P, LL, I, P])
    b200_latent_append = (I, [P, LL, I, I, I, P, P, F, P, P, P, P, P, P, I, P, P, LL, P, P, P])
    b200_rotary_heads = (I, [P, LL, I, I, I, I, I, I, P, P, P, I, P, P])
    b200_latent_gather = (I, [P, P, P, I, I, P, P, P])
    b200_attn_latent_any = (I, [P, LL, P, LL, I, P, LL, I, P, F, P, P, P, P, P, P])
    b200_attn_latent_fits = (I, [I, I])
    b200_attn_latent = (I, [P, LL, P, LL, I, P, LL, I, P, F, P, I, I, P, P, P, P, P, I, P, I, P, P])
    b200_attn_prefill_latent_fits = (I, [I, I, I])
    b200_attn_prefill_latent = (I, [P, LL, I, I, I, I, P, LL, P, LL, I, P, LL, I, I, I, F, P, P, P, P, LL, P, P])
    b200_rotary_paged = (I, [P, LL, I, I, P, P, P, P, I, I, I, P, P, P])
    b200_embed_norm = (I, [P, P, LL, I, I, F, I, I, P, P, P, P])
    b200_attn_paged = (I, [P, LL, P, LL, I, I, P, P, P, P, P, P, P])
    b200_attn_prefill_paged = (I, [P, LL, P, LL, I, I, I, I, P, P, P, P, P, P, P])
    b200_attn_decode_paged = (I, [P, LL, P, LL, I, I, P, P, P, P, I, I, I, P, P, I, P, P])
    b200_argmax_merge = (I, [P, P, I, I, P, P])
    b200_attn_decode_scratch_floats = (c_size_t, [I, I, I])
    b200_attn_decode = (I, [P, P, P, P, P, P, P, I, I, I, I, I, I, F, P, P])
    b200_attn_decode_noalloc = (I, [P, P, P, P, P, I, I, I, I, I, I, F, P])
    b200_attn_decode_tma = (I, [P, P, I, P, P, P, P, P, I, I, I, I, I, I, F, P, P])
    b200_attn_decode_tc = (I, [P, P, I, P, P, P, P, P, I, I, I, I, I, I, F, P, P])
    b200_attn_decode_tc_min_splits = (I, [I])
    b200_attn_decode_fused = (I, [P, LL, P, P, P, I, P, P, F, P, I, P, P, P, P, LL, P, P, P, P, P, P, I, I, I, I, I, I, F, P, P, c_uint64, P])
    b200_attn_decode_tcp = (I, [P, P, I, P, P, P, P, P, I, I, I, I, I, I, F, P, I, P])
    b200_attn_prefill = (I, [P, LL, P, LL, P, LL, P, P, I, I, I, I, I, F, P, P])
    b200_attn_prefill_split = (I, [P, LL, P, LL, P, LL, P, P, I, I, I, I, I, F, I, P, P, P])
    b200_attn_prefill_split_scratch_floats = (c_size_t, [I, I, I, I])


class QuantProlog(ctypes.Structure):
    """``b200_quant_prolog`` of csrc/kernels/api.h: the activation prologue a decode GEMM launch carries itself."""
    _fields_ = [("mode", c_int), ("x", c_void_p), ("ldx", c_longlong), ("residual", c_void_p), ("ldr", c_longlong),
                ("gamma", c_void_p), ("eps", c_float), ("q", c_void_p), ("scale", c_void_p), ("flags", c_void_p),
                ("step", c_void_p), ("residual_out", c_void_p), ("ldro", c_longlong), ("allow_inline", c_int)]


class DenseEpilogue(ctypes.Structure):
    """``b200_dense_epilogue`` of csrc/kernels/api.h: what a dense linear does with its result."""
    _fields_ = [("mode", c_int), ("out_f32", c_int), ("exact", c_int), ("y", c_void_p), ("ldy", c_longlong), ("x", c_void_p),
                ("ldx", c_longlong), ("add", c_void_p), ("mult", c_float), ("norm_w", c_void_p), ("norm_b", c_void_p),
                ("norm_alpha", c_float), ("limit", c_float), ("act", c_int), ("gate", c_void_p), ("ldg", c_longlong),
                ("y_group", c_longlong)]


class GemmGroups(ctypes.Structure):
    """``b200_gemm_groups`` of csrc/kernels/api.h: several linears in one launch."""
    _fields_ = [("groups", c_int), ("x_group", c_longlong), ("offsets", c_void_p), ("counts", c_void_p), ("tiles", c_void_p),
                ("num_tiles", c_void_p), ("max_tiles", c_int), ("expected", c_int)]


class StreamRows(ctypes.Structure):
    """``b200_stream_rows`` of csrc/kernels/api.h: rows of the residual stream between two sub-layers."""
    _fields_ = [("ids", c_void_p), ("table", c_void_p), ("ldt", c_longlong), ("vocab", c_int), ("table_f32", c_int), ("scale", c_float),
                ("x", c_void_p), ("ldx", c_longlong), ("index", c_void_p), ("y", c_void_p), ("ldy", c_longlong), ("slot", c_void_p),
                ("chosen", c_void_p), ("weight", c_void_p), ("top", c_int), ("experts", c_int), ("through", c_void_p),
                ("ldt2", c_longlong), ("add", c_void_p), ("x_out", c_void_p), ("gain", c_float), ("eps", c_float), ("h", c_void_p),
                ("ldh", c_longlong), ("f32", c_int), ("shift", c_void_p), ("state", c_void_p), ("state_ld", c_longlong),
                ("num_seqs", c_int), ("positions", c_void_p), ("seq_ids", c_void_p), ("active", c_void_p), ("cu", c_void_p),
                ("portions", c_int), ("max_len", c_int)]


class LatentDims(ctypes.Structure):
    """``b200_latent_dims`` of csrc/kernels/api.h."""
    _fields_ = [("heads", c_int), ("rank", c_int), ("rot", c_int), ("true_rank", c_int), ("true_rot", c_int)]


class PagedCacheDesc(ctypes.Structure):
    """``b200_paged_cache`` of csrc/kernels/api.h."""
    _fields_ = [("data", c_void_p), ("f32", c_int), ("kv_heads", c_int), ("page_size", c_int), ("dk", c_int), ("dv", c_int),
                ("num_pages", c_int), ("page_table", c_void_p), ("num_seqs", c_int), ("max_pages", c_int)]


class AttnSpecDesc(ctypes.Structure):
    """``b200_attn_spec`` of csrc/kernels/api.h."""
    _fields_ = [("scale", c_float), ("chunk", c_int), ("sink", c_void_p), ("gate", c_void_p), ("ldg", c_longlong)]


def ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def stream() -> int:
    return torch.cuda.current_stream().cuda_stream


LAUNCHES = [0]     # kernels of this library launched (or captured into a CUDA graph) by this process


def check(rc: int, what: str) -> None:
    if rc != 0:
        raise KernelError(f"{what} failed with code {rc}")
    LAUNCHES[0] += 1


@lru_cache(maxsize=None)
def num_sms(device_index: int) -> int:
    return torch.cuda.get_device_properties(device_index).multi_processor_count
