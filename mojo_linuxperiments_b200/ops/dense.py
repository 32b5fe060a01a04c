"""Dense (unquantised) linears in bf16 or fp32 whose epilogue finishes the step around them.

``store`` writes the product, ``glu`` applies a bounded gated activation to interleaved gate / up columns, ``residual``
adds the product to the fp32 residual stream and hands the normalised rows to the next linear - the norm is
element-wise, so it costs no launch of its own."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from .workspace import default_workspace

DECODE_MAX_M = 64              # up to this many tokens the weight-streaming kernel runs


def padded(n: int) -> int:
    """Row pitch of an activation / weight buffer: 16-byte rows for TMA in bf16, four-column groups for the epilogues."""
    return (n + 7) // 8 * 8


def rows(m: int, n: int, dtype: torch.dtype, device) -> torch.Tensor:
    """Uninitialised [m, padded(n)] buffer: the pitch every op here expects."""
    return torch.empty((m, padded(n)), dtype=dtype, device=device)


@dataclass
class DenseW:
    """[n, k] weight stored with a padded row pitch (padding zero)."""
    data: torch.Tensor
    n: int
    k: int

    @staticmethod
    def of(w: torch.Tensor, dtype: torch.dtype, device) -> "DenseW":
        n, k = w.shape
        d = torch.zeros((n, padded(k)), dtype=dtype, device=device)
        d[:, :k] = w.to(device=device, dtype=dtype)
        return DenseW(d, n, k)


@dataclass
class DynamicTanh:
    """Element-wise norm tanh(alpha x) w + b; w and b fp32 on the device, padded."""
    alpha: float
    w: torch.Tensor
    b: torch.Tensor

    @staticmethod
    def of(alpha: float, w: torch.Tensor, b: torch.Tensor, device) -> "DynamicTanh":
        def vec(t):
            v = torch.zeros(padded(t.numel()), dtype=torch.float32, device=device)
            v[: t.numel()] = t.to(device=device, dtype=torch.float32)
            return v
        return DynamicTanh(float(alpha), vec(w), vec(b))


EPI_STORE, EPI_RESIDUAL, EPI_GLU = 0, 1, 2


def _run(x: torch.Tensor, w: DenseW, epi, force: int = 0) -> None:
    M = x.shape[0]
    if M == 0:
        return
    assert x.dtype == w.data.dtype and x.stride(1) == 1 and x.shape[1] >= w.k
    if x.dtype == torch.float32:
        rc = _lib.lib().b200_f32_gemm(x.data_ptr(), x.stride(0), w.data.data_ptr(), w.data.stride(0), M, w.n, w.k,
                                      ctypes.byref(epi), _lib.stream())
        _lib.check(rc, "f32_gemm")
        return
    assert x.dtype == torch.bfloat16
    fn, name = (_lib.lib().b200_bf16_gemm_decode, "bf16_gemm_decode") if M <= DECODE_MAX_M else (_lib.lib().b200_bf16_gemm, "bf16_gemm")
    rc = fn(x.data_ptr(), x.stride(0), w.data.data_ptr(), w.data.stride(0), M, w.n, w.k, ctypes.byref(epi),
            default_workspace(x.device).status.data_ptr(), _lib.num_sms(x.device.index), force, _lib.stream())
    _lib.check(rc, name)


def linear(x: torch.Tensor, w: DenseW, out_dtype: torch.dtype | None = None, force: int = 0) -> torch.Tensor:
    """x [M, >= k] -> [M, padded(n)] (columns beyond n are padding)."""
    y = rows(x.shape[0], w.n, out_dtype or x.dtype, x.device)
    epi = _lib.DenseEpilogue(mode=EPI_STORE, out_f32=int(y.dtype == torch.float32), y=y.data_ptr(), ldy=y.stride(0))
    _run(x, w, epi, force)
    return y


def linear_glu(x: torch.Tensor, w: DenseW, limit: float, force: int = 0) -> torch.Tensor:
    """w holds gate / up rows interleaved -> [M, padded(n / 2)]: g sigmoid(1.702 g) (u + 1), g bounded above by ``limit``,
    u on both sides."""
    y = rows(x.shape[0], w.n // 2, x.dtype, x.device)
    f32 = int(x.dtype == torch.float32)
    epi = _lib.DenseEpilogue(mode=EPI_GLU, out_f32=f32, exact=f32, y=y.data_ptr(), ldy=y.stride(0), limit=float(limit))
    _run(x, w, epi, force)
    return y


def linear_residual(x: torch.Tensor, w: DenseW, stream: torch.Tensor, mult: float, norm: DynamicTanh | None,
                    out: torch.Tensor | None, add: torch.Tensor | None = None, force: int = 0) -> None:
    """stream (fp32, in place) += mult * (x w^T) (+ add); ``out`` receives norm(stream) when a norm is given."""
    assert stream.dtype == torch.float32 and (add is None or add.stride(0) == stream.stride(0))
    assert (norm is None) == (out is None)
    f32 = int(x.dtype == torch.float32)
    epi = _lib.DenseEpilogue(mode=EPI_RESIDUAL, out_f32=f32, exact=f32, y=_lib.ptr(out), ldy=out.stride(0) if out is not None else 0,
                             x=stream.data_ptr(), ldx=stream.stride(0), add=_lib.ptr(add), mult=float(mult),
                             norm_w=_lib.ptr(norm.w) if norm else None, norm_b=_lib.ptr(norm.b) if norm else None,
                             norm_alpha=norm.alpha if norm else 0.0)
    _run(x, w, epi, force)


def embed_norm(ids: torch.Tensor, table: torch.Tensor, d: int, scale: float, stream: torch.Tensor, copy: torch.Tensor | None,
               norm: DynamicTanh, out: torch.Tensor) -> None:
    """stream (and ``copy``) = table[ids] * scale in fp32; out = norm(stream)."""
    assert ids.dtype == torch.int64 and stream.dtype == torch.float32
    f32 = int(out.dtype == torch.float32)
    epi = _lib.DenseEpilogue(mode=EPI_RESIDUAL, out_f32=f32, exact=f32, y=out.data_ptr(), ldy=out.stride(0), ldx=stream.stride(0),
                             norm_w=norm.w.data_ptr(), norm_b=norm.b.data_ptr(), norm_alpha=norm.alpha)
    rc = _lib.lib().b200_embed_norm(ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0], int(table.dtype == torch.float32),
                                    float(scale), ids.numel(), d, stream.data_ptr(), _lib.ptr(copy), ctypes.byref(epi), _lib.stream())
    _lib.check(rc, "embed_norm")
