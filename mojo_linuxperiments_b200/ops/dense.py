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
HEADS_MAX_M = 8192             # tokens per launch of a linear per head


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


@dataclass
class GroupedW:
    """Weights of several linears stacked row by row, [groups * n, k] with a padded row pitch."""
    data: torch.Tensor
    groups: int
    n: int
    k: int

    @staticmethod
    def of(ws, groups: int, dtype: torch.dtype, device, n: int | None = None) -> "GroupedW":
        """``ws``: ``groups`` matrices [rows <= n, k], taken one at a time; missing rows are zero."""
        data = None
        for g, w in enumerate(ws):
            rows_, k = w.shape
            n = n or rows_
            if data is None:
                data = torch.zeros((groups * n, padded(k)), dtype=dtype, device=device)
            data[g * n:g * n + rows_, :k] = w.to(device=device, dtype=dtype)
        return GroupedW(data, groups, n, k)


EPI_STORE, EPI_RESIDUAL, EPI_GLU = 0, 1, 2
ACTIVATIONS = {None: 0, "relu2": 1}


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


def linear_heads(x: torch.Tensor, w: GroupedW, x_group: int, y_group: int, gate: torch.Tensor | None = None,
                 out_dtype: torch.dtype | None = None, splits: int = 0) -> torch.Tensor:
    """One linear per head in one launch: group g takes columns g * x_group .. of x and writes columns g * y_group .. of the
    result; ``gate`` fp32 [M, groups] (row stride free): logits of a sigmoid on each head's result."""
    y = rows(x.shape[0], w.groups * y_group, out_dtype or x.dtype, x.device)
    for a in range(0, x.shape[0], HEADS_MAX_M):             # what one launch's grid can count
        _linear_heads(x[a:a + HEADS_MAX_M], w, x_group, y_group, gate[a:a + HEADS_MAX_M] if gate is not None else None,
                      y[a:a + HEADS_MAX_M], splits)
    return y


def _linear_heads(x, w, x_group, y_group, gate, y, splits) -> None:
    M = x.shape[0]
    assert x.dtype == w.data.dtype and x.stride(1) == 1 and x_group % 8 == 0 and y_group % 8 == 0 and y_group >= (w.n + 3) // 4 * 4
    assert x.shape[1] >= (w.groups - 1) * x_group + w.k and (gate is None or gate.dtype == torch.float32)
    epi = _lib.DenseEpilogue(mode=EPI_STORE, out_f32=int(y.dtype == torch.float32), exact=int(x.dtype == torch.float32), y=y.data_ptr(),
                             ldy=y.stride(0), gate=_lib.ptr(gate), ldg=gate.stride(0) if gate is not None else 0, y_group=y_group)
    g = _lib.GemmGroups(groups=w.groups, x_group=x_group)
    if x.dtype == torch.float32:
        rc = _lib.lib().b200_f32_gemm_grouped(x.data_ptr(), x.stride(0), w.data.data_ptr(), w.data.stride(0), M, w.n, w.k,
                                              ctypes.byref(epi), ctypes.byref(g), _lib.stream())
        _lib.check(rc, "f32_gemm_grouped")
    else:
        rc = _lib.lib().b200_bf16_gemm_decode_grouped(
            x.data_ptr(), x.stride(0), w.data.data_ptr(), w.data.stride(0), M, M, w.n, w.k, ctypes.byref(epi), ctypes.byref(g),
            default_workspace(x.device).status.data_ptr(), _lib.num_sms(x.device.index), splits, _lib.stream())
        _lib.check(rc, "bf16_gemm_decode_grouped")


def linear_experts(x: torch.Tensor, w: GroupedW, work, act: str | None = None, force: int = 0) -> torch.Tensor:
    """x: rows in the slot order of ``work`` (ops.moe.MoEWorkList); every expert multiplies its own rows."""
    y = rows(x.shape[0], w.n, x.dtype, x.device)
    if work.M == 0:
        return y
    assert x.dtype == w.data.dtype and x.stride(1) == 1 and x.shape[1] >= w.k and w.groups == work.n_local
    f32 = int(x.dtype == torch.float32)
    epi = _lib.DenseEpilogue(mode=EPI_STORE, out_f32=f32, exact=f32, y=y.data_ptr(), ldy=y.stride(0), act=ACTIVATIONS[act])
    g = _lib.GemmGroups(groups=w.groups, offsets=work.offsets.data_ptr(), counts=work.counts.data_ptr(), tiles=work.tiles.data_ptr(),
                        num_tiles=work.meta[1:].data_ptr(), max_tiles=work.max_tiles, expected=min(w.groups, work.max_slots))
    args = (x.data_ptr(), x.stride(0), w.data.data_ptr(), w.data.stride(0))
    if f32:
        rc = _lib.lib().b200_f32_gemm_grouped(*args, work.M, w.n, w.k, ctypes.byref(epi), ctypes.byref(g), _lib.stream())
        _lib.check(rc, "f32_gemm_grouped")
        return y
    tail = (ctypes.byref(epi), ctypes.byref(g), default_workspace(x.device).status.data_ptr(), _lib.num_sms(x.device.index), force, _lib.stream())
    if work.M <= DECODE_MAX_M:
        _lib.check(_lib.lib().b200_bf16_gemm_decode_grouped(*args, work.M, x.shape[0], w.n, w.k, *tail), "bf16_gemm_decode_grouped")
    else:
        _lib.check(_lib.lib().b200_bf16_gemm_grouped(*args, x.shape[0], w.n, w.k, *tail), "bf16_gemm_grouped")
    return y


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
