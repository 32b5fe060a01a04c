"""Rows of the fp32 residual stream between two sub-layers: what is still to be added, a norm over the row, a token shift."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib


@dataclass
class ExpertSum:
    """What a mixture adds to every row: expert results ``y`` in slot order, weights per choice; choices numbered
    ``experts`` or more hand the row of ``through`` on."""
    y: torch.Tensor
    slot: torch.Tensor            # int32 [M, top], -1: none here
    chosen: torch.Tensor          # int32 [M, top]
    weight: torch.Tensor          # fp32 [M, top]
    experts: int
    through: torch.Tensor


@dataclass
class Shift:
    """Token shift of consecutive tokens: portions ``cu`` of sequences ``seq_ids`` (None: one token per row, sequence = row);
    ``state`` fp32 [sequences, >= d] holds each sequence's previous row, ``active`` says whose may change."""
    mix: torch.Tensor
    state: torch.Tensor
    positions: torch.Tensor
    seq_ids: torch.Tensor | None = None
    active: torch.Tensor | None = None
    cu: torch.Tensor | None = None
    max_len: int = 1


def stream_rows(d: int, gain: float, eps: float, h: torch.Tensor, *, x: torch.Tensor | None = None, x_out: torch.Tensor | None = None,
                ids: torch.Tensor | None = None, table: torch.Tensor | None = None, scale: float = 1.0, index: torch.Tensor | None = None,
                experts: ExpertSum | None = None, add: torch.Tensor | None = None, shift: Shift | None = None) -> torch.Tensor:
    """x' = table[ids] * scale or x (rows ``index`` of it), plus ``experts``, plus ``add`` -> ``x_out`` (another buffer than x);
    h = x' / rms(x') * gain, moved towards the previous token's by ``shift``."""
    r = _lib.StreamRows(gain=gain, eps=eps, h=h.data_ptr(), ldh=h.stride(0), f32=int(h.dtype == torch.float32), add=_lib.ptr(add))
    ld = x.stride(0) if x is not None else (x_out.stride(0) if x_out is not None else (d + 3) // 4 * 4)
    r.ldx, r.x, r.x_out = ld, _lib.ptr(x), _lib.ptr(x_out)
    assert x is None or x_out is None or x.stride(0) == x_out.stride(0)
    if ids is not None:
        assert ids.dtype == torch.int64
        r.ids, r.table, r.ldt, r.vocab = ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0]
        r.table_f32, r.scale = int(table.dtype == torch.float32), scale
    if index is not None:
        assert index.dtype == torch.int64
        r.index = index.data_ptr()
    if experts is not None:
        e = experts
        assert e.y.dtype == e.through.dtype == h.dtype
        r.y, r.ldy, r.slot, r.chosen, r.weight = e.y.data_ptr(), e.y.stride(0), e.slot.data_ptr(), e.chosen.data_ptr(), e.weight.data_ptr()
        r.top, r.experts, r.through, r.ldt2 = e.slot.shape[1], e.experts, e.through.data_ptr(), e.through.stride(0)
    if shift is not None:
        s = shift
        r.shift, r.state, r.state_ld, r.num_seqs = s.mix.data_ptr(), s.state.data_ptr(), s.state.stride(0), s.state.shape[0]
        r.positions, r.seq_ids, r.active, r.cu = s.positions.data_ptr(), _lib.ptr(s.seq_ids), _lib.ptr(s.active), _lib.ptr(s.cu)
        r.portions, r.max_len = (s.cu.numel() - 1 if s.cu is not None else 0), int(s.max_len)
    M = h.shape[0]
    _lib.check(_lib.lib().b200_stream_rows_launch(ctypes.byref(r), M, d, _lib.num_sms(h.device.index), _lib.stream()), "stream_rows")
    return h
