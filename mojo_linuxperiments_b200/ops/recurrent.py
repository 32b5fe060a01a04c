"""Gated linear recurrence over time (minGRU) with a state per sequence."""
from __future__ import annotations

import torch

from . import _lib
from .dense import rows


def mingru(zxg: torch.Tensor, zb: torch.Tensor, xb: torch.Tensor, width: int, state: torch.Tensor, positions: torch.Tensor, *,
           out_dtype: torch.dtype, seq_ids: torch.Tensor | None = None, active: torch.Tensor | None = None,
           cu: torch.Tensor | None = None, max_len: int = 1) -> torch.Tensor:
    """zxg fp32 [M, 3 * width]: gate, candidate and output-gate projections -> S * silu(g), [M, padded(width)].

    ``cu``: portions of consecutive tokens (sequence ``seq_ids`` of their first row); None: one token per sequence, row =
    sequence.  ``state`` fp32 [sequences, >= width] continues where position > 0 and is replaced (where ``active``)."""
    M = zxg.shape[0]
    assert zxg.dtype == torch.float32 and zxg.stride(1) == 1 and state.dtype == torch.float32 and positions.dtype == torch.int32
    out = rows(M, width, out_dtype, zxg.device)
    portions = cu.numel() - 1 if cu is not None else 0
    scratch = None
    if cu is not None:
        scratch = torch.empty(_lib.lib().b200_mingru_scratch_floats(portions, int(max_len), width), dtype=torch.float32, device=zxg.device)
    _lib.check(_lib.lib().b200_mingru(
        zxg.data_ptr(), zxg.stride(0), zb.data_ptr(), xb.data_ptr(), M, width, state.data_ptr(), state.stride(0), state.shape[0],
        positions.data_ptr(), _lib.ptr(seq_ids), _lib.ptr(active), _lib.ptr(cu), portions, int(max_len), _lib.ptr(scratch),
        out.data_ptr(), out.stride(0), int(out_dtype == torch.float32), _lib.stream()), "mingru")
    if cu is not None and M:
        _lib.LAUNCHES[0] += 1                    # two kernels
    return out
