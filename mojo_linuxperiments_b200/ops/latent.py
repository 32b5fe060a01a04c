"""Latent attention over the paged cache: one normalised latent and one rotated key part per token, shared by all heads."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from .attention import PAGE, PagedKVCache
from .dense import rows
from .workspace import default_workspace


MAX_ROWS = 32 * 65535          # (token, head) pairs of a portion that ``attend`` takes


def dims(heads: int, rank: int, rot: int) -> "_lib.LatentDims":
    up = lambda n: (n + 7) // 8 * 8
    return _lib.LatentDims(heads, up(rank), up(rot), rank, rot)


def _status(t: torch.Tensor) -> int:
    return default_workspace(t.device).status.data_ptr()


def append(x: torch.Tensor, q_rank: int, q_gain: torch.Tensor, c_gain: torch.Tensor, eps: float, dm, positions: torch.Tensor,
           seq_ids: torch.Tensor | None, cos: torch.Tensor, sin: torch.Tensor, cache: PagedKVCache, page_table: torch.Tensor, *,
           seq_lens: torch.Tensor | None = None, want_latents: bool = False):
    """x fp32 [M, q latent | latent | key part | ...] (each padded to eight): both norms, rotation of the key part, cache append.
    Returns the normalised query latent and (``want_latents``) the rows that went to the cache."""
    M, dt = x.shape[0], cache.data.dtype
    assert x.dtype == torch.float32 and x.stride(1) == 1 and positions.dtype == torch.int32
    qp = (q_rank + 7) // 8 * 8
    cq = rows(M, qp, dt, x.device)
    lat = torch.empty((M, dm.rank + dm.rot), dtype=dt, device=x.device) if want_latents else None
    _lib.check(_lib.lib().b200_latent_append(
        x.data_ptr(), x.stride(0), M, qp, q_rank, q_gain.data_ptr(), c_gain.data_ptr(), float(eps), ctypes.byref(dm), positions.data_ptr(),
        _lib.ptr(seq_ids), _lib.ptr(seq_lens), cos.data_ptr(), sin.data_ptr(), cos.shape[0], ctypes.byref(cache.desc(page_table)),
        cq.data_ptr(), cq.stride(0), _lib.ptr(lat), _status(x), _lib.stream()), "latent_append")
    return cq, lat


def rotary_heads(q: torch.Tensor, heads: int, head_ld: int, offset: int, rot: int, positions: torch.Tensor, cos: torch.Tensor,
                 sin: torch.Tensor) -> None:
    """q [M, heads * head_ld], in place: the ``rot`` elements at ``offset`` of every head turn (neighbouring pairs)."""
    _lib.check(_lib.lib().b200_rotary_heads(
        q.data_ptr(), q.stride(0), int(q.dtype == torch.float32), q.shape[0], heads, head_ld, offset, rot, positions.data_ptr(),
        cos.data_ptr(), sin.data_ptr(), cos.shape[0], _status(q), _lib.stream()), "rotary_heads")


def gather(cache: PagedKVCache, page_table: torch.Tensor, ctx: torch.Tensor, seqs: torch.Tensor, total: int, longest: int) -> torch.Tensor:
    """Cached rows 0 .. of sequences ``seqs`` one after the other (``ctx``: cumulative counts) -> [total, dk]."""
    lat = torch.empty((total, cache.dk), dtype=cache.data.dtype, device=cache.data.device)
    _lib.check(_lib.lib().b200_latent_gather(ctypes.byref(cache.desc(page_table)), ctx.data_ptr(), seqs.data_ptr(), seqs.numel(), longest,
                                             lat.data_ptr(), _status(cache.data), _lib.stream()), "latent_gather")
    return lat


def attend_any(q: torch.Tensor, q_rot: torch.Tensor, rot_head_ld: int, dm, scale: float, positions: torch.Tensor, seq_ids: torch.Tensor | None,
               cache: PagedKVCache, page_table: torch.Tensor, *, seq_lens: torch.Tensor | None = None) -> torch.Tensor:
    """General form (bf16 or fp32).  q [M, heads * rank] against the latents, q_rot (turned; first element of head 0, heads
    ``rot_head_ld`` apart) against the key parts -> weighted latents [M, heads * rank]."""
    out = rows(q.shape[0], dm.heads * dm.rank, q.dtype, q.device)
    _lib.check(_lib.lib().b200_attn_latent_any(
        q.data_ptr(), q.stride(0), q_rot.data_ptr(), q_rot.stride(0), rot_head_ld, out.data_ptr(), out.stride(0), q.shape[0],
        ctypes.byref(dm), float(scale), positions.data_ptr(), _lib.ptr(seq_ids), _lib.ptr(seq_lens), ctypes.byref(cache.desc(page_table)),
        _status(q), _lib.stream()), "attn_latent_any")
    return out


def fits(dm, dtype: torch.dtype, page_size: int) -> bool:
    """Whether ``attend`` takes these sizes (``attend_any`` takes all)."""
    return dtype == torch.bfloat16 and page_size == PAGE and bool(_lib.lib().b200_attn_latent_fits(dm.rank, dm.rot))


def pick_splits(batch: int, row_tiles: int, keys: int, slots: int) -> int:
    """CTAs per row tile: as many as still make one wave, with at least one tile of 128 keys each."""
    pairs = max(1, batch * row_tiles)
    return max(1, min(8, slots // pairs, keys // 128))


def attend(q: torch.Tensor, q_raw: torch.Tensor, raw_head_ld: int, dm, scale: float, positions: torch.Tensor, seq_ids: torch.Tensor | None,
           cos: torch.Tensor, sin: torch.Tensor, cache: PagedKVCache, page_table: torch.Tensor, *, cu: torch.Tensor | None = None,
           max_len: int = 1, seq_lens: torch.Tensor | None = None, keys: int | None = None, splits: int | None = None) -> torch.Tensor:
    """bf16: q [M, heads * rank] against the latents, q_raw (its second part, not yet turned) against the key parts -> weighted
    latents [M, heads * rank].  ``cu``: portions of consecutive tokens; None: one token per sequence.  ``keys``: most keys a
    row sees (default: what the page table can hold)."""
    M = q.shape[0]
    out = rows(M, dm.heads * dm.rank, q.dtype, q.device)
    if splits is None:
        longest, batch = (int(max_len), cu.numel() - 1) if cu is not None else (1, M)
        per_cta = 32 if longest * dm.heads > 16 else 16
        splits = pick_splits(batch, -(-longest * dm.heads // per_cta), keys or page_table.shape[1] * cache.page_size, _lib.num_sms(q.device.index))
    _lib.check(_lib.lib().b200_attn_latent(
        q.data_ptr(), q.stride(0), q_raw.data_ptr(), q_raw.stride(0), raw_head_ld, out.data_ptr(), out.stride(0), M, ctypes.byref(dm),
        float(scale), _lib.ptr(cu), cu.numel() - 1 if cu is not None else 0, int(max_len), positions.data_ptr(), _lib.ptr(seq_ids),
        _lib.ptr(seq_lens), cos.data_ptr(), sin.data_ptr(), cos.shape[0], ctypes.byref(cache.desc(page_table)), splits, _status(q),
        _lib.stream()), "attn_latent")
    return out


def expanded_fits(dn: int, dr: int, dv: int) -> bool:
    return bool(_lib.lib().b200_attn_prefill_latent_fits(dn, dr, dv))


def attend_expanded(q: torch.Tensor, heads: int, dn: int, dr: int, dv: int, kv: torch.Tensor, k_rot: torch.Tensor, scale: float,
                    cu: torch.Tensor, ctx: torch.Tensor, positions: torch.Tensor, max_len: int, gate: torch.Tensor | None = None) -> torch.Tensor:
    """q [M, heads * (dn + dr)] (turned) against kv [rows, heads * dn + heads * dv] and k_rot [rows, >= dr], rows ctx[b] .. of
    portion b's sequence from its first token on -> [M, heads * dv], times the sigmoid of ``gate`` fp32 [M, heads]."""
    M = q.shape[0]
    out = rows(M, heads * dv, q.dtype, q.device)
    assert gate is None or gate.dtype == torch.float32
    _lib.check(_lib.lib().b200_attn_prefill_latent(
        q.data_ptr(), q.stride(0), heads, dn, dr, dv, kv.data_ptr(), kv.stride(0), k_rot.data_ptr(), k_rot.stride(0), kv.shape[0],
        out.data_ptr(), out.stride(0), M, cu.numel() - 1, int(max_len), float(scale), cu.data_ptr(), ctx.data_ptr(), positions.data_ptr(),
        _lib.ptr(gate), gate.stride(0) if gate is not None else 0, _status(q), _lib.stream()), "attn_prefill_latent")
    return out
