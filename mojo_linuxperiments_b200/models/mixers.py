"""Mixers of layer-by-layer decoders: normalised rows in, what the output projection multiplies out.

Every mixer is called with the number of the layer run (its cache and state are the run's own), the rows, the layer's weights
and the ``Call``; it appends to the cache / moves the state on and returns [M, padded] rows for ``W["o"]``."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops import attention as A
from ..ops import dense as D
from ..ops import latent as LT
from ..ops import recurrent as R
from .kvcache import KVState
from .layered_config import AttentionSpec, LatentSpec, MinGRUSpec


@dataclass
class Call:
    """One forward pass: which tokens these rows are."""
    mode: str                              # "prefill": portions of sequences; "decode": one token per sequence slot
    positions: torch.Tensor                # int32 [M]
    kv: KVState
    cu_seqlens: torch.Tensor | None = None
    max_len: int = 0
    seq_ids: torch.Tensor | None = None
    portions: list | None = None           # host: (first position, tokens) of every portion; None: all start at 0
    _context: tuple | None = None

    @property
    def decode(self) -> bool:
        return self.mode == "decode"

    @property
    def carried(self) -> dict:
        """How kernels with a state per sequence find it."""
        if self.decode:
            return {"active": self.kv.active}
        return {"seq_ids": self.seq_ids, "cu": self.cu_seqlens, "max_len": self.max_len}

    @property
    def fresh(self) -> bool:
        """Every portion starts its sequence."""
        return self.portions is None or all(a == 0 for a, _ in self.portions)

    @property
    def context(self):
        """Portions that continue sequences: cumulative numbers of tokens up to each portion's end, the sequences, the total and
        the longest (on the device and on the host; made once per call)."""
        if self._context is None:
            ends = [a + n for a, n in self.portions]
            ctx = torch.tensor([0] + ends).cumsum(0).to(torch.int32).to(self.positions.device, non_blocking=True)
            seqs = self.seq_ids.index_select(0, self.cu_seqlens[:-1].to(torch.int64))
            self._context = ctx, seqs, sum(ends), max(ends)
        return self._context


class Attention:
    """Grouped heads over keys and values: rotary embedding, chunk mask, sink, output gate."""

    def __init__(self, spec: AttentionSpec, dtype: torch.dtype, tables):
        self.m, self.dtype = spec, dtype
        self.cos, self.sin = tables(spec.rot) if spec.rot is not None else (None, None)

    def __call__(self, run: int, h: torch.Tensor, W: dict, c: Call) -> torch.Tensor:
        m, cache = self.m, c.kv.layers[run]
        qkvg = D.linear(h, W["qkvg"])
        g0 = (m.heads + m.kv_heads) * m.dk + m.kv_heads * m.dv
        spec = A.attn_spec(m.scale, chunk=m.chunk, sink=W["sink"], gate=qkvg[:, g0:g0 + m.heads])
        out = D.rows(qkvg.shape[0], m.heads * m.dv, self.dtype, qkvg.device)
        if c.decode:
            return A.attn_decode_paged(qkvg, m.heads, c.positions, c.kv.seq_lens, self.cos, self.sin, cache, c.kv.page_table, spec, out)
        A.rotary_paged(qkvg, m.heads, c.positions, c.seq_ids, self.cos, self.sin, cache, c.kv.page_table)
        return A.attn_prefill_paged(qkvg, m.heads, c.positions, c.seq_ids, c.cu_seqlens, c.max_len, cache, c.kv.page_table, spec, out)


class LatentAttention:
    """The cache holds latents.  Decoding and short portions move the queries into the latent space and attend to the latents
    themselves; long portions expand the latents into keys and values, which costs less per query but something per key."""

    def __init__(self, spec: LatentSpec, dtype: torch.dtype, tables, eps: float, page_size: int):
        self.m, self.dtype, self.eps = spec, dtype, eps
        self.cos, self.sin = tables(spec.rot)
        self.dims = LT.dims(spec.heads, spec.kv_rank, spec.rot_dim)
        self.in_latent_space = LT.fits(self.dims, dtype, page_size)
        self.can_expand = dtype == torch.bfloat16 and LT.expanded_fits(spec.dn, spec.dr, spec.dv)

    def expands(self, longest: int) -> bool:
        """Portions of up to ``longest`` tokens: multiplications per key and head, those of the first form twice as dear (the
        expanded form's run on the tcgen05 units)."""
        m = self.m
        return self.can_expand and 2 * longest * (2 * m.rank + m.dr) > m.rank * (m.dn + m.dv) + longest * (m.dn + m.dr + m.dv)

    def __call__(self, run: int, h: torch.Tensor, W: dict, c: Call) -> torch.Tensor:
        m, kv, cache = self.m, c.kv, c.kv.layers[run]
        seq_ids, seq_lens = (None, kv.seq_lens) if c.decode else (c.seq_ids, None)
        expand = not c.decode and self.expands(c.max_len)
        low = D.linear(h, W["down"], out_dtype=torch.float32)          # query latent | latent | key part | gates
        cq, lat = LT.append(low, m.q_rank, W["q_gain"], W["c_gain"], self.eps, self.dims, c.positions, seq_ids, self.cos, self.sin,
                            cache, kv.page_table, seq_lens=seq_lens, want_latents=expand and c.fresh)
        g0 = m.qr + m.rank + m.dr
        gate = low[:, g0:g0 + m.heads]
        q = D.linear(cq, W["uq"])
        if expand:
            ctx = c.cu_seqlens
            if not c.fresh:
                ctx, seqs, total, longest = c.context
                lat = LT.gather(cache, kv.page_table, ctx, seqs, total, longest)
            LT.rotary_heads(q, m.heads, m.dn + m.dr, m.dn, m.rot.dims, c.positions, self.cos, self.sin)
            return LT.attend_expanded(q, m.heads, m.dn, m.dr, m.dv, D.linear(lat, W["ukv"]), lat[:, m.rank:], m.scale, c.cu_seqlens, ctx,
                                      c.positions, c.max_len, gate)
        qa = D.linear_heads(q, W["uk"], m.dn + m.dr, m.rank)
        if self.in_latent_space and (c.decode or c.max_len * m.heads <= LT.MAX_ROWS):
            keys = None if c.decode else (c.max_len if c.portions is None else max(a + n for a, n in c.portions))
            o = LT.attend(qa, q[:, m.dn:], m.dn + m.dr, self.dims, m.scale, c.positions, seq_ids, self.cos, self.sin, cache, kv.page_table,
                          cu=c.cu_seqlens, max_len=c.max_len, seq_lens=seq_lens, keys=keys)
        else:
            LT.rotary_heads(q, m.heads, m.dn + m.dr, m.dn, m.rot.dims, c.positions, self.cos, self.sin)
            o = LT.attend_any(qa, q[:, m.dn:], m.dn + m.dr, self.dims, m.scale, c.positions, seq_ids, cache, kv.page_table, seq_lens=seq_lens)
        return D.linear_heads(o, W["uv"], m.rank, m.dv, gate=gate)


class MinGRU:
    def __init__(self, spec: MinGRUSpec, dtype: torch.dtype):
        self.m, self.dtype = spec, dtype

    def __call__(self, run: int, h: torch.Tensor, W: dict, c: Call) -> torch.Tensor:
        zxg = D.linear(h, W["zxg"], out_dtype=torch.float32)
        return R.mingru(zxg, W["zb"], W["xb"], self.m.channels, c.kv.states[run]["recurrent"], c.positions, out_dtype=self.dtype,
                        **c.carried)
