"""Forward pass of layer-by-layer decoders as a sequence of sm_100a kernels.

The residual stream ``x`` is fp32 and lives in one buffer that the output and down projections update in their epilogue;
the same epilogue applies the next sub-layer's element-wise norm, so a layer is four launches in decoding and five in
prefill:

    qkvg linear | (rotary + cache append |) attention with sink and gate | o linear: x += m y, h = norm2(x)
    | gate/up linear with the gated activation | down linear: x += m y (+ embedding rows before a repeated pass), h = next norm

``rt.dtype`` "float32" runs the same sequence on the 32-bit kernels."""
from __future__ import annotations

import torch

from ..ops import attention as A
from ..ops import dense as D
from ..parallel.comm import Comm
from ..utils.trace import op_range
from .config import RuntimeConfig
from .kvcache import KVState
from .layered_config import LayeredConfig

_DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class LayeredDecoder:
    supports_portions = True      # a prompt may be cut anywhere: attention reads the paged cache

    def __init__(self, cfg: LayeredConfig, rt: RuntimeConfig, weights: dict, comm: Comm | None = None, device=None, tp_ctx=None):
        if rt.tp != 1 or rt.ep != 1 or (comm is not None and comm.world > 1):
            raise ValueError("layer-by-layer decoders run on one GPU")
        self.cfg, self.rt, self.w = cfg, rt, weights
        self.device = device or weights["embed"].device
        self.dtype = _DTYPES[rt.dtype]
        self.runs = cfg.runs
        self.tp_ctx = self.moe = None
        self.last_logits: torch.Tensor | None = None       # fp32 [rows, vocab] of the latest call
        self.observer = None      # called with (run index, x) after every layer run; x then already holds the embedding
                                  # rows if the next run starts a repeated pass
        self._decode_scratch: dict = {}
        self._rope: dict = {}
        for l in cfg.layers:
            r = l.mixer.rot
            if r is not None and r not in self._rope:
                self._rope[r] = A.rope_tables(rt.max_seq_len, r.base, self.device, r.dims, r.scaling)

    def _attention(self, run: int, qkvg, positions, kv: KVState, mode, cu_seqlens, max_len, seq_ids):
        m = self.cfg.layers[self.runs[run].layer].mixer
        W = self.w["layers"][self.runs[run].layer]
        cache = kv.layers[run]
        cos, sin = self._rope[m.rot] if m.rot is not None else (None, None)
        g0 = (m.heads + m.kv_heads) * m.dk + m.kv_heads * m.dv
        spec = A.attn_spec(m.scale, chunk=m.chunk, sink=W["sink"], gate=qkvg[:, g0:g0 + m.heads])
        out = D.rows(qkvg.shape[0], m.heads * m.dv, self.dtype, qkvg.device)
        if mode == "decode":
            return A.attn_decode_paged(qkvg, m.heads, positions, kv.seq_lens, cos, sin, cache, kv.page_table, spec, out)
        A.rotary_paged(qkvg, m.heads, positions, seq_ids, cos, sin, cache, kv.page_table)
        return A.attn_prefill_paged(qkvg, m.heads, positions, seq_ids, cu_seqlens, max_len, cache, kv.page_table, spec, out)

    def _norm_before(self, run: int):
        return self.w["final_norm"] if run >= len(self.runs) else self.w["layers"][self.runs[run].layer]["norm1"]

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, kv: KVState, *, mode: str,
                cu_seqlens: torch.Tensor | None = None, max_len: int = 0, seq_ids: torch.Tensor | None = None,
                last_idx: torch.Tensor | None = None) -> torch.Tensor | None:
        """token_ids int64 [M], positions int32 [M] -> greedy next token of the rows ``last_idx`` (all rows if None).

        mode "prefill": portions of sequences, concatenated (cu_seqlens), starting at any position, earlier tokens in
        the cache; mode "decode": one token per sequence slot, kv.seq_lens already counts it.  ``last_idx`` may be
        empty: the call then only fills the cache and returns None."""
        cfg, M, d = self.cfg, token_ids.shape[0], self.cfg.d_model
        dev = token_ids.device
        x = D.rows(M, d, torch.float32, dev)
        emb = D.rows(M, d, torch.float32, dev) if any(r.add_embedding for r in self.runs) else None
        h = D.rows(M, d, self.dtype, dev)
        D.embed_norm(token_ids, self.w["embed"], d, cfg.embed_scale, x, emb, self._norm_before(0), h)
        for r, run in enumerate(self.runs):
            W, mlp = self.w["layers"][run.layer], cfg.layers[run.layer].mlp
            # what follows this run: its norm, and the embedding rows if a repeated pass starts there
            nxt = self._norm_before(r + 1)
            add = emb if r + 1 < len(self.runs) and self.runs[r + 1].add_embedding else None
            qkvg = D.linear(h, W["qkvg"])
            with op_range(f"run{r}.attention.{mode}"):
                attn = self._attention(r, qkvg, positions, kv, mode, cu_seqlens, max_len, seq_ids)
            if mlp is None:
                D.linear_residual(attn, W["o"], x, cfg.residual_mult, nxt, h, add=add)
            else:
                D.linear_residual(attn, W["o"], x, cfg.residual_mult, W["norm2"], h)
                with op_range(f"run{r}.mlp"):
                    act = D.linear_glu(h, W["gate_up"], mlp.limit)
                    D.linear_residual(act, W["down"], x, cfg.residual_mult, nxt, h, add=add)
            if self.observer is not None:
                self.observer(r, x[:, :d])
        if last_idx is not None:
            if last_idx.numel() == 0:
                self.last_logits = None
                return None
            h = h.index_select(0, last_idx)
        with op_range("head+argmax"):
            logits = D.linear(h, self.w["head"], out_dtype=torch.float32)[:, :cfg.vocab]
            self.last_logits = logits
            val, idx = A.argmax_rows(logits, index_offset=self.w["vocab_offset"])
            return A.argmax_merge(val, idx)
