"""Forward pass of layer-by-layer decoders as a sequence of sm_100a kernels.

Every layer run is mixer -> output projection -> feed-forward -> down projection around an fp32 residual stream that lives in
one buffer; ``streams`` holds the stream and its norms, ``mixers`` the mixers, ``moe`` the mixture of experts.  With an
element-wise norm a layer is four launches in decoding and five in prefill:

    qkvg linear | (rotary + cache append |) attention with sink and gate | o linear: x += m y, h = norm2(x)
    | gate/up linear with the gated activation | down linear: x += m y (+ embedding rows before a repeated pass), h = next norm

``rt.dtype`` "float32" runs the same sequence on the 32-bit kernels."""
from __future__ import annotations

import torch

from ..ops import attention as A
from ..ops import dense as D
from ..parallel.comm import Comm
from ..utils.trace import op_range
from . import mixers as X
from .config import RuntimeConfig
from .kvcache import KVState
from .layered_config import AttentionSpec, LatentSpec, LayeredConfig, MoE
from .moe import GroupedExperts
from .streams import STREAMS

_DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class LayeredDecoder:
    supports_portions = True      # a prompt may be cut anywhere: attention reads the paged cache, the rest its states

    def __init__(self, cfg: LayeredConfig, rt: RuntimeConfig, weights: dict, comm: Comm | None = None, device=None, tp_ctx=None):
        if rt.tp != 1 or rt.ep != 1 or (comm is not None and comm.world > 1):
            raise ValueError("layer-by-layer decoders run on one GPU")
        self.cfg, self.rt, self.w = cfg, rt, weights
        self.device = device or weights["embed"].device
        self.dtype = _DTYPES[rt.dtype]
        self.runs = cfg.runs
        self.tp_ctx = self.moe = None
        self.last_logits: torch.Tensor | None = None       # fp32 [rows, vocab] of the latest call
        self.observer = None      # called with (run index, x) after every layer run; x then already holds what joins the
                                  # stream before the next run (embedding rows or step vector of a pass)
        self.stream = STREAMS[cfg.design.norm]
        if cfg.design.norm == "dynamic_tanh" and any(isinstance(l.mlp, MoE) for l in cfg.layers):
            raise ValueError("a mixture of experts needs a stream whose norm sees whole rows")
        self._decode_scratch: dict = {}
        self._rope: dict = {}
        self.mixers = [self._mixer(l.mixer) for l in cfg.layers]
        self.experts = [GroupedExperts(l.mlp) if isinstance(l.mlp, MoE) else None for l in cfg.layers]

    def _tables(self, r):
        if r not in self._rope:
            self._rope[r] = A.rope_tables(self.rt.max_seq_len, r.base, self.device, r.dims, r.scaling)
        return self._rope[r]

    def _mixer(self, m):
        if isinstance(m, AttentionSpec):
            return X.Attention(m, self.dtype, self._tables)
        if isinstance(m, LatentSpec):
            return X.LatentAttention(m, self.dtype, self._tables, self.cfg.eps, self.rt.page_size)
        return X.MinGRU(m, self.dtype)

    def observe(self, run: int, x: torch.Tensor) -> None:
        if self.observer is not None:
            self.observer(run, x[:, :self.cfg.d_model])

    def forward(self, token_ids: torch.Tensor, positions: torch.Tensor, kv: KVState, *, mode: str,
                cu_seqlens: torch.Tensor | None = None, max_len: int = 0, seq_ids: torch.Tensor | None = None,
                last_idx: torch.Tensor | None = None, portions: list | None = None) -> torch.Tensor | None:
        """token_ids int64 [M], positions int32 [M] -> greedy next token of the rows ``last_idx`` (all rows if None).

        mode "prefill": portions of sequences, concatenated (cu_seqlens), starting at any position, earlier tokens in
        the cache; mode "decode": one token per sequence slot, kv.seq_lens already counts it.  ``portions``: first position
        and length of every portion on the host (None: whole prompts).  ``last_idx`` may be empty: the call then only fills
        the cache and returns None."""
        cfg = self.cfg
        call = X.Call(mode, positions, kv, cu_seqlens, max_len, seq_ids, portions)
        s = self.stream(self, token_ids, call)
        for r, run in enumerate(self.runs):
            W, mlp = self.w["layers"][run.layer], cfg.layers[run.layer].mlp
            h = s.mixer_input(r)
            with op_range(f"run{r}.{cfg.layers[run.layer].mixer.kind}.{mode}"):
                a = self.mixers[run.layer](r, h, W, call)
            s.add_mixer(r, a, W, last=mlp is None)
            if mlp is None:
                continue
            with op_range(f"run{r}.mlp"):
                h = s.mlp_input(r, W)
                s.add_mlp(r, self.experts[run.layer](h, W) if isinstance(mlp, MoE) else D.linear_glu(h, W["gate_up"], mlp.limit), W)
        if last_idx is not None and last_idx.numel() == 0:
            if self.observer is not None:
                s.final(None)
            self.last_logits = None
            return None
        with op_range("head+argmax"):
            h = s.final(last_idx)
            logits = D.linear(h, self.w["head"], out_dtype=torch.float32)[:, :cfg.vocab]
            self.last_logits = logits
            val, idx = A.argmax_rows(logits, index_offset=self.w["vocab_offset"])
            return A.argmax_merge(val, idx)
