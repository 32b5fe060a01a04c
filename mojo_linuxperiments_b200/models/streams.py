"""The fp32 residual stream of layer-by-layer decoders, from embedding rows to the rows the head multiplies.

Two forms with the same calls, chosen by the design's norm.  ``ElementwiseStream``: the norm needs no statistics, so the
projections that update the stream also hand the next sub-layer its normalised rows (no launch of its own).  ``RowStream``: the
norm needs the whole row, so one launch between two sub-layers adds what is still pending (embedding rows, expert results, the
step vector of a pass), normalises and shifts."""
from __future__ import annotations

import torch

from ..ops import dense as D
from ..ops import rows as RW
from .mixers import Call


class ElementwiseStream:
    def __init__(self, model, ids: torch.Tensor, call: Call):
        self.model, self.w, self.cfg = model, model.w, model.cfg
        M, d, dev = ids.shape[0], self.cfg.d_model, ids.device
        runs = model.runs
        self.x = D.rows(M, d, torch.float32, dev)
        self.emb = D.rows(M, d, torch.float32, dev) if any(r.add_embedding for r in runs) else None
        self.h = D.rows(M, d, model.dtype, dev)
        D.embed_norm(ids, self.w["embed"], d, self.cfg.embed_scale, self.x, self.emb, self._norm_before(0), self.h)

    def _norm_before(self, run: int):
        runs = self.model.runs
        return self.w["final_norm"] if run >= len(runs) else self.w["layers"][runs[run].layer]["norm1"]

    def _close(self, r: int, a, w) -> None:
        """The run's last update: the next run's norm, and the embedding rows if a repeated pass starts there."""
        runs = self.model.runs
        add = self.emb if r + 1 < len(runs) and runs[r + 1].add_embedding else None
        D.linear_residual(a, w, self.x, self.cfg.residual_mult, self._norm_before(r + 1), self.h, add=add)
        self.model.observe(r, self.x)

    def mixer_input(self, r: int) -> torch.Tensor:
        return self.h

    def add_mixer(self, r: int, a, W: dict, last: bool) -> None:
        if last:
            self._close(r, a, W["o"])
        else:
            D.linear_residual(a, W["o"], self.x, self.cfg.residual_mult, W["norm2"], self.h)

    def mlp_input(self, r: int, W: dict) -> torch.Tensor:
        return self.h

    def add_mlp(self, r: int, act, W: dict) -> None:
        self._close(r, act, W["down_proj"])

    def final(self, last_idx: torch.Tensor | None) -> torch.Tensor:
        return self.h if last_idx is None else self.h.index_select(0, last_idx)


class RowStream:
    def __init__(self, model, ids: torch.Tensor, call: Call):
        self.model, self.w, self.cfg, self.call = model, model.w, model.cfg, call
        M, d, dev = ids.shape[0], self.cfg.d_model, ids.device
        self.ids = ids                                      # until the embedding rows are in x
        self.x, self.spare = D.rows(M, d, torch.float32, dev), None
        self.h1, self.h2 = D.rows(M, d, model.dtype, dev), D.rows(M, d, model.dtype, dev)
        self.experts: RW.ExpertSum | None = None            # the mixture that is still to be added
        self.opened = -1

    def _rows(self, gain: float, h: torch.Tensor, add=None, shift=None, index=None, keep: bool = True) -> None:
        src = {}
        if self.ids is not None:
            src = {"ids": self.ids, "table": self.w["embed"], "scale": self.cfg.embed_scale, "x_out": self.x if keep else None}
        else:
            src = {"x": self.x}
            if keep and (self.experts is not None or add is not None):
                if self.spare is None:
                    self.spare = torch.empty_like(self.x)
                src["x_out"] = self.spare
        RW.stream_rows(self.cfg.d_model, gain, self.cfg.eps, h, experts=self.experts, add=add, shift=shift, index=index, **src)
        if keep:
            if self.ids is None and "x_out" in src:
                self.x, self.spare = self.spare, self.x
            self.ids = self.experts = None

    def mixer_input(self, r: int) -> torch.Tensor:
        run, c = self.model.runs[r], self.call
        W = self.w["layers"][run.layer]
        shift = None
        if "shift" in W:
            shift = RW.Shift(W["shift"], c.kv.states[r]["shift"], c.positions, **c.carried)
        self._rows(W["norm1"], self.h1, add=self.w["step"][run.step] if run.step is not None else None, shift=shift)
        if r > 0:
            self.model.observe(r - 1, self.x)
        return self.h1

    def add_mixer(self, r: int, a, W: dict, last: bool) -> None:
        D.linear_residual(a, W["o"], self.x, self.cfg.residual_mult, None, None)

    def mlp_input(self, r: int, W: dict) -> torch.Tensor:
        self._rows(W["norm2"], self.h2)
        return self.h2

    def add_mlp(self, r: int, act, W: dict) -> None:
        if isinstance(act, RW.ExpertSum):
            self.experts = act
        else:
            D.linear_residual(act, W["down_proj"], self.x, self.cfg.residual_mult, None, None)

    def final(self, last_idx: torch.Tensor | None) -> torch.Tensor:
        if self.model.observer is not None:
            self._rows(self.w["final_norm"], self.h1)
            self.model.observe(len(self.model.runs) - 1, self.x)
        h = self.h1 if last_idx is None else D.rows(last_idx.numel(), self.cfg.d_model, self.model.dtype, self.x.device)
        self._rows(self.w["final_norm"], h, index=last_idx, keep=False)
        return h


STREAMS = {"dynamic_tanh": ElementwiseStream, "scalar_rms": RowStream}
