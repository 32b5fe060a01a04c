"""Replays a trace of given token ids through the engine, step by step, and hands out logits.

A trace step names requests, their next tokens, the places whose logits are wanted and the requests that end with it.
Everything runs through ``Engine.step``: the model, cache, batching and kernels that generation uses; nothing is sampled."""
from __future__ import annotations

import json
import os

import torch

from ..models import registry
from ..models.config import RuntimeConfig
from .engine import Engine


class TraceReplay:
    def __init__(self, model_path: str, dtype: str, max_tokens: int, slots: int = 4, device=None):
        """``max_tokens``: the most tokens all live requests hold together (sizes the cache); ``slots``: the most requests
        that are live at once."""
        ps = RuntimeConfig().page_size
        rt = RuntimeConfig.from_env(dtype=dtype, max_batch=slots, max_seq_len=max(ps, (max_tokens + ps - 1) // ps * ps),
                                    kv_pool_tokens=max(1, max_tokens))
        device = torch.device(device) if device is not None else torch.device("cuda", torch.cuda.current_device())
        cfg, weights = registry.open_model(model_path, rt, device)
        self.engine = Engine(cfg, rt, weights=weights, device=device)
        self.engine.start_batch(slots, rt.max_seq_len)
        self.slot_of: dict[str, int] = {}
        self.free = list(range(slots - 1, -1, -1))

    def step(self, step: dict) -> torch.Tensor | None:
        """-> fp32 [wanted, vocab] on the host in the order of the entries and their places, or None if nothing is wanted."""
        entries = []
        for e in step["entries"]:
            if e["id"] not in self.slot_of:
                if not self.free:
                    raise RuntimeError(f"more than {self.engine.batch} requests live at once")
                self.slot_of[e["id"]] = self.free.pop()
            entries.append((self.slot_of[e["id"]], e["tokens"], e.get("want", [])))
        rows = [r for r in self.engine.step(entries) if r.shape[0]]
        for rid in step.get("end", []):
            slot = self.slot_of.pop(rid)
            self.engine.release_sequence(slot)
            self.free.append(slot)
        self.engine.check_status()
        return torch.cat(rows).cpu() if rows else None


def run(model_path: str, dtype: str, out_dir: str, max_tokens: int, lines, emit) -> None:
    """``lines``: JSON steps; writes ``out_dir``/<step>.f32 (little-endian) and calls ``emit("done <step>")`` after each."""
    replay = TraceReplay(model_path, dtype, max_tokens)
    os.makedirs(out_dir, exist_ok=True)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step)
        if logits is not None:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
        emit(f"done {step['step']}")
