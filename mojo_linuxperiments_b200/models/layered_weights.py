"""Weights of layer-by-layer decoders: checkpoint folder (config.json + model.safetensors) -> the layouts the kernels read.

Tensor names: ``embed``, ``head``, ``final.norm``; per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.{q,k,v,g,o,sink}``,
``l<i>.mlp.{gate,up,down}``; a norm ``x`` also has ``x.alpha`` and ``x.b``.  Matrices are [out, in].

On the device q, k, v and the gate are one matrix (rows of a head padded to a multiple of eight with zeros, the columns of
the output projection likewise), gate and up are interleaved row by row, norms and sinks are fp32."""
from __future__ import annotations

import json
import os

import torch

from ..ops.dense import DenseW, DynamicTanh
from .config import RuntimeConfig
from .layered_config import AttentionSpec, LayeredConfig

_DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def read_config(path: str) -> LayeredConfig:
    with open(os.path.join(path, "config.json")) as f:
        return LayeredConfig.from_dict(json.load(f))


class _Checkpoint:
    """Reads one tensor at a time (a model never exists twice on the host)."""

    def __init__(self, path: str):
        from safetensors import safe_open
        self._ctx = safe_open(os.path.join(path, "model.safetensors"), framework="pt")
        self._f = self._ctx.__enter__()

    def __getitem__(self, name: str) -> torch.Tensor:
        return self._f.get_tensor(name)

    def close(self) -> None:
        self._ctx.__exit__(None, None, None)


def _expect(t: torch.Tensor, shape: tuple, name: str) -> torch.Tensor:
    if tuple(t.shape) != shape:
        raise ValueError(f"{name} is {tuple(t.shape)}, the configuration says {shape}")
    return t


def _pad_head_rows(w: torch.Tensor, heads: int, size: int, to: int) -> torch.Tensor:
    """[heads * size, k] -> [heads * to, k] with zero rows after each head."""
    if size == to:
        return w
    out = w.new_zeros((heads, to, w.shape[1]))
    out[:, :size] = w.view(heads, size, -1)
    return out.view(heads * to, -1)


def qkvg_matrix(q, k, v, g, m: AttentionSpec) -> torch.Tensor:
    return torch.cat([_pad_head_rows(q, m.heads, m.dim, m.dk), _pad_head_rows(k, m.kv_heads, m.dim, m.dk),
                      _pad_head_rows(v, m.kv_heads, m.vdim, m.dv), g])


def place(cfg: LayeredConfig, rt: RuntimeConfig, t, device) -> dict:
    """``t[name]``: checkpoint tensors (a dict or an open file) -> device weights."""
    dt = _DTYPES[rt.dtype]
    d = cfg.d_model

    def get(name, *shape):
        return _expect(t[name], shape, name)

    def norm(name):
        return DynamicTanh.of(float(get(name + ".alpha").float()), get(name, d), get(name + ".b", d), device)

    table = DenseW.of(get("embed", cfg.vocab, d), dt, device)
    w = {"embed": table.data, "head": DenseW.of(get("head", cfg.vocab, d), dt, device), "final_norm": norm("final.norm"),
         "vocab_offset": 0, "layers": []}
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        x = p + "mix."
        L = {"norm1": norm(p + "norm1"),
             "qkvg": DenseW.of(qkvg_matrix(get(x + "q", m.heads * m.dim, d), get(x + "k", m.kv_heads * m.dim, d),
                                           get(x + "v", m.kv_heads * m.vdim, d), get(x + "g", m.heads, d), m), dt, device),
             "sink": get(x + "sink", m.heads).to(device=device, dtype=torch.float32).contiguous(),
             "o": DenseW.of(_pad_head_rows(get(x + "o", d, m.heads * m.vdim).t().contiguous(), m.heads, m.vdim, m.dv).t(), dt, device)}
        if layer.mlp is not None:
            ff = layer.mlp.ff
            gate, up = get(p + "mlp.gate", ff, d), get(p + "mlp.up", ff, d)
            L["norm2"] = norm(p + "norm2")
            L["gate_up"] = DenseW.of(torch.stack([gate, up], 1).reshape(2 * ff, d), dt, device)
            L["down"] = DenseW.of(get(p + "mlp.down", d, ff), dt, device)
        w["layers"].append(L)
    return w


def load(path: str, rt: RuntimeConfig, device):
    """Checkpoint folder -> (config, device weights)."""
    cfg = read_config(path)
    ck = _Checkpoint(path)
    try:
        return cfg, place(cfg, rt, ck, device)
    finally:
        ck.close()


def save(path: str, cfg: LayeredConfig, tensors: dict) -> None:
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        f.write(cfg.to_json())
    save_file({k: v.contiguous().cpu() for k, v in tensors.items()}, os.path.join(path, "model.safetensors"))


def init_master(cfg: LayeredConfig, seed: int = 0, device="cpu") -> dict:
    """Random bf16 checkpoint tensors by name (tests, smoke runs)."""
    g = torch.Generator(device=device).manual_seed(seed)
    d = cfg.d_model

    def w(n, k, gain=1.0):
        return (torch.randn((n, k), generator=g, device=device) * (gain * k ** -0.5)).to(torch.bfloat16)

    t = {"embed": torch.randn((cfg.vocab, d), generator=g, device=device).to(torch.bfloat16), "head": w(cfg.vocab, d)}

    def norm(name):
        t[name] = (1 + 0.2 * torch.randn(d, generator=g, device=device)).to(torch.bfloat16)
        t[name + ".b"] = (0.1 * torch.randn(d, generator=g, device=device)).to(torch.bfloat16)
        t[name + ".alpha"] = (0.4 + 0.4 * torch.rand((), generator=g, device=device)).to(torch.bfloat16)

    norm("final.norm")
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        norm(p + "norm1")
        t[p + "mix.q"], t[p + "mix.k"] = w(m.heads * m.dim, d, 1.5), w(m.kv_heads * m.dim, d, 1.5)
        t[p + "mix.v"], t[p + "mix.g"] = w(m.kv_heads * m.vdim, d), w(m.heads, d)
        t[p + "mix.o"] = w(d, m.heads * m.vdim)
        t[p + "mix.sink"] = torch.randn(m.heads, generator=g, device=device).to(torch.bfloat16)
        if layer.mlp is not None:
            norm(p + "norm2")
            t[p + "mlp.gate"], t[p + "mlp.up"] = w(layer.mlp.ff, d, 2.0), w(layer.mlp.ff, d, 2.0)
            t[p + "mlp.down"] = w(d, layer.mlp.ff)
    return t


def random_weights(cfg: LayeredConfig, rt: RuntimeConfig, device, seed: int = 0) -> dict:
    """Random weights made on the device, one layer's tensors at a time (benchmarks)."""
    class Lazy:
        def __getitem__(self, name):
            gen = torch.Generator(device=device).manual_seed(seed * 1000003 + sum((i + 1) * b for i, b in enumerate(name.encode())))
            part = name.split(".")
            d = cfg.d_model

            def w(n, k):
                return torch.randn((n, k), generator=gen, device=device, dtype=torch.bfloat16).mul_(k ** -0.5)
            if part[-1] == "alpha":
                return torch.tensor(0.5)
            if part[-1] in ("norm", "norm1", "norm2"):
                return torch.ones(d, device=device)
            if part[-1] == "b":
                return torch.zeros(d, device=device)
            if name in ("embed", "head"):
                return w(cfg.vocab, d).mul_(d ** 0.5 if name == "embed" else 1.0)
            layer = cfg.layers[int(part[0][1:])]
            m = layer.mixer
            if part[1] == "mix":
                return {"q": lambda: w(m.heads * m.dim, d), "k": lambda: w(m.kv_heads * m.dim, d), "v": lambda: w(m.kv_heads * m.vdim, d),
                        "g": lambda: w(m.heads, d), "o": lambda: w(d, m.heads * m.vdim),
                        "sink": lambda: torch.zeros(m.heads, device=device)}[part[2]]()
            return w(d, layer.mlp.ff) if part[2] == "down" else w(layer.mlp.ff, d)
    return place(cfg, rt, Lazy(), device)
