"""Weights of layer-by-layer decoders: checkpoint folder (config.json + model.safetensors) -> the layouts the kernels read.

Tensor names: ``embed``, ``head``, ``final.norm``; per layer ``l<i>.norm1``, ``l<i>.norm2``, the mixer's ``l<i>.mix.*`` (attention
q, k, v, g, o, sink; latent attention dq, uq, dkv, uk, uv, g, o and the gains dq.norm, dkv.norm; minGRU z, x, g, o and the biases
z.b, x.b) and the feed-forward's ``l<i>.mlp.*`` (gate, up, down; a mixture router, correction, e<j>.up, e<j>.down).  A dynamic-tanh
norm ``x`` also has ``x.alpha`` and ``x.b``; a scalar norm is one number.  Designs with a token shift have ``l<i>.shift``, those
with a step vector per pass ``loop.step``.  Matrices are [out, in].

On the device matrices that read the same rows are one matrix (rows of a head padded to a multiple of eight with zeros, the
columns of the output projection likewise), gate and up are interleaved row by row, experts are stacked, norms, gains, biases
and sinks are fp32.  The latent's key map is kept both ways round: per head transposed (queries into the latent space) and, with
the value map, as it is (latents into keys and values)."""
from __future__ import annotations

import json
import os

import torch

from ..ops.dense import DenseW, DynamicTanh, GroupedW, padded
from .config import RuntimeConfig
from .layered_config import AttentionSpec, GatedMLP, LatentSpec, LayeredConfig, MinGRUSpec, MoE

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


def _pad_rows(w: torch.Tensor, to: int) -> torch.Tensor:
    return _pad_head_rows(w, 1, w.shape[0], to)


def _o_matrix(o: torch.Tensor, heads: int, size: int, to: int) -> torch.Tensor:
    """[d, heads * size] -> [d, heads * to] with zero columns after each head."""
    return _pad_head_rows(o.t().contiguous(), heads, size, to).t()


class _Placer:
    """Checkpoint tensors (checked against the configuration) -> device weights."""

    def __init__(self, cfg: LayeredConfig, rt: RuntimeConfig, t, device):
        self.cfg, self.dt, self.t, self.device, self.d = cfg, _DTYPES[rt.dtype], t, device, cfg.d_model

    def get(self, name, *shape) -> torch.Tensor:
        return _expect(self.t[name], shape, name)

    def dense(self, w) -> DenseW:
        return DenseW.of(w, self.dt, self.device)

    def vector(self, v, to: int | None = None) -> torch.Tensor:
        out = torch.zeros(to or padded(v.numel()), dtype=torch.float32, device=self.device)
        out[:v.numel()] = v.to(device=self.device, dtype=torch.float32)
        return out

    def norm(self, name):
        if self.cfg.design.norm == "scalar_rms":
            return float(self.get(name).float())
        return DynamicTanh.of(float(self.get(name + ".alpha").float()), self.get(name, self.d), self.get(name + ".b", self.d), self.device)

    def attention(self, x: str, m: AttentionSpec) -> dict:
        get, d = self.get, self.d
        return {"qkvg": self.dense(qkvg_matrix(get(x + "q", m.heads * m.dim, d), get(x + "k", m.kv_heads * m.dim, d),
                                               get(x + "v", m.kv_heads * m.vdim, d), get(x + "g", m.heads, d), m)),
                "sink": self.vector(get(x + "sink", m.heads), m.heads),
                "o": self.dense(_o_matrix(get(x + "o", d, m.heads * m.vdim), m.heads, m.vdim, m.dv))}

    def latent(self, x: str, m: LatentSpec) -> dict:
        get, d, H = self.get, self.d, m.heads
        dkv = get(x + "dkv", m.kv_rank + m.rot_dim, d)
        uq = get(x + "uq", H * (m.dim + m.rot_dim), m.q_rank).view(H, m.dim + m.rot_dim, m.q_rank)
        uk, uv = get(x + "uk", H * m.dim, m.kv_rank), get(x + "uv", H * m.vdim, m.kv_rank)
        head = torch.cat([_pad_head_rows(uq[:, :m.dim].reshape(-1, m.q_rank), H, m.dim, m.dn).view(H, m.dn, -1),
                          _pad_head_rows(uq[:, m.dim:].reshape(-1, m.q_rank), H, m.rot_dim, m.dr).view(H, m.dr, -1)], 1)
        ukv = self.dense(torch.cat([_pad_head_rows(uk, H, m.dim, m.dn), _pad_head_rows(uv, H, m.vdim, m.dv)]))
        return {"down": self.dense(torch.cat([_pad_rows(get(x + "dq", m.q_rank, d), m.qr), _pad_rows(dkv[:m.kv_rank], m.rank),
                                              _pad_rows(dkv[m.kv_rank:], m.dr), get(x + "g", H, d)])),
                "q_gain": self.vector(get(x + "dq.norm", m.q_rank)), "c_gain": self.vector(get(x + "dkv.norm", m.kv_rank)),
                "uq": self.dense(head.reshape(H * (m.dn + m.dr), m.q_rank)), "ukv": ukv,
                "uk": GroupedW.of((w.t() for w in uk.view(H, m.dim, m.kv_rank)), H, self.dt, self.device, n=m.rank),
                "uv": GroupedW(ukv.data[H * m.dn:], H, m.dv, m.kv_rank),
                "o": self.dense(_o_matrix(get(x + "o", d, H * m.vdim), H, m.vdim, m.dv))}

    def mingru(self, x: str, m: MinGRUSpec) -> dict:
        get, d, c = self.get, self.d, m.channels
        return {"zxg": self.dense(torch.cat([_pad_rows(get(x + n, m.width, d), c) for n in "zxg"])),
                "zb": self.vector(get(x + "z.b", m.width), c), "xb": self.vector(get(x + "x.b", m.width), c),
                "o": self.dense(get(x + "o", d, m.width))}

    def gated(self, x: str, m: GatedMLP) -> dict:
        gate, up = self.get(x + "gate", m.ff, self.d), self.get(x + "up", m.ff, self.d)
        return {"gate_up": self.dense(torch.stack([gate, up], 1).reshape(2 * m.ff, self.d)),
                "down_proj": self.dense(self.get(x + "down", self.d, m.ff))}

    def mixture(self, x: str, m: MoE) -> dict:
        get, d = self.get, self.d
        return {"router": self.dense(get(x + "router", m.outputs, d)), "correction": self.vector(get(x + "correction", m.outputs)),
                "experts_up": GroupedW.of((get(f"{x}e{e}.up", m.ff, d) for e in range(m.experts)), m.experts, self.dt, self.device, n=padded(m.ff)),
                "experts_down": GroupedW.of((get(f"{x}e{e}.down", d, m.ff) for e in range(m.experts)), m.experts, self.dt, self.device, n=padded(d))}


def place(cfg: LayeredConfig, rt: RuntimeConfig, t, device) -> dict:
    """``t[name]``: checkpoint tensors (a dict or an open file) -> device weights."""
    p, d = _Placer(cfg, rt, t, device), cfg.d_model
    w = {"embed": p.dense(p.get("embed", cfg.vocab, d)).data, "head": p.dense(p.get("head", cfg.vocab, d)), "final_norm": p.norm("final.norm"),
         "vocab_offset": 0, "layers": []}
    if cfg.loop and cfg.design.pass_addend == "step":
        w["step"] = [p.vector(v) for v in p.get("loop.step", cfg.loop.times, d)]
    for i, layer in enumerate(cfg.layers):
        l = f"l{i}."
        place_mixer = {AttentionSpec: p.attention, LatentSpec: p.latent, MinGRUSpec: p.mingru}[type(layer.mixer)]
        L = {"norm1": p.norm(l + "norm1"), **place_mixer(l + "mix.", layer.mixer)}
        if cfg.design.token_shift:
            L["shift"] = p.vector(p.get(l + "shift", d))
        if layer.mlp is not None:
            L["norm2"] = p.norm(l + "norm2")
            L.update({GatedMLP: p.gated, MoE: p.mixture}[type(layer.mlp)](l + "mlp.", layer.mlp))
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


def tensor_shapes(cfg: LayeredConfig) -> dict[str, tuple[str, tuple]]:
    """Every tensor of a checkpoint: name -> (role, shape).  Roles: matrix, gain, alpha, bias, sink, shift, step, correction."""
    d = cfg.d_model
    out = {"embed": ("matrix", (cfg.vocab, d)), "head": ("matrix", (cfg.vocab, d))}

    def norm(name):
        if cfg.design.norm == "scalar_rms":
            out[name] = ("gain", ())
        else:
            out.update({name: ("gain", (d,)), name + ".b": ("bias", (d,)), name + ".alpha": ("alpha", ())})

    norm("final.norm")
    if cfg.loop and cfg.design.pass_addend == "step":
        out["loop.step"] = ("step", (cfg.loop.times, d))
    for i, layer in enumerate(cfg.layers):
        m, f, l = layer.mixer, layer.mlp, f"l{i}."
        norm(l + "norm1")
        if cfg.design.token_shift:
            out[l + "shift"] = ("shift", (d,))
        if isinstance(m, AttentionSpec):
            mix = {"q": (m.heads * m.dim, d), "k": (m.kv_heads * m.dim, d), "v": (m.kv_heads * m.vdim, d), "g": (m.heads, d),
                   "o": (d, m.heads * m.vdim)}
            out[l + "mix.sink"] = ("sink", (m.heads,))
        elif isinstance(m, LatentSpec):
            mix = {"dq": (m.q_rank, d), "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank), "dkv": (m.kv_rank + m.rot_dim, d),
                   "uk": (m.heads * m.dim, m.kv_rank), "uv": (m.heads * m.vdim, m.kv_rank), "g": (m.heads, d), "o": (d, m.heads * m.vdim)}
            out.update({l + "mix.dq.norm": ("gain", (m.q_rank,)), l + "mix.dkv.norm": ("gain", (m.kv_rank,))})
        else:
            mix = {**{n: (m.width, d) for n in "zxg"}, "o": (d, m.width)}
            out.update({l + "mix.z.b": ("bias", (m.width,)), l + "mix.x.b": ("bias", (m.width,))})
        out.update({l + "mix." + n: ("matrix", s) for n, s in mix.items()})
        if f is None:
            continue
        norm(l + "norm2")
        if isinstance(f, GatedMLP):
            ff = {"gate": (f.ff, d), "up": (f.ff, d), "down": (d, f.ff)}
        else:
            ff = {"router": (f.outputs, d)}
            for e in range(f.experts):
                ff.update({f"e{e}.up": (f.ff, d), f"e{e}.down": (d, f.ff)})
            out[l + "mlp.correction"] = ("correction", (f.outputs,))
        out.update({l + "mlp." + n: ("matrix", s) for n, s in ff.items()})
    return out


# matrices that come out of init_master larger than 1 / sqrt(columns), so that scores, gates and choices differ clearly
_INIT_GAIN = {"q": 1.5, "k": 1.5, "uq": 1.5, "uk": 1.5, "gate": 2.0, "up": 2.0, "router": 3.0}


def init_master(cfg: LayeredConfig, seed: int = 0, device="cpu") -> dict:
    """Random bf16 checkpoint tensors by name (tests, smoke runs)."""
    g = torch.Generator(device=device).manual_seed(seed)

    def make(name: str, role: str, shape: tuple) -> torch.Tensor:
        n = torch.randn(shape, generator=g, device=device)
        if role == "matrix":
            return n if name == "embed" else n * (_INIT_GAIN.get(name.split(".")[-1], 1.0) * shape[1] ** -0.5)
        if role == "alpha":
            return 0.4 + 0.4 * torch.rand(shape, generator=g, device=device)
        if role == "shift":
            return torch.rand(shape, generator=g, device=device)
        return {"gain": 1 + 0.2 * n, "bias": 0.1 * n if cfg.design.norm == "dynamic_tanh" else n, "sink": n, "step": n,
                "correction": 0.1 * n}[role]
    return {name: make(name, *rs).to(torch.bfloat16) for name, rs in tensor_shapes(cfg).items()}


def random_weights(cfg: LayeredConfig, rt: RuntimeConfig, device, seed: int = 0) -> dict:
    """Random weights made on the device, one layer's tensors at a time (benchmarks)."""
    shapes = tensor_shapes(cfg)

    class Lazy:
        def __getitem__(self, name):
            gen = torch.Generator(device=device).manual_seed(seed * 1000003 + sum((i + 1) * b for i, b in enumerate(name.encode())))
            role, shape = shapes[name]
            if role == "matrix":
                w = torch.randn(shape, generator=gen, device=device, dtype=torch.bfloat16).mul_(shape[1] ** -0.5)
                return w.mul_(shape[1] ** 0.5) if name == "embed" else w
            fixed = {"alpha": 0.5, "gain": 1.0, "shift": 0.5}.get(role, 0.0)
            return torch.full(shape, fixed, device=device)
    return place(cfg, rt, Lazy(), device)
