"""Configuration of decoders that are described layer by layer in a config.json (every layer has its own mixer, sizes and
feed-forward; a span of layers may run several times in a row).

The dataclasses name mechanisms with their constants (rotary embedding with YaRN scaling, chunk mask, softmax sink, output
gate, bounded gated feed-forward, repeated layers); ``Volonex`` is the design that combines them.  ``from_dict`` reads its
config.json, ``to_dict`` writes it."""
from __future__ import annotations

import json
from dataclasses import dataclass

from .config import CacheSpec, RuntimeConfig


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class Yarn:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotary:
    base: float
    dims: int                     # leading dimensions of a head that turn; pairs are neighbours (2i, 2i + 1)
    scaling: Yarn | None = None


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                      # query / key size per head
    vdim: int                     # value size per head
    scale: float
    rot: Rotary | None = None
    chunk: int | None = None      # a position sees only its own block of this many positions

    @property
    def dk(self) -> int:          # stored sizes: padded to 16-byte rows with zero dimensions
        return _pad8(self.dim)

    @property
    def dv(self) -> int:
        return _pad8(self.vdim)


@dataclass(frozen=True)
class GatedMLP:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    mlp: GatedMLP | None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: its cache is its own, its weights are the layer's."""
    layer: int
    add_embedding: bool           # first layer of a repeated pass: the embedding rows join the residual stream before it


@dataclass(frozen=True)
class LayeredConfig:
    architecture: str
    vocab: int
    d_model: int
    layers: tuple[LayerSpec, ...]
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    eps: float = 1e-6             # of norms that compute statistics (none in this design)
    loop: Loop | None = None

    @property
    def name(self) -> str:
        return self.architecture.lower()

    @property
    def runs(self) -> list[LayerRun]:
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [LayerRun(i, False) for i in range(n)]
        out = [LayerRun(i, False) for i in range(lp.start)]
        for t in range(lp.times):
            out += [LayerRun(i, t > 0 and i == lp.start) for i in range(lp.start, lp.stop)]
        return out + [LayerRun(i, False) for i in range(lp.stop, n)]

    def cache_layout(self, rt: RuntimeConfig) -> list[CacheSpec]:
        """One entry per layer *run*."""
        return [CacheSpec(m.kv_heads, m.dk, m.dv, rt.dtype, m.chunk) for m in (self.layers[r.layer].mixer for r in self.runs)]

    @staticmethod
    def from_dict(c: dict) -> "LayeredConfig":
        def mixer(kind: str, m: dict) -> AttentionSpec:
            if kind != "attention":
                raise ValueError(f"unknown mixer type {kind!r}")
            rot = m.get("rot")
            if rot is not None:
                sc = rot.get("scaling")
                rot = Rotary(float(rot["base"]), int(rot["dims"]),
                             Yarn(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None)
                if rot.dims % 2 or rot.dims > m["dim"]:
                    raise ValueError(f"{rot.dims} rotated dimensions do not fit a head of {m['dim']}")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{m['heads']} query heads over {m['kv_heads']} key/value heads")
            mask = m.get("mask")
            return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), rot,
                                 int(mask["size"]) if mask else None)

        def mlp(m: dict | None) -> GatedMLP | None:
            if m is None:
                return None
            if m.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
            return GatedMLP(int(m["ff"]), float(m["limit"]))

        layers = tuple(LayerSpec(mixer(l.get("type", "attention"), l["mixer"]), mlp(l.get("mlp"))) for l in c["layers"])
        lp = c.get("loop")
        loop = Loop(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return LayeredConfig(c["architecture"], int(c["vocab"]), int(c["width"]), layers, float(c["embedding"]["scale"]),
                             float(c["residual_mult"]), float(c.get("norm", {}).get("eps", 1e-6)), loop)

    def to_dict(self) -> dict:
        def mixer(m: AttentionSpec) -> dict:
            d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.chunk:
                d["mask"] = {"size": m.chunk}
            if m.rot:
                d["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.scaling:
                    s = m.rot.scaling
                    d["rot"]["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
            return d
        c = {"architecture": self.architecture, "vocab": self.vocab, "width": self.d_model, "embedding": {"scale": self.embed_scale},
             "residual_mult": self.residual_mult, "norm": {"eps": self.eps},
             "layers": [{"type": "attention", "mixer": mixer(l.mixer),
                         "mlp": {"kind": "dense", "ff": l.mlp.ff, "limit": l.mlp.limit} if l.mlp else None} for l in self.layers]}
        if self.loop:
            c["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return c

    def to_json(self) -> str:
        return json.dumps(self.to_dict())

    @staticmethod
    def from_json(text: str) -> "LayeredConfig":
        return LayeredConfig.from_dict(json.loads(text))

    def weight_bytes(self, elem: int = 2) -> int:
        """Bytes of the matrices (each layer once, however often it runs)."""
        d = self.d_model
        n = 2 * self.vocab * d
        for l in self.layers:
            m = l.mixer
            n += d * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim) + m.heads + m.heads * m.vdim)
            n += 3 * d * l.mlp.ff if l.mlp else 0
        return n * elem


def volonex(width: int, n_layers: int, heads: int, kv_heads: int, ff: int, vocab: int, *, dim: int = 128, vdim: int = 128,
            chunk: int = 8192, rot_dims: int = 64, base: float = 500000.0, scaling: Yarn | None = Yarn(8.0, 8192.0, 32.0, 1.0),
            limit: float = 7.0, scale: float | None = None, residual_mult: float = 1.0, embed_scale: float = 1.0,
            loop: Loop | None = None) -> LayeredConfig:
    """A Volonex whose layers are all alike."""
    m = AttentionSpec(heads, kv_heads, dim, vdim, scale if scale is not None else dim ** -0.5, Rotary(base, rot_dims, scaling), chunk)
    return LayeredConfig("Volonex", vocab, width, (LayerSpec(m, GatedMLP(ff, limit)),) * n_layers, embed_scale, residual_mult, 1e-6, loop)


def volonex_8b() -> LayeredConfig:
    """Layers as wide as the 8B Llama shape."""
    return volonex(4096, 32, 32, 8, 14336, 128256)


def volonex_1b() -> LayeredConfig:
    return volonex(2048, 16, 32, 8, 8192, 128256, dim=64, vdim=64, rot_dims=32)


def tiny_volonex() -> LayeredConfig:
    """Miniature for smoke runs: uneven layers, one without feed-forward, two of them run twice."""
    a = AttentionSpec(4, 2, 64, 48, 0.11, Rotary(10000.0, 24, Yarn(2.0, 64.0, 16.0, 1.0)), 40)
    b = AttentionSpec(6, 1, 40, 64, 0.2, Rotary(1000.0, 40, Yarn(4.0, 128.0, 8.0, 2.0)), 24)
    layers = (LayerSpec(a, GatedMLP(320, 3.0)), LayerSpec(b, None), LayerSpec(a, GatedMLP(200, 1.5)))
    return LayeredConfig("Volonex", 500, 256, layers, 4.0, 0.7, 1e-6, Loop(1, 3, 2))
