"""Configuration of decoders that are described layer by layer in a config.json (every layer has its own mixer, sizes and
feed-forward; a span of layers may run several times in a row).

The dataclasses name mechanisms with their constants: attention (rotary embedding with YaRN scaling, chunk mask, softmax
sink, output gate), latent attention, a gated linear recurrence, a bounded gated feed-forward, a mixture of experts, repeated
layers.  A ``Design`` says what all layers of an architecture have in common (norm, token shift, what joins the residual
stream before a pass through repeated layers).  ``from_dict`` reads a config.json, ``to_dict`` writes it."""
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


    kind = "attention"

    def cache(self, dtype: str) -> CacheSpec:
        return CacheSpec(self.kv_heads, self.dk, self.dv, dtype, self.chunk)

    def state(self) -> dict[str, int]:
        return {}

    def matrix_elements(self, d: int) -> int:
        return d * (self.heads * self.dim + self.kv_heads * (self.dim + self.vdim) + self.heads + self.heads * self.vdim)


@dataclass(frozen=True)
class LatentSpec:
    """Attention whose keys and values are linear maps of one latent per token; queries go through a latent of their own."""
    heads: int
    dim: int                      # unrotated query / key size per head
    rot_dim: int                  # rotated query size per head = size of the one rotated key part all heads share
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotary
    kind = "latent_attention"

    @property
    def dn(self) -> int:          # stored sizes: padded to 16-byte rows with zero dimensions
        return _pad8(self.dim)

    @property
    def dr(self) -> int:
        return _pad8(self.rot_dim)

    @property
    def dv(self) -> int:
        return _pad8(self.vdim)

    @property
    def rank(self) -> int:
        return _pad8(self.kv_rank)

    @property
    def qr(self) -> int:
        return _pad8(self.q_rank)

    def cache(self, dtype: str) -> CacheSpec:
        return CacheSpec(1, self.rank + self.dr, 0, dtype, None)

    def state(self) -> dict[str, int]:
        return {}

    def matrix_elements(self, d: int) -> int:
        return (d * (self.q_rank + self.kv_rank + self.rot_dim + self.heads) + self.q_rank * self.heads * (self.dim + self.rot_dim) +
                self.heads * (self.kv_rank * (self.dim + self.vdim) + self.vdim * d))


@dataclass(frozen=True)
class MinGRUSpec:
    """Gated linear recurrence; ``width`` channels of fp32 state per sequence."""
    width: int
    kind = "mingru"

    @property
    def channels(self) -> int:
        return _pad8(self.width)

    def cache(self, dtype: str) -> None:
        return None

    def state(self) -> dict[str, int]:
        return {"recurrent": self.channels}

    def matrix_elements(self, d: int) -> int:
        return 4 * d * self.width


@dataclass(frozen=True)
class GatedMLP:
    ff: int
    limit: float

    def matrix_elements(self, d: int) -> int:
        return 3 * d * self.ff


@dataclass(frozen=True)
class MoE:
    """Mixture of ungated experts.  The router has ``experts + identity`` outputs in ``groups`` equal groups of neighbours, of
    which the best ``keep`` are eligible; the last ``identity`` outputs hand the input through."""
    experts: int
    top: int
    ff: int
    scale: float = 1.0
    identity: int = 0
    groups: int = 1
    keep: int = 1

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def matrix_elements(self, d: int) -> int:
        return d * (self.outputs + 2 * self.experts * self.ff)


Mixer = AttentionSpec | LatentSpec | MinGRUSpec


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    mlp: GatedMLP | MoE | None


@dataclass(frozen=True)
class Design:
    """What the layers of an architecture share."""
    norm: str                     # "dynamic_tanh": element-wise; "scalar_rms": root mean square times one number
    token_shift: bool = False     # what a mixer reads leans on the token before
    pass_addend: str = "embedding"      # joins the stream "embedding": before every repeated pass; "step": a vector per pass


DESIGNS = {"Volonex": Design("dynamic_tanh"), "Rakelorn": Design("scalar_rms", token_shift=True, pass_addend="step")}


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
    step: int | None = None       # first layer of a pass: the number of the step vector that joins the stream before it


@dataclass(frozen=True)
class LayeredConfig:
    architecture: str
    vocab: int
    d_model: int
    layers: tuple[LayerSpec, ...]
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    eps: float = 1e-6             # of norms that compute statistics
    loop: Loop | None = None

    @property
    def name(self) -> str:
        return self.architecture.lower()

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def runs(self) -> list[LayerRun]:
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [LayerRun(i, False) for i in range(n)]
        step = self.design.pass_addend == "step"
        out = [LayerRun(i, False) for i in range(lp.start)]
        for t in range(lp.times):
            out += [LayerRun(i, not step and t > 0 and i == lp.start, t if step and i == lp.start else None)
                    for i in range(lp.start, lp.stop)]
        return out + [LayerRun(i, False) for i in range(lp.stop, n)]

    def cache_layout(self, rt: RuntimeConfig) -> list[CacheSpec | None]:
        """One entry per layer *run*; None where a run keeps nothing per token."""
        return [self.layers[r.layer].mixer.cache(rt.dtype) for r in self.runs]

    def state_layout(self) -> list[dict[str, int]]:
        """Per layer *run*: what it carries from token to token of a sequence, name -> fp32 numbers."""
        shift = {"shift": _pad8(self.d_model)} if self.design.token_shift else {}
        return [{**shift, **self.layers[r.layer].mixer.state()} for r in self.runs]

    @staticmethod
    def from_dict(c: dict) -> "LayeredConfig":
        if c["architecture"] not in DESIGNS:
            raise ValueError(f"unknown architecture {c['architecture']!r}")

        def rotary(rot: dict, limit: int) -> Rotary:
            sc = rot.get("scaling")
            r = Rotary(float(rot["base"]), int(rot["dims"]),
                       Yarn(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None)
            if r.dims % 2 or r.dims > limit:
                raise ValueError(f"{r.dims} rotated dimensions do not fit a vector of {limit}")
            return r

        def mixer(kind: str, m: dict) -> Mixer:
            if kind == "mingru":
                return MinGRUSpec(int(m["width"]))
            if kind == "latent_attention":
                return LatentSpec(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")), float(m["scale"]),
                                  rotary(m["rot"], int(m["rot_dim"])))
            if kind != "attention":
                raise ValueError(f"unknown mixer type {kind!r}")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{m['heads']} query heads over {m['kv_heads']} key/value heads")
            mask = m.get("mask")
            return AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                                 rotary(m["rot"], int(m["dim"])) if m.get("rot") else None, int(mask["size"]) if mask else None)

        def mlp(m: dict | None) -> GatedMLP | MoE | None:
            if m is None:
                return None
            kind = m.get("kind", "dense")
            if kind == "moe":
                r = m["router"]
                g = r.get("groups") or {"count": 1, "keep": 1}
                moe = MoE(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), float(r.get("scale", 1.0)), int(r.get("identity") or 0),
                          int(g["count"]), int(g["keep"]))
                if moe.outputs % moe.groups or not 0 < moe.keep <= moe.groups or not 0 < moe.top <= moe.keep * (moe.outputs // moe.groups):
                    raise ValueError(f"{moe.top} of {moe.outputs} outputs in {moe.keep} of {moe.groups} groups")
                return moe
            if kind != "dense":
                raise ValueError(f"unknown feed-forward kind {kind!r}")
            return GatedMLP(int(m["ff"]), float(m["limit"]))

        layers = tuple(LayerSpec(mixer(l.get("type", "attention"), l["mixer"]), mlp(l.get("mlp"))) for l in c["layers"])
        lp = c.get("loop")
        loop = Loop(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None
        if loop and not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return LayeredConfig(c["architecture"], int(c["vocab"]), int(c["width"]), layers, float(c["embedding"]["scale"]),
                             float(c.get("residual_mult", 1.0)), float(c.get("norm", {}).get("eps", 1e-6)), loop)

    def to_dict(self) -> dict:
        def rotary(r: Rotary) -> dict:
            d = {"base": r.base, "dims": r.dims}
            if r.scaling:
                s = r.scaling
                d["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
            return d

        def mixer(m: Mixer) -> dict:
            if isinstance(m, MinGRUSpec):
                return {"width": m.width}
            if isinstance(m, LatentSpec):
                return {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                        "scale": m.scale, "rot": rotary(m.rot)}
            d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.chunk:
                d["mask"] = {"size": m.chunk}
            if m.rot:
                d["rot"] = rotary(m.rot)
            return d

        def mlp(m: GatedMLP | MoE | None) -> dict | None:
            if isinstance(m, MoE):
                return {"kind": "moe", "expert": {"ff": m.ff},
                        "router": {"experts": m.experts, "identity": m.identity, "top": m.top, "scale": m.scale,
                                   "groups": {"count": m.groups, "keep": m.keep}}}
            return {"kind": "dense", "ff": m.ff, "limit": m.limit} if m else None
        c = {"architecture": self.architecture, "vocab": self.vocab, "width": self.d_model, "embedding": {"scale": self.embed_scale},
             "norm": {"eps": self.eps},
             "layers": [{"type": l.mixer.kind, "mixer": mixer(l.mixer), "mlp": mlp(l.mlp)} for l in self.layers]}
        if self.design.norm == "dynamic_tanh":
            c["residual_mult"] = self.residual_mult
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
        n = 2 * self.vocab * self.d_model
        for l in self.layers:
            n += l.mixer.matrix_elements(self.d_model) + (l.mlp.matrix_elements(self.d_model) if l.mlp else 0)
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


def rakelorn(width: int, n_layers: int, heads: int, vocab: int, *, dim: int = 128, rot_dim: int = 64, vdim: int = 128, q_rank: int = 1536,
             kv_rank: int = 512, recurrent: int | None = None, every: int = 3, moe: MoE | None = None, base: float = 1e6,
             embed_scale: float = 1.0, loop: Loop | None = None) -> LayeredConfig:
    """A Rakelorn whose every ``every``-th layer is recurrent (``recurrent`` channels, as wide as the stream by default) and whose
    other layers are latent attention."""
    a = LatentSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, (dim + rot_dim) ** -0.5, Rotary(base, rot_dim))
    r = MinGRUSpec(recurrent or width)
    layers = tuple(LayerSpec(r if (i + 1) % every == 0 else a, moe) for i in range(n_layers))
    return LayeredConfig("Rakelorn", vocab, width, layers, embed_scale, 1.0, 1e-6, loop)


def rakelorn_16b() -> LayeredConfig:
    """Many small experts of which a few are active, attention and recurrent layers two to one."""
    return rakelorn(2048, 27, 16, 102400, recurrent=3072, moe=MoE(64, 6, 2048, 2.0, 8, 8, 4))


def rakelorn_2b() -> LayeredConfig:
    return rakelorn(2048, 12, 16, 65536, dim=64, rot_dim=32, vdim=64, q_rank=512, kv_rank=256, moe=MoE(24, 4, 1024, 2.0, 4, 4, 2))


def tiny_rakelorn() -> LayeredConfig:
    """Miniature for smoke runs: uneven layers, one without feed-forward, the middle two run three times."""
    a = LatentSpec(6, 40, 16, 24, 72, 88, 0.13, Rotary(5000.0, 16))
    b = LatentSpec(3, 24, 32, 56, 96, 56, 0.16, Rotary(900.0, 32))
    layers = (LayerSpec(a, MoE(6, 3, 112, 1.3, 3, 3, 2)), LayerSpec(MinGRUSpec(200), None), LayerSpec(b, MoE(8, 2, 80, 0.8, 2, 5, 2)),
              LayerSpec(MinGRUSpec(168), MoE(5, 1, 96, 2.0)))
    return LayeredConfig("Rakelorn", 512, 192, layers, 0.7, 1.0, 1e-5, Loop(1, 3, 3))
