"""Plain PyTorch statement of the Volonex decoder, one function per mechanism, one sequence at a time, no cache.

Numerical oracle of the tests: everything is computed from scratch in one precision (``dtype``, float64 by default) from
the equations alone; nothing here is shared with the kernels or with the model code.  ``cfg`` is the parsed config.json,
``t`` the tensors of the checkpoint by name."""
from __future__ import annotations

import math

import torch


def dynamic_tanh(x, alpha, w, b):
    """Normalisation without statistics: a scaled tanh with an affine map."""
    return torch.tanh(alpha * x) * w + b


def yarn_frequencies(dims: int, base: float, scaling: dict | None):
    """Rotation frequency of each of the dims/2 pairs and the factor on cos and sin.

    Slow pairs (those that turn less than ``slow`` times within ``original`` positions) are interpolated by ``factor``,
    fast ones are kept, with a linear ramp over the pair index in between."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return torch.tensor(freq, dtype=torch.float64), 1.0

    def index_of(turns):      # the (fractional) pair index that makes this many turns
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_interleaved(x, positions, freq, mag):
    """x [T, heads, dim]: pairs (2i, 2i+1) of the first 2 * len(freq) dimensions turn by position * freq[i]."""
    n = freq.numel()
    ang = positions.to(torch.float64)[:, None] * freq[None, :].to(positions.device)
    c = (ang.cos() * mag).to(x.dtype)[:, None, :]
    s = (ang.sin() * mag).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


def chunk_mask(T: int, size: int | None, device="cpu"):
    """visible[i, j]: j is not after i and both lie in the same block of ``size`` positions."""
    i = torch.arange(T, device=device)
    vis = i[None, :] <= i[:, None]
    if size is not None:
        vis &= (i[None, :] // size) == (i[:, None] // size)
    return vis


def sink_softmax(scores, visible, sink):
    """scores [H, T, T] -> weights; exp(sink[h]) takes part in the denominator only."""
    s = scores.masked_fill(~visible[None], float("-inf"))
    m = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = (s - m).exp()
    return e / (e.sum(-1, keepdim=True) + (sink[:, None, None] - m).exp())


def attention(h, mix: dict, m: dict):
    """h [T, width] -> [T, width].  ``mix``: q, k, v, o, g, sink of the layer; ``m``: its sizes and constants."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ mix["q"].t()).view(T, H, d)
    k = (h @ mix["k"].t()).view(T, G, d)
    v = (h @ mix["v"].t()).view(T, G, dv)
    if m.get("rot"):
        pos = torch.arange(T, device=h.device)
        freq, mag = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_interleaved(q, pos, freq, mag), rotate_interleaved(k, pos, freq, mag)
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    size = m["mask"]["size"] if m.get("mask") else None
    w = sink_softmax(scores, chunk_mask(T, size, h.device), mix["sink"])
    o = torch.einsum("hij,jhd->ihd", w, v)
    gate = torch.sigmoid(h @ mix["g"].t())
    return (o * gate[:, :, None]).reshape(T, H * dv) @ mix["o"].t()


def clamped_glu(h, mlp: dict, limit: float):
    """Gated feed-forward whose gate is bounded above and whose other branch is bounded on both sides, then shifted."""
    g = (h @ mlp["gate"].t()).clamp(max=limit)
    u = (h @ mlp["up"].t()).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ mlp["down"].t()


def layer_schedule(cfg: dict):
    """[(layer index, first layer of a repeated pass?)] in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for p in range(times):
        order += [(i, p > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def forward(cfg: dict, t: dict, ids, dtype=torch.float64, collect: list | None = None):
    """ids int64 [T] -> logits [T, vocab]; ``collect`` receives the residual stream after every layer run."""
    t = {k: v.to(dtype) for k, v in t.items()}

    def norm(name, x):
        return dynamic_tanh(x, t[name + ".alpha"], t[name], t[name + ".b"])

    emb = t["embed"][ids] * cfg["embedding"]["scale"]
    x, mult = emb, cfg["residual_mult"]
    for i, again in layer_schedule(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + emb
        mix = {n: t[p + "mix." + n] for n in ("q", "k", "v", "o", "g", "sink")}
        x = x + mult * attention(norm(p + "norm1", x), mix, L["mixer"])
        if L["mlp"] is not None:
            mlp = {n: t[p + "mlp." + n] for n in ("gate", "up", "down")}
            x = x + mult * clamped_glu(norm(p + "norm2", x), mlp, L["mlp"]["limit"])
        if collect is not None:
            collect.append(x)
    return norm("final.norm", x) @ t["head"].t()


def greedy(cfg: dict, t: dict, prompt, n_new: int, dtype=torch.float64):
    """Greedy continuation by full recomputation: (tokens, logits of each step)."""
    ids, toks, logs = prompt.clone(), [], []
    for _ in range(n_new):
        lg = forward(cfg, t, ids, dtype)[-1]
        toks.append(int(lg.argmax()))
        logs.append(lg)
        ids = torch.cat([ids, torch.tensor([toks[-1]], device=ids.device)])
    return toks, logs
