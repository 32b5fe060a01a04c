"""Plain PyTorch statement of the Rakelorn decoder, one function per mechanism, one sequence at a time, no cache.

Numerical oracle of the tests: everything is computed from scratch in one precision (``dtype``, float64 by default) from
the equations alone; nothing here is shared with the kernels or with the model code.  ``cfg`` is the parsed config.json,
``t`` the tensors of the checkpoint by name."""
from __future__ import annotations

import torch


def rms(x, eps):
    """x over its root mean square (eps inside the root)."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    """The whole row is scaled by one number."""
    return rms(x, eps) * gain


def token_shift(h, mix):
    """Row i moves the share ``mix`` (per coordinate) towards row i - 1; before the first row there are zeros."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return (1.0 - mix) * h + mix * prev


def rotate_pairs(x, positions, base: float, dims: int):
    """x [T, ..., >= dims]: pair (2i, 2i+1) of the first ``dims`` coordinates turns by position * base^(-2i/dims)."""
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=x.device)
    ang = positions.to(torch.float64)[:, None] * freq[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (dims // 2,)
    c, s = ang.cos().to(x.dtype).view(shape), ang.sin().to(x.dtype).view(shape)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = u * s + v * c
    return out


def causal_softmax(scores):
    """[H, T, T] -> weights over the keys that are not later than the query."""
    T = scores.shape[-1]
    later = torch.ones((T, T), dtype=torch.bool, device=scores.device).triu(1)
    return torch.softmax(scores.masked_fill(later, float("-inf")), -1)


def latent_attention(h, mix: dict, m: dict, eps: float):
    """Keys and values are linear maps of one normalised latent per token; one rotated key part is common to all heads."""
    T, H, n, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T, device=h.device)
    cq = rms(h @ mix["dq"].t(), eps) * mix["dq.norm"]
    q = (cq @ mix["uq"].t()).view(T, H, n + r)
    qn, qr = q[..., :n], rotate_pairs(q[..., n:], pos, m["rot"]["base"], m["rot"]["dims"])
    down = h @ mix["dkv"].t()
    c = rms(down[:, :rank], eps) * mix["dkv.norm"]
    kr = rotate_pairs(down[:, rank:], pos, m["rot"]["base"], m["rot"]["dims"])
    kn = (c @ mix["uk"].t()).view(T, H, n)
    v = (c @ mix["uv"].t()).view(T, H, dv)
    scores = (torch.einsum("ihd,jhd->hij", qn, kn) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", causal_softmax(scores), v)
    o = o * torch.sigmoid(h @ mix["g"].t())[:, :, None]
    return o.reshape(T, H * dv) @ mix["o"].t()


def mingru_candidate(u):
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def mingru_states(z, cand):
    """S_t = (1 - z_t) S_(t-1) + z_t cand_t, from zero, row by row."""
    s, out = torch.zeros_like(z[0]), []
    for zt, ct in zip(z, cand):
        s = (1 - zt) * s + zt * ct
        out.append(s)
    return torch.stack(out)


def mingru(h, mix: dict):
    z = torch.sigmoid(h @ mix["z"].t() + mix["z.b"])
    s = mingru_states(z, mingru_candidate(h @ mix["x"].t() + mix["x.b"]))
    g = h @ mix["g"].t()
    return (s * (g * torch.sigmoid(g))) @ mix["o"].t()


def route(logits, correction, router: dict):
    """-> (chosen [T, top], weights [T, top]).  The correction decides who is chosen, the weights do without it; only the
    best groups of neighbours (by their best member) are eligible."""
    s = torch.softmax(logits, -1)
    choice = s + correction
    groups = router.get("groups") or {"count": 1, "keep": 1}
    T, n, size = s.shape[0], groups["count"], s.shape[1] // groups["count"]
    best = choice.view(T, n, size).amax(-1)
    kept = torch.zeros((T, n), dtype=torch.bool, device=s.device).scatter_(1, best.topk(groups["keep"], -1).indices, True)
    eligible = kept.repeat_interleave(size, 1)
    chosen = choice.masked_fill(~eligible, float("-inf")).topk(router["top"], -1).indices
    return chosen, s.gather(1, chosen) * router["scale"]


def squared_relu_expert(h, up, down):
    return torch.relu(h @ up.t()).pow(2) @ down.t()


def mixture(h, mlp: dict, router: dict):
    """Weighted sum over each token's experts; the last ``identity`` of the router's outputs hand h through."""
    chosen, w = route(h @ mlp["router"].t(), mlp["correction"], router)
    out = torch.zeros_like(h)
    for e in range(router["experts"] + router.get("identity", 0)):
        share = (w * (chosen == e)).sum(-1, keepdim=True)
        rows = (chosen == e).any(-1)
        if rows.any():
            x = h[rows]
            y = squared_relu_expert(x, mlp[f"e{e}.up"], mlp[f"e{e}.down"]) if e < router["experts"] else x
            out[rows] += share[rows] * y
    return out


def schedule(cfg: dict):
    """[(layer, pass)] in running order; pass is None except on the first layer of a pass through the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for p in range(loop["times"]):
        order += [(i, p if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


MIX = {"latent_attention": ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "g", "o"),
       "mingru": ("z", "z.b", "x", "x.b", "g", "o")}


def forward(cfg: dict, t: dict, ids, dtype=torch.float64, collect: list | None = None):
    """ids int64 [T] -> logits [T, vocab]; ``collect`` receives the residual stream after every layer run."""
    t = {k: v.to(dtype) for k, v in t.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][ids] * cfg["embedding"]["scale"]
    for i, p in schedule(cfg):
        L, l = cfg["layers"][i], f"l{i}."
        if p is not None:
            x = x + t["loop.step"][p]
        h = token_shift(scalar_norm(x, t[l + "norm1"], eps), t[l + "shift"])
        mix = {n: t[l + "mix." + n] for n in MIX[L["type"]]}
        x = x + (latent_attention(h, mix, L["mixer"], eps) if L["type"] == "latent_attention" else mingru(h, mix))
        if L["mlp"] is not None:
            mlp = {k[len(l) + 4:]: v for k, v in t.items() if k.startswith(l + "mlp.")}
            x = x + mixture(scalar_norm(x, t[l + "norm2"], eps), mlp, L["mlp"]["router"])
        if collect is not None:
            collect.append(x)
    return scalar_norm(x, t["final.norm"], eps) @ t["head"].t()


def greedy(cfg: dict, t: dict, prompt, n_new: int, dtype=torch.float64):
    """Greedy continuation by full recomputation: (tokens, logits of each step)."""
    ids, toks, logs = prompt.clone(), [], []
    for _ in range(n_new):
        lg = forward(cfg, t, ids, dtype)[-1]
        toks.append(int(lg.argmax()))
        logs.append(lg)
        ids = torch.cat([ids, torch.tensor([toks[-1]], device=ids.device)])
    return toks, logs
