"""Volonex on the GPU: every mechanism of the kernels alone and the model through the engine, against the plain oracle.

Comparisons of whole models use the root mean square over a row of logits relative to that of the logits: the 32-bit form
must agree to a few 1e-6, the bf16 form to what rounding the activations costs."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from mojo_linuxperiments_b200.models import layered_config as LC
from mojo_linuxperiments_b200.models import layered_weights as LW
from mojo_linuxperiments_b200.models.config import RuntimeConfig
from mojo_linuxperiments_b200.oracle import volonex as V

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 4e-2}
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rel(got, want):
    """largest row error: rms(got - want) / rms(want)"""
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-12)).max().item()


# ---------------------------------------------------------------------------------------------------------
# linears with their epilogues
# ---------------------------------------------------------------------------------------------------------
SHAPES = [(1, 40, 24), (3, 200, 136), (16, 130, 1000), (17, 384, 640), (33, 96, 520), (64, 1000, 77), (65, 72, 200), (128, 256, 512),
          (300, 515, 333), (777, 1100, 264)]


def _operands(M, N, K, dtype, seed=0):
    from mojo_linuxperiments_b200.ops import dense as D
    g = torch.Generator(device=DEV).manual_seed(seed)
    x = D.rows(M, K, DT[dtype], DEV)
    x.fill_(float("nan"))                                    # the padding must not matter
    x[:, :K] = torch.randn((M, K), generator=g, device=DEV)
    w = (torch.randn((N, K), generator=g, device=DEV) * K ** -0.5).to(torch.bfloat16)
    return x, x[:, :K].double(), D.DenseW.of(w, DT[dtype], DEV), w.double(), g


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear(M, N, K, dtype):
    from mojo_linuxperiments_b200.ops import dense as D
    x, xd, w, wd, _ = _operands(M, N, K, dtype)
    y = D.linear(x, w, out_dtype=torch.float32)[:, :N]
    assert rel(y, xd @ wd.t()) < 2e-6
    if dtype == "bfloat16":
        assert rel(D.linear(x, w)[:, :N].float(), xd @ wd.t()) < 4e-3
        for force in ((1, 2, 3, 4, 5, 6, 7, 8) if M <= 64 else (64, 128, 256)):
            assert rel(D.linear(x, w, out_dtype=torch.float32, force=force)[:, :N], xd @ wd.t()) < 2e-6, force


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear_glu(M, N, K, dtype):
    from mojo_linuxperiments_b200.ops import dense as D
    N -= N % 2
    x, xd, w, wd, _ = _operands(M, N, K, dtype, 1)
    for limit in (0.4, 7.0):
        y = D.linear_glu(x, w, limit)[:, :N // 2]
        eye = torch.eye(N // 2, dtype=torch.float64, device=DEV)
        want = V.clamped_glu(xd, {"gate": wd[0::2], "up": wd[1::2], "down": eye}, limit)
        assert rel(y, want) < (3e-6 if dtype == "float32" else 4e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear_residual_with_norm_and_second_addend(M, N, K, dtype):
    from mojo_linuxperiments_b200.ops import dense as D
    x, xd, w, wd, g = _operands(M, N, K, dtype, 2)
    base, emb = D.rows(M, N, torch.float32, DEV), D.rows(M, N, torch.float32, DEV)
    base.normal_(generator=g), emb.normal_(generator=g)
    nw, nb = torch.randn(N, generator=g, device=DEV), torch.randn(N, generator=g, device=DEV)
    norm = D.DynamicTanh.of(0.8, nw, nb, DEV)
    for add in (None, emb):
        for mult in (1.0, 0.37):
            s, h = base.clone(), D.rows(M, N, DT[dtype], DEV)
            D.linear_residual(x, w, s, mult, norm, h, add=add)
            want = base[:, :N].double() + mult * (xd @ wd.t()) + (add[:, :N].double() if add is not None else 0)
            assert rel(s[:, :N], want) < 2e-6
            hn = V.dynamic_tanh(want, 0.8, nw.double(), nb.double())
            assert rel(h[:, :N], hn) < (2e-6 if dtype == "float32" else 4e-3)
    s = base.clone()
    D.linear_residual(x, w, s, 1.0, None, None)
    assert rel(s[:, :N], base[:, :N].double() + xd @ wd.t()) < 2e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_rows_scale_copy_and_norm(dtype):
    from mojo_linuxperiments_b200.ops import dense as D
    g = torch.Generator(device=DEV).manual_seed(3)
    V_, d = 37, 150
    table = D.DenseW.of(torch.randn((V_, d), generator=g, device=DEV).to(torch.bfloat16), DT[dtype], DEV)
    nw, nb = torch.randn(d, generator=g, device=DEV), torch.randn(d, generator=g, device=DEV)
    ids = torch.tensor([0, 36, 5, 5], device=DEV)
    x, c, h = D.rows(4, d, torch.float32, DEV), D.rows(4, d, torch.float32, DEV), D.rows(4, d, DT[dtype], DEV)
    D.embed_norm(ids, table.data, d, 3.25, x, c, D.DynamicTanh.of(-0.6, nw, nb, DEV), h)
    want = table.data[ids, :d].double() * 3.25
    assert rel(x[:, :d], want) < 1e-6 and torch.equal(x[:, :d], c[:, :d])
    assert rel(h[:, :d], V.dynamic_tanh(want, -0.6, nw.double(), nb.double())) < (2e-6 if dtype == "float32" else 4e-3)


# ---------------------------------------------------------------------------------------------------------
# rotary embedding and attention over the paged cache
# ---------------------------------------------------------------------------------------------------------
class Paged:
    """Sequences of given lengths whose raw q, k, v (and gate) are random; a cache with shuffled pages."""

    def __init__(self, lens, H, G, dk, dv, dtype, *, pairs=0, mag=1.0, seed=0, chunk=None, sink=True, gate=True, scale=None, cap=None):
        from mojo_linuxperiments_b200.ops import attention as A
        self.A, self.lens, self.H, self.G, self.dk, self.dv, self.chunk = A, lens, H, G, dk, dv, chunk
        g = torch.Generator(device=DEV).manual_seed(seed)
        self.width = H * dk + G * (dk + dv) + H
        self.pitch = (self.width + 7) // 8 * 8
        self.raw = [torch.randn((n, self.pitch), generator=g, device=DEV).to(DT[dtype]) for n in lens]
        self.cap = cap or max(lens) + 40
        mp = (self.cap + 15) // 16
        self.cache = A.PagedKVCache(len(lens) * mp + 1, G, 16, DEV, dk=dk, dv=dv, dtype=DT[dtype])
        self.cache.data.normal_(generator=g)                                    # stale contents of reused pages
        perm = torch.randperm(len(lens) * mp, generator=torch.Generator().manual_seed(seed))
        self.table = perm.to(torch.int32).view(len(lens), mp).to(DEV)
        self.cos, self.sin = A.rope_tables(self.cap, 300.0, DEV, 2 * pairs) if pairs else (None, None)
        if pairs:
            self.cos, self.sin = self.cos * mag, self.sin * mag
        self.pairs, self.mag = pairs, mag
        self.sink = torch.randn(H, generator=g, device=DEV) if sink else None
        self.gate = gate
        self.scale = scale if scale is not None else dk ** -0.5
        self.dtype = DT[dtype]

    def spec(self, rows):
        at = self.H * self.dk + self.G * (self.dk + self.dv)
        return self.A.attn_spec(self.scale, chunk=self.chunk, sink=self.sink, gate=rows[:, at:at + self.H] if self.gate else None)

    def parts(self, b):
        """fp64 q, k (rotated), v, gate logits of sequence b"""
        H, G, dk, dv = self.H, self.G, self.dk, self.dv
        r = self.raw[b].double()
        q, k, v, gt = r[:, :self.width].split([H * dk, G * dk, G * dv, H], 1)
        q, k = q.reshape(-1, H, dk), k.reshape(-1, G, dk)
        if self.pairs:
            f = 300.0 ** (-torch.arange(0, 2 * self.pairs, 2, dtype=torch.float64) / (2 * self.pairs))
            pos = torch.arange(r.shape[0], device=DEV)
            q, k = V.rotate_interleaved(q, pos, f.to(DEV), self.mag), V.rotate_interleaved(k, pos, f.to(DEV), self.mag)
        return q, k, v.reshape(-1, G, dv), gt

    def want(self, b):
        q, k, v, gt = self.parts(b)
        n = q.shape[0]
        k, v = k.repeat_interleave(self.H // self.G, 1), v.repeat_interleave(self.H // self.G, 1)
        s = torch.einsum("ihd,jhd->hij", q, k) * self.scale
        vis = V.chunk_mask(n, self.chunk, DEV)
        sink = self.sink.double() if self.sink is not None else torch.full((self.H,), -1e30, device=DEV, dtype=torch.float64)
        o = torch.einsum("hij,jhd->ihd", V.sink_softmax(s, vis, sink), v)
        if self.gate:
            o = o * torch.sigmoid(gt)[:, :, None]
        return o.reshape(n, -1)

    def portion(self, spans):
        """{sequence: (first, count)}: rotary + cache append + prefill attention of these tokens, one call"""
        bs = list(spans)
        rows = torch.cat([self.raw[b][a:a + n] for b, (a, n) in spans.items()]).clone()
        pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for a, n in spans.values()]).to(DEV)
        sid = torch.cat([torch.full((n,), b, dtype=torch.int32) for b, (a, n) in spans.items()]).to(DEV)
        cu = torch.tensor([0] + [n for _, n in spans.values()]).cumsum(0).to(torch.int32).to(DEV)
        self.A.rotary_paged(rows, self.H, pos, sid, self.cos, self.sin, self.cache, self.table)
        out = torch.full((rows.shape[0], self.H * self.dv), float("nan"), dtype=self.dtype, device=DEV)
        self.A.attn_prefill_paged(rows, self.H, pos, sid, cu, max(n for _, n in spans.values()), self.cache, self.table, self.spec(rows), out)
        return dict(zip(bs, out.split([n for _, n in spans.values()])))

    def decode(self, at, splits=None, live=None):
        """one new token at position at[b] of every sequence"""
        rows = torch.stack([self.raw[b][p] for b, p in enumerate(at)])
        pos = torch.tensor(at, dtype=torch.int32, device=DEV)
        lens = torch.tensor([p + 1 if live is None or live[b] else 0 for b, p in enumerate(at)], dtype=torch.int32, device=DEV)
        out = torch.full((len(at), self.H * self.dv), float("nan"), dtype=self.dtype, device=DEV)
        kw = {} if splits is None else {"splits": splits}
        self.A.attn_decode_paged(rows, self.H, pos, lens, self.cos, self.sin, self.cache, self.table, self.spec(rows), out, **kw)
        return out

    def ok(self):
        from mojo_linuxperiments_b200.ops.workspace import default_workspace
        default_workspace(torch.device(DEV)).check_status()


ATOL = {torch.float32: 1e-5, torch.bfloat16: 2.5e-2}
HEADS = [(4, 2, 64, 48, 12), (6, 1, 40, 64, 20), (4, 4, 128, 128, 64), (3, 3, 24, 96, 0), (8, 2, 104, 16, 8), (20, 1, 16, 24, 8), (2, 1, 200, 136, 50)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dk,dv,pairs", HEADS)
def test_whole_prompts_and_decoding_of_many_head_shapes(H, G, dk, dv, pairs, dtype):
    for chunk, sink, gate in ((None, True, True), (50, True, False), (37, False, True), (16, True, True), (300, False, False)):
        P = Paged([1, 130, 300, 77], H, G, dk, dv, dtype, pairs=pairs, mag=1.2 if pairs else 1.0, chunk=chunk, sink=sink, gate=gate)
        got = P.portion({b: (0, n) for b, n in enumerate(P.lens)})
        last = [n - 1 for n in P.lens]
        dec = P.decode(last)                            # the last token once more, as a decoding step
        P.ok()
        for b in range(4):
            want = P.want(b)
            assert (got[b].double() - want).abs().max().item() < ATOL[P.dtype], (chunk, b)
            assert (dec[b].double() - want[-1]).abs().max().item() < ATOL[P.dtype], (chunk, b)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rotary_writes_the_cache_where_the_page_table_says(dtype):
    P = Paged([90, 33], 4, 2, 64, 48, dtype, pairs=12, mag=0.9)
    before = P.cache.data.clone()
    P.portion({0: (0, 90), 1: (0, 33)})
    P.ok()
    for b, n in enumerate(P.lens):
        _, k, v, _ = P.parts(b)
        for p in (0, 15, 16, 31, 32, n - 1):
            page = int(P.table[b, p // 16])
            assert (P.cache.keys()[page, :, p % 16].double() - k[p]).abs().max() < (1e-5 if dtype == "float32" else 3e-2)
            assert torch.equal(P.cache.values()[page, :, p % 16].double(), v[p])
    # nothing beyond the last token of a sequence was touched
    page, tail = int(P.table[1, 2]), slice(33 % 16, 16)
    ref = type(P.cache)(P.cache.num_pages, 2, 16, DEV, storage=before, dk=64, dv=48)
    assert torch.equal(P.cache.keys()[page][:, tail], ref.keys()[page][:, tail])


@pytest.mark.parametrize("halves", [False, True])
def test_rotary_pairings(halves):
    from mojo_linuxperiments_b200.ops import attention as A
    P = Paged([20], 2, 1, 32, 16, "float32", pairs=16)
    rows = P.raw[0].clone()
    pos = torch.arange(20, dtype=torch.int32, device=DEV)
    A.rotary_paged(rows, 2, pos, torch.zeros_like(pos), P.cos, P.sin, P.cache, P.table, interleaved=not halves)
    x = P.raw[0][:, :64].double().view(20, 2, 32)
    c, s = P.cos[:20].double()[:, None], P.sin[:20].double()[:, None]
    u, v = (x[..., :16], x[..., 16:]) if halves else (x[..., 0::2], x[..., 1::2])
    a, b = u * c - v * s, v * c + u * s
    want = torch.cat([a, b], -1) if halves else torch.stack([a, b], -1).reshape(20, 2, 32)
    assert (rows[:, :64].double().view(20, 2, 32) - want).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [None, 24, 100, 160])
def test_portions_of_any_size_equal_the_whole_prompt(chunk, dtype):
    P = Paged([420, 260], 4, 2, 64, 64, dtype, pairs=16, chunk=chunk)
    want = [P.want(0), P.want(1)]
    sizes = [2, 3, 2, 9, 16, 17, 31, 64, 2, 100, 129, 2, 43]
    a = b = 0
    for n in sizes:
        m = min(max(2, n // 2), 260 - b)
        n = min(n, 420 - a)
        span = {0: (a, n)}
        if m > 0:
            span = {1: (b, m), 0: (a, n)}             # ragged, not in slot order
        got = P.portion(span)
        P.ok()
        for i, (f, k) in span.items():
            assert (got[i].double() - want[i][f:f + k]).abs().max().item() < ATOL[P.dtype], (i, f, k)
        a, b = a + n, b + m
    assert a == 420


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [None, 16, 40, 96 + 7])
def test_decoding_token_by_token_over_page_and_chunk_edges(chunk, dtype):
    P = Paged([230, 131, 60], 6, 2, 48, 80, dtype, pairs=10, chunk=chunk)
    want = [P.want(b) for b in range(3)]
    start = [100, 1, 0]
    P.portion({0: (0, 100), 1: (0, 1)})
    for t in range(60):
        got = P.decode([s + t for s in start], splits=1 + t % 8 if dtype == "bfloat16" else None)
        for b in range(3):
            assert (got[b].double() - want[b][start[b] + t]).abs().max().item() < ATOL[P.dtype], (b, start[b] + t)
    P.ok()


def _spotlight(P, b, q_pos, k_pos, gain=9.0):
    """Make key k_pos match query q_pos (every head) so strongly that the output is that key's value, if it is visible."""
    H, G, dk, dv = P.H, P.G, P.dk, P.dv
    base = torch.zeros(dk, device=DEV)
    base[2 * P.pairs:] = gain / math.sqrt(dk - 2 * P.pairs) * math.sqrt(math.sqrt(dk))        # unrotated dimensions only
    P.raw[b][q_pos, :H * dk] = base.repeat(H).to(P.dtype)
    P.raw[b][k_pos, H * dk:(H + G) * dk] = base.repeat(G).to(P.dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [24, 64, 100, None])
def test_one_outstanding_key_just_inside_and_just_outside(chunk, dtype):
    """A single key with a score far above all others: at the chunk's first position (seen), at the last position of the
    chunk before (not seen), at the very first token, at page borders; in a prompt, in portions and in decoding."""
    c = chunk or 1 << 30
    n = 330
    for q_pos in sorted({c - 1, c, 2 * c - 1, 2 * c + 3, 3 * c - 1, 17, 127, 128, 300, 329} & set(range(n))):
        lo = q_pos // c * c
        for k_pos in sorted({lo, lo - 1, lo + 1, 0, q_pos, q_pos - 1, (q_pos // 16) * 16, max(0, (q_pos // 16) * 16 - 1)}):
            if not 0 <= k_pos <= q_pos:
                continue
            P = Paged([n], 4, 2, 64, 32, dtype, pairs=16, chunk=chunk, sink=True, gate=False, seed=q_pos)
            _spotlight(P, 0, q_pos, k_pos)
            want = P.want(0)[q_pos]
            value = P.parts(0)[2][k_pos].repeat_interleave(2, 0).reshape(-1)
            seen = lo <= k_pos
            assert ((want - value).abs().max().item() < 0.05) == seen          # the test itself is sharp
            whole = P.portion({0: (0, n)})[0][q_pos]
            assert (whole.double() - want).abs().max().item() < ATOL[P.dtype], (q_pos, k_pos)
            cut = P.portion({0: (q_pos, min(2, n - q_pos))})[0][0]             # the same row at the start of a two-token portion
            assert (cut.double() - want).abs().max().item() < ATOL[P.dtype], (q_pos, k_pos)
            dec = P.decode([q_pos])[0]
            assert (dec.double() - want).abs().max().item() < ATOL[P.dtype], (q_pos, k_pos)
    P.ok()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sink_counts_once_and_is_not_scaled(dtype):
    """Equal scores make the weights countable: m visible keys and a sink of log(m) leave half of the mean value."""
    P = Paged([200], 4, 1, 32, 16, dtype, chunk=64, gate=False, scale=0.01)
    P.raw[0][:, :4 * 32] = 0
    for m, pos in ((1, 64), (10, 73), (64, 63), (8, 199)):
        P.sink = torch.tensor([math.log(m), -40.0, 60.0, math.log(3 * m)], device=DEV)
        lo = pos // 64 * 64
        assert pos - lo + 1 == m
        mean = P.parts(0)[2][lo:pos + 1, 0].mean(0)
        rows = {"whole": P.portion({0: (0, 200)})[0][pos], "decoded": P.decode([pos])[0]}
        for how, r in rows.items():
            r = r.double().view(4, 16)
            for h, f in enumerate((0.5, 1.0, 0.0, 0.25)):
                assert (r[h] - f * mean).abs().max().item() < 1.5e-2, (how, m, h)
    P.ok()


@pytest.mark.parametrize("splits", [1, 2, 3, 5, 8])
def test_decode_splits_agree_and_empty_slots_stay_silent(splits):
    P = Paged([1, 20, 515, 900, 64], 8, 2, 128, 128, "bfloat16", pairs=32)
    P.portion({b: (0, n) for b, n in enumerate(P.lens)})
    before = P.cache.data.clone()
    got = P.decode([n - 1 for n in P.lens], splits=splits, live=[1, 1, 1, 0, 1])
    P.ok()
    for b in (0, 1, 2, 4):
        assert (got[b].double() - P.want(b)[-1]).abs().max().item() < 2.5e-2, b
    assert got[3].abs().max().item() == 0
    assert (P.cache.data.float() - before.float()).abs().max().item() < 1e-6      # the same tokens were written again


def test_positions_outside_the_pages_are_refused():
    P = Paged([30], 2, 1, 32, 32, "bfloat16", pairs=8, cap=64)
    rows = P.raw[0][:1].clone()
    out = torch.zeros((1, 64), dtype=torch.bfloat16, device=DEV)
    pos = torch.tensor([64], dtype=torch.int32, device=DEV)
    before = P.cache.data.clone()
    P.A.rotary_paged(rows, 2, pos, torch.zeros_like(pos), P.cos, P.sin, P.cache, P.table)
    with pytest.raises(RuntimeError, match="rotary_paged"):
        P.ok()
    P.A.attn_decode_paged(rows, 2, pos, pos + 1, P.cos, P.sin, P.cache, P.table, P.spec(rows), out)
    with pytest.raises(RuntimeError, match="attn_decode_paged"):
        P.ok()
    assert torch.equal(P.cache.data, before)
    P.ok()


def test_fp32_argmax_matches_torch():
    from mojo_linuxperiments_b200.ops import attention as A
    g = torch.Generator(device=DEV).manual_seed(4)
    x = torch.randn((9, 5003), generator=g, device=DEV)
    x[3, 17] = x[3, 4000] = 99.0
    for chunks in (1, 4, 64):
        assert A.argmax_merge(*A.argmax_rows(x[:, :5001], chunks=chunks)).tolist() == x[:, :5001].argmax(-1).tolist()


# ---------------------------------------------------------------------------------------------------------
# the model through the engine
# ---------------------------------------------------------------------------------------------------------
def uneven() -> LC.LayeredConfig:
    """Layers that differ in everything, one without feed-forward, no scaling / no rotation / no chunk somewhere, a loop that
    starts inside."""
    y = LC.Yarn(3.0, 50.0, 10.0, 1.0)
    a = LC.AttentionSpec(4, 2, 48, 64, 0.21, LC.Rotary(2000.0, 20, y), 36)
    b = LC.AttentionSpec(3, 3, 20, 12, 0.5, LC.Rotary(100.0, 20), 23)
    c = LC.AttentionSpec(10, 1, 128, 24, 0.09, None, None)
    layers = (LC.LayerSpec(a, LC.GatedMLP(130, 0.8)), LC.LayerSpec(b, None), LC.LayerSpec(c, LC.GatedMLP(77, 2.0)),
              LC.LayerSpec(a, LC.GatedMLP(64, 5.0)))
    return LC.LayeredConfig("Volonex", 203, 108, layers, 2.5, 0.6, 1e-6, LC.Loop(1, 3, 3))


def bare() -> LC.LayeredConfig:
    """Odd sizes everywhere, the whole stack repeated, its last layer without feed-forward."""
    a = LC.AttentionSpec(5, 5, 18, 22, 0.3, LC.Rotary(50.0, 18, LC.Yarn(2.0, 40.0, 4.0, 1.0)), 19)
    b = LC.AttentionSpec(7, 1, 33, 9, 0.2, LC.Rotary(900.0, 6), 64)
    return LC.LayeredConfig("Volonex", 131, 93, (LC.LayerSpec(a, LC.GatedMLP(51, 1.0)), LC.LayerSpec(b, None)), 1.7, 1.0, 1e-6, LC.Loop(0, 2, 2))


def even(chunk=40, **kw) -> LC.LayeredConfig:
    kw = {"dim": 64, "vdim": 32, "rot_dims": 32, "base": 1e4, "scaling": LC.Yarn(2.0, 100.0, 8.0, 1.0), "limit": 1.5, "embed_scale": 3.0,
          "residual_mult": 0.8, **kw}
    return LC.volonex(160, 3, 4, 2, 192, 301, chunk=chunk, **kw)


class Model:
    def __init__(self, cfg, dtype, seed=0, slots=3, max_len=512, **rt):
        from mojo_linuxperiments_b200.engine.engine import Engine
        self.cfg, self.t = cfg, LW.init_master(cfg, seed)
        self.rt = RuntimeConfig(dtype=dtype, max_seq_len=max_len, **rt)
        self.eng = Engine(cfg, self.rt, weights=LW.place(cfg, self.rt, self.t, DEV), device=DEV)
        self.eng.start_batch(slots, max_len)
        self.td = {k: v.to(DEV) for k, v in self.t.items()}
        self.d = cfg.to_dict()

    def ids(self, n, seed=0):
        return torch.randint(0, self.cfg.vocab, (n,), generator=torch.Generator().manual_seed(seed))

    def want(self, ids):
        return V.forward(self.d, self.td, ids.to(DEV))

    def run(self, slot, ids, sizes=None):
        """feed ids in portions (sizes cycle; None: all at once) and return every position's logits"""
        out, a, i = [], 0, 0
        while a < len(ids):
            n = len(ids) - a if sizes is None else min(sizes[i % len(sizes)], len(ids) - a)
            out.append(self.eng.step([(slot, ids[a:a + n], list(range(n)))])[0])
            a, i = a + n, i + 1
        self.eng.check_status()
        return torch.cat(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("make", [uneven, bare, even, LC.tiny_volonex])
def test_whole_prompt_layers_and_logits(make, dtype):
    M = Model(make(), dtype)
    for n in (1, 2, 23, 150):
        ids = M.ids(n, n)
        M.eng.release_sequence(0)
        got, seen = [], []
        M.eng.model.observer = lambda r, x: got.append(x.double().clone())
        lg = M.run(0, ids)
        M.eng.model.observer = None
        want = V.forward(M.d, M.td, ids.to(DEV), collect=seen)
        emb = M.td["embed"][ids.to(DEV)].double() * M.cfg.embed_scale
        assert len(got) == len(seen) == len(M.cfg.runs)
        for r, (x, y) in enumerate(zip(got, seen)):
            if r + 1 < len(seen) and M.cfg.runs[r + 1].add_embedding:
                y = y + emb
            assert rel(x, y) < TOL[dtype], r
        assert rel(lg, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("make", [uneven, bare, even])
def test_cuts_do_not_matter(make, dtype):
    """whole prompt = token by token = portions of changing size, down to two tokens, started anywhere in a chunk"""
    M = Model(make(), dtype)
    ids = M.ids(130, 5)
    want = M.want(ids)
    for sizes in (None, [1], [2], [3, 2, 17], [16, 2, 40], [100, 1, 1, 1, 2], [23], [36, 35, 2]):
        M.eng.release_sequence(1)
        assert rel(M.run(1, ids, sizes), want) < TOL[dtype], sizes


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_equal_each_alone(dtype):
    """Portions and single tokens of several sequences in the same step, sequences that pause, slots and pages that are
    released and used again."""
    M = Model(uneven(), dtype, slots=3, kv_pool_tokens=420)
    seqs = [M.ids(n, 10 + n) for n in (140, 61, 200, 33, 90)]
    want = [M.want(s) for s in seqs]
    at, slot_of, waiting, got = {}, {}, [0, 1, 2, 3, 4], {i: [] for i in range(5)}
    free, g = [2, 0, 1], torch.Generator().manual_seed(1)
    steps = 0
    while waiting or slot_of:
        while waiting and free:
            i = waiting.pop(0)
            slot_of[i], at[i] = free.pop(), 0
        who = [i for i in slot_of if torch.rand((), generator=g) < 0.75] or list(slot_of)[:1]
        single = steps % 3 == 2
        entries = []
        for i in who:
            n = 1 if single else int(torch.randint(1, 45, (), generator=g))
            n = min(n, len(seqs[i]) - at[i])
            entries.append((slot_of[i], seqs[i][at[i]:at[i] + n], list(range(n))))
            at[i] += n
        for i, l in zip(who, M.eng.step(entries)):
            got[i].append(l)
        for i in list(slot_of):
            if at[i] == len(seqs[i]):
                M.eng.release_sequence(slot_of[i])
                free.append(slot_of.pop(i))
        steps += 1
    M.eng.check_status()
    assert steps > 12 and M.eng.kv.pages_in_use() == 0
    for i in range(5):
        assert rel(torch.cat(got[i]), want[i]) < TOL[dtype], i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_gives_old_chunks_back(dtype):
    M = Model(even(chunk=48), dtype, slots=2, max_len=1024, max_prefill_tokens=64)
    ids = M.ids(700, 3)
    want = M.want(ids)
    got = [M.run(1, ids[:150], [150])]                    # cut into three calls by max_prefill_tokens
    held = []
    for p in range(150, 700):
        got.append(M.eng.step([(1, ids[p:p + 1], [0])])[0])
        held.append(M.eng.kv.pages_in_use())
    M.eng.check_status()
    assert rel(torch.cat(got), want) < TOL[dtype]
    assert max(held) <= 3 + 1 and M.eng.kv.num_pages < 2 * 64


def test_a_chunk_knows_nothing_of_the_one_before():
    """All layers share one chunk size: another token in an earlier chunk changes nothing, the chunk's first token does."""
    M = Model(even(chunk=40), "float32")
    a = M.ids(120, 1)
    b, c = a.clone(), a.clone()
    b[39], c[40] = (a[39] + 1) % 301, (a[40] + 1) % 301
    for sizes in (None, [1], [2, 39, 7]):
        la, lb, lc = (M.run(s, x, sizes) for s, x in enumerate((a, b, c)))
        assert rel(lb[40:], la[40:]) < 1e-6 and rel(lb[39:40], la[39:40]) > 1e-2
        assert rel(lc[79:80], la[79:80]) > 1e-4 and rel(lc[80:], la[80:]) < 1e-6 and rel(lc[:40], la[:40]) < 1e-6
        for s in range(3):
            M.eng.release_sequence(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("make", [uneven, even])
def test_greedy_generation_through_the_engine(make, dtype):
    M = Model(make(), dtype)
    prompts = torch.stack([M.ids(37, 20), M.ids(37, 21), M.ids(37, 22)])
    new = 30
    for graph in (True, False):
        out = M.eng.generate(prompts, new, use_graph=graph)
        same = 0
        for b in range(3):
            toks, logs = V.greedy(M.d, M.td, prompts[b].to(DEV), new)
            for i in range(new):
                if int(out[b, i]) != toks[i]:
                    top = logs[i].topk(2).values
                    assert (top[0] - top[1]).item() < 4 * TOL[dtype] * logs[i].pow(2).mean().sqrt().item(), (b, i)
                    break
                same += 1
        assert same > (3 * new - 3 if dtype == "float32" else new)


def test_ragged_prefill_and_admission_between_decode_steps():
    M = Model(even(chunk=32), "float32", slots=3, max_prefill_tokens=48)
    eng, prompts, late = M.eng, [M.ids(5, 1), M.ids(70, 2), M.ids(31, 3)], M.ids(55, 4)
    new = 24
    want = [V.greedy(M.d, M.td, p.to(DEV), new)[0] for p in prompts]
    want_late = V.greedy(M.d, M.td, late.to(DEV), new - 6)[0]
    eng.start_batch(3, 128)
    got = [[t] for t in eng.prefill(prompts).tolist()]
    for step in range(1, new):
        if step == 6:
            eng.release_sequence(0)
            got_late = [int(eng.admit_sequence(0, late)[0])]
        toks = eng.decode_step().tolist()
        for b in range(3):
            (got_late if b == 0 and step >= 6 else got[b]).append(toks[b])
    eng.check_status()
    assert got[0] == want[0][:6] and got[1] == want[1] and got[2] == want[2] and got_late[:new - 6] == want_late


def test_given_tokens_then_greedy_decoding():
    """step() leaves the engine ready for decode_step when the last place was asked for; a paused sequence keeps its token."""
    M = Model(even(), "float32", slots=2)
    a, b = M.ids(20, 1), M.ids(45, 2)
    ta, tb = V.greedy(M.d, M.td, a.to(DEV), 6)[0], V.greedy(M.d, M.td, b.to(DEV), 6)[0]
    M.eng.step([(0, a, [19]), (1, b[:40], [])])
    for p in range(40, 45):                                   # sequence 0 waits
        M.eng.step([(1, b[p:p + 1], [0])])
    assert M.eng.tokens.tolist() == [ta[0], tb[0]]
    for i in range(1, 6):
        assert M.eng.decode_step().tolist() == [ta[i], tb[i]]
    with pytest.raises(ValueError):
        M.eng.step([(0, [1], [1])])
    with pytest.raises(ValueError):
        M.eng.step([(0, [1], [0]), (0, [2], [0])])


def test_w8a8_models_take_explicit_steps_too():
    from mojo_linuxperiments_b200.engine.engine import Engine
    from mojo_linuxperiments_b200.models import config as C
    eng = Engine(C.tiny_dense(), C.RuntimeConfig(max_seq_len=128), seed=0, device=DEV)
    p = torch.randint(0, 1024, (2, 20), generator=torch.Generator().manual_seed(0))
    out = eng.generate(p, 4)
    eng.start_batch(2, 64)
    lg = eng.step([(0, p[0], [19]), (1, p[1], [19])])
    assert [int(l.argmax()) for l in lg] == out[:, 0].tolist()
    lg = eng.step([(0, out[0, :1], [0]), (1, out[1, :1], [0])])
    assert [int(l.argmax()) for l in lg] == out[:, 1].tolist()
    with pytest.raises(ValueError, match="whole prompts"):
        eng.step([(0, p[0], [])])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(tmp_path, dtype):
    cfg = uneven()
    t = LW.init_master(cfg, 9)
    LW.save(str(tmp_path / "m"), cfg, t)
    g = torch.Generator().manual_seed(2)
    a, b = (torch.randint(0, cfg.vocab, (n,), generator=g) for n in (80, 30))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:50].tolist(), "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[50:51].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b.tolist(), "want": [0, 29]}, {"id": "x", "tokens": a[51:53].tolist(), "want": [1]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": a[53:54].tolist(), "want": [0]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "o"),
                        "--max-tokens", "100"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = (V.forward(cfg.to_dict(), t, s) for s in (a, b))
    want = {0: wa[[49, 3]], 2: torch.stack([wb[0], wb[29], wa[52]]), 3: wa[53:54]}
    assert sorted(os.listdir(tmp_path / "o")) == [f"{i}.f32" for i in want]
    for i, w in want.items():
        got = torch.frombuffer(bytearray((tmp_path / "o" / f"{i}.f32").read_bytes()), dtype=torch.float32).view(w.shape)
        assert rel(got, w) < TOL[dtype], i


def test_generate_command(tmp_path):
    r = subprocess.run([sys.executable, "-m", "mojo_linuxperiments_b200", "generate", "--model", "tiny-volonex", "--dtype", "float32",
                        "--prompt-ids", "1,2,3", "7,8,9,10,11", "--max-new-tokens", "5"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = r.stdout.strip().splitlines()
    assert len(lines) == 2 and all(len(l.split(",")) == 5 for l in lines)
