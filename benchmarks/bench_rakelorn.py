"""Prefill and decode throughput of the Rakelorn design beside the framework's closest models of equal size, and each of its
kernels beside the like kernel of those models, both as a fraction of their own roofline.

``python bench.py --layered rakelorn`` runs it (random weights, synthetic ids).  Closest models: Volonex (the other unquantised
layer-by-layer decoder; same width, layers, heads and vocabulary, a dense feed-forward with as many multiplications per token as
the chosen experts) and the W8A8 mixture-of-experts decoder (int8; same width, layers, experts and choices).  Kernel numbers and
rooflines as in ``bench_layered``; the roofline of an attention is that of its cheapest form (bytes of the cached rows, or the
multiplications of the expanded form)."""
from __future__ import annotations

import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

from benchmarks.bench_layered import INT8_OPS, peaks, per_launch, timed  # noqa: E402

# width, layers, heads, own / shared / value size per head, query latent, latent, recurrent channels, experts, identity, top, expert
# feed-forward, groups, kept groups, vocabulary
SIZES = {
    "2048": dict(width=2048, layers=12, heads=16, dim=128, rot=64, vdim=128, q_rank=1536, rank=512, rec=3072, experts=64, identity=8, top=6,
                 ff=1536, groups=8, keep=4, vocab=102400),
    "4096": dict(width=4096, layers=6, heads=32, dim=96, rot=32, vdim=96, q_rank=1024, rank=384, rec=4096, experts=16, identity=2, top=2,
                 ff=4096, groups=6, keep=3, vocab=128256),
}


def config(kind: str, z: dict):
    from mojo_linuxperiments_b200.models import config as C
    from mojo_linuxperiments_b200.models import layered_config as LC
    dense = -(-z["top"] * z["ff"] * 2 // 3 // 128) * 128
    if kind == "rakelorn":
        return LC.rakelorn(z["width"], z["layers"], z["heads"], z["vocab"], dim=z["dim"], rot_dim=z["rot"], vdim=z["vdim"], q_rank=z["q_rank"],
                           kv_rank=z["rank"], recurrent=z["rec"],
                           moe=LC.MoE(z["experts"], z["top"], z["ff"], 1.5, z["identity"], z["groups"], z["keep"]))
    if kind == "volonex":
        return LC.volonex(z["width"], z["layers"], z["heads"], max(1, z["heads"] // 4), dense, z["vocab"])
    return C.ModelConfig("w8a8-moe", z["layers"], z["width"], z["width"] // 128, max(1, z["width"] // 512), 0, z["vocab"], n_experts=z["experts"],
                         top_k=z["top"], moe_ffn=max(128, z["ff"] * 2 // 3 // 128 * 128), qk_norm=True)


def throughput(kind: str, z: dict, decode_batches=(1, 32), prompt=1024, steps=32) -> dict:
    from mojo_linuxperiments_b200.engine.engine import Engine
    from mojo_linuxperiments_b200.models.config import RuntimeConfig
    out, cfg = {}, config(kind, z)
    for batch in decode_batches:
        rt = RuntimeConfig(max_batch=batch, max_seq_len=(prompt + 2 * steps + 159) // 128 * 128, max_prefill_tokens=16384)
        eng = Engine(cfg, rt, seed=0)
        ids = torch.randint(0, cfg.vocab, (batch, prompt), generator=torch.Generator().manual_seed(1)).cuda()
        eng.start_batch(batch, prompt + 2 * steps + 16)
        t = []
        for _ in range(6):                       # the first call captures the graph
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            a.record()
            eng.prefill(ids)
            b.record()
            torch.cuda.synchronize()
            t.append(a.elapsed_time(b))
        t = sorted(t[3:])[1]
        out[f"prefill_{batch}x{prompt}"] = {"ms": round(t, 3), "tokens_per_s": round(batch * prompt / t * 1e3)}
        eng.check_status()
        sec = timed(eng.decode_step, steps, 4)
        eng.check_status()
        out[f"decode_bs{batch}"] = {"ms": round(sec * 1e3, 4), "tokens_per_s": round(batch / sec, 1), "kernels": eng.kernels_per_step}
        eng.close()
        del eng
        torch.cuda.empty_cache()
    return out


def kernels(z: dict, batch=32, ctx=1024, seqs=4, prompt=2048) -> dict:
    from mojo_linuxperiments_b200.ops import attention as A
    from mojo_linuxperiments_b200.ops import dense as D
    from mojo_linuxperiments_b200.ops import latent as LT
    from mojo_linuxperiments_b200.ops import linear as L
    from mojo_linuxperiments_b200.ops import moe as MO
    from mojo_linuxperiments_b200.ops import recurrent as RC
    from mojo_linuxperiments_b200.ops import rows as RW
    hbm, bf16, note = peaks()
    w, H, n, r, dv, qr, rank, rec = (z[k] for k in ("width", "heads", "dim", "rot", "vdim", "q_rank", "rank", "rec"))
    E, I, top, ff = z["experts"], z["identity"], z["top"], z["ff"]
    g = torch.Generator(device="cuda").manual_seed(0)
    bf = torch.bfloat16
    res: dict = {}

    def put(phase, name, sec, nbytes, ops=0.0, peak=bf16):
        roof = max(nbytes / hbm, ops / peak)
        res.setdefault(phase, {})[name] = {"us": round(sec * 1e6, 2), "roofline_us": round(roof * 1e6, 2), "fraction": round(roof / sec, 3)}

    def rnd(*shape, dtype=bf):
        return torch.randn(shape, generator=g, device="cuda", dtype=dtype)

    def weights(N, K, reps):
        return [D.DenseW(rnd(N, D.padded(K)).mul_(K ** -0.5), N, K) for _ in range(reps)]

    Mp = seqs * prompt
    for phase, M in (("decode", batch), ("prefill", Mp)):
        reps = 16 if phase == "decode" else 4
        # plain linears
        for name, N, K, f32 in (("down linear (latents, gates)", qr + rank + r + H, w, True), ("query linear", H * (n + r), qr, False),
                                ("recurrent linear", 3 * rec, w, True)):
            ws, x = weights(N, K, reps), rnd(M, K)
            od = torch.float32 if f32 else bf
            put(phase, "rakelorn " + name, per_launch(lambda l: D.linear(x, ws[l], out_dtype=od), reps), N * K * 2 + M * K * 2 + M * N * (4 if f32 else 2), 2.0 * M * N * K)
            del ws
        qkv = ((H + 2 * max(1, H // 4)) * 128 + H)
        ws, x = weights(qkv, w, reps), rnd(M, w)
        put(phase, "volonex qkvg linear", per_launch(lambda l: D.linear(x, ws[l]), reps), qkv * w * 2 + M * w * 2 + M * qkv * 2, 2.0 * M * qkv * w)
        del ws
        stream = D.rows(M, w, torch.float32, "cuda").zero_()
        h = D.rows(M, w, bf, "cuda")
        norm = D.DynamicTanh.of(0.5, torch.ones(w), torch.zeros(w), "cuda")
        for name, K in (("attention output", H * dv), ("recurrent output", rec)):
            ws, x = weights(w, K, reps), rnd(M, K)
            put(phase, f"rakelorn {name} + residual", per_launch(lambda l: D.linear_residual(x, ws[l], stream, 1.0, None, None), reps),
                w * K * 2 + M * K * 2 + M * w * 8, 2.0 * M * w * K)
            del ws
        ws, x = weights(w, H * 128, reps), rnd(M, H * 128)
        put(phase, "volonex attention output + residual + norm", per_launch(lambda l: D.linear_residual(x, ws[l], stream, 0.5, norm, h), reps),
            w * H * 128 * 2 + M * H * 256 + M * w * 10, 2.0 * M * w * H * 128)
        del ws
        if phase == "decode":
            q = rnd(M, H * (n + r))
            wk = [D.GroupedW(rnd(H * rank, n), H, rank, n) for _ in range(24)]
            put(phase, "rakelorn queries into the latent space (per head)", per_launch(lambda l: D.linear_heads(q, wk[l], n + r, rank), 24),
                H * rank * n * 2 + M * H * (n + rank) * 2, 2.0 * M * H * n * rank)
            o, gate = rnd(M, H * rank), rnd(M, H, dtype=torch.float32)
            wv = [D.GroupedW(rnd(H * dv, rank), H, dv, rank) for _ in range(24)]
            put(phase, "rakelorn values out of the latent space (per head, gate)", per_launch(lambda l: D.linear_heads(o, wv[l], rank, dv, gate=gate), 24),
                H * rank * dv * 2 + M * H * (dv + rank) * 2, 2.0 * M * H * dv * rank)
            del wk, wv
        else:
            lat = rnd(M, rank + r)
            ws = weights(H * (n + dv), rank, reps)
            put(phase, "rakelorn latents into keys and values", per_launch(lambda l: D.linear(lat, ws[l]), reps),
                H * (n + dv) * rank * 2 + M * rank * 2 + M * H * (n + dv) * 2, 2.0 * M * H * (n + dv) * rank)
            del ws
        torch.cuda.empty_cache()

        # mixture of experts beside the int8 one
        x = rnd(M, w)
        wr = weights(E + I, w, 4)
        put(phase, "rakelorn router linear", per_launch(lambda l: D.linear(x, wr[l], out_dtype=torch.float32), 4), (E + I) * w * 2 + M * w * 2 + M * (E + I) * 4, 2.0 * M * (E + I) * w)
        e128 = -(-E // 16) * 16
        xq, sx = torch.randint(-127, 128, (M, w), generator=g, device="cuda", dtype=torch.int8), torch.full((M,), 0.01, device="cuda")
        wq, sw = torch.randint(-127, 128, (4, e128, w), generator=g, device="cuda", dtype=torch.int8), torch.full((e128,), 0.01, device="cuda")
        put(phase, "w8a8 router linear", per_launch(lambda l: L.w8a8_gemm(xq, sx, wq[l], sw, out_dtype=torch.float32, narrow=True), 4), e128 * w + M * w + M * e128 * 4, 2.0 * M * e128 * w, INT8_OPS)
        lg = rnd(M, E + I, dtype=torch.float32)
        corr = torch.zeros(E + I, device="cuda")
        put(phase, "rakelorn routing", per_launch(lambda l: MO.route_grouped(lg, corr, top, z["groups"], z["keep"], 1.5, E + I), 8), M * ((E + I) * 4 + top * 8))
        lge = lg[:, :E].contiguous()
        put(phase, "w8a8 routing", per_launch(lambda l: MO.router_topk(lge, top), 8), M * (E * 4 + top * 8))
        ids, wts = MO.route_grouped(lg, corr, top, z["groups"], z["keep"], 1.5, E + I)
        work = MO.moe_align(ids, 0, E)
        ids8, wts8 = MO.router_topk(lge, top)
        work8 = MO.moe_align(ids8, 0, E)
        pairs, pairs8 = int(work.meta[0]), int(work8.meta[0])
        live, live8 = int((work.counts > 0).sum()), int((work8.counts > 0).sum())
        put(phase, "rakelorn work list", per_launch(lambda l: MO.moe_align(ids, 0, E), 8), M * top * 12 + pairs * 4)
        put(phase, "w8a8 work list", per_launch(lambda l: MO.moe_align(ids8, 0, E), 8), M * top * 12 + pairs8 * 4)
        put(phase, "rakelorn gather", per_launch(lambda l: MO.gather_rows(x, work), 8), pairs * w * 4)
        put(phase, "w8a8 gather", per_launch(lambda l: MO.moe_gather(xq, sx, work8), 8), pairs8 * w * 2)
        xp = MO.gather_rows(x, work)
        up = [D.GroupedW(rnd(E * ff, w).mul_(w ** -0.5), E, ff, w) for _ in range(2)]
        put(phase, "rakelorn experts up + activation", per_launch(lambda l: D.linear_experts(xp, up[l % 2], work, act="relu2"), 4),
            live * ff * w * 2 + pairs * (w + ff) * 2, 2.0 * pairs * ff * w)
        u = D.linear_experts(xp, up[0], work, act="relu2")
        del up
        down = [D.GroupedW(rnd(E * w, ff).mul_(ff ** -0.5), E, w, ff) for _ in range(2)]
        put(phase, "rakelorn experts down", per_launch(lambda l: D.linear_experts(u, down[l % 2], work), 4), live * ff * w * 2 + pairs * (w + ff) * 2, 2.0 * pairs * ff * w)
        y = D.linear_experts(u, down[0], work)
        del down, u, xp
        torch.cuda.empty_cache()
        xp8, sp8 = MO.moe_gather(xq, sx, work8)
        wg = torch.randint(-127, 128, (2, E, ff, w), generator=g, device="cuda", dtype=torch.int8)
        sg = torch.full((E, ff), 0.01, device="cuda")
        put(phase, "w8a8 experts (same shape as up)", per_launch(lambda l: MO.grouped_gemm(xp8, sp8, wg[l % 2], sg, work8), 4),
            live8 * ff * w + pairs8 * (w + 2 * ff), 2.0 * pairs8 * ff * w, INT8_OPS)
        wg, sg = wg.view(2, E, w, ff), torch.full((E, w), 0.01, device="cuda")
        hq, sh = torch.randint(-127, 128, (work8.max_slots, ff), generator=g, device="cuda", dtype=torch.int8), torch.full((work8.max_slots,), 0.01, device="cuda")
        put(phase, "w8a8 experts (same shape as down)", per_launch(lambda l: MO.grouped_gemm(hq, sh, wg[l % 2], sg, work8), 4),
            live8 * ff * w + pairs8 * (ff + 2 * w), 2.0 * pairs8 * ff * w, INT8_OPS)
        y8 = MO.grouped_gemm(hq, sh, wg[0], sg, work8)
        del wg, hq
        put(phase, "w8a8 weighted sum of experts", per_launch(lambda l: MO.moe_combine(y8, work8, wts8), 8), pairs8 * w * 2 + M * w * 2)

        # rows between sub-layers
        st2, mixv, state = torch.empty_like(stream), torch.full((w,), 0.5, device="cuda"), torch.zeros((max(batch, seqs), w), device="cuda")
        sums = RW.ExpertSum(y, work.inv, ids, wts, E, x)
        ident = int((ids >= E).sum())
        if phase == "decode":
            pos = torch.full((M,), 5, dtype=torch.int32, device="cuda")
            shift = RW.Shift(mixv, state, pos)
        else:
            pos = torch.arange(prompt, dtype=torch.int32, device="cuda").repeat(seqs)
            sid = torch.arange(seqs, dtype=torch.int32, device="cuda").repeat_interleave(prompt)
            cu = torch.arange(0, M + 1, prompt, dtype=torch.int32, device="cuda")
            shift = RW.Shift(mixv, state, pos, seq_ids=sid, cu=cu, max_len=prompt)
        put(phase, "rakelorn rows: experts + norm + shift", per_launch(lambda l: RW.stream_rows(w, 1.0, 1e-6, h, x=stream, x_out=st2, experts=sums, shift=shift), 8),
            (pairs + ident) * w * 2 + M * w * 10)
        put(phase, "rakelorn rows: norm", per_launch(lambda l: RW.stream_rows(w, 1.0, 1e-6, h, x=stream), 8), M * w * 6)
        gam = torch.ones(w, device="cuda", dtype=bf)
        put(phase, "w8a8 norm + quantisation", per_launch(lambda l: L.act_quant(x, mode=L.AQ_NORM, gamma=gam, eps=1e-6), 8), M * w * 3)
        del y, y8, st2
        # recurrence
        zxg, zb = rnd(M, 3 * rec, dtype=torch.float32), torch.zeros(rec, device="cuda")
        rs = torch.zeros((max(batch, seqs), rec), device="cuda")
        if phase == "decode":
            put(phase, "rakelorn recurrence", per_launch(lambda l: RC.mingru(zxg, zb, zb, rec, rs, pos, out_dtype=bf), 8), M * rec * (12 + 2 + 8))
        else:
            put(phase, "rakelorn recurrence (two launches)", per_launch(lambda l: RC.mingru(zxg, zb, zb, rec, rs, pos, out_dtype=bf, seq_ids=sid, cu=cu, max_len=prompt), 8), M * rec * (12 + 2))
        del zxg, stream, h
        torch.cuda.empty_cache()

    # attention: decoding over the paged cache, a short and a long context
    G = max(1, H // 4)
    dm = LT.dims(H, rank, r)
    qkv_n = (H + 2 * G) * 128
    sink = torch.zeros(H, device="cuda")
    scale = (n + r) ** -0.5
    gq, gc = torch.ones(qr, device="cuda"), torch.ones(rank, device="cuda")
    for c_len, reps in ((ctx, 8), (8 * ctx, 2)):
        note_ctx = f", {c_len} keys"
        mp = c_len // 16
        table = torch.arange(batch * mp, dtype=torch.int32, device="cuda").view(batch, mp)
        pos = torch.full((batch,), c_len - 1, dtype=torch.int32, device="cuda")
        lens = pos + 1
        caches = [A.PagedKVCache(batch * mp, 1, 16, "cuda", dk=rank + r, dv=0) for _ in range(reps)]
        for c in caches:
            c.data.normal_()
        cos, sin = A.rope_tables(c_len, 1e6, "cuda", r)
        qa, q = rnd(batch, H * rank), rnd(batch, H * (n + r))
        put("decode", "rakelorn attention" + note_ctx, per_launch(lambda l: LT.attend(qa, q[:, n:], n + r, dm, scale, pos, None, cos, sin, caches[l % reps], table, seq_lens=lens), 8),
            batch * c_len * (rank + r) * 2 + batch * H * (2 * rank + r) * 2, 2.0 * batch * c_len * H * (2 * rank + r))
        if c_len == ctx:
            low = rnd(batch, qr + rank + r + H, dtype=torch.float32)
            put("decode", "rakelorn norms + cache append", per_launch(lambda l: LT.append(low, qr, gq, gc, 1e-6, dm, pos, None, cos, sin, caches[l], table, seq_lens=lens), 8),
                batch * (qr + rank + r) * 6)
        del caches
        caches = [A.PagedKVCache(batch * mp, G, 16, "cuda") for _ in range(reps)]
        for c in caches:
            c.data.normal_()
        qkvg = rnd(batch, D.padded(qkv_n + H))
        c2, s2 = A.rope_tables(c_len, 1e4, "cuda", 64)
        out = torch.empty((batch, H * 128), dtype=bf, device="cuda")
        spec = A.attn_spec(128 ** -0.5, sink=sink, gate=qkvg[:, qkv_n:qkv_n + H])
        put("decode", "volonex attention (rotary, append, sink, gate)" + note_ctx, per_launch(lambda l: A.attn_decode_paged(qkvg, H, pos, lens, c2, s2, caches[l % reps], table, spec, out), 8),
            batch * c_len * G * 512, 4.0 * batch * c_len * H * 128)
        del caches
        torch.cuda.empty_cache()
    c2, s2 = A.rope_tables(prompt, 1e4, "cuda", 64)
    cos, sin = A.rope_tables(prompt, 1e6, "cuda", r)
    # prefill, and a short portion at the end of a long context
    mp = prompt // 16
    table = torch.arange(seqs * mp, dtype=torch.int32, device="cuda").view(seqs, mp)
    pos = torch.arange(prompt, dtype=torch.int32, device="cuda").repeat(seqs)
    sid = torch.arange(seqs, dtype=torch.int32, device="cuda").repeat_interleave(prompt)
    cu = torch.arange(0, Mp + 1, prompt, dtype=torch.int32, device="cuda")
    cache = A.PagedKVCache(seqs * mp, 1, 16, "cuda", dk=rank + r, dv=0)
    low = rnd(Mp, qr + rank + r + H, dtype=torch.float32)
    put("prefill", "rakelorn norms + cache append", per_launch(lambda l: LT.append(low, qr, gq, gc, 1e-6, dm, pos, sid, cos, sin, cache, table, want_latents=True), 4),
        Mp * ((qr + rank + r) * 6 + (rank + r) * 2))
    q, kv, lat = rnd(Mp, H * (n + r)), rnd(Mp, H * (n + dv)), rnd(Mp, rank + r)
    put("prefill", "rakelorn rotary of the queries", per_launch(lambda l: LT.rotary_heads(q, H, n + r, n, r, pos, cos, sin), 4), Mp * H * r * 4)
    gate = rnd(Mp, H, dtype=torch.float32)
    tri = seqs * prompt * (prompt + 1) / 2
    put("prefill", "rakelorn attention (expanded)", per_launch(lambda l: LT.attend_expanded(q, H, n, r, dv, kv, lat[:, rank:], scale, cu, cu, pos, prompt, gate), 4),
        Mp * H * (2 * n + 2 * r + 2 * dv) * 2, 2.0 * tri * H * (n + r + dv))
    put("prefill", "rakelorn gather of cached latents", per_launch(lambda l: LT.gather(cache, table, cu, torch.arange(seqs, dtype=torch.int32, device="cuda"), Mp, prompt), 4), Mp * (rank + r) * 4)
    short = 64
    ps = torch.arange(prompt - short, prompt, dtype=torch.int32, device="cuda").repeat(seqs)
    ss = torch.arange(seqs, dtype=torch.int32, device="cuda").repeat_interleave(short)
    cs = torch.arange(0, seqs * short + 1, short, dtype=torch.int32, device="cuda")
    qa, q = rnd(seqs * short, H * rank), rnd(seqs * short, H * (n + r))
    put("prefill", f"rakelorn attention, portions of {short} (latent space)", per_launch(
        lambda l: LT.attend(qa, q[:, n:], n + r, dm, scale, ps, ss, cos, sin, cache, table, cu=cs, max_len=short, keys=prompt), 4),
        seqs * prompt * (rank + r) * 2, 2.0 * seqs * short * prompt * H * (2 * rank + r))
    cache = A.PagedKVCache(seqs * mp, G, 16, "cuda")
    qkvg = rnd(Mp, D.padded(qkv_n + H))
    out = torch.empty((Mp, H * 128), dtype=bf, device="cuda")
    put("prefill", "volonex rotary + cache append", per_launch(lambda l: A.rotary_paged(qkvg, H, pos, sid, c2, s2, cache, table), 4), Mp * (2 * H * 128 + 2 * G * 512))
    spec = A.attn_spec(128 ** -0.5, chunk=8192, sink=sink, gate=qkvg[:, qkv_n:qkv_n + H])
    put("prefill", "volonex attention", per_launch(lambda l: A.attn_prefill_paged(qkvg, H, pos, sid, cu, prompt, cache, table, spec, out), 4),
        Mp * (2 * H + 2 * G) * 256, 4.0 * tri * H * 128)
    spec = A.attn_spec(128 ** -0.5, chunk=8192, sink=sink, gate=qkvg[:seqs * short, qkv_n:qkv_n + H])
    put("prefill", f"volonex attention, portions of {short}", per_launch(
        lambda l: A.attn_prefill_paged(qkvg[:seqs * short], H, ps, ss, cs, short, cache, table, spec, out[:seqs * short]), 4),
        seqs * prompt * G * 512, 4.0 * seqs * short * prompt * H * 128)
    table_ = rnd(z["vocab"], w)
    ids = torch.randint(0, z["vocab"], (Mp,), generator=g, device="cuda")
    st, h = D.rows(Mp, w, torch.float32, "cuda"), D.rows(Mp, w, bf, "cuda")
    put("prefill", "rakelorn rows: embedding + norm + shift", per_launch(lambda l: RW.stream_rows(w, 1.0, 1e-6, h, ids=ids, table=table_, x_out=st,
        shift=RW.Shift(torch.full((w,), 0.5, device="cuda"), torch.zeros((seqs, w), device="cuda"), pos, seq_ids=sid, cu=cu, max_len=prompt)), 4), Mp * w * 8)
    norm = D.DynamicTanh.of(0.5, torch.ones(w), torch.zeros(w), "cuda")
    put("prefill", "volonex embedding + norm", per_launch(lambda l: D.embed_norm(ids, table_, w, 2.0, st, None, norm, h), 4), Mp * w * 8)
    return {"note": note, **res}


def run(sizes=tuple(SIZES), parts=("model", "kernels")) -> dict:
    out = {"metric": "Rakelorn prefill and decode beside the closest models of equal size", "data": "synthetic, random weights", "gpu": torch.cuda.get_device_name()}
    for s in sizes:
        r = {"config": SIZES[s]}
        if "model" in parts:
            for kind in ("rakelorn", "volonex", "w8a8-moe"):
                r[kind] = throughput(kind, SIZES[s])
        if "kernels" in parts:
            r["kernels"] = kernels(SIZES[s])
        out[s] = r
        torch.cuda.empty_cache()
    return out


if __name__ == "__main__":
    print(json.dumps(run()))
