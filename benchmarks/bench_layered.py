"""Prefill and decode throughput of the Volonex design beside the W8A8 decoder of equal size, and each of its kernels beside
the like kernel of that decoder, both as a fraction of their own roofline.

``python bench.py --layered`` runs it (random weights, synthetic ids).  Equal size means equal widths, heads, feed-forward,
vocabulary and context; Volonex streams bf16 weights (twice the bytes) and keeps an fp32 residual stream.  Whole-model
numbers go through ``Engine`` (captured graphs).  Kernel numbers: a graph with one launch per layer (weights and caches
larger than the 126 MB L2 in total, so nothing is re-read from L2), CUDA events around several replays after warm-up.
Rooflines: the larger of bytes / measured copy bandwidth and operations / peak (bf16: measured; int8: nominal 4.5 POPS)."""
from __future__ import annotations

import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

INT8_OPS = 4.5e15
SIZES = {   # width, layers, heads, kv heads, feed-forward, vocabulary
    "4096": (4096, 8, 32, 8, 14336, 128256),
    "2048": (2048, 16, 16, 8, 8192, 128256),
}


def peaks():
    try:
        with open(os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "of measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "of fallback"


def timed(fn, iters=5, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e-3 / iters


def per_launch(fn, layers):
    """Seconds per call of fn(layer): all layers in one graph."""
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        for l in range(layers):
            fn(l)
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=s):
        for l in range(layers):
            fn(l)
    t = timed(g.replay) / layers
    del g
    return t


def engine(kind, size, batch, max_len, max_prefill=16384):
    from mojo_linuxperiments_b200.engine.engine import Engine
    from mojo_linuxperiments_b200.models import config as C
    from mojo_linuxperiments_b200.models import layered_config as LC
    w, n, h, kv, ff, vocab = SIZES[size]
    rt = C.RuntimeConfig(max_batch=batch, max_seq_len=(max_len + 127) // 128 * 128, max_prefill_tokens=max_prefill)
    cfg = LC.volonex(w, n, h, kv, ff, vocab) if kind == "volonex" else C.ModelConfig("w8a8", n, w, h, kv, ff, vocab)
    return cfg, Engine(cfg, rt, seed=0)


def throughput(kind, size, decode_batches=(1, 32), prompt=1024, steps=32):
    out = {}
    for batch in decode_batches:
        cfg, eng = engine(kind, size, batch, prompt + 2 * steps + 32)
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


def kernels(size, batch=32, ctx=1024, prompt_seqs=4, prompt=2048):
    from mojo_linuxperiments_b200.models.config import RuntimeConfig
    from mojo_linuxperiments_b200.ops import attention as A
    from mojo_linuxperiments_b200.ops import dense as D
    from mojo_linuxperiments_b200.ops import linear as L
    hbm, bf16, note = peaks()
    w, n, H, G, ff, vocab = SIZES[size]
    n = max(n, 12)
    gen = torch.Generator(device="cuda").manual_seed(0)
    res = {}

    def put(name, phase, sec, nbytes, ops, peak):
        roof = max(nbytes / hbm, ops / peak)
        res.setdefault(phase, {})[name] = {"us": round(sec * 1e6, 2), "roofline_us": round(roof * 1e6, 2), "fraction": round(roof / sec, 3)}

    shapes = {"qkv": ((H + 2 * G) * 128, w), "o": (w, H * 128), "gate_up": (2 * ff, w), "down": (w, ff)}
    for phase, M in (("decode", batch), ("prefill", prompt_seqs * prompt)):
        for name, (N, K) in shapes.items():
            reps = n if phase == "decode" else 4
            extra = H if name == "qkv" else 0
            ws = [D.DenseW(torch.randn((N + extra, D.padded(K)), generator=gen, device="cuda", dtype=torch.bfloat16) * K ** -0.5, N + extra, K) for _ in range(reps)]
            x = torch.randn((M, K), generator=gen, device="cuda", dtype=torch.bfloat16)
            if name in ("o", "down"):
                stream = D.rows(M, N, torch.float32, "cuda").zero_()
                norm = D.DynamicTanh.of(0.5, torch.ones(N), torch.zeros(N), "cuda")
                h = D.rows(M, N, torch.bfloat16, "cuda")
                fn = lambda l: D.linear_residual(x, ws[l], stream, 0.5, norm, h)
                act = M * K * 2 + M * N * (8 + 2)
            elif name == "gate_up":
                fn = lambda l: D.linear_glu(x, ws[l], 7.0)
                act = M * K * 2 + M * N
            else:
                fn = lambda l: D.linear(x, ws[l])
                act = M * K * 2 + M * (N + extra) * 2
            put("volonex " + name, phase, per_launch(fn, reps), (N + extra) * K * 2 + act, 2.0 * M * (N + extra) * K, bf16)
            del ws
            # the W8A8 decoder's linear of the same shape (its norm / activation prologue is a launch of its own)
            wq = [torch.randint(-127, 128, (N, K), generator=gen, device="cuda", dtype=torch.int8) for _ in range(max(reps, 2 * n if phase == "decode" else 4))]
            sw = torch.full((N,), 0.01, device="cuda")
            xq = torch.randint(-127, 128, (M, K), generator=gen, device="cuda", dtype=torch.int8)
            sx = torch.full((M,), 0.01, device="cuda")
            put("w8a8 " + name, phase, per_launch(lambda l: L.w8a8_gemm(xq, sx, wq[l], sw), len(wq)), N * K + M * K + M * N * 2, 2.0 * M * N * K, INT8_OPS)
            del wq
            torch.cuda.empty_cache()
    # head, sampling and embedding rows
    head = [D.DenseW(torch.randn((vocab, w), generator=gen, device="cuda", dtype=torch.bfloat16) * w ** -0.5, vocab, w) for _ in range(2)]
    x = torch.randn((batch, w), generator=gen, device="cuda", dtype=torch.bfloat16)
    put("volonex head (fp32 logits)", "decode", per_launch(lambda l: D.linear(x, head[l % 2], out_dtype=torch.float32), 4),
        vocab * w * 2 + batch * (vocab * 4 + w * 2), 2.0 * batch * vocab * w, bf16)
    lg = [torch.randn((batch, vocab), generator=gen, device="cuda") for _ in range(12)]
    put("volonex argmax", "decode", per_launch(lambda l: A.argmax_rows(lg[l]), 12), batch * vocab * 4, 0.0, bf16)
    lg = [v.to(torch.bfloat16) for v in lg + lg]
    put("w8a8 argmax", "decode", per_launch(lambda l: A.argmax_rows(lg[l]), 24), batch * vocab * 2, 0.0, bf16)
    wq = [torch.randint(-127, 128, (vocab, w), generator=gen, device="cuda", dtype=torch.int8) for _ in range(2)]
    sw, sx = torch.full((vocab,), 0.01, device="cuda"), torch.full((batch,), 0.01, device="cuda")
    xq = torch.randint(-127, 128, (batch, w), generator=gen, device="cuda", dtype=torch.int8)
    put("w8a8 head", "decode", per_launch(lambda l: L.w8a8_gemm(xq, sx, wq[l % 2], sw), 4), vocab * w + batch * (vocab * 2 + w), 2.0 * batch * vocab * w, INT8_OPS)
    Mp = prompt_seqs * prompt
    ids = torch.randint(0, vocab, (Mp,), generator=gen, device="cuda")
    st, h = D.rows(Mp, w, torch.float32, "cuda"), D.rows(Mp, w, torch.bfloat16, "cuda")
    norm = D.DynamicTanh.of(0.5, torch.ones(w), torch.zeros(w), "cuda")
    put("volonex embedding + norm", "prefill", per_launch(lambda l: D.embed_norm(ids, head[l % 2].data, w, 2.0, st, None, norm, h), 4), Mp * w * 8, 0.0, bf16)
    put("w8a8 embedding", "prefill", per_launch(lambda l: A.embed_gather(ids, head[l % 2].data, out=h), 4), Mp * w * 4, 0.0, bf16)
    del head, wq, lg, st, h
    torch.cuda.empty_cache()
    # attention
    qkv_n = (H + 2 * G) * 128
    mp = (ctx + 127) // 128 * 128 // 16
    caches = [A.PagedKVCache(batch * mp, G, 16, "cuda") for _ in range(4)]
    for c in caches:
        c.data.normal_()
    table = torch.arange(batch * mp, dtype=torch.int32, device="cuda").view(batch, mp)
    pos = torch.full((batch,), ctx - 1, dtype=torch.int32, device="cuda")
    lens = pos + 1
    qkvg = torch.randn((batch, D.padded(qkv_n + H)), generator=gen, device="cuda", dtype=torch.bfloat16)
    sink = torch.zeros(H, device="cuda")
    cos, sin = A.rope_tables(ctx, 10000.0, "cuda", 64)
    out = torch.empty((batch, H * 128), dtype=torch.bfloat16, device="cuda")
    kv_bytes = batch * ctx * G * 128 * 2 * 2
    spec = A.attn_spec(128 ** -0.5, chunk=8192, sink=sink, gate=qkvg[:, qkv_n:qkv_n + H])
    put("volonex attention", "decode", per_launch(lambda l: A.attn_decode_paged(qkvg, H, pos, lens, cos, sin, caches[l], table, spec, out), 4),
        kv_bytes, 4.0 * batch * ctx * H * 128, bf16)
    cos2, sin2 = A.rope_tables(ctx, 10000.0, "cuda")
    qkv = qkvg[:, :qkv_n].contiguous()
    sp = A.pick_decode_splits_tc(batch, G, mp * 16, fused=True)
    sc = A.DecodeAttnScratch(batch, H, G, sp, "cuda")
    put("w8a8 attention", "decode", per_launch(lambda l: A.attn_decode_fused(qkv, pos, cos2, sin2, H, G, caches[l], table, lens, scratch=sc, splits=sp), 4),
        kv_bytes, 4.0 * batch * ctx * H * 128, bf16)
    del caches
    torch.cuda.empty_cache()
    M, B = prompt_seqs * prompt, prompt_seqs
    mp = prompt // 16
    cache = A.PagedKVCache(B * mp, G, 16, "cuda")
    table = torch.arange(B * mp, dtype=torch.int32, device="cuda").view(B, mp)
    qkvg = torch.randn((M, D.padded(qkv_n + H)), generator=gen, device="cuda", dtype=torch.bfloat16)
    pos = torch.arange(prompt, dtype=torch.int32, device="cuda").repeat(B)
    sid = torch.arange(B, dtype=torch.int32, device="cuda").repeat_interleave(prompt)
    cu = torch.arange(0, M + 1, prompt, dtype=torch.int32, device="cuda")
    cos, sin = A.rope_tables(prompt, 10000.0, "cuda", 64)
    out = torch.empty((M, H * 128), dtype=torch.bfloat16, device="cuda")
    put("volonex rotary + cache append", "prefill", per_launch(lambda l: A.rotary_paged(qkvg, H, pos, sid, cos, sin, cache, table), 4),
        M * (2 * H * 64 * 2 + 2 * G * 256 * 2), 0.0, bf16)
    qk = qkvg[:, :qkv_n].contiguous()
    kb, ob = torch.empty((M, G, 128), dtype=torch.bfloat16, device="cuda"), torch.empty((M, H, 128), dtype=torch.bfloat16, device="cuda")
    cos2, sin2 = A.rope_tables(prompt, 10000.0, "cuda")
    put("w8a8 rotary + cache append", "prefill", per_launch(lambda l: A.rope_kv_write(qk, pos, cos2, sin2, H, G, q_out=ob, k_out=kb, cache=cache, page_table=table, seq_ids=sid), 4),
        M * (2 * H * 128 * 2 + 2 * G * 256 * 2 + G * 256), 0.0, bf16)
    flops = 4.0 * B * H * 128 * prompt * (prompt + 1) / 2
    io = M * (2 * H * 128 + 2 * G * 128) * 2
    for chunk in (8192, 512):
        spec = A.attn_spec(128 ** -0.5, chunk=chunk, sink=sink, gate=qkvg[:, qkv_n:qkv_n + H])
        pairs = sum(min(i % chunk, i) + 1 for i in range(prompt))
        put("volonex attention" + ("" if chunk > prompt else f" (chunks of {chunk})"), "prefill",
            per_launch(lambda l: A.attn_prefill_paged(qkvg, H, pos, sid, cu, prompt, cache, table, spec, out), 4), io, 4.0 * B * H * 128 * pairs, bf16)
    q3, v3 = ob, qk.view(M, H + 2 * G, 128)[:, H + G:]
    put("w8a8 attention", "prefill", per_launch(lambda l: A.attn_prefill(q3, kb, v3, cu, prompt, kv_chunk=0), 4), io, flops, bf16)
    return {"note": note, **res}


def run(sizes=("4096", "2048"), parts=("model", "kernels")) -> dict:
    out = {"metric": "Volonex prefill and decode beside the W8A8 decoder of equal size", "data": "synthetic, random weights", "gpu": torch.cuda.get_device_name()}
    for s in sizes:
        w, n, h, kv, ff, vocab = SIZES[s]
        r = {"config": {"width": w, "layers": n, "heads": h, "kv_heads": kv, "ff": ff, "vocab": vocab, "head_dim": 128}}
        if "model" in parts:
            r["volonex"], r["w8a8"] = throughput("volonex", s), throughput("w8a8", s)
        if "kernels" in parts:
            r["kernels"] = kernels(s)
        out[s] = r
        torch.cuda.empty_cache()
    return out


if __name__ == "__main__":
    print(json.dumps(run()))
