"""Kernel microbenchmarks with roofline fractions (CUDA-event timing, L2 flushed between runs).

    python -m cuteafd_b200.bench.microbench gemm --tokens 8192 --features 5120 --k 2048
    python -m cuteafd_b200.bench.microbench attn-prefill --len 8192
    python -m cuteafd_b200.bench.microbench attn-decode --seqs 32 --len 8192
    python -m cuteafd_b200.bench.microbench mla --seqs 8 --len 8192 --qlen 1 --heads 128 [--topk 2048]
    python -m cuteafd_b200.bench.microbench w4 --tokens 8 --features 7168 --k 2048 --fmt nvfp4
    python -m cuteafd_b200.bench.microbench hybrid --size base
    python -m cuteafd_b200.bench.microbench parallel --size base
    python -m cuteafd_b200.bench.microbench sampler --rows 32 --vocab 151936
    python -m cuteafd_b200.bench.microbench moe --tokens 1,16,128,1024,8192 --hidden 7168 --ffn 2048 \
        --experts 256 --top-k 8 --scoring sigmoid

Small kernels (a few microseconds) are timed as a CUDA graph of many launches cycling over more
weight copies than fit in L2, so host launch cost does not pollute the number.  Roofline
denominators come from MEASURED_PEAKS.json at the repository root when present (measured copy
bandwidth and cuBLAS bf16 throughput), else 6650 GB/s and 1590 TFLOP/s.

The MoE mode is the dispatch -> expert -> combine benchmark of the reference's exchange path
(rust/crates/cuteafd-daemon/src/families/glm5/engine.rs:2489-2512 plus the expert worker), here
plan + dispatch + grouped fc1/SwiGLU + grouped fc2/combine kernels on one GPU or, under torchrun,
with the experts on the other ranks.
"""
from __future__ import annotations

import argparse
import json
import os

import torch

from ..ops import kernels as K

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))


def peaks() -> dict:
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return {"hbm_gbs": d["hbm_gbs"], "bf16_tflops": d["bf16_tflops"], "kind": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "kind": "fallback"}


_flush = None


def flush_l2(dev) -> None:
    global _flush
    if _flush is None:
        _flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    _flush.zero_()


def time_eager(fn, dev, iters: int = 10, warm: int = 3) -> float:
    """Median milliseconds of one call, L2 flushed before each timed call."""
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(iters):
        flush_l2(dev)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record(); fn(); b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return sorted(ts)[len(ts) // 2]


def time_graph(fns, reps: int = 5) -> float:
    """Median milliseconds per call for a list of calls captured into one CUDA graph."""
    for f in fns:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in fns:
            f()
    g.replay()
    torch.cuda.synchronize()
    ts = []
    for _ in range(reps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record(); g.replay(); b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return sorted(ts)[len(ts) // 2] / len(fns)


def report(name: str, ms: float, flops: float, byts: float, pk: dict) -> dict:
    tf, gb = flops / ms / 1e9, byts / ms / 1e6
    r = {"case": name, "us": round(ms * 1e3, 2), "tflops": round(tf, 1), "gbs": round(gb, 0),
         "frac_compute": round(tf / pk["bf16_tflops"], 3), "frac_hbm": round(gb / pk["hbm_gbs"], 3), "of": pk["kind"]}
    print(json.dumps(r), flush=True)
    return r


def bench_gemm(a, dev, pk):
    T, N, Kd = a.tokens, a.features, a.k
    x = torch.randn(T, Kd, device=dev).bfloat16()
    out = torch.empty(T, N, dtype=torch.bfloat16, device=dev)
    per = N * Kd * 2 * (2 if a.dual else 1)
    copies = 1 if T > 256 else max(2, min(24, int(200e6 // per) + 1))
    ws = [(torch.randn(N, Kd, device=dev) * 0.02).bfloat16() for _ in range(copies)]
    us = [(torch.randn(N, Kd, device=dev) * 0.02).bfloat16() if a.dual else None for _ in range(copies)]
    if T > 256:
        ms = time_eager(lambda: K.linear(x, ws[0], out=out, w_up=us[0]), dev, iters=a.iters)
    else:
        ms = time_graph([(lambda w=w, u=u: K.linear(x, w, out=out, w_up=u)) for w, u in zip(ws, us)] * 2)
    flops = 2.0 * T * N * Kd * (2 if a.dual else 1)
    report(f"gemm T={T} N={N} K={Kd} dual={a.dual}", ms, flops, per + (T * Kd + T * N) * 2, pk)
    assert K.read_status() == 0


def bench_attn_prefill(a, dev, pk):
    Hq, Hkv, D, n = a.heads, a.kv_heads, 128, a.len
    pages = (n + 63) // 64 + 1
    kc = torch.randn(pages, Hkv, 64, D, device=dev).bfloat16()
    vc = torch.randn_like(kc)
    kc[0] = 0; vc[0] = 0
    table = torch.arange(1, pages, dtype=torch.int32, device=dev).view(1, -1).contiguous()
    q = torch.randn(n, Hq, D, device=dev).bfloat16()
    out = torch.empty_like(q)
    sl = torch.tensor([n], dtype=torch.int32, device=dev)
    qs = torch.tensor([0, n], dtype=torch.int32, device=dev)
    w = a.window
    ms = time_eager(lambda: K.attn_prefill(q, kc, vc, table, sl, qs, out, n, window=w), dev, iters=a.iters)
    # visible (query, key) pairs: the causal triangle, or the band of a sliding window
    pairs = n * n / 2 if not w or w >= n else n * w - w * w / 2
    report(f"attn_prefill len={n} Hq={Hq} Hkv={Hkv}" + (f" window={w}" if w else ""), ms, 4.0 * pairs * D * Hq,
           (2 * n * Hq * D + 2 * n * Hkv * D) * 2, pk)
    assert K.read_status() == 0


def bench_attn_decode(a, dev, pk):
    Hq, Hkv, D, S, n = a.heads, a.kv_heads, 128, a.seqs, a.len
    pps = (n + 63) // 64
    pages = S * pps + 1
    kcs = [torch.randn(pages, Hkv, 64, D, device=dev).bfloat16() for _ in range(2 if S >= 16 else 4)]
    table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
    q = torch.randn(S, Hq, D, device=dev).bfloat16()
    out = torch.empty_like(q)
    sl = torch.full((S,), n, dtype=torch.int32, device=dev)
    qs = torch.arange(S + 1, dtype=torch.int32, device=dev)
    splits = a.splits or K.attn_decode_splits(S, 1, Hkv, pps, a.window)
    scratch = torch.empty(K.attn_decode_scratch_floats(S, 1, Hq, Hkv, splits), dtype=torch.float32, device=dev)
    w = a.window
    seen = min(n, w) if w else n                                       # positions a row reads
    ms = time_graph([(lambda kc=kc: K.attn_decode(q, kc, kc, table, sl, qs, out, scratch, 1, splits, window=w)) for kc in kcs] * 3)
    report(f"attn_decode seqs={S} len={n} splits={splits}" + (f" window={w}" if w else ""), ms, 4.0 * S * seen * D * Hq,
           S * seen * Hkv * D * 2 * 2.0, pk)


def bench_moe(a, dev, pk):
    from ..parallel.moe_exchange import ExchangeGeometry, LocalExchange
    H, I, E, k = a.hidden, a.ffn, a.experts, a.top_k
    sets = []
    n_sets = 1 if E * 3 * H * I * 2 > 2e9 else 2
    for _ in range(n_sets):
        sets.append(tuple((torch.randn(E, r, c, device=dev) * 0.02).bfloat16() for r, c in ((I, H), (I, H), (H, I))))
    kw = dict(scoring=a.scoring, num_groups=a.groups, topk_groups=a.topk_groups)
    for T in [int(t) for t in a.tokens.split(",")]:
        ex = LocalExchange(ExchangeGeometry(H, I, E, k, T, 1), dev)
        x = torch.randn(T, H, device=dev).bfloat16()
        res = torch.randn(T, H, device=dev).bfloat16()
        logits = torch.randn(T, E, device=dev)
        out = torch.empty(T, H, dtype=torch.bfloat16, device=dev)
        fns = [(lambda s=s: ex.forward(x, logits, kw, s[0], s[1], s[2], out, residual=res)) for s in sets]
        if T <= 256:
            ms = time_graph(fns * 3)
        else:
            ms = time_eager(fns[0], dev, iters=a.iters)
        idx = ex.att.idx[:T]
        active = int(torch.unique(idx).numel())
        byts = active * 3 * H * I * 2 + T * k * H * 2 * 2 + T * k * I * 2 * 2 + T * k * H * 2 * 2
        report(f"moe T={T} H={H} I={I} E={E} k={k} active={active}", ms, 2.0 * T * k * 3 * H * I, byts, pk)
        assert K.read_status() == 0


def bench_mla(a, dev, pk):
    """Absorbed MLA attention: decode (one row per sequence) when --qlen 1, prefill / verify rows otherwise."""
    import math
    heads, S, n, ql = a.heads, a.seqs, a.len, a.qlen
    pps = (n + 63) // 64
    pages = S * pps + 1
    caches = [torch.randn(pages, 64, 576, device=dev).bfloat16() for _ in range(1 if pages * 64 * 576 * 2 > 150e6 else 3)]
    table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
    T = S * ql
    q = (torch.randn(T, heads, 576, device=dev) * 0.3).bfloat16()
    out = torch.empty(T, heads, 512, dtype=torch.bfloat16, device=dev)
    sl = torch.full((S,), n, dtype=torch.int32, device=dev)
    qs = torch.arange(S + 1, dtype=torch.int32, device=dev) * ql
    i32 = dict(dtype=torch.int32, device=dev)
    sparse = None
    if a.topk:
        base = torch.arange(a.topk, **i32) * max(1, n // a.topk)
        sparse = base[None, :].repeat(T, 1).contiguous()
        bs, bt = K.mla_blocks([ql] * S, 128)
    else:
        bs, bt = K.mla_blocks([ql] * S, heads)
    nb = len(bs)
    tiles = (a.topk or n) // 32
    splits = a.splits or max(1, min(K.num_sms() // max(1, nb * 2), max(1, tiles // 8), 32))
    scratch = torch.empty(K.mla_scratch_floats(nb, splits), dtype=torch.float32, device=dev) if splits > 1 else None
    bsd, btd = torch.tensor(bs, **i32), torch.tensor(bt, **i32)
    scale = 1.0 / math.sqrt(192)
    fns = [(lambda c=c: K.mla_attention(q, c, table, sl, qs, bsd, btd, out, scale, splits, scratch, sparse_idx=sparse)) for c in caches]
    ms = time_graph(fns * 3) if T <= 512 else time_eager(fns[0], dev, iters=a.iters)
    kv = a.topk or n
    avg_kv = kv if (ql == 1 or a.topk) else (n - ql / 2)
    flops = 2.0 * T * heads * avg_kv * (576 + 512)
    byts = (S * n if not a.topk else T * kv) * 576 * 2.0 + T * heads * (576 + 512) * 2.0
    report(f"mla seqs={S} len={n} qlen={ql} heads={heads} topk={a.topk} splits={splits}", ms, flops, byts, pk)
    assert K.read_status() == 0


def bench_mla_prefill_expanded(a, dev, pk):
    """MLA prefill in expanded form (per-head K_nope / V from kv_b, shared rope keys from the latent cache)."""
    import math
    heads, n = a.heads, a.len
    pages = (n + 63) // 64 + 1
    cache = torch.randn(pages, 64, 576, device=dev).bfloat16(); cache[0] = 0
    table = torch.arange(1, pages, dtype=torch.int32, device=dev).view(1, -1).contiguous()
    q = (torch.randn(n, heads * 192, device=dev) * 0.3).bfloat16()
    qr = (torch.randn(n, heads, 576, device=dev) * 0.3).bfloat16()
    rows = ((n + 63) // 64) * 64
    kx = (torch.randn(rows, heads * 128, device=dev) * 0.3).bfloat16(); vx = torch.randn_like(kx)
    out = torch.empty(n, heads, 128, dtype=torch.bfloat16, device=dev)
    i32 = dict(dtype=torch.int32, device=dev)
    sl, qs, z = torch.tensor([n], **i32), torch.tensor([0, n], **i32), torch.zeros(1, **i32)
    ms = time_eager(lambda: K.attn_prefill_mla(q, qr, kx, vx, z, cache, table, sl, qs, out, n, heads, 1.0 / math.sqrt(192)), dev, iters=a.iters)
    report(f"mla_prefill_expanded len={n} heads={heads}", ms, 2.0 * n * n / 2 * heads * (192 + 128), (n * heads * (192 + 128 + 256)) * 2.0, pk)
    assert K.read_status() == 0


def bench_w4(a, dev, pk):
    """4-bit weight GEMM at decode sizes against the bf16 kernel on the same logical weights."""
    from ..quant import codecs
    T, N, Kd = a.tokens, a.features, a.k
    x = torch.randn(T, Kd, device=dev).bfloat16()
    out = torch.empty(T, N, dtype=torch.bfloat16, device=dev)
    copies = max(2, min(16, int(300e6 // (N * Kd // 2)) + 1))
    g = torch.Generator().manual_seed(0)
    w = torch.randn(N, Kd, generator=g) * 0.05
    if a.fmt == "mxfp4":
        pq, sq = codecs.mxfp4_quant(w)
        ws = [(pq.to(dev).clone(), sq.to(dev).clone(), None) for _ in range(copies)]
    else:
        pq, sq, gq = codecs.nvfp4_quant(w)
        ws = [(pq.to(dev).clone(), sq.view(torch.uint8).to(dev).clone(), gq.to(dev)) for _ in range(copies)]
    ms = time_graph([(lambda w_=w_: K.linear_w4(x, w_, a.fmt, out=out)) for w_ in ws] * 2)
    per = N * Kd // 2 + N * Kd // (32 if a.fmt == "mxfp4" else 16)
    report(f"gemm_w4 {a.fmt} T={T} N={N} K={Kd}", ms, 2.0 * T * N * Kd, per + (T * Kd + T * N) * 2, pk)
    wb = [(torch.randn(N, Kd, device=dev) * 0.05).bfloat16() for _ in range(max(2, copies // 4))]
    ms_b = time_graph([(lambda w_=w_: K.linear(x, w_, out=out)) for w_ in wb] * 2)
    report(f"gemm bf16 twin T={T} N={N} K={Kd}", ms_b, 2.0 * T * N * Kd, N * Kd * 2 + (T * Kd + T * N) * 2, pk)
    assert K.read_status() == 0


def bench_exl3(a, dev, pk):
    """EXL3 trellis GEMM at decode sizes (Hadamard rotations + in-kernel trellis decode + tcgen05)."""
    from ..quant import codecs
    T, N, Kd, bits = a.tokens, a.features, a.k, a.bits
    x = torch.randn(T, Kd, device=dev).bfloat16()
    copies = max(2, min(16, int(300e6 // (N * Kd * bits // 8)) + 1))
    g = torch.Generator().manual_seed(0)
    ws = []
    for _ in range(copies):
        t, su, sv = codecs.exl3_random(Kd, N, bits, g)
        ws.append((t.to(dev), su.to(dev), sv.to(dev)))
    out = torch.empty(T, N, dtype=torch.bfloat16, device=dev)
    ms = time_graph([(lambda w=w: K.linear_exl3(x, w[0], w[1], w[2], out=out)) for w in ws] * 2)
    per = N * Kd * bits // 8 + (N + Kd) * 2
    report(f"gemm_exl3 k{bits} T={T} N={N} K={Kd}", ms, 2.0 * T * N * Kd, per + (T * Kd + T * N) * 2, pk)
    assert K.read_status() == 0


def bench_gemm_fp8(a, dev, pk):
    """Block-scaled E4M3 GEMM (128 x 128 weight scales, 1 x 128 activation scales)."""
    from ..quant import codecs
    T, N, Kd = a.tokens, a.features, a.k
    x = torch.randn(T, Kd, device=dev).bfloat16()
    xq = torch.empty(T, Kd, dtype=torch.float8_e4m3fn, device=dev)
    xs = torch.empty(T, Kd // 128, dtype=torch.float32, device=dev)
    K.quant_rows_fp8(x, xq, xs)
    copies = 1 if T > 256 else max(2, min(24, int(200e6 // (N * Kd)) + 1))
    ws = []
    for i in range(copies):
        q, sc = codecs.fp8_quant_block128(torch.randn(N, Kd, generator=torch.Generator().manual_seed(i)) * 0.05)
        ws.append((q.to(dev), sc.to(dev)))
    out = torch.empty(T, N, dtype=torch.bfloat16, device=dev)
    if T > 256:
        ms = time_eager(lambda: K.linear_fp8(xq, xs, ws[0][0], ws[0][1], out=out), dev, iters=a.iters)
    else:
        ms = time_graph([(lambda w=w: K.linear_fp8(xq, xs, w[0], w[1], out=out)) for w in ws] * 2)
    report(f"gemm_fp8 T={T} N={N} K={Kd}", ms, 2.0 * T * N * Kd, N * Kd + T * Kd + T * N * 2, pk)
    assert K.read_status() == 0


def bench_indexer(a, dev, pk):
    """Lightning indexer: scores of every cached position for each query token, then the radix top-k."""
    heads, S, n, topk = a.heads, a.seqs, a.len, a.topk
    pps = (n + 63) // 64
    pages = S * pps + 1
    kc = torch.randn(pages, 64, 128, device=dev).bfloat16()
    table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
    q = (torch.randn(S, heads, 128, device=dev) * 0.3).bfloat16()
    hw = torch.rand(S, heads, device=dev).bfloat16()
    sl = torch.full((S,), n, dtype=torch.int32, device=dev)
    qs = torch.arange(S + 1, dtype=torch.int32, device=dev)
    bs, bt = K.mla_blocks([1] * S, heads // 2)
    i32 = dict(dtype=torch.int32, device=dev)
    bsd, btd = torch.tensor(bs, **i32), torch.tensor(bt, **i32)
    ld = ((pps * 64 + 127) // 128) * 128
    scores = torch.empty(S, ld, dtype=torch.float32, device=dev)
    sel = torch.empty(S, topk, dtype=torch.int32, device=dev)
    splits = max(1, min(K.num_sms() // max(1, len(bs)), max(1, (pps + 1) // 4), 64))
    ms = time_graph([lambda: K.indexer_scores(q, kc, hw, table, sl, qs, bsd, btd, scores, splits, w_scale=heads ** -0.5)] * 6)
    report(f"indexer_scores seqs={S} len={n} heads={heads} splits={splits}", ms, 2.0 * S * heads * n * 128, S * n * 128 * 2.0, pk)
    ms2 = time_graph([lambda: K.index_topk(scores, topk, sel, seq_lens=sl, q_start=qs)] * 6)
    report(f"index_topk seqs={S} len={n} k={topk}", ms2, 0.0, S * n * 4.0, pk)
    assert K.read_status() == 0


def bench_sampler(a, dev, pk):
    from ..runtime.sampling import SamplingParams
    n, V = a.rows, a.vocab
    logits = torch.randn(n, V, device=dev) * 3
    params = [SamplingParams(temperature=0.8, top_k=a.top_k or None, top_p=a.top_p, seed=i) for i in range(n)]
    rows = K.pack_sample_rows(params, list(range(n))).to(dev)
    tok = torch.empty(n, dtype=torch.int32, device=dev); st = torch.empty(n, dtype=torch.int32, device=dev)
    ms = time_graph([lambda: K.sample_rows(logits, rows, tok, st)] * 8)
    report(f"sample_rows rows={n} V={V} top_k={a.top_k} top_p={a.top_p}", ms, 0.0, n * V * 4.0, pk)


def bench_hybrid(a, dev, pk) -> None:
    """The per-layer hybrids' own kernels beside the like kernels of the MLA decoder, at one of the benchmark sizes."""
    from ..config import KARUSUN_SIZES, DeltaSpec, LayerSpec, hybrid_config
    from ..models.hybrid import HybridCache, HybridWeights
    H, _, heads, _ = KARUSUN_SIZES[a.size]
    bf, T, k = torch.bfloat16, a.tokens, 6

    def i32(v):
        return torch.tensor(list(v), dtype=torch.int32, device=dev)

    def run(name, fn, nbytes, flops=0.0):
        report(name, time_eager(fn, dev, a.iters), flops, nbytes, pk)
    for n in (8, T):
        S = n if n == 8 else 1
        x, xo, y, h = torch.randn(n, H, device=dev), torch.empty(n, H, device=dev), torch.randn(n, H, device=dev, dtype=bf), torch.empty(n, H, device=dev, dtype=bf)
        w, c, st = torch.ones(H, device=dev, dtype=bf), (torch.randn(4, H, device=dev) * 0.1).to(bf), torch.zeros(2 + 2 * S, 3 * H, device=dev)
        kw = dict(x_in=x, w_b=w, x_out=xo, conv=c, state=st, state_in=i32(range(2, 2 + S)), state_out=i32(range(2 + S, 2 + 2 * S)),
                  q_start=i32(range(S + 1) if S > 1 else (0, n)))
        ys, idx = torch.randn(n * k, H, device=dev, dtype=bf), torch.randint(0, 64, (n, k), device=dev, dtype=torch.int32)
        sw = torch.rand(n, k, device=dev)
        own = S * 6 * H * 4 if S > 1 else 0
        run(f"norm_conv {n} rows", lambda: K.norm_conv(h, w, 4, 1e-5, y=y, **kw), n * H * 12 + own)
        run(f"norm_conv {n} rows, top-{k} routed sum", lambda: K.norm_conv(h, w, 4, 1e-5, y=ys, slots=(sw, idx, 56, y), **kw), n * H * (10 + 2 * k) + own)
        run(f"(MLA) rmsnorm {n} rows", lambda: K.rmsnorm(y, w, 1e-5, out=h), n * H * 4)
        run(f"(MLA) combine + norm {n} rows", lambda: K.moe_combine(ys, sw, h, residual=y, norm_w=w, eps=1e-5, x_out=ys[:n]), n * H * (6 + 2 * k))
    m = DeltaSpec(heads, heads // 2, 128, 128, 4)
    cfg = hybrid_config("bench", 128, H, [LayerSpec(m)], 4, 4, 1e-5)
    L = HybridWeights.random_init(cfg, dev).layers[0]
    n_in = L.w_in.shape[0]
    for B in (1, 8, 32):
        kv = HybridCache(cfg, 4, dev, 2 + 2 * B)
        p, out = torch.randn(B, n_in, device=dev, dtype=bf), torch.empty(B, heads, 128, device=dev, dtype=bf)
        args = (p, L.offs, m, L, kv.state, kv.offsets[0]["S"], kv.offsets[0]["conv"], i32(range(2, 2 + B)), i32(range(2 + B, 2 + 2 * B)), i32(range(B + 1)))
        run(f"delta_step {B} sequences x {heads} heads", lambda: K.delta_step(*args, out, None, 1e-5), B * heads * 128 * 128 * 8)
    kv = HybridCache(cfg, 4, dev, 4)
    p, out, raw = torch.randn(T, n_in, device=dev, dtype=bf), torch.empty(T, heads, 128, device=dev, dtype=bf), torch.empty(T * heads * 128, device=dev)
    scratch = torch.empty(128 << 20, dtype=torch.uint8, device=dev)
    args = (p, L.offs, m, L, kv.state, kv.offsets[0]["S"], kv.offsets[0]["conv"], i32([0]), i32([2]), i32([0, T]))
    macs = T / 64 * heads * 64 * (64 * 128 * 5 + 128 * 128 * 3)
    run(f"delta_chunked {T} tokens x {heads} heads", lambda: K.delta_chunked(scratch, *args, out, raw, 1e-5), T * n_in * 2 + T * heads * 256, 2 * macs)
    run(f"latent_gate {T} rows", lambda: K.latent_gate(out, p, 0, heads, 128), T * heads * 128 * 6)


def bench_parallel(a, dev, pk) -> None:
    """The kernels of parallel layers with differential attention beside the like kernels of the dense GQA decoder, at one of the
    benchmark sizes."""
    from ..config import GUBERAX_SIZES, guberax_bench
    from ..models.hybrid import rope_frequencies
    H, _, heads, kvh, ffn = GUBERAX_SIZES[a.size]
    cfg, bf, T = guberax_bench(a.size), torch.bfloat16, a.tokens
    m = cfg.layer_specs[0].mixer
    w = m.window
    freq = rope_frequencies(m.rope).to(dev)

    def i32(v):
        return torch.tensor(list(v), dtype=torch.int32, device=dev)

    def run(name, fn, nbytes, flops=0.0):
        report(name, time_eager(fn, dev, a.iters), flops, nbytes, pk)
    diff = dict(scale=m.scale, window=w, keep=m.keep_first, maps=2, lam=0.5, out_scale=0.5, eps=1e-6)
    for n in (1, 8, 32, T):
        S = n if n < T else 1
        x, xo, y, h = torch.randn(n, H, device=dev), torch.empty(n, H, device=dev), torch.randn(n, H, device=dev, dtype=bf), torch.empty(n, H, device=dev, dtype=bf)
        wt = torch.zeros(H, device=dev, dtype=bf)
        run(f"norm_conv, plain add, {n} rows", lambda: K.norm_conv(h, wt, 1, 1e-6, x_in=x, y=y, x_out=xo, w_offset=1.0), n * H * 12)
        run(f"(GQA) rmsnorm {n} rows", lambda: K.rmsnorm(y, wt, 1e-6, out=h), n * H * 4)
        C = m.conv_channels
        ctx = T
        pps = (ctx + 63) // 64
        kc, vc = (torch.randn(S * pps + 1, kvh, 64, 128, device=dev, dtype=bf) for _ in range(2))
        table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
        a_ = torch.randn(n, C, device=dev, dtype=bf)
        offs = dict(q=0, k=m.q_channels, v=m.q_channels + m.k_channels)
        pos = i32([ctx - 1] * S) if n < T else i32(range(T))
        slots = (table[:, -1] * 64 + 63).int() if n < T else i32(range(64, 64 + T))
        cw, st = torch.randn(m.conv, C, device=dev), torch.zeros(2 + 2 * S, 3 * C, device=dev)
        tab, q = torch.empty(n, 32, 2, device=dev), torch.randn(n, heads, 128, device=dev, dtype=bf)
        K.rope_table(pos, freq, tab)
        qs, sl = (i32(range(S + 1)), i32([ctx] * S)) if n < T else (i32([0, T]), i32([T]))
        si, so = i32(range(2, 2 + S)), i32(range(2 + S, 2 + 2 * S))
        run(f"conv_rope_kv {n} rows", lambda: K.conv_rope_kv(a_, offs, m, cw, tab, slots, q, kc, vc, state=st, state_in=si, state_out=so, q_start=qs),
            n * C * 4 + S * C * 24)
        f64 = torch.ones(64, device=dev)
        run(f"(GQA) qk_rope_kv {n} rows", lambda: K.qk_rope_kv(a_, None, None, f64, pos, slots, q, kc, vc, heads, kvh, 128, 1e-6, False), n * C * 4)
        out, wide = torch.empty(n, heads, 128, device=dev, dtype=bf), torch.empty(n, heads * 128 + ffn, device=dev, dtype=bf)
        if n == T:
            pairs = T * w - w * w / 2 + max(0, T - w - m.keep_first) * m.keep_first
            run(f"attn_prefill, two maps, {T} tokens, window {w} + {m.keep_first}", lambda: K.attn_prefill(q, kc, vc, table, sl, qs, wide, T, **diff),
                T * C * 4, pairs * heads * 2 * (2 * 64 + 2 * 128))
            pairs = T * w - w * w / 2
            run(f"(GQA) attn_prefill {T} tokens, window {w}", lambda: K.attn_prefill(q, kc, vc, table, sl, qs, out, T, window=w), T * C * 4, pairs * heads * 4 * 128)
            logits = torch.randn(32, cfg.vocab_size, device=dev)
            run("softcap 32 rows", lambda: K.softcap(logits, 30.0), logits.numel() * 8)
            run(f"rope_table {T} rows", lambda: K.rope_table(pos, freq, tab), T * 32 * 8)
        else:
            for tag, kw, keep, hm in ((", two maps", diff, m.keep_first, 2), ("(GQA) ", dict(window=w), 0, 1)):
                sp = K.attn_decode_splits(S, 1, kvh, pps, w, keep)
                sc = torch.empty(K.attn_decode_scratch_floats(S, 1, hm * heads, kvh, sp), device=dev)
                o = wide if hm == 2 else out
                run((tag + "attn_decode" if hm == 1 else "attn_decode" + tag) + f", {S} x {ctx}, window {w} + {keep}, {sp} splits",
                    lambda: K.attn_decode(q, kc, vc, table, sl, qs, o, sc, 1, sp, **kw), S * (w + keep) * kvh * 512)
        g, u, wo = (torch.randn(r, c, device=dev, dtype=bf) * 0.02 for r, c in ((ffn, H), (ffn, H), (H, heads * 128 + ffn)))
        flop = 2.0 * n * H
        run(f"gate / up product {n} rows", lambda: K.linear(h, g, out=wide[:, heads * 128:], w_up=u), 4 * ffn * H + n * (H + ffn) * 2, flop * 2 * ffn)
        run(f"[o | down] product {n} rows", lambda: K.linear(wide, wo, out=y), 2 * wo.numel() + n * (H + wo.shape[1]) * 2, flop * wo.shape[1])
        o1, d1 = wo[:, :heads * 128].contiguous(), wo[:, heads * 128:].contiguous()
        on, dn = out.view(n, -1), torch.randn(n, ffn, device=dev, dtype=bf)
        run(f"(GQA) o product + residual {n} rows", lambda: K.linear(on, o1, out=y, residual=y), 2 * o1.numel() + n * (2 * H + heads * 128) * 2, flop * heads * 128)
        run(f"(GQA) down product + residual {n} rows", lambda: K.linear(dn, d1, out=y, residual=y), 2 * d1.numel() + n * (2 * H + ffn) * 2, flop * ffn)
    assert K.read_status() == 0


def bench_two_norm(a, dev, pk) -> None:
    """The kernels of two-norm parallel layers (norms over heads or projections, values out of keys, sinks, head gates, scaled latent
    rotation, joined passes) beside the like kernels of the GQA + MoE and MLA decoders, at one of the benchmark sizes."""
    from ..config import ROFAPEL_SIZES, rofapel_bench
    from ..models.hybrid import rope_frequencies
    H, _, heads, kvh, ffn = ROFAPEL_SIZES[a.size]
    cfg, bf, T, top, E = rofapel_bench(a.size), torch.bfloat16, a.tokens, 6, 64
    lat, win, att = (s.mixer for s in cfg.layer_specs[:3])

    def i32(v):
        return torch.tensor(list(v), dtype=torch.int32, device=dev)

    def rand(*s):
        return torch.randn(*s, device=dev, dtype=bf)

    def run(name, fn, nbytes, flops=0.0):
        report(name, time_eager(fn, dev, a.iters), flops, nbytes, pk)
    w = torch.zeros(H, device=dev, dtype=bf)
    for n in (1, 8, 32, T):
        S = n if n < T else 1
        x, xo, y, yo, h, h2, ys = torch.randn(n, H, device=dev), torch.empty(n, H, device=dev), *(rand(n, H) for _ in range(4)), rand(n * top, H)
        idx, sw = torch.randint(0, E, (n, top), device=dev, dtype=torch.int32), torch.rand(n, top, device=dev)
        run(f"norm_conv, two outputs, routed + plain rows, {n} rows",
            lambda: K.norm_conv(h, w, 1, 1e-5, x_in=x, y=ys, base=y, slots=(sw, idx, E, h2), x_out=xo, w_offset=1.0, w2=w, h2_out=h2), n * H * (14 + 2 * top))
        run(f"(GQA) combine + norm {n} rows", lambda: K.moe_combine(ys, sw, h, shared=y, residual=h2, norm_w=w, eps=1e-5, x_out=yo), n * H * (8 + 2 * top))
        both, wj = rand(n, 2 * H), rand(H, 2 * H)
        run(f"norm_conv, rows of a join, {n} rows", lambda: K.norm_conv(both, None, 1, 1e-5, x_in=x, y=ys, base=y, slots=(sw, idx, E, h2)), n * H * (8 + 2 * top))
        run(f"join product, fp32 out, {n} rows", lambda: K.linear(both, wj, out=xo, out_f32=True), 4 * H * H + n * H * 8, 4.0 * n * H * H)
        run(f"(GQA) a product of the same size {n} rows", lambda: K.linear(both, wj, out=h), 4 * H * H + n * H * 6, 4.0 * n * H * H)
        rw, rb, z = rand(E, H), torch.zeros(E, device=dev), torch.empty(n, E, device=dev)
        i_, w_ = torch.empty(n, top, dtype=torch.int32, device=dev), torch.empty(n, top, device=dev)
        for tag, kw in (("", dict(scoring="softmax_bias", bias=rb)), ("(GQA) ", dict(scoring="softmax"))):
            if n <= 64:
                run(f"{tag}norm_route {n} rows", lambda: K.norm_route(h, None, 0.0, rw, None, i_, w_, top, **kw), E * H * 2 + n * H * 2)
            else:
                run(f"{tag}route_topk {n} rows", lambda: K.route_topk(z, top, out_idx=i_, out_w=w_, **kw), n * E * 4 + n * top * 8)
        ctx, pps = T, (T + 63) // 64
        kc, vc = rand(S * pps + 1, kvh, 64, 128), rand(S * pps + 1, kvh, 64, 128)
        table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
        pos = i32([ctx - 1] * S) if n < T else i32(range(T))
        slots = (table[:, -1] * 64 + 63).int() if n < T else i32(range(64, 64 + T))
        qs, sl = (i32(range(S + 1)), i32([ctx] * S)) if n < T else (i32([0, T]), i32([T]))
        q, gate = rand(n, heads, 128), rand(n, heads + 8)[:, :heads]
        n1, f64, tab = torch.ones(heads * 128, device=dev), torch.ones(64, device=dev), torch.empty(n, 64, 2, device=dev)
        nb = torch.ones(128, device=dev, dtype=bf)
        si, so, st = i32(range(2, 2 + S)), i32(range(2 + S, 2 + 2 * S)), torch.zeros(2 + 2 * S, 3 * win.conv_channels, device=dev)
        C = att.conv_channels
        proj = rand(n, C + 8 * (1 + heads // 8))
        for tag, m in (("norms per head, convolution, values out of keys", win), ("norms over the projection", att)):
            offs = dict(q=0, k=m.q_channels, v=m.q_channels + m.k_channels)
            K.rope_table(pos, rope_frequencies(m.rope).to(dev), tab.view(-1)[:n * m.rope.dims])
            cw = torch.randn(m.conv, m.conv_channels, device=dev) if m.conv else None
            nq, nk = (n1[:128], n1[:128]) if m.qk_norm == "head" else (n1, n1[:m.k_channels])
            run(f"conv_norm_rope_kv, {tag}, {n} rows",
                lambda: K.conv_rope_kv(proj, offs, m, cw, tab, slots, q, kc, vc, state=st, state_in=si, state_out=so, q_start=qs, q_norm=nq, k_norm=nk, eps=1e-5),
                n * (m.conv_channels + C) * 2 + (S * m.conv_channels * 24 if m.conv else 0))
        qkv = rand(n, C)
        run(f"(GQA) qk_rope_kv with norms {n} rows", lambda: K.qk_rope_kv(qkv, nb, nb, f64, pos, slots, q, kc, vc, heads, kvh, 128, 1e-5, False), n * C * 4)
        out, wide = rand(n, heads, 128), rand(n, heads * 128 + ffn)
        sink = torch.zeros(heads, device=dev)
        for tag, kw, o in (("sinks and gates, ", dict(sink=sink, gate=gate), wide), ("(GQA) ", {}, out)):
            for wn in (win.window, 0):
                if n == T:
                    pairs = T * wn - wn * wn / 2 if wn else T * T / 2
                    run(f"attn_prefill, {tag}{T} tokens, window {wn}", lambda: K.attn_prefill(q, kc, vc, table, sl, qs, o, T, window=wn, **kw), T * C * 4, pairs * heads * 512)
                else:
                    sp = K.attn_decode_splits(S, 1, kvh, pps, wn)
                    sc = torch.empty(K.attn_decode_scratch_floats(S, 1, heads, kvh, sp), device=dev)
                    run(f"attn_decode, {tag}{S} x {ctx}, window {wn}, {sp} splits", lambda: K.attn_decode(q, kc, vc, table, sl, qs, o, sc, 1, sp, window=wn, **kw),
                        S * (wn or ctx) * kvh * 512)
        if n < T:
            continue
        rec, kn, knb, fl = 576, torch.ones(512, device=dev), torch.ones(512, device=dev, dtype=bf), torch.ones(32, device=dev)
        la, lq, lc, cache, qa = rand(n, heads * 192 + rec), rand(n, heads * 192), rand(n, rec), rand(S * pps + 1, 64, rec), rand(n, heads, rec)
        lo, slab, kx, vx, z0 = rand(n, 512), rand(heads, n, 128), rand(n, heads * 128), rand(n, heads * 128), i32([0])
        run(f"latent_prep {n} rows", lambda: K.latent_prep(la, 0, heads * 192, heads, 128, 64, kn, fl, pos, slots, cache, None, qa, 1e-5, lat_out=lo, halves=False,
                                                           magnitude=1.2), n * (rec * 4 + 1024 + heads * 256))
        run(f"(MLA) mla_prep_a {n} rows", lambda: K.mla_prep_a(lc, 0, None, knb, fl, pos, slots, None, cache, 1e-5, True, lat_out=lo), n * (rec * 4 + 1024))
        run(f"(MLA) mla_q_split {n} rows", lambda: K.mla_q_split(lq, fl, pos, slab, qa, heads, True), n * heads * 192 * 4)
        for tag, o in (("into longer rows, ", wide), ("(MLA) ", out)):
            run(f"attn_prefill_mla, {tag}{n} tokens", lambda: K.attn_prefill_mla(lq, qa, kx, vx, z0, cache, table, sl, qs, o, n, heads, lat.scale),
                n * heads * 192 * 4, n * n / 2 * heads * 2 * 320)
    assert K.read_status() == 0


def bench_post_norm(a, dev, pk) -> None:
    """The kernels of layers normed after their sublayers (averages over depth, gated linear recurrences, attention with capped scores and
    turned values beside linear attention) beside the like kernels of the GQA + MoE decoder and of the delta-rule hybrid, at one of the
    benchmark sizes."""
    from ..config import BUZARAX_SIZES, DeltaSpec, LayerSpec, buzarax_bench, hybrid_config, scaled_down
    from ..models.hybrid import HybridCache, HybridEngine, HybridWeights, pad8, rope_frequencies
    H, layers, heads, kvh, ffn = BUZARAX_SIZES[a.size]
    cfg, bf, T, top, E = buzarax_bench(a.size), torch.bfloat16, a.tokens, 6, 64
    att, lin, rec = cfg.layer_specs[0].mixer.left, cfg.layer_specs[0].mixer.right, cfg.layer_specs[1].mixer

    def i32(v):
        return torch.tensor(list(v), dtype=torch.int32, device=dev)

    def rand(*s):
        return torch.randn(*s, device=dev, dtype=bf)

    def run(name, fn, nbytes, flops=0.0):
        report(name, time_eager(fn, dev, a.iters), flops, nbytes, pk)
    small = scaled_down(cfg, 2, 128)
    W = HybridWeights.random_init(small, dev)
    L0, L1 = W.layers
    delta = DeltaSpec(heads, heads // 2, 128, 128, 4)
    dcfg = hybrid_config("bench", 128, H, [LayerSpec(delta)], 4, 4, 1e-5)
    Ld = HybridWeights.random_init(dcfg, dev).layers[0]
    w = torch.ones(H, device=dev, dtype=bf)
    for n in (1, 8, 32, T):
        S = n if n < T else 1
        x, xo, y, yo, h, ys = torch.randn(n, H, device=dev), torch.empty(n, H, device=dev), *(rand(n, H) for _ in range(3)), rand(n * top, H)
        idx, sw = torch.randint(0, E, (n, top), device=dev, dtype=torch.int32), torch.rand(n, top, device=dev)
        half = layers // 2
        past, pw = torch.randn(half + 1, n, H, device=dev), torch.rand(half + 1, device=dev)
        run(f"norm_conv, norm of the sublayer, {n} rows", lambda: K.norm_conv(h, None, 1, 1e-5, x_in=x, y=y, w_b=w, x_out=xo), n * H * 12)
        run(f"(GQA) rmsnorm {n} rows", lambda: K.rmsnorm(y, w, 1e-5, out=h), n * H * 4)
        run(f"norm_conv, routed rows, average over {half} + 1 results, {n} rows",
            lambda: K.norm_conv(h, None, 1, 1e-5, x_in=x, y=ys, slots=(sw, idx, E, y), w_b=w, x_out=xo, past=(past[:half], pw, past[half])),
            n * H * (14 + 2 * top + 4 * half))
        run(f"(GQA) combine + norm {n} rows", lambda: K.moe_combine(ys, sw, h, residual=y, norm_w=w, eps=1e-5, x_out=yo), n * H * (6 + 2 * top))
        ctx, pps = T, (T + 63) // 64
        kc, vc = rand(S * pps + 1, kvh, 64, 128), rand(S * pps + 1, kvh, 64, 128)
        table = (torch.arange(S * pps, dtype=torch.int32, device=dev) + 1).view(S, pps).contiguous()
        pos = i32([ctx - 1] * S) if n < T else i32(range(T))
        slots = (table[:, -1] * 64 + 63).int() if n < T else i32(range(64, 64 + T))
        qs, sl = (i32(range(S + 1)), i32([ctx] * S)) if n < T else (i32([0, T]), i32([T]))
        si, so = i32(range(2, 2 + S)), i32(range(2 + S, 2 + 2 * S))
        q, tab, vtab = rand(n, heads, 128), torch.empty(n, att.rope.dims // 2, 2, device=dev), torch.empty(n, 64, 2, device=dev)
        K.rope_table(pos, rope_frequencies(att.rope).to(dev), tab, att.rope.magnitude)
        K.rope_table(pos, rope_frequencies(att.v_rope).to(dev), vtab)
        proj = rand(n, L0.w_in.shape[0])
        C = att.conv_channels
        run(f"conv_norm_rope_kv, norms after rotation, turned values, {n} rows",
            lambda: K.conv_rope_kv(proj, L0.offs, att, None, tab, slots, q, kc, vc, eps=1e-5, v_table=vtab), n * C * 4)
        nb, f64, qkv = torch.ones(128, device=dev, dtype=bf), torch.ones(64, device=dev), rand(n, C)
        run(f"(GQA) qk_rope_kv with norms {n} rows", lambda: K.qk_rope_kv(qkv, nb, nb, f64, pos, slots, q, kc, vc, heads, kvh, 128, 1e-5, False), n * C * 4)
        out, wide = rand(n, heads, 128), rand(n, L0.w_out.shape[1])
        kw = dict(scale=att.scale, sink=torch.zeros(heads, device=dev), cap=att.softcap, v_table=vtab, out_scale=0.8)
        qn = torch.nn.functional.rms_norm(q.float(), (128,)).to(bf)
        for tag, k2, o in (("capped, turned, ", kw, wide), ("(GQA) ", {}, out)):
            if n == T:
                run(f"attn_prefill, {tag}{T} tokens", lambda: K.attn_prefill(qn, kc, vc, table, sl, qs, o, T, **k2), T * C * 4, T * T / 2 * heads * 512)
            else:
                sp = K.attn_decode_splits(S, 1, kvh, pps)
                sc = torch.empty(K.attn_decode_scratch_floats(S, 1, heads, kvh, sp), device=dev)
                run(f"attn_decode, {tag}{S} x {ctx}, {sp} splits", lambda: K.attn_decode(qn, kc, vc, table, sl, qs, o, sc, 1, sp, **k2), S * ctx * kvh * 512)
        eng = HybridEngine(small, W, HybridCache(small, 4, dev, 2 + 2 * S), max_tokens=n, max_seqs=S)
        off, act = eng.kv.offsets, wide[:, heads * pad8(128):]
        args = (proj, {k: L0.offs["right." + k] for k in "qkvg"}, lin, L0, eng.kv.state, off[0]["S"], si, so, qs, eng.ws.raw, act, 128, 1e-5)
        dproj, dout = rand(n, Ld.w_in.shape[0]), torch.empty(n, heads, 128, device=dev, dtype=bf)
        dkv = HybridCache(dcfg, 4, dev, 2 + 2 * S)
        dargs = (dproj, Ld.offs, delta, Ld, dkv.state, dkv.offsets[0]["S"], dkv.offsets[0]["conv"], si, so, qs)
        rproj, rw = rand(n, L1.w_in.shape[0]), eng._rglru[rec]
        state_bytes = heads * 128 * 128 * 8
        if n < T:
            run(f"linear attention + norm, {S} sequences x {heads} heads", lambda: K.lightning_step(*args), S * state_bytes + n * heads * 128 * 10)
            run(f"(delta) delta_step {S} sequences x {heads} heads", lambda: K.delta_step(*dargs, dout, None, 1e-5), S * state_bytes + n * heads * 128 * 8)
        else:
            sc = torch.empty(K.lightning_scratch_bytes(lin, T, 1), dtype=torch.uint8, device=dev)
            flops = 2.0 * T * heads * (2 * 128 * 128 + 2 * 64 * 128)
            run(f"linear attention in chunks + norm, {T} tokens x {heads} heads", lambda: K.lightning_chunked(*args, sc), T * heads * 128 * 10, flops)
            raw, scd = torch.empty(T * heads * 128, device=dev), torch.empty(128 << 20, dtype=torch.uint8, device=dev)
            run(f"(delta) delta_chunked {T} tokens x {heads} heads", lambda: K.delta_chunked(scd, *dargs, dout, raw, 1e-5), T * heads * 128 * 8,
                2.0 * T * heads * (64 * 128 * 5 + 128 * 128 * 3))
            del raw, scd, sc
        from ..models.mla_moe import _HeadTiles
        ht = _HeadTiles(n, rec.blocks, dev)
        u = rw.u[:rec.blocks * ht.t_pad * 128].view(rec.blocks, ht.t_pad, 128)
        gates = rw.gates[:rec.blocks * ht.t_pad * 256].view(rec.blocks, ht.t_pad, 256)
        rargs = (rproj, L1.offs, rec, L1, u, gates, eng.kv.state, off[1]["S"], off[1]["conv"], si, so, qs, rw.out[:n], T if n == T else 1)
        gate_w = rec.width * 128 * 4
        if K.rglru_step_ok(rec, bf, n):
            run(f"recurrence in one launch, {n} rows", lambda: K.rglru_step(*rargs), gate_w + S * rec.width * 32 + n * rec.width * 6)
        run(f"recurrence: convolution {n} rows", lambda: K.rglru_conv(*rargs), n * rec.width * 4)
        run(f"recurrence: products of the gates {n} rows", lambda: K.grouped_linear(u.view(-1, 128), L1.w_gates, gates.view(-1, 256), ht.tile_expert, ht.tile_row0,
                                                                                    ht.num_tiles, ht.max_tiles, ht.tile_rows, split_k=False),
            gate_w + n * rec.width * 10, 2.0 * n * rec.width * 256)
        run(f"recurrence: scan {n} rows", lambda: K.rglru_scan(*rargs), n * rec.width * 14)
        del eng
        z, i_, w_ = torch.empty(n, E, device=dev), torch.empty(n, top, dtype=torch.int32, device=dev), torch.empty(n, top, device=dev)
        rwt, rb = rand(E, H), torch.zeros(E, device=dev)
        for tag, k2 in (("sigmoid ", dict(scoring="sigmoid", bias=rb, normalize=False)), ("(GQA) ", dict(scoring="softmax"))):
            if n <= 64:
                run(f"{tag}norm_route {n} rows", lambda: K.norm_route(h, None, 0.0, rwt, None, i_, w_, top, **k2), E * H * 2 + n * H * 2)
            else:
                run(f"{tag}route_topk {n} rows", lambda: K.route_topk(z, top, out_idx=i_, out_w=w_, **k2), n * E * 4 + n * top * 8)
        F = 6 * ffn
        o = rand(n, F)
        for tag, k2 in (("clipped ", dict(glu=(7.0, 1.702, 1.0))), ("(GQA) ", {})):
            run(f"{tag}gate / up product {n} rows", lambda: K.linear(h, L0.d_gate, out=o, w_up=L0.d_up, **k2), 4 * F * H + n * (H + F) * 2, 4.0 * n * H * F)
    assert K.read_status() == 0


def main() -> None:
    ap = argparse.ArgumentParser()
    sub = ap.add_subparsers(dest="cmd", required=True)
    ex = sub.add_parser("exl3")
    ex.add_argument("--tokens", type=int, default=8); ex.add_argument("--features", type=int, default=7168)
    ex.add_argument("--k", type=int, default=2048); ex.add_argument("--bits", type=int, default=4)
    f8 = sub.add_parser("gemm-fp8")
    f8.add_argument("--tokens", type=int, default=8); f8.add_argument("--features", type=int, default=7168)
    f8.add_argument("--k", type=int, default=2048); f8.add_argument("--iters", type=int, default=10)
    ix = sub.add_parser("indexer")
    ix.add_argument("--seqs", type=int, default=8); ix.add_argument("--len", type=int, default=32768)
    ix.add_argument("--heads", type=int, default=64); ix.add_argument("--topk", type=int, default=2048)
    g = sub.add_parser("gemm")
    g.add_argument("--tokens", type=int, default=8192); g.add_argument("--features", type=int, default=5120)
    g.add_argument("--k", type=int, default=2048); g.add_argument("--dual", action="store_true")
    p = sub.add_parser("attn-prefill")
    p.add_argument("--len", type=int, default=8192); p.add_argument("--heads", type=int, default=32)
    p.add_argument("--kv-heads", type=int, default=4); p.add_argument("--window", type=int, default=0, help="sliding window in tokens (0 = none)")
    d = sub.add_parser("attn-decode")
    d.add_argument("--seqs", type=int, default=32); d.add_argument("--len", type=int, default=8192)
    d.add_argument("--heads", type=int, default=32); d.add_argument("--kv-heads", type=int, default=4)
    d.add_argument("--splits", type=int, default=0); d.add_argument("--window", type=int, default=0, help="sliding window in tokens (0 = none)")
    m = sub.add_parser("moe")
    m.add_argument("--tokens", default="1,16,128,1024,8192"); m.add_argument("--hidden", type=int, default=2048)
    m.add_argument("--ffn", type=int, default=768); m.add_argument("--experts", type=int, default=128)
    m.add_argument("--top-k", type=int, default=8); m.add_argument("--scoring", default="softmax")
    m.add_argument("--groups", type=int, default=1); m.add_argument("--topk-groups", type=int, default=1)
    ml = sub.add_parser("mla")
    ml.add_argument("--seqs", type=int, default=8); ml.add_argument("--len", type=int, default=8192)
    ml.add_argument("--qlen", type=int, default=1); ml.add_argument("--heads", type=int, default=128)
    ml.add_argument("--topk", type=int, default=0); ml.add_argument("--splits", type=int, default=0)
    mp_ = sub.add_parser("mla-prefill")
    mp_.add_argument("--len", type=int, default=8192); mp_.add_argument("--heads", type=int, default=128)
    w4 = sub.add_parser("w4")
    w4.add_argument("--tokens", type=int, default=8); w4.add_argument("--features", type=int, default=7168)
    w4.add_argument("--k", type=int, default=2048); w4.add_argument("--fmt", default="mxfp4")
    sm = sub.add_parser("sampler")
    sm.add_argument("--rows", type=int, default=32); sm.add_argument("--vocab", type=int, default=151936)
    sm.add_argument("--top-k", type=int, default=50); sm.add_argument("--top-p", type=float, default=0.9)
    hy = sub.add_parser("hybrid")
    hy.add_argument("--size", default="base", choices=["small", "base", "large"]); hy.add_argument("--tokens", type=int, default=8192)
    pa = sub.add_parser("parallel")
    pa.add_argument("--size", default="base", choices=["small", "base", "large"]); pa.add_argument("--tokens", type=int, default=8192)
    tn = sub.add_parser("two-norm")
    tn.add_argument("--size", default="base", choices=["small", "base", "large"]); tn.add_argument("--tokens", type=int, default=8192)
    pn = sub.add_parser("post-norm")
    pn.add_argument("--size", default="base", choices=["small", "base", "large"]); pn.add_argument("--tokens", type=int, default=8192)
    for s in (g, p, d, m, ml, mp_, w4, sm, hy, pa, tn, pn):
        s.add_argument("--iters", type=int, default=10)
    a = ap.parse_args()
    dev = torch.device("cuda", int(os.environ.get("LOCAL_RANK", "0")))
    torch.cuda.set_device(dev)
    pk = peaks()
    {"exl3": bench_exl3, "gemm-fp8": bench_gemm_fp8, "indexer": bench_indexer, "gemm": bench_gemm, "attn-prefill": bench_attn_prefill, "attn-decode": bench_attn_decode, "moe": bench_moe,
     "mla": bench_mla, "mla-prefill": bench_mla_prefill_expanded, "w4": bench_w4, "sampler": bench_sampler, "hybrid": bench_hybrid,
     "parallel": bench_parallel, "two-norm": bench_two_norm, "post-norm": bench_post_norm}[a.cmd](a, dev, pk)


if __name__ == "__main__":
    main()
