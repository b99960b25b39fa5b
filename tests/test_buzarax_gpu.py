"""Kernels of the layers normed after their sublayers on the GPU against the plain oracle, one mechanism at a time (the engine is with the
other per-layer designs in test_guberax_gpu.py, greedy generation through the scheduler in test_hybrid_gpu.py)."""
import dataclasses
from types import SimpleNamespace

import pytest
import torch

from cuteafd_b200.config import RglruSpec, RopeSpec
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import averaged_config, dual_config, err, fading, oracle_logits, params, tokens, turned
from tests.test_guberax_gpu import _pages
from tests.test_hybrid_gpu import DTYPES, SPREAD, backend, close, dev, i32, rnd, run_cut

pytestmark = pytest.mark.gpu


def pad8(n):
    return -(-n // 8) * 8


def starts(lens):
    out = [0]
    for n in lens:
        out.append(out[-1] + n)
    return out


# ---- between sublayers -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,n", [(5, 104, 1), (5, 90, 4), (70, 2048, 9), (300, 1536, 3), (900, 4096, 6), (3, 4608, 25), (20, 8192, 2), (400, 90, 5), (300, 100, 7)])
@pytest.mark.parametrize("slots", [False, True])
def test_average_over_depth(dtype, T, H, n, slots):
    """A sublayer's output added under its norm (one number for all channels), kept for later, then averaged with earlier results; rows as
    they leave are the sum itself."""
    from cuteafd_b200.ops import kernels as K
    Hp, top, E = pad8(H), 3, 5
    x, past = rnd(T, H, seed=1), torch.stack([rnd(T, H, seed=20 + j) for j in range(n)])
    w = rnd(n + 1, seed=3)
    wb = torch.full((H,), 0.75)
    pad = lambda v: torch.nn.functional.pad(v, (0, Hp - H)).to(dev(), dtype)    # noqa: E731
    kw, y = {}, rnd(T, H, seed=2, dtype=dtype)
    if slots:
        g = torch.Generator().manual_seed(4)
        idx, wt, ex = torch.randint(0, E, (T, top), generator=g), torch.rand(T, top, generator=g), rnd(T * top, H, seed=5, dtype=dtype)
        y = (wt[..., None] * ex.view(T, top, H)).sum(1)
        kw = dict(y=pad(ex), slots=(wt.to(dev()), i32(idx.tolist()), E, pad(ex[:T])))
    else:
        kw = dict(y=pad(y))
    buf = torch.full((n + 1, T + 3, H), 7.0, device=dev())                      # rows of a longer buffer
    buf[:n, :T] = past.to(dev())
    h, xo = torch.full((T, Hp), 9.0, dtype=dtype, device=dev()), torch.empty(T, H, device=dev())
    kw.update(x_in=x.to(dev()), w_b=wb.to(dev(), dtype))
    K.norm_conv(h, None, 1, 1e-5, x_out=xo, past=(buf[:n], w.to(dev()), buf[n, :T]), **kw)
    mine = x + R.rms(y, 1e-5) * 0.75
    want = R.depth_average(w, [*past, mine])
    close(buf[n, :T], mine, torch.float32)
    close(xo, want, torch.float32)
    close(h[:, :H], want, dtype)
    assert (h[:, H:] == 9.0).all() and (buf[:, T:] == 7.0).all()
    rows = [T - 1, 0, T // 2]                                                   # the output's norm over picked rows
    hf = torch.empty(3, Hp, dtype=dtype, device=dev())[:, :H]
    K.norm_conv(hf, wb.to(dev(), dtype), 1, 1e-5, rows=i32(rows), past=(buf[:n], w.to(dev()), None), **kw)
    close(hf, R.rms(want[rows], 1e-5) * 0.75, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bigram", [(53, 11, 3), (1, 3, 1), (65521, 1000003, 7919)], ids=str)
def test_bigram_rows(dtype, bigram):
    """Portions of three sequences over three steps, the token before a portion coming from its slot; products past 32 bits; then both
    tables' rows added."""
    from cuteafd_b200.ops import kernels as K
    vocab, H = 70000, 40
    seqs = [tokens(40, vocab, 1), [0] * 20, tokens(3, vocab, 2)]
    cuts = [[7, 1, 2], [1, 18, 1], [32, 1]]
    state = torch.full((10, 64), 3.0, device=dev())
    state[0] = 0
    emb, table = rnd(vocab, H, seed=1, dtype=dtype).to(dev(), dtype), rnd(bigram[0] + 1, H, seed=2, dtype=dtype).to(dev(), dtype)
    at, slots = [0, 0, 0], [0, 0, 0]
    for step, lens in enumerate(cuts):
        parts = [s[o:o + n] for s, o, n in zip(seqs, at, lens)]
        want = sum((R.bigram_rows(p, seqs[i][at[i] - 1] if at[i] else -1, *bigram) for i, p in enumerate(parts)), [])
        T, outs = len(want), [2 + 3 * (step & 1) + i for i in range(len(lens))]
        toks, rows = i32(sum(parts, [])), torch.empty(T, dtype=torch.int32, device=dev())
        K.bigram_rows(toks, bigram, state, 32, i32(slots[:len(lens)]), i32(outs), i32(starts(lens)), rows)
        assert rows.tolist() == want
        h, xo = torch.empty(T, H, dtype=dtype, device=dev()), torch.empty(T, H, device=dev())
        K.norm_conv(h, None, 1, 1e-5, tokens=toks, embed=emb, second=(rows, table), x_out=xo)
        assert torch.equal(xo, emb.float()[toks.long()] + table.float()[rows.long()])
        at = [o + n for o, n in zip(at, lens)]
        slots = outs


# ---- queries, keys, values ---------------------------------------------------------------------------------------------------
SPECS = [turned(), turned(3, 3, 8, 24, RopeSpec(8, 300.0, halves=True)), turned(1, 1, 6, 2, RopeSpec(6, 100.0, halves=True)),
         turned(5, 5, 80, 64, RopeSpec(40, 1e4, 2.5, 1.0, 16.0, 512, "yarn", halves=True)),
         turned(4, 2, 128, 128, RopeSpec(64, 1e4, 4.0, 1.0, 32.0, 256, "yarn", halves=True)), turned(7, 7, 128, 128, RopeSpec(128, 1e5, halves=True))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", SPECS, ids=lambda m: f"{m.heads}x{m.dim}x{m.vdim}")
@pytest.mark.parametrize("T", [1, 3, 150, 700])
def test_norm_after_rotation_and_rotated_values(dtype, m, T):
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    g = torch.Generator().manual_seed(T)
    offs, ld = dict(q=8, k=8 + pad8(m.q_channels), v=16 + pad8(m.q_channels) + pad8(m.k_channels)), 24 + pad8(m.q_channels) + pad8(m.k_channels) + pad8(m.v_channels)
    a = rnd(T, ld, seed=1, dtype=dtype)
    a[T // 2, offs["k"]:offs["k"] + m.dim] *= 1e-3                              # where the norm's epsilon shows
    a = a.to(dtype).float()
    pos = torch.randint(0, 9000, (T,), generator=g)
    pages = T // 64 + 3
    slots = torch.randperm(pages * 64, generator=g)[:T]
    slots[T // 3] = -1 if T > 1 else slots[0]                                   # a row that caches nothing
    kc, vc = (torch.full((pages, m.kv_heads, 64, w), 5.0, dtype=dtype, device=dev()) for w in (m.dim, m.vdim))
    tabs = []
    for r in (m.rope, m.v_rope):
        tab = torch.empty(T, max(1, r.dims // 2), 2, device=dev())
        K.rope_table(i32(pos.tolist()), rope_frequencies(r).to(dev()), tab, r.magnitude)
        tabs.append(tab)
    q = torch.empty(T, m.q_channels, dtype=dtype, device=dev())
    K.conv_rope_kv(a.to(dev(), dtype), offs, m, None, tabs[0], i32(slots.tolist()), q, kc, vc, eps=1e-3, v_table=tabs[1])
    cut = lambda n, c, w: a[:, offs[n]:offs[n] + c].double().view(T, -1, w)     # noqa: E731
    want_q = R.rms(R.rotate(cut("q", m.q_channels, m.dim), pos, m.rope), 1e-3)
    want_k = R.rms(R.rotate(cut("k", m.k_channels, m.dim), pos, m.rope), 1e-3)
    want_v = R.rotate(cut("v", m.v_channels, m.vdim), pos, m.v_rope)
    tol = 1e-3 if dtype == torch.float32 else 2e-2                              # angles of thousands of radians in fp32
    for got, want in ((q.view(T, m.heads, m.dim), want_q),):
        assert (got.cpu().double() - want).abs().max() < tol * want.abs().max()
    used = torch.zeros(pages * 64, dtype=torch.bool)
    for t, s in enumerate(slots.tolist()):
        if s < 0:
            continue
        used[s] = True
        for c, want in ((kc, want_k), (vc, want_v)):
            assert (c[s // 64, :, s % 64].cpu().double() - want[t]).abs().max() < tol * want.abs().max()
    free = kc.permute(0, 2, 1, 3).reshape(pages * 64, -1).cpu()[~used]
    assert (free == 5.0).all()


# ---- attention ---------------------------------------------------------------------------------------------------------------
WIDE = [turned(4, 2, 128, 128, cap=6.0, scale=0.12), turned(8, 1, 128, 128, cap=30.0, scale=0.3), turned(2, 2, 128, 128, cap=0.0, scale=0.1),
        turned(16, 1, 128, 128, cap=50.0, scale=0.02)]
NARROW = [turned(), turned(3, 3, 8, 24, cap=2.0), turned(1, 1, 6, 2, cap=0.0), turned(4, 1, 30, 10, cap=20.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", NARROW + WIDE, ids=lambda m: f"{m.heads}x{m.dim}x{m.vdim}-{m.softcap}")
@pytest.mark.parametrize("edge", ["first", "page_before", "page", "itself", "none"])
def test_capped_scores_sinks_and_turned_outputs(dtype, m, edge):
    """Ragged portions; one query's score for one key stands out: the first one, the last of the page before, the first of this page, its
    own; or all scores are far below the sink's."""
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    g = torch.Generator().manual_seed(3)
    lens, q_lens = [300, 64, 65, 129, 200, 515], [70, 1, 65, 2, 1, 5]
    rep, q_all, ks, vs, want, posn = m.heads // m.kv_heads, [], [], [], [], []
    T, out_scale = sum(q_lens), 0.7
    for n, ql in zip(lens, q_lens):
        k, v = torch.randn(n, m.kv_heads, m.dim, generator=g), torch.randn(n, m.kv_heads, m.vdim, generator=g)
        q = torch.randn(ql, m.heads, m.dim, generator=g) * 0.2
        for t in range(ql):
            i = n - ql + t
            at = {"first": 0, "page_before": i // 64 * 64 - 1, "page": i // 64 * 64, "itself": i, "none": -1}[edge]
            if 0 <= at <= i:
                q[t] += 9.0 / (m.scale * m.dim) * k[at].repeat_interleave(rep, 0) * (1 + 0.05 * torch.arange(m.heads))[:, None]
            elif edge == "none":                                                # every score strongly negative
                k[:i + 1, :, 0] = -3.0
                q[t, :, 0] = 2.0 / m.scale
        q, k, v = (x.to(dtype).float() for x in (q, k, v))
        pos = torch.arange(n - ql, n)
        o = R.sink_attention(q.double(), k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1), n - ql, 0, 0, m.scale,
                             torch.zeros(m.heads, dtype=torch.float64), m.softcap)
        want.append(out_scale * R.rotate(o, -pos, m.v_rope))
        q_all.append(q); ks.append(k); vs.append(v); posn += pos.tolist()
    want = torch.cat(want).float()
    (kc, table), (vc, _) = _pages(ks, lens, dtype), _pages(vs, lens, dtype)
    tab = torch.empty(T, m.vdim // 2, 2, device=dev())
    K.rope_table(i32(posn), rope_frequencies(m.v_rope).to(dev()), tab)
    qs, sink = i32(starts(q_lens)), torch.zeros(m.heads, device=dev())
    q = torch.cat(q_all).reshape(T, -1).to(dev(), dtype)
    pitch = pad8(m.vdim)
    out = torch.full((T, m.heads * pitch + 16), 5.0, dtype=dtype, device=dev())
    K.paged_attn(q, kc, vc, m, table, i32(posn), qs, out, pitch, sink=sink, v_table=tab, out_scale=out_scale)
    tol = 4.0 if dtype == torch.float32 else 1.0                                # fp32: angles and exponentials of large arguments
    close(out[:, :m.heads * pitch].reshape(T, m.heads, pitch)[..., :m.vdim], want, dtype, tol)
    assert (out[:, m.heads * pitch:] == 5.0).all()
    if dtype != torch.bfloat16 or m not in WIDE:
        return
    kw = dict(scale=m.scale, sink=sink, cap=m.softcap, v_table=tab, out_scale=out_scale)
    q = q.view(T, m.heads, 128)
    for splits, fixed in ((0, 0), (1, 0), (2, 0), (5, 0), (9, 64), (5, 128)):
        out = torch.full((T, m.heads * 128 + 16), 5.0, dtype=dtype, device=dev())
        if splits == 0:
            K.attn_prefill(q, kc, vc, table, i32(lens), qs, out, max(q_lens), **kw)
        else:
            sc = torch.empty(K.attn_decode_scratch_floats(len(lens), max(q_lens), m.heads, m.kv_heads, splits), device=dev())
            K.set_fixed_kv_split(fixed)
            try:
                K.attn_decode(q, kc, vc, table, i32(lens), qs, out, sc, max(q_lens), splits, **kw)
            finally:
                K.set_fixed_kv_split(0)
        close(out[:, :m.heads * 128].view(T, m.heads, 128), want, dtype)
        assert (out[:, m.heads * 128:] == 5.0).all()
    assert K.read_status() == 0


# ---- linear attention -----------------------------------------------------------------------------------------------------------
LINEAR = [fading(), fading(2, 40, 136), fading(1, 1, 1), fading(3, 7, 5, 0.0), fading(2, 200, 260), fading(3, 64, 64), fading(4, 128, 128, 0.6, 0.999),
          fading(2, 32, 64), fading(2, 96, 192, 0.9), dataclasses.replace(fading(2, 64, 128), decay=(1.0, 0.0))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", LINEAR, ids=lambda m: f"{m.heads}x{m.dim}x{m.vdim}")
def test_linear_attention(dtype, m):
    """Ragged portions over three steps, the state handed from slot to slot; then the norm over all heads and the gate."""
    from cuteafd_b200.ops import kernels as K
    offs, ld, o = {}, 0, 8
    for n, c in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
        offs[n], o = o, o + pad8(c)
    ld, C, pitch = o + 8, m.heads * m.vdim, pad8(m.vdim)
    w = SimpleNamespace(decay=torch.tensor(m.decay, device=dev()), out_norm=(1 + rnd(C, seed=9, scale=0.3)).to(dev()))
    per = m.heads * m.dim * m.vdim
    state = torch.full((12, 32 + -(-per // 4) * 4), 3.0, device=dev())
    state[0] = 0
    S = [torch.zeros(m.heads, m.dim, m.vdim, dtype=torch.float64) for _ in range(4)]
    slots = [0] * 4
    big = K.lightning_chunk_ok(m, dtype)
    for step, lens in enumerate([[70, 1, 33, 2], [1, 1, 1, 1], [200 if big else 20, 64, 3, 129 if big else 9], [2, 5, 1, 1]]):
        T, qs, outs = sum(lens), starts(lens), [2 + 4 * (step & 1) + i for i in range(4)]
        a = rnd(T, ld, seed=step, scale=1.5, dtype=dtype)
        raw, act = torch.full((T, C), 9.0, device=dev()), torch.full((T, 16 + m.heads * pitch), 5.0, dtype=dtype, device=dev())
        args = (a.to(dev(), dtype), offs, m, w, state, 32, i32(slots), i32(outs), i32(qs))
        calls = [lambda: K.lightning_step(*args, raw, act[:, 16:], pitch, 1e-5)]
        if big and max(lens) >= 32:
            sc = torch.empty(K.lightning_scratch_bytes(m, T, 4), dtype=torch.uint8, device=dev())
            calls.append(lambda: K.lightning_chunked(*args, raw, act[:, 16:], pitch, 1e-5, sc, max(lens)))
        before = [s.clone() for s in S]
        for call in calls:
            raw.fill_(9.0); act.fill_(5.0)
            state[outs] = 3.0
            call()
            for s in range(4):
                x = a[qs[s]:qs[s + 1]].double()
                part = lambda n, d: x[:, offs[n]:offs[n] + m.heads * d].view(-1, m.heads, d)             # noqa: E731
                q, k, v = R.silu(part("q", m.dim)), R.silu(part("k", m.dim)), R.silu(part("v", m.vdim))
                if call is not calls[0]:                                        # chunks round them to bf16
                    q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
                want, S[s] = R.decayed_products(q, k, v, m.decay, before[s])
                tol = 2e-5 if call is calls[0] else 3e-4
                got = raw[qs[s]:qs[s + 1]].view(-1, m.heads, m.vdim).cpu().double()
                assert (got - want).abs().max() < tol * want.abs().max()
                assert (state[outs[s], 32:32 + per].view(S[s].shape).cpu().double() - S[s]).abs().max() < tol * S[s].abs().max()
                normed = R.rms(raw[qs[s]:qs[s + 1]].cpu().double(), 1e-5) * w.out_norm.cpu().double()
                out = normed * torch.sigmoid(x[:, offs["g"]:offs["g"] + C])
                close(act[qs[s]:qs[s + 1], 16:].reshape(-1, m.heads, pitch)[..., :m.vdim].reshape(-1, C), out.float(), dtype)
            assert (act[:, :16] == 5.0).all() and (state[outs, :32] == 3.0).all()
        for s in range(4):
            state[outs[s], 32:32 + per] = S[s].float().reshape(-1).to(dev())
        slots = outs


# ---- gated linear recurrence ------------------------------------------------------------------------------------------------------
RECS = [RglruSpec(72, 3, 3), RglruSpec(60, 5, 5), RglruSpec(35, 7, 1), RglruSpec(10, 1, 2), RglruSpec(256, 2, 4), RglruSpec(384, 3, 9), RglruSpec(1280, 5, 4),
        dataclasses.replace(RglruSpec(64, 1, 4), c=3.0)]


def rec_weights(m, dtype):
    r = lambda *s, seed, scale=1.0: rnd(*s, seed=seed, scale=scale, dtype=torch.bfloat16)                # noqa: E731
    p = {"x.b": r(m.width, seed=1, scale=0.5), "y.b": r(m.width, seed=2, scale=0.5), "conv": r(m.width, m.conv, seed=3, scale=0.6), "conv.b": r(m.width, seed=4, scale=0.3),
         "lam": r(m.width, seed=5, scale=1.5) - 3}
    for n in ("ra", "ri"):
        p[n], p[n + ".b"] = r(m.blocks, m.block, m.block, seed=6 + len(p), scale=m.block ** -0.5), r(m.blocks, m.block, seed=8 + len(p), scale=0.5)
    bp = pad8(m.block)
    w = SimpleNamespace(x_bias=p["x.b"].to(dev()), y_bias=p["y.b"].to(dev()), conv_b=p["conv.b"].to(dev()), lam=p["lam"].to(dev()), conv_w=p["conv"].T.contiguous().to(dev()))
    g, b = torch.zeros(m.blocks, 2, bp, bp), torch.zeros(m.blocks, 2, bp)
    for j, n in enumerate(("ra", "ri")):
        g[:, j, :m.block, :m.block], b[:, j, :m.block] = p[n], p[n + ".b"]
    w.w_gates, w.gate_bias = g.view(m.blocks, 2 * bp, bp).to(dev(), dtype), b.view(m.blocks, 2 * bp).to(dev())
    return p, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", RECS, ids=lambda m: f"{m.width}-{m.blocks}-{m.conv}")
def test_gated_linear_recurrence(dtype, m):
    """Ragged portions over steps of every size class (one row per sequence, a few rows, prompts in chunks), the state and the convolution's
    inputs handed from slot to slot."""
    from cuteafd_b200.models.mla_moe import _HeadTiles
    from cuteafd_b200.ops import kernels as K
    p, w = rec_weights(m, dtype)
    bp, ld = pad8(m.block), 8 + 2 * pad8(m.width)
    offs = dict(x=8, y=8 + pad8(m.width))
    conv_at = 32 + pad8(m.width)
    state = torch.full((12, conv_at + (m.conv - 1) * m.width + 4 - (m.conv - 1) * m.width % 4), 3.0, device=dev())
    state[0] = 0
    S, past, slots = [torch.zeros(m.width, dtype=torch.float64)] * 4, [torch.zeros(m.conv - 1, m.width, dtype=torch.float64)] * 4, [0] * 4
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for step, lens in enumerate([[300, 1, 129, 2], [1, 1, 1, 1], [2, 5, 1, 3], [20, 64, 3, 128], [1, 1, 1, 1]]):
        T, qs, outs = sum(lens), starts(lens), [2 + 4 * (step & 1) + i for i in range(4)]
        a = rnd(T, ld, seed=step, dtype=dtype)
        ht = _HeadTiles(T, m.blocks, dev())
        u, gates = torch.zeros(m.blocks, ht.t_pad, bp, dtype=dtype, device=dev()), torch.empty(m.blocks, ht.t_pad, 2 * bp, device=dev())
        out = torch.full((T, pad8(m.width)), 5.0, dtype=dtype, device=dev())
        args = (a.to(dev(), dtype), offs, m, w, u, gates, state, 32, conv_at, i32(slots), i32(outs), i32(qs), out, max(lens))

        def three():
            K.rglru_conv(*args)
            K.grouped_linear(u.view(-1, bp), w.w_gates, gates.view(-1, 2 * bp), ht.tile_expert, ht.tile_row0, ht.num_tiles, ht.max_tiles, ht.tile_rows, split_k=False)
            K.rglru_scan(*args)
        calls = [three] + ([lambda: K.rglru_step(*args)] if K.rglru_step_ok(m, dtype, T) else [])
        before, before_past = list(S), list(past)
        for call in calls:
            out.fill_(5.0)
            state[outs] = 3.0
            call()
            for s in range(4):
                x = a[qs[s]:qs[s + 1]].double()
                cut = lambda n: x[:, offs[n]:offs[n] + m.width]                 # noqa: E731
                q = {k: v.double() for k, v in p.items()}
                v, past[s] = R.causal_conv(cut("x") + q["x.b"], q["conv"], before_past[s])
                v = v + q["conv.b"]
                r, i = (torch.sigmoid(R.block_products(v, q[n], q[n + ".b"])) for n in ("ra", "ri"))
                seq, S[s] = R.gated_recurrence(v, r, i, q["lam"], m.c, before[s])
                want = seq * R.gelu_tanh(cut("y") + q["y.b"])
                got = out[qs[s]:qs[s + 1], :m.width].cpu().double()
                assert (got - want).abs().max() < tol * want.abs().max()
                assert (state[outs[s], 32:32 + m.width].cpu().double() - S[s]).abs().max() < tol * S[s].abs().max().clamp_min(1e-3)
                assert torch.allclose(state[outs[s], conv_at:conv_at + (m.conv - 1) * m.width].view(m.conv - 1, m.width).cpu().double(), past[s], atol=2e-5)
            assert (out[:, m.width:] == 5.0).all() and (state[outs, :32] == 3.0).all()
        slots = outs


# ---- feed-forward -----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,F", [(1, 64, 40), (5, 96, 200), (40, 256, 136), (100, 512, 384), (300, 128, 264), (7, 2048, 512)])
@pytest.mark.parametrize("glu", [(1.1, 1.702, 1.0), (0.3, 2.5, -0.5), (float("inf"), 1.702, 1.0)], ids=str)
def test_clipped_gated_unit(dtype, T, H, F, glu):
    """Split and whole products, rows on either side of the tensor core."""
    from cuteafd_b200.ops import kernels as K
    x, g, u = rnd(T, H, seed=1, dtype=dtype), rnd(F, H, seed=2, scale=2 * H ** -0.5, dtype=dtype), rnd(F, H, seed=3, scale=2 * H ** -0.5, dtype=dtype)
    a, b = (x.double() @ g.double().T).clamp_max(glu[0]), (x.double() @ u.double().T).clamp(-glu[0], glu[0])
    want = (a * torch.sigmoid(glu[1] * a) * (b + glu[2])).float()
    close(K.linear(x.to(dev(), dtype), g.to(dev(), dtype), w_up=u.to(dev(), dtype), glu=glu), want, dtype)


@pytest.mark.parametrize("T,H,E,top", [(5, 64, 6, 3), (200, 64, 6, 1), (3, 256, 64, 6), (33, 128, 130, 32), (2, 64, 1, 1), (7, 64, 9, 9)])
def test_sigmoid_routing_without_renormalising(T, H, E, top):
    from cuteafd_b200.ops import kernels as K
    bf = torch.bfloat16
    h, w, b = rnd(T, H, seed=1, dtype=bf), rnd(E, H, seed=2, scale=H ** -0.5, dtype=bf), rnd(E, seed=3, scale=0.5)
    ids, wt = R.route_by_sigmoid(h.double(), w.double(), b.double(), top)
    kw = dict(scoring="sigmoid", bias=b.to(dev()), num_groups=1, topk_groups=1, normalize=False, routed_scale=1.0, group_score="max")
    got = [K.route_topk((h @ w.T).to(dev()).contiguous(), top, **kw)]
    if T <= 64:
        i, x = torch.empty(T, top, dtype=torch.int32, device=dev()), torch.empty(T, top, device=dev())
        K.norm_route(h.to(dev(), bf), None, 0.0, w.to(dev(), bf), None, i, x, top, **kw)
        got.append((i, x))
    for i, x in got:
        assert torch.equal(i.cpu().long(), ids)
        assert torch.allclose(x.cpu().double(), wt, atol=1e-5)


# ---- whole model --------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["averaged", "dual"])
def test_far_keys_and_decays_in_the_engine(name):
    """Sharpened scores: what an engine computes must lie far nearer to its own model than to one whose cap, sink, rotation, scale or decay
    is off by a little."""
    cfg = averaged_config() if name == "averaged" else dual_config()
    dtype = "f32" if name == "averaged" else "bf16"
    p, toks = params(cfg, spread=SPREAD[dtype]), tokens(260, cfg.vocab_size, 6)
    want = oracle_logits(cfg, p, toks)
    e = err(run_cut(backend(cfg, p, dtype), toks, [200] + [1] * 60), want)
    assert e.median() < (1e-4 if dtype == "f32" else 0.05)

    def other(left=lambda m: {}, right=lambda m: {}, **own):
        def pair(m):
            return dataclasses.replace(m, left=dataclasses.replace(m.left, **left(m.left)), right=dataclasses.replace(m.right, **right(m.right)), **own)
        specs = tuple(dataclasses.replace(s, mixer=pair(s.mixer)) if hasattr(s.mixer, "right") else s for s in cfg.layer_specs)
        return err(oracle_logits(cfg.replace(layer_specs=specs), p, toks), want)[150:].median()
    factor, base = (20 if dtype == "f32" else 1.5), e[150:].median()
    assert other(left=lambda m: dict(v_rope=None)) > factor * base
    assert other(left=lambda m: dict(rope=dataclasses.replace(m.rope, base=m.rope.base * 1.5))) > factor * base
    assert other(right=lambda m: dict(decay=tuple(d * 0.97 for d in m.decay))) > factor * base
    assert other(right_scale=0.2) > factor * base
    if dtype == "f32":
        assert other(left=lambda m: dict(unit_sink=False)) > factor * base
        assert other(left=lambda m: dict(softcap=m.softcap * 1.1)) > factor * base
