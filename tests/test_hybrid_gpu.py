"""Per-layer hybrid decoders on the GPU against the plain oracle: every kernel alone, then the engine through its serving
backend (prompts, portions, mixed batches, reused pages and slots, long decoding, greedy generation)."""
import json
import subprocess

import numpy as np
import pytest
import torch

from cuteafd_b200.config import RouterSpec
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import averaged_config, delta, err, latent, joined_config, looped_config, narrow_config, odd_config, oracle_logits, params, plain_config, tokens, wide_config, write_model

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


def dev():
    return torch.device("cuda:0")


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=dev())


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    x = torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale
    return x.to(dtype).float()


def close(got, want, dtype, k=1.0):
    d = (got.float().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert d < k * TOL[dtype], float(d)


# ---- mechanisms --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,groups,taps", [(96, 3, 3), (90, 3, 4), (256, 1, 1), (2048, 4, 4), (4608, 2, 5), (8192, 8, 2), (24, 6, 9), (600, 120, 2)])
def test_norm_conv(dtype, H, groups, taps):
    """Embedding rows, then a sublayer's output added under its own norm, over ragged portions whose convolution inputs
    come from the state, then from earlier rows of the step."""
    from cuteafd_b200.ops import kernels as K
    eps, V = 1e-5, 50
    lens = [[40, 1, 2, 19], [1, 33, 2, 1]]                    # two steps of four sequences
    T = [sum(x) for x in lens]
    emb = rnd(V, H, seed=1, dtype=dtype)
    w, wb, c = (x.to(dtype).float() for x in (1 + rnd(H, seed=2, scale=0.2), 1 + rnd(H, seed=3, scale=0.2), rnd(H, taps, seed=4, scale=0.4)))
    toks = [tokens(n, V, 5 + i) for i, n in enumerate(T)]
    ys = [rnd(n, H, seed=7 + i, dtype=dtype) for i, n in enumerate(T)]
    second = 32 + -(-(taps - 1) * H // 32) * 32
    state = torch.full((12, 2 * second), 7.0, device=dev())
    state[0] = 0
    ins, outs = [0, 0, 0, 0], [3, 5, 2, 9]
    past = [torch.zeros(taps - 1, H) for _ in range(4)]
    past_y = [torch.zeros(taps - 1, H) for _ in range(4)]
    cd = c.T.contiguous().to(dev(), dtype)
    wd, wbd = w.to(dev(), dtype), wb.to(dev(), dtype)
    for step in range(2):
        qs, n = [0], T[step]
        for x in lens[step]:
            qs.append(qs[-1] + x)
        hp = torch.full((n, -(-H // 8) * 8), 9.0, dtype=dtype, device=dev())
        h, x0 = hp[:, :H], torch.empty(n, H, device=dev())
        ypad = torch.nn.functional.pad(ys[step], (0, hp.shape[1] - H)).to(dev(), dtype)
        kw = dict(state=state, state_in=i32(ins), state_out=i32(outs), q_start=i32(qs), conv=cd)
        K.norm_conv(h, wd, groups, eps, tokens=i32(toks[step]), embed=emb.to(dev(), dtype), x_out=x0, state_off=32, **kw)
        x = emb[torch.tensor(toks[step])]
        assert torch.equal(x0.cpu(), x)
        for s in range(4):
            g = R.group_rms(x[qs[s]:qs[s + 1]], w, groups, eps)
            y, past[s] = R.causal_conv(g, c, past[s])
            close(h[qs[s]:qs[s + 1]], g + y, dtype)
            if taps > 1:
                assert torch.allclose(state[outs[s], 32:32 + (taps - 1) * H].view(taps - 1, H).cpu(), past[s], atol=2e-5)
        x1 = torch.empty_like(x0)
        K.norm_conv(h, wd, groups, eps, x_in=x0, y=ypad, w_b=wbd, x_out=x1, state_off=second, run=7, **kw)
        x = x + R.group_rms(ys[step], wb, groups, eps)
        close(x1, x, torch.float32)
        for s in range(4):
            g = R.group_rms(x[qs[s]:qs[s + 1]], w, groups, eps)
            y, past_y[s] = R.causal_conv(g, c, past_y[s])
            close(h[qs[s]:qs[s + 1]], g + y, dtype)
        rows = [n - 1, 0, n // 2]
        assert (hp[:, H:] == 9.0).all()
        hf = torch.empty(3, hp.shape[1], dtype=dtype, device=dev())[:, :H]
        K.norm_conv(hf, wd, groups, eps, x_in=x0, y=ypad, w_b=wbd, rows=i32(rows))
        close(hf, R.group_rms(x[rows], w, groups, eps), dtype)
        ins, outs = outs, [1, 6, 7, 10] if step == 0 else outs


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,k,H", [(37, 3, 72), (600, 6, 256), (300, 9, 2560), (5, 12, 4096)])
def test_norm_conv_sums_routed_rows_and_identity_slots(dtype, T, k, H):
    from cuteafd_b200.ops import kernels as K
    E = 4
    y, ident, x = rnd(T * k, H, seed=1, dtype=dtype), rnd(T, H, seed=2, dtype=dtype), rnd(T, H, seed=3)
    idx = torch.randint(0, E + 2, (T, k), generator=torch.Generator().manual_seed(4))
    wts, wb, w = rnd(T, k, seed=5).abs(), (1 + rnd(H, seed=6, scale=0.2)).to(dtype).float(), (1 + rnd(H, seed=7, scale=0.2)).to(dtype).float()
    h, xo = torch.empty(T, H, dtype=dtype, device=dev()), torch.empty(T, H, device=dev())
    K.norm_conv(h, w.to(dev(), dtype), 2, 1e-5, x_in=x.to(dev()), y=y.to(dev(), dtype), w_b=wb.to(dev(), dtype), x_out=xo,
                slots=(wts.to(dev()), i32(idx.tolist()), E, ident.to(dev(), dtype)))
    rows = torch.where((idx >= E)[..., None], ident[:, None], y.view(T, k, H))
    want = x + R.group_rms((wts[..., None] * rows).sum(1), wb, 2, 1e-5)
    close(xo, want, torch.float32)
    close(h, R.group_rms(want, w, 2, 1e-5), dtype)


def _paged(rows, lens, rec, dtype, seed=0, scatter=True):
    """Records of several sequences in shuffled pages: (cache, page table)."""
    pages = [-(-n // 64) for n in lens]
    order = torch.randperm(sum(pages), generator=torch.Generator().manual_seed(seed)) + 1
    cache = torch.zeros(sum(pages) + 1, 64, rec)
    table = torch.zeros(len(lens), max(pages), dtype=torch.int32)
    o = 0
    for s, n in enumerate(lens):
        for j in range(pages[s]):
            pg = int(order[o]); o += 1
            table[s, j] = pg
            part = rows[s][64 * j:64 * (j + 1)]
            cache[pg, :part.shape[0], :part.shape[1]] = part
    return cache.to(dev(), dtype), table.to(dev())


def _planted(m, lens, q_lens, seed, edge):
    """Queries and records where, for every query row, one record just inside (``edge`` 0), just outside (1) its window or
    at its far end in the page before (2) outscores the rest by far."""
    g = torch.Generator().manual_seed(seed)
    rec = m.record
    rows = [torch.randn(n, rec, generator=g) for n in lens]
    qs = []
    for n, ql, r in zip(lens, q_lens, rows):
        q = torch.randn(ql, m.heads, rec, generator=g) * 0.2
        for t in range(ql):
            at = n - ql + t - m.window + (1 if edge == 0 else 0)
            if edge == 2:
                at = max(0, (n - ql + t) // 64 * 64 - 1)
            if at >= 0:
                q[t] += 0.6 * r[at] * (1 + 0.1 * torch.arange(m.heads)[:, None])
        qs.append(q)
    return torch.cat(qs), rows


@pytest.mark.parametrize("edge", [0, 1, 2])
@pytest.mark.parametrize("dtype,m", [(d, m) for d in DTYPES for m in (latent(3, 24, 8, 20, 40, 37), latent(2, 8, 4, 8, 12, 1),
                                                                      latent(5, 16, 12, 24, 200, 130), latent(9, 64, 64, 64, 512, 64))]
                         + [(torch.bfloat16, latent(8, 128, 64, 128, 512, 100)), (torch.bfloat16, latent(16, 128, 64, 128, 512, 65))])
def test_latent_attention_windows(dtype, m, edge):
    from cuteafd_b200.ops import kernels as K
    lens, q_lens = [300, 64, 65, 129, 200], [70, 1, 65, 2, 1]
    q, rows = _planted(m, lens, q_lens, 3, edge)
    rec = -(-m.record // 8) * 8
    cache, table = _paged(rows, lens, rec, dtype)
    T = sum(q_lens)
    qp = torch.zeros(T, m.heads, rec)
    qp[..., :m.record] = q
    qp = qp.to(dev(), dtype)
    q_start = [0]
    pos = []
    for n, ql in zip(lens, q_lens):
        pos += list(range(n - ql, n))
        q_start.append(q_start[-1] + ql)
    o, want = 0, []
    qf = qp.float().cpu()[..., :m.record]
    for s, (n, ql) in enumerate(zip(lens, q_lens)):
        r = rows[s].to(dtype).float()
        want.append(R.window_attention(qf[o:o + ql], r[:, None].expand(n, m.heads, m.record), r[:, None, :m.kv_rank].expand(n, m.heads, m.kv_rank),
                                       n - ql, m.window, m.scale))
        o += ql
    want = torch.cat(want)
    t_pad = 256
    out = torch.zeros(m.heads, t_pad, m.kv_rank, dtype=dtype, device=dev())
    K.latent_attn(qp, cache, m.kv_rank, m.rot_dim, table, i32(pos), i32(q_start), out, m.scale, m.window)
    close(out[:, :T].transpose(0, 1), want, dtype)
    if rec == 576 and 128 % m.heads == 0:
        bs, bt = K.mla_blocks(q_lens, m.heads)
        for splits in (1, 3):
            sc = torch.empty(K.mla_scratch_floats(len(bs), splits), device=dev())
            out = torch.zeros(m.heads, t_pad, 512, dtype=dtype, device=dev())
            K.mla_attention(qp, cache, table, i32(lens), i32(q_start), i32(bs), i32(bt), out, m.scale, splits, sc, out_tpad=t_pad, window=m.window)
            close(out[:, :T].transpose(0, 1), want, dtype)
        assert K.read_status() == 0


@pytest.mark.parametrize("edge", [0, 1, 2])
@pytest.mark.parametrize("window", [1, 64, 100, 129, 1000])
def test_expanded_prompt_attention_windows(window, edge):
    """The expanded form (per-head keys and values of the whole prompt, shared rotated part from the cache) under a
    sliding window, one key outscoring the rest just inside, just outside or in the page before."""
    from cuteafd_b200.ops import kernels as K
    n, heads, scale = 330, 4, 192 ** -0.5 * 1.5
    q, k, v = rnd(n, heads, 192, seed=1, scale=0.2), rnd(n, heads, 192, seed=2), rnd(n, heads, 128, seed=3)
    k[..., 128:] = k[:, :1, 128:]                                    # all heads share the rotated part
    for t in range(n):
        at = t // 64 * 64 - 1 if edge == 2 else t - window + (1 if edge == 0 else 0)
        if at >= 0:
            q[t] += 0.7 * k[at]
    q, k, v = (x.to(torch.bfloat16).float() for x in (q, k, v))
    lat = torch.zeros(n, 576)
    lat[:, 512:] = k[:, 0, 128:]
    cache, table = _paged([lat], [n], 576, torch.bfloat16)
    rows = -(-n // 64) * 64
    kx, vx = (torch.zeros(rows, heads * 128, dtype=torch.bfloat16, device=dev()) for _ in range(2))
    kx[:n], vx[:n] = k[..., :128].reshape(n, -1), v.reshape(n, -1)
    qa = torch.zeros(n, heads, 576, dtype=torch.bfloat16, device=dev())
    qa[..., 512:] = q[..., 128:]
    wide = torch.zeros(n, heads * 192 + 40, dtype=torch.bfloat16, device=dev())      # query columns inside longer rows
    wide[:, 8:8 + heads * 192] = q.reshape(n, -1)
    out = torch.zeros(n, heads, 128, dtype=torch.bfloat16, device=dev())
    K.attn_prefill_mla(wide[:, 8:8 + heads * 192], qa, kx, vx, i32([0]), cache, table, i32([n]), i32([0, n]), out, n, heads, scale, window=window)
    close(out, R.window_attention(q, k, v, 0, window, scale), torch.bfloat16)
    assert K.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_prep(dtype):
    from cuteafd_b200.ops import kernels as K
    m, T, eps = latent(3, 20, 12, 20, 36, 50), 21, 1e-4
    a = rnd(T, 400, seed=1, dtype=dtype)
    w = 1 + rnd(m.kv_rank, seed=2, scale=0.3)
    pos = [0, 1, 2, 63, 64, 1000, 5000] * 3
    slots = [64 + 3 * i for i in range(T)]
    slots[4] = -1
    f = torch.tensor(R.scaled_frequencies(m.rope))
    cache = torch.zeros(4, 64, 48, dtype=dtype, device=dev())
    slab, qa = torch.zeros(3, 32, 24, dtype=dtype, device=dev()), torch.zeros(T, 3, 48, dtype=dtype, device=dev())
    lat = torch.zeros(T, m.kv_rank, dtype=dtype, device=dev())
    K.latent_prep(a.to(dev(), dtype), 8, 200, 3, 20, 12, w.to(dev()), f.to(dev()), i32(pos), i32(slots), cache, slab, qa, eps, lat_out=lat)
    q = a[:, 8:8 + 96].view(T, 3, 32)
    c = R.rms(a[:, 200:236], eps) * w
    kr = R.rotate(a[:, 236:248], torch.tensor(pos), m.rope)
    got = cache.view(-1, 48).float().cpu()
    for t in range(T):
        if slots[t] >= 0:
            close(got[slots[t], :48], torch.cat([c[t], kr[t]]), dtype)
    assert got[0].abs().max() == 0
    close(lat, c, dtype)
    close(slab[:, :T, :20].transpose(0, 1), q[..., :20], dtype)
    close(qa[..., 36:], R.rotate(q[..., 20:], torch.tensor(pos), m.rope), dtype)


def _delta_layer(m, seed=0):
    class W:
        pass
    w = W()
    w.conv_w, w.A_log = rnd(m.conv_channels, m.conv, seed=seed, scale=0.5), rnd(m.heads, seed=seed + 1) - 1
    w.dt_bias, w.out_norm = rnd(m.heads, seed=seed + 2), 1 + rnd(m.vdim, seed=seed + 3, scale=0.2)
    return w


def _delta_oracle(m, w, x, st, eps):
    """x: the projection's sections by name, per token."""
    n, kd = x["q"].shape[0], m.kv_heads * m.dim
    cw = dict(q=w.conv_w[:kd], k=w.conv_w[kd:2 * kd], v=w.conv_w[2 * kd:])
    y = {}
    for s in "qkv":
        z, st[s] = R.causal_conv(x[s], cw[s], st[s])
        y[s] = R.silu(z)
    rep = m.heads // m.kv_heads
    q = R.unit(y["q"].view(n, m.kv_heads, m.dim)).repeat_interleave(rep, 1) * m.dim ** -0.5
    k = R.unit(y["k"].view(n, m.kv_heads, m.dim)).repeat_interleave(rep, 1)
    g = torch.exp(-torch.exp(w.A_log) * torch.nn.functional.softplus(x["a"] + w.dt_bias))
    o, st["S"] = R.delta_recurrence(q, k, y["v"].view(n, m.heads, m.vdim), torch.sigmoid(x["b"]), g, st["S"])
    return (R.rms(o, eps) * w.out_norm) * R.silu(x["g"].view(n, m.heads, m.vdim))


DELTAS = [delta(), delta(4, 4, 64, 128, 3), delta(2, 2, 40, 136, 5), delta(1, 1, 16, 16, 1), delta(3, 1, 33, 7, 2), delta(4, 2, 128, 128, 4), delta(2, 1, 256, 64, 4),
          delta(2, 2, 64, 300, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", DELTAS, ids=str)
def test_delta_rule(dtype, m):
    """Ragged portions over three steps, the state handed from slot to slot."""
    from cuteafd_b200.ops import kernels as K
    eps, w = 1e-5, _delta_layer(m)
    kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
    widths = dict(q=kd, k=kd, v=vd, g=vd, b=m.heads, a=m.heads)
    offs, o = {}, 0
    for n, c in widths.items():
        offs[n] = o
        o += -(-c // 8) * 8
    s_sz, c_sz = m.heads * m.dim * m.vdim, (m.conv - 1) * m.conv_channels
    state = torch.full((12, s_sz + c_sz + 50), 3.0, device=dev())
    state[0] = 0
    st = [dict(S=torch.zeros(m.heads, m.dim, m.vdim), q=torch.zeros(m.conv - 1, kd), k=torch.zeros(m.conv - 1, kd), v=torch.zeros(m.conv - 1, vd))
          for _ in range(3)]
    class D:
        pass
    wd = D()
    for n in ("conv_w", "A_log", "dt_bias", "out_norm"):
        setattr(wd, n, getattr(w, n).to(dev()))
    ins, outs = [0, 0, 0], [2, 3, 4]
    for step, lens in enumerate([[30, 1, 2], [1, 17, 1], [2, 1, 70]]):
        T, qs = sum(lens), [0]
        for n in lens:
            qs.append(qs[-1] + n)
        a = rnd(T, o, seed=20 + step, dtype=dtype)
        out = torch.zeros(T, m.heads, -(-m.vdim // 8) * 8, dtype=dtype, device=dev())
        raw = torch.empty(T, vd, device=dev()) if m.vdim > 128 else None
        K.delta_step(a.to(dev(), dtype), offs, m, wd, state, 8, 8 + s_sz, i32(ins), i32(outs), i32(qs), out, raw, eps)
        for s in range(3):
            x = {n: a[qs[s]:qs[s + 1], offs[n]:offs[n] + c] for n, c in widths.items()}
            want = _delta_oracle(m, w, x, st[s], eps)
            close(out[qs[s]:qs[s + 1], :, :m.vdim], want, dtype, 3)
            close(state[outs[s], 8:8 + s_sz].view(m.heads, m.dim, m.vdim), st[s]["S"], torch.float32, 3)
            if m.conv > 1:
                close(state[outs[s], 8 + s_sz:8 + s_sz + c_sz].view(m.conv - 1, -1), torch.cat([st[s][n] for n in "qkv"], 1), torch.float32)
        ins, outs = outs, [5, 6, 7] if step == 0 else [2, 8, 9]


@pytest.mark.parametrize("slab", [1, 3, 64])
@pytest.mark.parametrize("m", [delta(4, 2, 128, 128, 4), delta(3, 3, 64, 32, 2), delta(2, 1, 64, 96, 4), delta(2, 2, 128, 32, 1)], ids=str)
def test_delta_rule_in_chunks(m, slab):
    """The chunked form over ragged portions (whole chunks, parts of one, single tokens), three steps in a row, in slabs of
    one, three and all chunks: rows and states against the token-by-token equations.  Decays from almost none to almost
    everything, and keys that repeat."""
    from cuteafd_b200.ops import kernels as K
    eps, w = 1e-5, _delta_layer(m)
    w.A_log = w.A_log + torch.linspace(-4, 5, m.heads)
    kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
    widths = dict(q=kd, k=kd, v=vd, g=vd, b=m.heads, a=m.heads)
    offs, o = {}, 0
    for n, c in widths.items():
        offs[n] = o
        o += -(-c // 8) * 8
    s_sz, c_sz = m.heads * m.dim * m.vdim, (m.conv - 1) * m.conv_channels
    state = torch.full((12, s_sz + c_sz + 32), 3.0, device=dev())
    state[0] = 0
    st = [dict(S=torch.zeros(m.heads, m.dim, m.vdim), q=torch.zeros(m.conv - 1, kd), k=torch.zeros(m.conv - 1, kd), v=torch.zeros(m.conv - 1, vd))
          for _ in range(3)]

    class D:
        pass
    wd = D()
    for n in ("conv_w", "A_log", "dt_bias", "out_norm"):
        setattr(wd, n, getattr(w, n).to(dev()))
    scratch = torch.empty(slab * K.delta_chunk_bytes(m), dtype=torch.uint8, device=dev())
    ins, outs = [0, 0, 0], [2, 3, 4]
    for step, lens in enumerate([[130, 1, 64], [2, 65, 63], [1, 200, 3]]):
        T, qs = sum(lens), [0]
        for n in lens:
            qs.append(qs[-1] + n)
        a = rnd(T, o, seed=20 + step, dtype=torch.bfloat16)
        if step == 1:
            a[10:50, offs["k"]:offs["k"] + kd] = a[10, offs["k"]:offs["k"] + kd]
        out = torch.zeros(T, m.heads, m.vdim, dtype=torch.bfloat16, device=dev())
        raw = torch.empty(T * vd, device=dev())
        K.delta_chunked(scratch, a.to(dev(), torch.bfloat16), offs, m, wd, state, 0, s_sz, i32(ins), i32(outs), i32(qs), out, raw, eps)
        for s in range(3):
            x = {n: a[qs[s]:qs[s + 1], offs[n]:offs[n] + c] for n, c in widths.items()}
            want = _delta_oracle(m, w, x, st[s], eps)
            close(out[qs[s]:qs[s + 1]], want, torch.bfloat16)
            got = state[outs[s], :s_sz].view(m.heads, m.dim, m.vdim).cpu()
            for hh in range(m.heads):
                close(got[hh], st[s]["S"][hh], torch.float32, 10)
            if m.conv > 1:
                close(state[outs[s], s_sz:s_sz + c_sz].view(m.conv - 1, -1), torch.cat([st[s][n] for n in "qkv"], 1), torch.float32)
        ins, outs = outs, [5, 6, 7] if step == 0 else [2, 8, 9]


@pytest.mark.parametrize("r", [RouterSpec(6, 1, 3, 2, 4, 2), RouterSpec(5, 1, 2), RouterSpec(40, 1, 6, 8, 6, 2), RouterSpec(100, 1, 8, 20, 8, 8)], ids=str)
def test_routes(r):
    from cuteafd_b200.ops import kernels as K
    T, H = 50, 64
    h, w = rnd(T, H, seed=1, dtype=torch.bfloat16), rnd(r.outputs, H, seed=2, scale=0.3, dtype=torch.bfloat16)
    c = rnd(r.outputs, seed=3, scale=0.5) - 0.4                     # choice scores on both sides of zero
    ids, wts = R.route(h, w, c, r)
    kw = dict(bias=c.to(dev()), num_groups=r.groups, topk_groups=r.groups_kept, normalize=False, group_score="max")
    i1, w1 = K.route_topk((h @ w.T).to(dev()), r.top, **kw)
    i2, w2 = torch.empty_like(i1), torch.empty_like(w1)
    K.norm_route(h.to(dev(), torch.bfloat16), None, 0.0, w.to(dev(), torch.bfloat16), None, i2, w2, r.top, **kw)
    for i, ww in ((i1, w1), (i2, w2)):
        assert (i.cpu() == ids).all(1).float().mean() > 0.95        # sums in another order may swap a close pair
        ok = (i.cpu() == ids).all(1)
        assert torch.allclose(ww.cpu()[ok], wts[ok], rtol=1e-4)


def test_matrix_products_in_32_bit():
    from cuteafd_b200.ops import kernels as K
    for T, N, Kd in ((1, 7, 5), (70, 130, 100), (200, 64, 33)):
        x, w, u = rnd(T, Kd, seed=1), rnd(N, Kd, seed=2), rnd(N, Kd, seed=3)
        assert torch.allclose(K.linear(x.to(dev()), w.to(dev())).cpu(), x @ w.T, atol=1e-4)
        assert torch.allclose(K.linear(x.to(dev()), w.to(dev()), w_up=u.to(dev())).cpu(), R.silu(x @ w.T) * (x @ u.T), rtol=1e-4, atol=1e-4)


# ---- engine ------------------------------------------------------------------------------------------------------------
def backend(cfg, p, dtype="f32", pages=40, chunk=512, rows=4, slots=12, graphs=False):
    from cuteafd_b200.models.hybrid import HybridCache, HybridEngine, HybridWeights
    from cuteafd_b200.runtime.backends import EngineBackend
    cfg = cfg.replace(compute_dtype=dtype)
    W = HybridWeights.from_params(cfg, p, dev())
    eng = HybridEngine(cfg, W, HybridCache(cfg, pages, dev(), slots), max_tokens=chunk, max_seqs=rows * 8)
    return EngineBackend(eng, pages, pages, prefill_chunk=chunk, max_decode_rows=rows, use_graphs=graphs)


def run_cut(be, toks, cuts):
    """Every row's logits of ``toks`` fed in portions of the sizes ``cuts`` cycles through."""
    h, out, o, i = be.open(toks, cold=True)[0], [], 0, 0
    while o < len(toks):
        n = min(cuts[i % len(cuts)], len(toks) - o)
        out.append(be.step([(h, toks[o:o + n], list(range(n)))])[0])
        o, i = o + n, i + 1
    be.release(h)
    return torch.cat(out)


def check(got, want, dtype):
    e = err(got, want)
    if dtype == "f32":
        assert e.max() < 1e-4, float(e.max())
    else:
        assert e.median() < 0.03 and e.max() < 0.15, (float(e.median()), float(e.max()))


SPREAD = {"f32": 0.4, "bf16": 2.0}
CASES = [(narrow_config(), "f32"), (narrow_config(), "bf16"), (odd_config(), "f32"), (odd_config(), "bf16"), (plain_config(), "f32"), (plain_config(), "bf16"), (wide_config(), "f32"),
         (wide_config(), "bf16")]
IDS = [f"{c.name}-{d}" for c, d in CASES]


@pytest.mark.parametrize("cfg,dtype", CASES, ids=IDS)
def test_prompts_portions_and_decoding(cfg, dtype):
    p, toks = params(cfg, spread=SPREAD[dtype]), tokens(333, cfg.vocab_size, 5)
    want = oracle_logits(cfg, p, toks)
    be = backend(cfg, p, dtype)
    for cuts in ([333], [300] + [1] * 33, [2], [3, 61, 1, 64, 17], [63, 2], [128, 5]):
        got = run_cut(be, toks, cuts)
        check(got, want, dtype)
    assert be.pool.free_pages == be.pool.usable_pages and be.states.free_slots == 10


@pytest.mark.parametrize("cfg,dtype", [(odd_config(), "f32"), (odd_config(), "bf16"), (wide_config(70), "bf16")], ids=["odd-f32", "odd-bf16", "wide-bf16"])
def test_mixed_batches_reuse_pages_and_slots(cfg, dtype):
    """Four live requests of unequal lengths, portions beside single tokens, in pools that only just hold them; every
    finished request's pages and slots serve the next."""
    p = params(cfg, spread=SPREAD[dtype])
    reqs = [tokens(n, cfg.vocab_size, 10 + i) for i, n in enumerate([150, 1, 90, 64, 65, 3, 128, 127, 2, 77])]
    want = [oracle_logits(cfg, p, t) for t in reqs]
    be = backend(cfg, p, dtype, pages=1 + 3 + 2 + 2 + 2, slots=2 + 8)
    g = torch.Generator().manual_seed(1)
    live, nxt, got = {}, 0, [[] for _ in reqs]
    while live or nxt < len(reqs):
        while nxt < len(reqs) and len(live) < 4 and sum(-(-len(reqs[i]) // 64) for i in live) + -(-len(reqs[nxt]) // 64) <= 9:
            live[nxt] = [be.open(reqs[nxt], cold=True)[0], 0]
            nxt += 1
        items, who = [], []
        for i in list(live):
            if torch.rand(1, generator=g) < 0.25:
                continue                                        # left out of this step
            h, o = live[i]
            n = [1, 2, 3, 16, 29, 64, 100][int(torch.randint(0, 7, (1,), generator=g))]
            part = reqs[i][o:o + n]
            items.append((h, part, list(range(len(part)))))
            who.append(i)
        if not items:
            continue
        for i, lg in zip(who, be.step(items)):
            got[i].append(lg)
            live[i][1] += lg.shape[0]
            if live[i][1] == len(reqs[i]):
                be.release(live.pop(i)[0])
    check(torch.cat([torch.cat(x) for x in got]), torch.cat(want), dtype)


def test_a_row_does_not_depend_on_the_cut_or_the_batch():
    """32-bit: the same row computed in other portions and beside other requests differs by rounding alone."""
    cfg = odd_config()
    p = params(cfg)
    be = backend(cfg, p)
    a, b = tokens(200, cfg.vocab_size, 1), tokens(130, cfg.vocab_size, 2)
    alone = run_cut(be, a, [200])
    h, k = be.open(a, cold=True)[0], be.open(b, cold=True)[0]
    got = []
    for o in range(0, 200, 40):
        part = b[o // 2:o // 2 + 20]
        items = [(k, part, []), (h, a[o:o + 40], list(range(40)))] if part else [(h, a[o:o + 40], list(range(40)))]
        got.append(be.step(items)[-1])
    assert err(torch.cat(got), alone).max() < 2e-6


def test_long_decoding_and_large_steps():
    cfg = plain_config()
    p, toks = params(cfg), tokens(900, cfg.vocab_size, 3)
    want = oracle_logits(cfg, p, toks)
    be = backend(cfg, p)
    check(run_cut(be, toks, [100] + [1] * 800), want, "f32")
    h = be.open(toks, cold=True)[0]                         # more tokens than the engine takes at once: the step is cut
    check(be.step([(h, toks, [0, 511, 512, 899])])[0], want[[0, 511, 512, 899]], "f32")


def _greedy(cfg, p, prompt, n):
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    st, out = m.new_state(), []
    with torch.no_grad():
        lg = m.forward(torch.tensor(prompt), st)[-1]
        for _ in range(n):
            out.append(int(lg.argmax()))
            lg = m.forward(torch.tensor(out[-1:]), st)[-1]
    return out


@pytest.mark.parametrize("cfg", [odd_config(), looped_config(), joined_config(), averaged_config()], ids=lambda c: c.name)
@pytest.mark.parametrize("draft,graphs", [(False, False), (False, True), (True, True)])
def test_scheduler_generates_like_the_oracle(draft, graphs, cfg):
    from cuteafd_b200.runtime.scheduler import Request, Scheduler, collect
    from cuteafd_b200.runtime.speculation import DrafterSpec

    class Drafter:
        """Proposes the true continuation with every fourth token wrong: full, partial and empty acceptance, long lags."""
        spec = DrafterSpec(4)

        def __init__(self, truth):
            self.truth, self.done = truth, {}

        def begin(self, rid, prompt, first):
            self.done[rid] = 1

        def draft(self, rid, _h, last, n):
            t = self.truth[rid - 1]
            o = self.done.get(rid, 1)
            return [(x + 1) % 7 if (o + j) % 4 == 3 else x for j, x in enumerate(t[o:o + n])], None

        def accept(self, rid, new):
            self.done[rid] += len(new)

        def forget(self, rid):
            pass
    p = params(cfg)
    prompts = [tokens(70, cfg.vocab_size, 1), tokens(5, cfg.vocab_size, 2), tokens(140, cfg.vocab_size, 3)]
    n = 40
    truth = [_greedy(cfg, p, q, n) for q in prompts]
    again = prompts[0] + truth[0][:n - 1] + [3, 4]
    truth.append(_greedy(cfg, p, again, 6))
    be = backend(cfg, p, pages=60, chunk=96, slots=2 + 24, graphs=graphs)
    sched = Scheduler(be, drafter=Drafter(truth) if draft else None, draft_control="fixed" if draft else "history")
    sched.policy.fixed = 4
    reqs = [sched.submit(Request(list(q), max_tokens=n)) for q in prompts]
    for _ in range(400):
        if not sched.step() and not sched.pending and sched.waiting.empty():
            break
    for t, r in zip(truth, reqs):
        got = collect(r, 1.0)
        assert got["error"] is None and got["tokens"] == t
        if draft:
            assert got["usage"]["speculation"]["accepted"] > 0 and got["usage"]["speculation"]["accepted"] < got["usage"]["speculation"]["proposed"]
    r = sched.submit(Request(list(again), max_tokens=6))           # resumes from a snapshot: pages and a state slot are shared
    while sched.step():
        pass
    got = collect(r, 1.0)
    assert got["tokens"] == truth[3] and got["usage"]["cached_tokens"] >= 70
    if graphs and not draft:
        assert be.graph_stats["replays"] > 10
    be.prefix.clear()
    assert be.pool.free_pages == be.pool.usable_pages and be.states.free_slots == 24


def test_generator_matches_the_backend_under_graphs():
    from cuteafd_b200.runtime.generate import Generator
    cfg = odd_config()
    p = params(cfg)
    be = backend(cfg, p, slots=20)
    gen = Generator(be.engine, be.pool, 20, 4, prefill_chunk=64, use_graphs=True)
    prompts = [tokens(100, cfg.vocab_size, 1), tokens(9, cfg.vocab_size, 2)]
    truth = [_greedy(cfg, p, q, 12) for q in prompts]
    seqs = [gen.table.new() for _ in prompts]
    last = [gen.prefill(s, q) for s, q in zip(seqs, prompts)]
    out = [[t] for t in last]
    for _ in range(11):
        last = gen.decode(seqs, last)
        for o, t in zip(out, last):
            o.append(t)
    assert out == truth


def test_serve_builds_over_a_snapshot(tmp_path):
    """``serve --snapshot``: loading, page and slot pools, scheduler with the n-gram drafter, decode graphs, sampling."""
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.sampling import SamplingParams
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    cfg = odd_config().replace(vocab_size=271)            # the byte tokenizer takes 260
    p = params(cfg, 3, spread=2.0)
    path = write_model(cfg, p, str(tmp_path / "m"))
    st = build_state(build_parser().parse_args(["serve", "--snapshot", path, "--max-context-tokens", "512", "--concurrency", "3",
                                                "--speculator", "ngram"]))
    st.sched.eos_ids = ()
    assert type(st.sched.be.engine).__name__ == "HybridEngine" and st.sched.be.tier is None
    prompt = (tokens(9, cfg.vocab_size, 3) * 12)[:100]
    greedy = [st.sched.submit(Request(list(prompt[i:]), max_tokens=24)) for i in range(3)]
    drawn = [st.sched.submit(Request(list(prompt), max_tokens=24, params=SamplingParams(temperature=1.0, seed=7))) for _ in range(2)]
    while st.sched.step():
        pass
    for i, r in enumerate(greedy):
        got = collect(r, 1.0)["tokens"]
        want = oracle_logits(cfg, p, prompt[i:] + got)[len(prompt) - i - 1:-1]
        best = want.max(-1).values
        assert len(got) == 24 and (best - want[torch.arange(24), got] < 0.05 * best.abs()).all()    # bf16: a near tie may go either way
    a, b = (collect(r, 1.0)["tokens"] for r in drawn)
    assert len(a) == 24 and a[0] == b[0]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(dtype, tmp_path):
    import os
    cfg = odd_config()
    p = params(cfg, spread=2.0)
    d = write_model(cfg, p, str(tmp_path / "m"))
    a, b = tokens(120, cfg.vocab_size, 1), tokens(30, cfg.vocab_size, 2)
    steps = [{"entries": [{"id": "a", "tokens": a[:50], "want": [49, 0]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"entries": [{"id": "a", "tokens": a[50:51], "want": []}], "end": []},
             {"entries": [{"id": "b", "tokens": b[2:], "want": [27]}, {"id": "a", "tokens": a[51:], "want": [3, 68]}], "end": ["a", "b"]},
             {"entries": [{"id": "c", "tokens": a, "want": [119]}], "end": ["c"]}]
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "192"],
                       input=text, capture_output=True, text=True, timeout=200)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = oracle_logits(cfg, p, a), oracle_logits(cfg, p, b)
    want = {0: wa[[49, 0]], 2: torch.stack([wb[29], wa[54], wa[119]]), 3: wa[119:]}
    assert not (tmp_path / "1.f32").exists()
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(w.shape).copy())
        assert err(got, w).max() < (1e-4 if dtype == "float32" else 0.08)
