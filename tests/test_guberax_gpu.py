"""Stacks of parallel layers on the GPU against the plain oracle: the kernels of differential attention alone (those of the two-norm
design are in test_rofapel_gpu.py, those of the design normed after its sublayers in test_buzarax_gpu.py), then the engine through its
serving backend, all three designs (greedy generation through the scheduler is with the other per-layer designs' in test_hybrid_gpu.py)."""
import dataclasses
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from cuteafd_b200.config import RopeSpec
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import (attention, averaged_config, bare_config, dual_config, err, faint_config, joined_config, joint_config, lone_config,
                                 looped_config, oracle_logits, paired_config, params, single_map_config, tokens, write_model)
from tests.test_hybrid_gpu import DTYPES, SPREAD, backend, check, close, dev, i32, rnd, run_cut

pytestmark = pytest.mark.gpu


# ---- mechanisms --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(5, 104), (5, 90), (70, 2048), (300, 1536), (900, 4096), (3, 4608), (20, 8192)])
def test_plain_residual_add_and_offset_norm(dtype, T, H):
    """x + y under a norm whose weight is stored around zero, and the embedding added once more."""
    from cuteafd_b200.ops import kernels as K
    x, y, emb = rnd(T, H, seed=1), rnd(T, H, seed=2, dtype=dtype), rnd(40, H, seed=3, dtype=dtype)
    w, ids = rnd(H, seed=4, scale=0.3, dtype=dtype), tokens(T, 40, 5)
    Hp = -(-H // 8) * 8
    yd = torch.nn.functional.pad(y, (0, Hp - H)).to(dev(), dtype)
    for add in (False, True):
        h, xo = torch.full((T, Hp), 9.0, dtype=dtype, device=dev()), torch.empty(T, H, device=dev())
        kw = dict(tokens=i32(ids), embed=emb.to(dev(), dtype)) if add else {}
        K.norm_conv(h[:, :H], w.to(dev(), dtype), 1, 1e-5, x_in=x.to(dev()), y=yd, x_out=xo, w_offset=1.0, **kw)
        want = x + y + (emb[torch.tensor(ids)] if add else 0)
        close(xo, want, torch.float32)
        close(h[:, :H], R.rms(want, 1e-5) * (1 + w), dtype)
        assert (h[:, H:] == 9.0).all()


SHAPES = [attention(), attention(3, 3, 8, 8, rope=RopeSpec(8, 300.0), conv=1), attention(5, 1, 15, 7, rope=RopeSpec(10, 1e4), conv=5),
          attention(4, 2, 64, 128, rope=RopeSpec(32, 1e5, 4.0, 1.0, 4.0, 256), conv=4), attention(2, 1, 24, 40, rope=RopeSpec(0, 1.0), conv=2),
          attention(16, 8, 64, 128, rope=RopeSpec(64, 1e5), conv=3), attention(8, 8, 16, 16, rope=RopeSpec(6, 1e2), conv=8),
          attention(2, 2, 16, 16, rope=RopeSpec(16, 1e2), conv=11), attention(2, 1, 32, 32, rope=RopeSpec(32, 1e2), conv=0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", SHAPES, ids=lambda m: f"{m.heads}.{m.kv_heads}.{m.dim}.{m.vdim}.r{m.rope.dims}.c{m.conv}")
def test_convolution_rotation_and_pages(dtype, m):
    """Ragged portions over two steps: convolution inputs from earlier rows of the step or from the state, positions far into a
    sequence, records in scattered pages, a row that caches nothing; a step of few rows and one of many."""
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    lens = [[90, 1, 2, 130], [1, 5, 1, 2], [40, 1, 700, 3]]
    C = m.conv_channels
    w = rnd(C, max(1, m.conv), seed=1, scale=0.6)
    off, halo = 32, max(0, m.conv - 1)
    state = torch.full((14, off + -(-halo * C // 32) * 32 + 32), 3.0, device=dev())
    state[0] = 0
    ins, free = [0] * 4, [3, 5, 2, 9, 1, 6, 7, 10, 11, 12, 13, 4]
    past, pos0 = [torch.zeros(halo, C) for _ in range(4)], [0, 70, 5000, 11]
    q8 = lambda n: -(-n // 8) * 8                                               # noqa: E731
    offs = dict(q=8, k=8 + q8(m.q_channels), v=8 + q8(m.q_channels) + q8(m.k_channels))
    ld = offs["v"] + q8(m.v_channels) + 8
    freq = rope_frequencies(m.rope).to(dev())
    kd, vd = (torch.zeros(16, m.kv_heads, 64, n, dtype=dtype, device=dev()) for n in (2 * m.dim, m.vdim))
    for step, ls in enumerate(lens):
        T, qs = sum(ls), [0]
        for n in ls:
            qs.append(qs[-1] + n)
        outs = free[4 * step:4 * step + 4]
        a = rnd(T, ld, seed=10 + step, dtype=dtype)
        pos = [p + i for p, n in zip(pos0, ls) for i in range(n)]
        slots = torch.randperm(15 * 64, generator=torch.Generator().manual_seed(step))[:T] + 64
        slots[3 % T] = -1
        table = torch.empty(T, max(1, m.rope.dims // 2), 2, device=dev())
        if m.rope.dims:
            K.rope_table(i32(pos), freq, table.view(-1)[:T * m.rope.dims])
        q = torch.zeros(T, m.q_channels, dtype=dtype, device=dev())
        K.conv_rope_kv(a.to(dev(), dtype), offs, m, w.T.contiguous().to(dev()) if m.conv else None, table, i32(slots.tolist()), q, kd, vd, state=state,
                       state_off=off, state_in=i32(ins), state_out=i32(outs), q_start=i32(qs))
        x = torch.cat([a[:, offs[n]:offs[n] + c] for n, c in (("q", m.q_channels), ("k", m.k_channels), ("v", m.v_channels))], 1)
        for s in range(4):
            xs, ps = x[qs[s]:qs[s + 1]], torch.tensor(pos[qs[s]:qs[s + 1]])
            y = xs
            if m.conv:
                y, past[s] = R.causal_conv(xs, w, past[s])
            n = ls[s]
            rot = lambda z, h: R.rotate(z.reshape(n, h, 2, m.dim).double(), ps, m.rope).float()      # noqa: E731
            wq = rot(y[:, :m.q_channels], m.heads).reshape(n, -1)
            wk = rot(y[:, m.q_channels:m.q_channels + m.k_channels], m.kv_heads).reshape(n, m.kv_heads, -1)
            wv = y[:, -m.v_channels:].reshape(n, m.kv_heads, m.vdim)
            k = 1.0 if dtype == torch.bfloat16 else 20.0                        # 5000 positions in: angles carry 2e-4 of rounding
            close(q[qs[s]:qs[s + 1]], wq, dtype, k)
            sl = slots[qs[s]:qs[s + 1]]
            on = sl >= 0
            if on.any():
                close(kd[sl[on] // 64, :, sl[on] % 64], wk[on], dtype, k)
                close(vd[sl[on] // 64, :, sl[on] % 64], wv[on], dtype)
            if halo:
                assert torch.equal(state[outs[s], off:off + halo * C].view(halo, C).cpu(), past[s])
            pos0[s] += n
        assert kd[0].abs().max() == 0 and (state[:, :off] == torch.where(torch.arange(14, device=dev())[:, None] == 0, 0.0, 3.0)).all()
        ins = outs


def _pages(rows, lens, dtype, seed=0):
    """[(tokens, heads, width)] per sequence in shuffled pages: (pool [pages, heads, 64, width], page table)."""
    pages = [-(-n // 64) for n in lens]
    order = torch.randperm(sum(pages), generator=torch.Generator().manual_seed(seed)) + 1
    pool = torch.zeros(sum(pages) + 1, rows[0].shape[1], 64, rows[0].shape[2])
    table, o = torch.zeros(len(lens), max(pages), dtype=torch.int32), 0
    for s, n in enumerate(lens):
        for j in range(pages[s]):
            part = rows[s][64 * j:64 * (j + 1)]
            pool[int(order[o]), :, :part.shape[0]] = part.transpose(0, 1)
            table[s, j], o = int(order[o]), o + 1
    return pool.to(dev(), dtype), table.to(dev())


def _loud_key(edge, i, m):
    """The position whose key outscores the rest for the query at position i."""
    return {"window_in": i - m.window + 1, "window_out": i - m.window, "kept_in": m.keep_first - 1, "kept_out": m.keep_first,
            "first": 0, "page_before": i // 64 * 64 - 1, "itself": i}[edge]


EDGES = ["window_in", "window_out", "kept_in", "kept_out", "first", "page_before", "itself"]
ANY = [attention(6, 2, 12, 20, 37, 5), attention(3, 3, 8, 8, 1, 2), attention(5, 1, 15, 7, 130, 70),
       attention(4, 2, 16, 24, 64, 64), attention(2, 1, 96, 160, 65, 33), attention(4, 1, 8, 8, 0, 0), attention(16, 1, 24, 144, 200, 1)]
PAIRED = [attention(4, 2, 64, 128, 100, 70), attention(8, 1, 64, 128, 65, 3), attention(2, 2, 64, 128, 128, 128), attention(8, 8, 64, 128, 1, 0),
          attention(4, 1, 64, 128, 0, 0), attention(4, 4, 64, 128, 130, 64), attention(8, 4, 64, 128, 200, 129)]


@pytest.mark.parametrize("edge", EDGES)
@pytest.mark.parametrize("dtype,m", [(d, m) for d in DTYPES for m in ANY] + [(torch.bfloat16, m) for m in PAIRED] + [(torch.float32, PAIRED[0])],
                         ids=lambda x: "f32" if x == torch.float32 else "bf16" if x == torch.bfloat16 else
                         f"{x.heads}.{x.kv_heads}.{x.dim}.{x.vdim}.w{x.window}.k{x.keep_first}")
def test_attention_windows_and_kept_tokens(dtype, m, edge):
    """One key just inside or just outside a window or the kept tokens, the first one, one across a page border or the query's
    own outscores the rest in map 1 (and half as loudly in map 2), for prompt portions and single rows."""
    from cuteafd_b200.ops import kernels as K
    g = torch.Generator().manual_seed(3)
    lens, q_lens, eps, lam = [300, 64, 65, 129, 200, 515], [70, 1, 65, 2, 1, 5], 1e-5, 0.7
    rep, q_all, ks, vs, want = m.heads // m.kv_heads, [], [], [], []
    for n, ql in zip(lens, q_lens):
        k, v = torch.randn(n, m.kv_heads, 2, m.dim, generator=g), torch.randn(n, m.kv_heads, m.vdim, generator=g)
        q = torch.randn(ql, m.heads, 2, m.dim, generator=g) * 0.2
        for t in range(ql):
            at = _loud_key(edge, n - ql + t, m)
            if 0 <= at <= n - ql + t:
                loud = 7.0 / (m.scale * m.dim)
                q[t] += loud * k[at].repeat_interleave(rep, 0) * torch.tensor([1.0, 0.5])[:, None] * (1 + 0.05 * torch.arange(m.heads))[:, None, None]
        q, k, v = (x.to(dtype).float() for x in (q, k, v))
        kr, vr = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
        a = [R.sink_attention(q[:, :, j], kr[:, :, j], vr, n - ql, m.window, m.keep_first, m.scale) for j in range(2)]
        want.append(R.rms(a[0] - lam * a[1], eps) * (1 - m.diff))
        q_all.append(q); ks.append(k.reshape(n, m.kv_heads, -1)); vs.append(v)
    want, T = torch.cat(want), sum(q_lens)
    (kc, table), (vc, _) = _pages(ks, lens, dtype), _pages(vs, lens, dtype)
    q_start = [0]
    for ql in q_lens:
        q_start.append(q_start[-1] + ql)
    pos = [n - ql + t for n, ql in zip(lens, q_lens) for t in range(ql)]
    q = torch.cat(q_all).reshape(T, -1).to(dev(), dtype)
    pitch = -(-m.vdim // 8) * 8
    # a row's norm divides by what is left after the subtraction: its error is relative to that
    k = 3.0 if dtype == torch.bfloat16 else 10.0
    out = torch.full((T, m.heads * pitch + 16), 5.0, dtype=dtype, device=dev())
    K.paged_attn(q, kc, vc, m, table, i32(pos), i32(q_start), out, pitch, lam, eps)
    got = out[:, :m.heads * pitch].reshape(T, m.heads, pitch)
    close(got[..., :m.vdim], want, dtype, k)
    assert (out[:, m.heads * pitch:] == 5.0).all()
    if not (dtype == torch.bfloat16 and m in PAIRED):
        return
    kw = dict(scale=m.scale, window=m.window, keep=m.keep_first, maps=2, lam=lam, out_scale=1 - m.diff, eps=eps)
    q = q.view(T, m.heads, 128)
    for splits, fixed in ((0, 0), (1, 0), (2, 0), (5, 0), (9, 64), (5, 128)):
        out = torch.full((T, m.heads * 128 + 16), 5.0, dtype=dtype, device=dev())
        if splits == 0:
            K.attn_prefill(q, kc, vc, table, i32(lens), i32(q_start), out, max(q_lens), **kw)
        else:
            sc = torch.empty(K.attn_decode_scratch_floats(len(lens), max(q_lens), 2 * m.heads, m.kv_heads, splits), device=dev())
            K.set_fixed_kv_split(fixed)
            try:
                K.attn_decode(q, kc, vc, table, i32(lens), i32(q_start), out, sc, max(q_lens), splits, **kw)
            finally:
                K.set_fixed_kv_split(0)
        close(out[:, :m.heads * 128].view(T, m.heads, 128), want, dtype, k)
        assert (out[:, m.heads * 128:] == 5.0).all()
    assert K.read_status() == 0


@pytest.mark.parametrize("keep", [0, 3, 64, 130])
@pytest.mark.parametrize("window", [1, 65, 128, 300])
def test_kept_tokens_with_one_map(window, keep):
    """The same mask in the plain (one map, 128-wide) form of the prompt and decode kernels, fixed-size splits included."""
    from cuteafd_b200.ops import kernels as K
    lens, q_lens, Hq, Hkv = [300, 70, 515], [90, 1, 3], 4, 2
    ks, vs, q_all, want = [], [], [], []
    for i, (n, ql) in enumerate(zip(lens, q_lens)):
        q, k, v = (rnd(*s, seed=10 * i + j, dtype=torch.bfloat16) for j, s in enumerate([(ql, Hq, 128), (n, Hkv, 128), (n, Hkv, 128)]))
        want.append(R.sink_attention(q, k.repeat_interleave(2, 1), v.repeat_interleave(2, 1), n - ql, window, keep, 0.1))
        q_all.append(q); ks.append(k); vs.append(v)
    (kc, table), (vc, _) = _pages(ks, lens, torch.bfloat16), _pages(vs, lens, torch.bfloat16)
    q, want, qs = torch.cat(q_all).to(dev(), torch.bfloat16), torch.cat(want), i32([0, 90, 91, 94])
    out = torch.empty_like(q)
    close(K.attn_prefill(q, kc, vc, table, i32(lens), qs, out, 90, scale=0.1, window=window, keep=keep), want, torch.bfloat16)
    for fixed, splits in ((0, 1), (0, 3), (128, 5)):
        K.set_fixed_kv_split(fixed)
        try:
            sc = torch.empty(K.attn_decode_scratch_floats(3, 90, Hq, Hkv, splits), device=dev())
            close(K.attn_decode(q, kc, vc, table, i32(lens), qs, out, sc, 90, splits, scale=0.1, window=window, keep=keep), want, torch.bfloat16)
        finally:
            K.set_fixed_kv_split(0)
    assert K.read_status() == 0


def test_softcap():
    from cuteafd_b200.ops import kernels as K
    for n in (7, 500, 4099):
        x = rnd(5, n + 13, seed=1, scale=40.0).to(dev())
        want, rest = R.softcap(x[:, :n].double().cpu(), 11.0), x[:, n:].clone()
        K.softcap(x[:, :n], 11.0)
        assert torch.allclose(x[:, :n].cpu().double(), want, atol=1e-5) and torch.equal(x[:, n:], rest)


# ---- engine ------------------------------------------------------------------------------------------------------------
CASES = [(c, d) for c in (looped_config(), bare_config(), paired_config(), single_map_config(), joined_config(), lone_config(), joint_config(),
                          averaged_config(), faint_config(), dual_config())
         for d in ("f32", "bf16")]
IDS = [f"{c.name}-{d}" for c, d in CASES]


@pytest.mark.parametrize("cfg,dtype", CASES, ids=IDS)
def test_prompts_portions_and_decoding(cfg, dtype):
    p, toks = params(cfg, spread=SPREAD[dtype]), tokens(333, cfg.vocab_size, 5)
    want = oracle_logits(cfg, p, toks)
    be = backend(cfg, p, dtype)
    for cuts in ([333], [300] + [1] * 33, [2], [3, 61, 1, 64, 17], [63, 2], [128, 5]):
        check(run_cut(be, toks, cuts), want, dtype)
    assert be.pool.free_pages == be.pool.usable_pages and be.states.free_slots == 10


@pytest.mark.parametrize("cfg,dtype", CASES, ids=IDS)
def test_residual_after_every_layer_run(cfg, dtype):
    """Layer by layer, one short prompt; a run's residual is what the oracle has before the next pass starts."""
    p, toks = params(cfg, spread=SPREAD[dtype]), tokens(41, cfg.vocab_size, 8)
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    m.trace = []
    with torch.no_grad():
        m.forward(torch.tensor(toks), m.new_state())
    be, got = backend(cfg, p, dtype), []
    be.engine.layer_hook = lambda n, x: got.append((n, x.float().cpu()))
    be.step([(be.open(toks, cold=True)[0], toks, [])])
    assert [n for n, _ in got] == list(range(len(cfg.layer_runs)))
    for (_, a), b in zip(got, m.trace):
        close(a, b, torch.float32 if dtype == "f32" else torch.bfloat16, 2.0)


@pytest.mark.parametrize("cfg", [looped_config(), paired_config(), joined_config(), joint_config(), averaged_config(), dual_config()],
                         ids=lambda c: c.name)
def test_decode_steps_match_prompt_steps(cfg):
    """The decode form (its own attention kernel, drafts as rows of one step) against prompt portions of the same tokens."""
    dtype = "f32" if cfg.name in ("looped", "joined", "averaged") else "bf16"
    p, seqs = params(cfg, spread=SPREAD[dtype]), [tokens(n, cfg.vocab_size, n) for n in (230, 66, 131)]
    want = [oracle_logits(cfg, p, t) for t in seqs]
    for rows in ([1, 1, 1], [4, 1, 3]):
        be = backend(cfg, p, dtype, pages=60, slots=20)
        hs = [be.open(t, cold=True)[0] for t in seqs]
        at = [40, 2, 100]
        for h, t, o in zip(hs, seqs, at):
            be.step([(h, t[:o], [])])
        got = [[] for _ in seqs]
        while all(o + r <= len(t) for o, r, t in zip(at, rows, seqs)):
            lg = be.verify(hs, [t[o:o + r] for t, o, r in zip(seqs, at, rows)])
            for i, part in enumerate(torch.split(lg.float().cpu(), rows)):
                at[i] += rows[i]
                be.commit(hs[i], at[i])
                got[i].append(part)
        for i, o in enumerate([40, 2, 100]):
            check(torch.cat(got[i]), want[i][o:at[i]], dtype)


@pytest.mark.parametrize("cfg,dtype", CASES, ids=IDS)
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


@pytest.mark.parametrize("cfg", [looped_config(), joined_config(), averaged_config()], ids=lambda c: c.name)
def test_a_row_does_not_depend_on_the_cut_or_the_batch(cfg):
    """32-bit: the same row computed in other portions and beside other requests differs by rounding alone."""
    p = params(cfg)
    be = backend(cfg, p)
    a, b = tokens(200, cfg.vocab_size, 1), tokens(130, cfg.vocab_size, 2)
    alone = run_cut(be, a, [200])
    h, k = be.open(a, cold=True)[0], be.open(b, cold=True)[0]
    got = []
    for o in range(0, 200, 40):
        part = b[o // 2:o // 2 + 20]
        got.append(be.step([(k, part, []), (h, a[o:o + 40], list(range(40)))])[-1])
    assert err(torch.cat(got), alone).max() < 2e-6


@pytest.mark.parametrize("cfg", [bare_config(), lone_config(), faint_config()], ids=lambda c: c.name)
def test_long_decoding_and_large_steps(cfg):
    p, toks = params(cfg), tokens(900, cfg.vocab_size, 3)
    want = oracle_logits(cfg, p, toks)
    be = backend(cfg, p)
    check(run_cut(be, toks, [100] + [1] * 800), want, "f32")
    h = be.open(toks, cold=True)[0]                         # more tokens than the engine takes at once: the step is cut
    check(be.step([(h, toks, [0, 511, 512, 899])])[0], want[[0, 511, 512, 899]], "f32")


@pytest.mark.parametrize("name", ["looped", "paired"])
def test_far_keys_and_kept_tokens_in_the_engine(name):
    """One query's row is made loud for one early token, so that a kept token that is dropped, or one past them that is seen,
    changes every logit: the same model with ``keep_first`` one more or one less must give something else."""
    cfg = looped_config() if name == "looped" else paired_config()
    dtype = "f32" if name == "looped" else "bf16"
    p, toks = params(cfg), tokens(260, cfg.vocab_size, 6)
    for i, s in enumerate(cfg.layer_specs):
        for n in ("q", "k"):
            p[f"l{i}.mix.{n}"] = (p[f"l{i}.mix.{n}"] * 1.7).to(torch.bfloat16).float()
    want = oracle_logits(cfg, p, toks)
    be = backend(cfg, p, dtype)
    got = run_cut(be, toks, [200] + [1] * 60)
    e = err(got, want)
    assert e.median() < (1e-4 if dtype == "f32" else 0.05)
    for d in (-1, 1):
        specs = tuple(dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, keep_first=s.mixer.keep_first + d))
                      if s.mixer.keep_first else s for s in cfg.layer_specs)
        other = err(oracle_logits(cfg.replace(layer_specs=specs), p, toks), want)
        if dtype == "f32":
            assert other[150:].median() > 20 * e[150:].median()


@pytest.mark.parametrize("cfg,dtype", [(looped_config(), "f32"), (paired_config(), "bf16"), (joined_config(), "f32"), (joint_config(), "bf16"),
                                       (averaged_config(), "f32"), (dual_config(), "bf16")],
                         ids=["looped", "paired", "joined", "joint", "averaged", "dual"])
def test_generator_and_device_loop(cfg, dtype):
    """Greedy generation under decode graphs, and the device-resident decode loop that benchmarks time."""
    from cuteafd_b200.runtime.generate import Generator
    p = params(cfg, spread=SPREAD[dtype])
    be = backend(cfg, p, dtype, slots=20)
    gen = Generator(be.engine, be.pool, 20, 4, prefill_chunk=64, use_graphs=True)
    prompts = [tokens(100, cfg.vocab_size, 1), tokens(9, cfg.vocab_size, 2)]
    seqs = [gen.table.new() for _ in prompts]
    last = [gen.prefill(s, q) for s, q in zip(seqs, prompts)]
    out = [[t] for t in last]
    for _ in range(11):
        last = gen.decode(seqs, last)
        for o, t in zip(out, last):
            o.append(t)
    for q, o in zip(prompts, out):
        want = oracle_logits(cfg, p, q + o)[len(q) - 1:-1]
        if dtype == "f32":
            assert o == want.argmax(-1).tolist()
        best = want.max(-1).values                            # bf16: a near tie may go either way
        assert (best - want[torch.arange(12), o] < 0.06 * best.abs() + 1e-6).all()


@pytest.mark.parametrize("cfg", [paired_config(), joint_config(), dual_config()], ids=lambda c: c.name)
def test_serve_builds_over_a_snapshot(tmp_path, cfg):
    """``serve --snapshot``: loading, page and slot pools, scheduler with the n-gram drafter, decode graphs, sampling."""
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.sampling import SamplingParams
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    p = params(cfg, 3, spread=2.0)
    path = write_model(cfg, p, str(tmp_path / "m"))
    st = build_state(build_parser().parse_args(["serve", "--snapshot", path, "--max-context-tokens", "512", "--concurrency", "3",
                                                "--speculator", "ngram"]))
    st.sched.eos_ids = ()
    assert type(st.sched.be.engine).__name__ == "HybridEngine" and st.sched.be.tier is None
    prompt = (tokens(9, cfg.vocab_size, 3) * 25)[:220]
    greedy = [st.sched.submit(Request(list(prompt[i:]), max_tokens=24)) for i in range(3)]
    drawn = [st.sched.submit(Request(list(prompt), max_tokens=24, params=SamplingParams(temperature=1.0, seed=7))) for _ in range(2)]
    while st.sched.step():
        pass
    for i, r in enumerate(greedy):
        got = collect(r, 1.0)["tokens"]
        want = oracle_logits(cfg, p, prompt[i:] + got)[len(prompt) - i - 1:-1]
        best = want.max(-1).values
        assert len(got) == 24 and (best - want[torch.arange(24), got] < 0.06 * best.abs()).all()
    a, b = (collect(r, 1.0)["tokens"] for r in drawn)
    assert len(a) == 24 and a[0] == b[0]


@pytest.mark.parametrize("cfg", [looped_config(), paired_config(), joined_config(), joint_config(), averaged_config(), dual_config()],
                         ids=lambda c: c.name)
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(dtype, cfg, tmp_path):
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
    wa, wb = oracle_logits(cfg, p, a), oracle_logits(cfg, p, b)
    want = {0: wa[[49, 0]], 2: torch.stack([wb[29], wa[54], wa[119]]), 3: wa[119:]}
    assert not (tmp_path / "1.f32").exists()
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(w.shape).copy())
        assert err(got, w).max() < (1e-4 if dtype == "float32" else 0.08)
