"""Kernels of the two-norm parallel layers on the GPU against the plain oracle, one mechanism at a time (the engine is with the other
parallel layers in test_guberax_gpu.py, greedy generation through the scheduler in test_hybrid_gpu.py)."""
import dataclasses

import pytest
import torch

from cuteafd_b200.config import RopeSpec
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import err, joined_config, joint_config, key_valued, normed, open_latent, oracle_logits, params, tokens
from tests.test_guberax_gpu import _pages
from tests.test_hybrid_gpu import DTYPES, SPREAD, backend, close, dev, i32, rnd, run_cut

pytestmark = pytest.mark.gpu


# ---- between layers ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(5, 104), (5, 90), (70, 2048), (300, 1536), (900, 4096), (3, 4608), (20, 8192), (400, 90)])
def test_two_outputs_of_one_norm_over_routed_and_plain_rows(dtype, T, H):
    """x + step + plain rows + weighted expert rows (some routes hand a row of the input through); two outputs under two weight
    vectors; scaled embedding rows; rows without a norm into one half of longer rows."""
    from cuteafd_b200.ops import kernels as K
    top, E, Hp = 3, 5, -(-H // 8) * 8
    x, base, ex = rnd(T, H, seed=1), rnd(T, H, seed=2, dtype=dtype), rnd(T * top, H, seed=3, dtype=dtype)
    ident, step, emb = rnd(T, H, seed=4, dtype=dtype), rnd(H, seed=5, dtype=dtype), rnd(40, H, seed=6, dtype=dtype)
    w1, w2 = rnd(H, seed=7, scale=0.3, dtype=dtype), rnd(H, seed=8, scale=0.3, dtype=dtype)
    g = torch.Generator().manual_seed(9)
    idx, wt = torch.randint(0, E + 1, (T, top), generator=g), torch.rand(T, top, generator=g)
    pad = lambda v, n=Hp: torch.nn.functional.pad(v, (0, n - H)).to(dev(), dtype)           # noqa: E731
    h1, h2 = (torch.full((T, Hp), 9.0, dtype=dtype, device=dev()) for _ in range(2))
    xo = torch.empty(T, H, device=dev())
    K.norm_conv(h1, w1.to(dev(), dtype), 1, 1e-5, x_in=x.to(dev()), y=pad(ex), base=pad(base, Hp + 8), slots=(wt.to(dev()), i32(idx.tolist()), E, pad(ident, Hp + 16)),
                x_out=xo, w_offset=1.0, step=step.to(dev(), dtype), w2=w2.to(dev(), dtype), h2_out=h2)
    rows = torch.where((idx >= E)[..., None], ident[:, None], ex.view(T, top, H))
    want = x + step + base + (wt[..., None] * rows).sum(1)
    close(xo, want, torch.float32)
    close(h1[:, :H], R.rms(want, 1e-5) * (1 + w1), dtype)
    close(h2[:, :H], R.rms(want, 1e-5) * (1 + w2), dtype)
    assert (h1[:, H:] == 9.0).all() and (h2[:, H:] == 9.0).all()
    ids = tokens(T, 40, 5)
    both = torch.full((T, 2 * Hp), 7.0, dtype=dtype, device=dev())
    K.norm_conv(both[:, Hp:], None, 1, 1e-5, tokens=i32(ids), embed=emb.to(dev(), dtype), embed_scale=6.5)
    K.norm_conv(both, None, 1, 1e-5, x_in=x.to(dev()), y=pad(base))
    close(both[:, Hp:Hp + H], emb[torch.tensor(ids)] * 6.5, dtype)
    close(both[:, :H], x + base, dtype)
    assert (both[:, H:Hp] == 7.0).all() and (both[:, Hp + H:] == 7.0).all()
    K.norm_conv(h1, w1.to(dev(), dtype), 1, 1e-5, tokens=i32(ids), embed=emb.to(dev(), dtype), embed_scale=6.5, x_out=xo, w_offset=1.0)
    close(xo, emb[torch.tensor(ids)] * 6.5, torch.float32)


# ---- queries, keys and values ----------------------------------------------------------------------------------------------
def _m(m, **kw):
    return dataclasses.replace(m, **kw)


SHAPES = [key_valued(), key_valued(3, 3, 8, 0, RopeSpec(8, 300.0, halves=True), 1), key_valued(4, 2, 128, 0, RopeSpec(64, 1e4, 2.0, kind="linear", halves=True), 4),
          key_valued(2, 1, 33, 0, RopeSpec(18, 1e3, halves=True), 9), key_valued(16, 8, 128, 0, RopeSpec(128, 1e6, halves=True), 4),
          key_valued(2, 2, 256, 0, RopeSpec(96, 1e4, 3.0, kind="linear", halves=True), 2),
          normed(), normed(4, 4, 16, 24, RopeSpec(16, 700.0, halves=True)), normed(16, 8, 128, 128, RopeSpec(128, 1e6, halves=True)),
          normed(32, 8, 128, 128, RopeSpec(48, 1e4, halves=True)), normed(3, 1, 200, 40, RopeSpec(0, 1e4, halves=True)),
          _m(normed(4, 2, 24, 16, RopeSpec(16, 100.0, halves=True)), conv=3), _m(normed(3, 1, 16, 20, RopeSpec(8, 100.0)), qk_norm="head", conv=2),
          _m(normed(4, 2, 12, 12, RopeSpec(12, 100.0, 4.0, 1.0, 8.0, 64, "yarn")), qk_norm="head"), _m(normed(2, 2, 32, 8, RopeSpec(32, 1e2, halves=True)), qk_norm=""),
          _m(normed(2, 1, 16, 16, RopeSpec(16, 1e2)), qk_norm="head", v_from_k=True),
          key_valued(3, 1, 128, 0, RopeSpec(128, 1e4, halves=True), 2), key_valued(2, 2, 128, 0, RopeSpec(32, 1e4), 3), key_valued(4, 2, 128, 0, RopeSpec(64, 1e4, halves=True), 5),
          key_valued(2, 2, 128, 0, RopeSpec(0, 1e4, halves=True), 1), normed(3, 3, 128, 128, RopeSpec(128, 1e4)), normed(6, 2, 128, 128, RopeSpec(64, 1e4, halves=True)),
          normed(34, 17, 128, 128, RopeSpec(64, 1e4, halves=True)), _m(normed(4, 2, 128, 128, RopeSpec(64, 1e4, halves=True)), qk_norm=""),
          _m(normed(5, 1, 128, 128, RopeSpec(24, 1e4, halves=True)), qk_norm="head", v_from_k=True), _m(normed(4, 4, 128, 128, RopeSpec(8, 1e4, halves=True)), conv=4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", SHAPES, ids=lambda m: f"{m.heads}.{m.kv_heads}.{m.dim}.{m.vdim}.r{m.rope.dims}{'h' if m.rope.halves else 'n'}.c{m.conv}.{m.qk_norm}{'.vk' if m.v_from_k else ''}")
def test_convolution_norm_rotation_and_pages(dtype, m):
    """Ragged portions over three steps: convolution inputs from earlier rows of the step or from the state, norms per head or over
    the projection, pairs of both kinds, values of their own or the convolved keys, scattered pages, a row that caches nothing."""
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    lens = [[90, 1, 2, 130], [1, 5, 1, 2], [40, 1, 700, 3]]
    C, own = m.conv_channels, ("q", "k") if m.v_from_k else ("q", "k", "v")
    rows = dict(q=m.q_channels, k=m.k_channels, v=m.v_channels)
    w = rnd(C, max(1, m.conv), seed=1, scale=0.6)
    nw = {n: 1 + rnd(m.dim if m.qk_norm == "head" else rows[n], seed=2, scale=0.3) for n in "qk"}
    off, halo, eps = 32, max(0, m.conv - 1), 1e-4
    state = torch.full((14, off + -(-halo * C // 32) * 32 + 32), 3.0, device=dev())
    state[0] = 0
    ins, free = [0] * 4, [3, 5, 2, 9, 1, 6, 7, 10, 11, 12, 13, 4]
    past, pos0 = [torch.zeros(halo, C) for _ in range(4)], [0, 70, 5000, 11]
    offs, ld = {}, 8
    for n in own:
        offs[n] = ld
        ld += -(-rows[n] // 8) * 8
    ld += 8
    freq = rope_frequencies(m.rope).to(dev())
    kd, vd = (torch.zeros(16, m.kv_heads, 64, n, dtype=dtype, device=dev()) for n in (m.dim, m.vdim))
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
            K.rope_table(i32(pos), freq, table.view(-1)[:T * m.rope.dims], m.rope.magnitude)
        q = torch.zeros(T, m.q_channels, dtype=dtype, device=dev())
        K.conv_rope_kv(a.to(dev(), dtype), offs, m, w.T.contiguous().to(dev()) if m.conv else None, table, i32(slots.tolist()), q, kd, vd, state=state,
                       state_off=off, state_in=i32(ins), state_out=i32(outs), q_start=i32(qs), q_norm=nw["q"].to(dev()), k_norm=nw["k"].to(dev()), eps=eps)
        x = torch.cat([a[:, offs[n]:offs[n] + rows[n]] for n in own], 1)
        for s in range(4):
            xs, ps, n = x[qs[s]:qs[s + 1]], torch.tensor(pos[qs[s]:qs[s + 1]]), ls[s]
            y = xs
            if m.conv:
                y, past[s] = R.causal_conv(xs, w, past[s])
            part = dict(zip(own, torch.split(y, [rows[o] for o in own], 1)))
            wv = part["k" if m.v_from_k else "v"].reshape(n, m.kv_heads, m.vdim)
            got = {}
            for o in "qk":
                z = part[o] if m.qk_norm != "head" else part[o].reshape(n, -1, m.dim)
                z = R.rms(z, eps) * nw[o] if m.qk_norm else z
                got[o] = R.rotate(z.reshape(n, -1, m.dim).double(), ps, m.rope).float()
            k = 1.0 if dtype == torch.bfloat16 else 20.0                        # 5000 positions in: angles carry 2e-4 of rounding
            close(q[qs[s]:qs[s + 1]], got["q"].reshape(n, -1), dtype, k)
            sl = slots[qs[s]:qs[s + 1]]
            on = sl >= 0
            if on.any():
                close(kd[sl[on] // 64, :, sl[on] % 64], got["k"][on], dtype, k)
                close(vd[sl[on] // 64, :, sl[on] % 64], wv[on], dtype)
            if halo:
                assert torch.equal(state[outs[s], off:off + halo * C].view(halo, C).cpu(), past[s])
            pos0[s] += n
        assert kd[0].abs().max() == 0 and vd[0].abs().max() == 0
        assert (state[:, :off] == torch.where(torch.arange(14, device=dev())[:, None] == 0, 0.0, 3.0)).all()
        ins = outs


# ---- latent attention -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("halves", [False, True])
def test_latent_records_with_neighbouring_pairs_and_a_magnitude(dtype, halves):
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    rope = RopeSpec(12, 300.0, 5.0, 1.5, 24.0, 700, "yarn", halves)
    T, eps = 21, 1e-4
    a, w = rnd(T, 400, seed=1, dtype=dtype), 1 + rnd(36, seed=2, scale=0.3)
    pos, slots = [0, 1, 2, 63, 64, 1000, 5000] * 3, [64 + 3 * i for i in range(T)]
    slots[4] = -1
    cache = torch.zeros(4, 64, 48, dtype=dtype, device=dev())
    slab, qa = torch.zeros(3, 32, 24, dtype=dtype, device=dev()), torch.zeros(T, 3, 48, dtype=dtype, device=dev())
    K.latent_prep(a.to(dev(), dtype), 8, 200, 3, 20, 12, w.to(dev()), rope_frequencies(rope).to(dev()), i32(pos), i32(slots), cache, slab, qa, eps,
                  halves=halves, magnitude=rope.magnitude)
    q = a[:, 8:8 + 96].view(T, 3, 32)
    want = torch.cat([R.rms(a[:, 200:236], eps) * w, R.rotate(a[:, 236:248].double(), torch.tensor(pos), rope).float()], 1)
    got = cache.view(-1, 48).float().cpu()
    k = 1.0 if dtype == torch.bfloat16 else 20.0
    for t in range(T):
        if slots[t] >= 0:
            close(got[slots[t], :48], want[t], dtype, k)
    assert got[0].abs().max() == 0
    close(slab[:, :T, :20].transpose(0, 1), q[..., :20], dtype)
    close(qa[..., 36:], R.rotate(q[..., 20:].double(), torch.tensor(pos), rope).float(), dtype, k)


def test_decode_sized_absorb_and_unabsorb():
    """A magnitude on the rotated part, and head outputs in longer rows."""
    from cuteafd_b200.models.hybrid import rope_frequencies
    from cuteafd_b200.ops import kernels as K
    bf, rope, T, heads = torch.bfloat16, RopeSpec(64, 1e5, 4.0, 1.0, 32.0, 256, "yarn"), 5, 16
    a, uk, uv = rnd(T, 24 + heads * 192, seed=1, dtype=bf), rnd(heads, 512, 128, seed=2, scale=0.1, dtype=bf), rnd(heads, 128, 512, seed=3, scale=0.05, dtype=bf)
    pos = [0, 3, 64, 999, 4000]
    qa = torch.zeros(T, heads, 576, dtype=bf, device=dev())
    K.mla_absorb_small(a.to(dev(), bf)[:, 16:16 + heads * 192], uk.to(dev(), bf), rope_frequencies(rope).to(dev()), i32(pos), qa, heads, True, rope.magnitude)
    q = a[:, 16:16 + heads * 192].view(T, heads, 192)
    close(qa[..., :512], torch.einsum("thd,hrd->thr", q[..., :128], uk), bf)
    close(qa[..., 512:], R.rotate(q[..., 128:].double(), torch.tensor(pos), rope).float(), bf)
    o = rnd(heads, 16, 512, seed=4, dtype=bf)
    out = torch.full((T, heads * 128 + 256), 5.0, dtype=bf, device=dev())
    K.mla_unabsorb_small(o.to(dev(), bf), uv.to(dev(), bf), out, T)
    close(out[:, :heads * 128].reshape(T, heads, 128), torch.einsum("htr,hdr->thd", o[:, :T], uv), bf)
    assert (out[:, heads * 128:] == 5.0).all()


# ---- attention ------------------------------------------------------------------------------------------------------------
EDGES = ["window_in", "window_out", "first", "page_before", "itself", "none"]
ANY = [key_valued(6, 2, 20, 37), key_valued(3, 3, 8, 1), key_valued(4, 1, 33, 130), normed(5, 1, 14, 7), normed(16, 1, 24, 144), normed(2, 2, 96, 200, window=64)]
WIDE = [key_valued(4, 2, 128, 100), key_valued(8, 1, 128, 65), key_valued(2, 2, 128, 128), key_valued(16, 1, 128, 1), normed(8, 4, 128, 128), normed(4, 1, 128, 128)]


@pytest.mark.parametrize("edge", EDGES)
@pytest.mark.parametrize("dtype,m", [(d, m) for d in DTYPES for m in ANY] + [(torch.bfloat16, m) for m in WIDE] + [(torch.float32, WIDE[0])],
                         ids=lambda x: "f32" if x == torch.float32 else "bf16" if x == torch.bfloat16 else f"{x.heads}.{x.kv_heads}.{x.dim}.{x.vdim}.w{x.window}")
def test_attention_with_sinks_and_gates(dtype, m, edge):
    """One key just inside or outside the window, the first one, one across a page border, the query's own or none outscores the
    rest; a head's sink is negligible, of the scores' size, as loud as the loud key, or louder than all; prompt portions and single
    rows, with and without splits."""
    from cuteafd_b200.ops import kernels as K
    g = torch.Generator().manual_seed(3)
    lens, q_lens = [300, 64, 65, 129, 200, 515], [70, 1, 65, 2, 1, 5]
    rep, q_all, ks, vs, want = m.heads // m.kv_heads, [], [], [], []
    sink = torch.tensor([[-60.0, 1.0, 7.0, 30.0, 4.0][h % 5] for h in range(m.heads)])
    T = sum(q_lens)
    gates = (torch.randn(T, m.heads, generator=g) * 2).to(dtype).float()
    for n, ql in zip(lens, q_lens):
        k, v = torch.randn(n, m.kv_heads, m.dim, generator=g), torch.randn(n, m.kv_heads, m.vdim, generator=g)
        q = torch.randn(ql, m.heads, m.dim, generator=g) * 0.2
        for t in range(ql):
            i = n - ql + t
            at = {"window_in": i - m.window + 1, "window_out": i - m.window, "first": 0, "page_before": i // 64 * 64 - 1, "itself": i, "none": -1}[edge]
            if 0 <= at <= i:
                q[t] += 7.0 / (m.scale * m.dim) * k[at].repeat_interleave(rep, 0) * (1 + 0.05 * torch.arange(m.heads))[:, None]
        q, k, v = (x.to(dtype).float() for x in (q, k, v))
        want.append(R.sink_attention(q, k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1), n - ql, m.window, 0, m.scale, sink if m.sink else None))
        q_all.append(q); ks.append(k); vs.append(v)
    want = torch.cat(want) * torch.sigmoid(gates)[..., None]
    (kc, table), (vc, _) = _pages(ks, lens, dtype), _pages(vs, lens, dtype)
    q_start = [0]
    for ql in q_lens:
        q_start.append(q_start[-1] + ql)
    pos = [n - ql + t for n, ql in zip(lens, q_lens) for t in range(ql)]
    q = torch.cat(q_all).reshape(T, -1).to(dev(), dtype)
    pitch = -(-m.vdim // 8) * 8
    wide = torch.zeros(T, 24 + m.heads, dtype=dtype, device=dev())              # gates inside longer rows
    gate = wide[:, 16:16 + m.heads]
    gate.copy_(gates)
    sd = sink.to(dev()) if m.sink else None
    out = torch.full((T, m.heads * pitch + 16), 5.0, dtype=dtype, device=dev())
    K.paged_attn(q, kc, vc, m, table, i32(pos), i32(q_start), out, pitch, sink=sd, gate=gate)
    close(out[:, :m.heads * pitch].reshape(T, m.heads, pitch)[..., :m.vdim], want, dtype)
    assert (out[:, m.heads * pitch:] == 5.0).all()
    if not (dtype == torch.bfloat16 and m in WIDE):
        return
    kw = dict(scale=m.scale, window=m.window, sink=sd, gate=gate)
    q = q.view(T, m.heads, 128)
    for splits, fixed in ((0, 0), (1, 0), (2, 0), (5, 0), (9, 64), (5, 128)):
        out = torch.full((T, m.heads * 128 + 16), 5.0, dtype=dtype, device=dev())
        if splits == 0:
            K.attn_prefill(q, kc, vc, table, i32(lens), i32(q_start), out, max(q_lens), **kw)
        else:
            sc = torch.empty(K.attn_decode_scratch_floats(len(lens), max(q_lens), m.heads, m.kv_heads, splits), device=dev())
            K.set_fixed_kv_split(fixed)
            try:
                K.attn_decode(q, kc, vc, table, i32(lens), i32(q_start), out, sc, max(q_lens), splits, **kw)
            finally:
                K.set_fixed_kv_split(0)
        close(out[:, :m.heads * 128].view(T, m.heads, 128), want, dtype)
        assert (out[:, m.heads * 128:] == 5.0).all()
    assert K.read_status() == 0


# ---- routing ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,H,E,top", [(5, 64, 6, 3), (200, 64, 6, 1), (3, 256, 64, 6), (33, 128, 130, 32), (2, 64, 1, 1), (7, 64, 9, 9)])
def test_bias_in_the_router_logits(T, H, E, top):
    from cuteafd_b200.ops import kernels as K
    bf = torch.bfloat16
    h, w, b = rnd(T, H, seed=1, dtype=bf), rnd(E, H, seed=2, scale=H ** -0.5, dtype=bf), rnd(E, seed=3, scale=1.5)
    ids, wt = R.route_by_logits(h.double(), w.double(), b.double(), top)
    kw = dict(scoring="softmax_bias", bias=b.to(dev()), num_groups=1, topk_groups=1, normalize=True, routed_scale=1.0, group_score="max")
    z = (h @ w.T).to(dev())
    got = [K.route_topk(z.contiguous(), top, **kw)]
    if T <= 64:
        i, x = torch.empty(T, top, dtype=torch.int32, device=dev()), torch.empty(T, top, device=dev())
        K.norm_route(h.to(dev(), bf), None, 0.0, w.to(dev(), bf), None, i, x, top, **kw)
        got.append((i, x))
    for i, x in got:
        assert torch.equal(i.cpu().long(), ids)
        assert torch.allclose(x.cpu().double(), wt, atol=1e-5)


# ---- whole model ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["joined", "joint"])
def test_far_keys_windows_and_sinks_in_the_engine(name):
    """Sharpened scores: what an engine computes must lie far nearer to its own model than to one whose window, sink, gate or
    scaling is off by a little."""
    cfg = joined_config() if name == "joined" else joint_config()
    dtype = "f32" if name == "joined" else "bf16"
    p, toks = params(cfg, spread=SPREAD[dtype]), tokens(260, cfg.vocab_size, 6)
    for k in p:
        if k.endswith((".mix.q.norm", ".mix.k.norm")):
            p[k] = (p[k] * 1.5).to(torch.bfloat16).float()
        elif k.endswith(".mix.sink"):
            p[k] = p[k] + 4
        elif k.endswith((".mix.uk", ".mix.dkv")):
            p[k] = (p[k] * 1.4).to(torch.bfloat16).float()
    want = oracle_logits(cfg, p, toks)
    e = err(run_cut(backend(cfg, p, dtype), toks, [200] + [1] * 60), want)
    assert e.median() < (1e-4 if dtype == "f32" else 0.05)

    def other(change, q=p):
        specs = tuple(dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, **change(s.mixer))) for s in cfg.layer_specs)
        return err(oracle_logits(cfg.replace(layer_specs=specs), q, toks), want)[150:].median()
    factor = 20 if dtype == "f32" else 1.5
    for d in (-1, 1):
        if dtype == "f32":
            assert other(lambda m: dict(window=m.window + d) if m.window > 1 else {}) > factor * e[150:].median()
    assert other(lambda m: dict(sink=False) if getattr(m, "sink", False) else {}) > factor * e[150:].median()
    assert other(lambda m: dict(rope=dataclasses.replace(m.rope, factor=1.0))) > factor * e[150:].median()
    assert other(lambda m: {}, {k: v * 0 if k == "loop.step" else v for k, v in p.items()}) > factor * e[150:].median()
