"""Parallel layers with a norm for each half (latent, windowed and plain attention beside dense or routed feed-forwards, passes that
start with a product of [x; embedding row]) on the CPU: configuration and loading, the oracle's mechanisms by hand and against
itself, planning, scheduler and serving over the oracle backend."""
import dataclasses
import json
import math

import pytest
import torch

from cuteafd_b200.config import ModelConfig, RopeSpec, RouterSpec, rofapel_bench, rofapel_bench_gqa, scaled_down
from cuteafd_b200.loader.load import load_params, open_snapshot
from cuteafd_b200.loader.snapshot import from_hf_config, to_hf_config, write_random_snapshot
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import err, joined_config, joint_config, key_valued, lone_config, normed, open_latent, oracle_logits, params, tokens, two_norms
from tests.test_guberax import greedy

CFGS = [joined_config(), lone_config(), joint_config()]


@pytest.mark.parametrize("cfg", CFGS + [rofapel_bench("base")], ids=lambda c: c.name)
def test_config_round_trips(cfg):
    d = json.loads(json.dumps(to_hf_config(cfg)))
    assert from_hf_config(d) == cfg
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg
    small = scaled_down(cfg, 2, 64)
    assert small.layer_specs == cfg.layer_specs[:2] and small.embed_scale == cfg.embed_scale and small.loop_join
    assert all(r.layer < 2 for r in small.layer_runs)


def test_config_keys():
    """The reader against a configuration written out by hand."""
    d = {"architecture": "Rofapel", "vocab": 99, "width": 48, "norm": {"eps": 1e-4}, "embedding": {"scale": 7.0}, "loop": {"start": 1, "stop": 3, "times": 2},
         "layers": [
             {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 31}, "mixer": {
                 "heads": 3, "dim": 10, "rot_dim": 6, "vdim": 9, "kv_rank": 20, "scale": 0.3,
                 "rot": {"base": 123.0, "dims": 6, "scaling": {"factor": 2.0, "original": 77, "fast": 9.0, "slow": 1.5}}}},
             {"type": "attention_2", "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 13}}, "mixer": {
                 "heads": 6, "kv_heads": 3, "dim": 14, "vdim": 14, "conv": 2, "scale": 0.4, "mask": {"size": 11},
                 "rot": {"base": 50.0, "dims": 8, "scaling": {"factor": 3.0}}}},
             {"type": "attention", "mlp": None, "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 1.0, "rot": {"base": 10.0, "dims": 4}}}]}
    c = from_hf_config(d)
    lat, win, att = (s.mixer for s in c.layer_specs)
    assert (lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank, lat.window, lat.scale, lat.gate) == (3, 10, 6, 9, 20, 0, 0.3, False)
    assert lat.rope == RopeSpec(6, 123.0, 2.0, 1.5, 9.0, 77, "yarn", halves=False)
    assert (win.heads, win.kv_heads, win.dim, win.vdim, win.conv, win.window, win.scale) == (6, 3, 14, 14, 2, 11, 0.4)
    assert (win.qk_norm, win.v_from_k, win.sink, win.gate) == ("head", True, True, True) and win.rope == RopeSpec(8, 50.0, 3.0, kind="linear", halves=True)
    assert (att.heads, att.kv_heads, att.dim, att.vdim, att.conv, att.window) == (4, 2, 6, 5, 0, 0)
    assert (att.qk_norm, att.v_from_k, att.sink, att.gate) == ("all", False, False, True) and att.rope == RopeSpec(4, 10.0, halves=True)
    assert c.layer_specs[0].dense.ffn == 31 and c.layer_specs[0].router is None
    assert c.layer_specs[1].router == RouterSpec(5, 12, 2, logit_bias=True, normalize=True) and c.layer_specs[1].dense.ffn == 13
    assert c.layer_specs[2].dense is None and all(s.parallel and s.two_norms for s in c.layer_specs)
    assert (c.vocab_size, c.hidden, c.rms_eps, c.embed_scale, c.norm_offset, c.loop) == (99, 48, 1e-4, 7.0, 1.0, (1, 3, 2))
    assert [(r.layer, r.add_embedding, r.join) for r in c.layer_runs] == [(0, False, -1), (1, False, 0), (2, False, -1), (1, False, 1), (2, False, -1)]
    d.pop("loop")
    assert [(r.layer, r.join) for r in from_hf_config(d).layer_runs] == [(0, -1), (1, -1), (2, -1)]


def test_unknown_parts_are_refused():
    d = to_hf_config(joined_config())
    for i, change in ((0, lambda e: e.update(type="delta")), (1, lambda e: e["mlp"].update(kind="other")), (0, lambda e: e["mixer"]["rot"].update(dims=22)),
                      (0, lambda e: e["mixer"].update(kv_heads=4)), (0, lambda e: e["mixer"].update(vdim=24)), (1, lambda e: e["mixer"]["rot"].update(dims=8)),
                      (1, lambda e: e["mixer"]["rot"].update(scaling={"factor": 2.0, "low": 1.0})), (1, lambda e: e["mlp"].update(act="gelu")),
                      (0, lambda e: e["mlp"]["router"].update(top=7))):
        bad = json.loads(json.dumps(d))
        change(bad["layers"][i])
        with pytest.raises(ValueError):
            from_hf_config(bad)
    with pytest.raises(ValueError):
        from_hf_config(dict(d, loop={"start": 2, "stop": 9, "times": 2}))


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_snapshot_is_recognised_and_sized(cfg, tmp_path):
    from cuteafd_b200.models.hybrid import HybridCache, HybridWeights, tensor_shapes
    path = write_random_snapshot(cfg, str(tmp_path / "m"))
    snap = open_snapshot(path)
    assert snap.family.id == "rofapel" and not snap.hints() and snap.cfg.layer_specs == cfg.layer_specs
    shapes = tensor_shapes(cfg)
    assert {n: tuple(e.shape) for n, e in snap.catalog.entries.items()} == shapes
    assert cfg.total_params() == sum(e.numel for e in snap.catalog.entries.values())
    assert snap.model.classify("l0.mlp.e0.up") == ("routed_expert", 0, 0) and snap.model.classify("l0.mlp.shared.up") == ("shared_expert", 0, None)
    assert {snap.model.classify(n)[0] for n in shapes} <= {"embedding", "head", "final_norm", "norm", "attention", "dense_ffn", "router", "routed_expert",
                                                           "shared_expert"}
    cpu = torch.device("cpu")
    W = HybridWeights.build(snap.cfg, snap.catalog.read, cpu)
    assert len(W.layers) == cfg.num_layers and W.loop_step.shape[0] == cfg.loop[2]
    kv = HybridCache(cfg, 3, cpu, 4)
    runs = [cfg.layer_specs[r.layer].mixer for r in cfg.layer_runs]
    pad8 = lambda n: -(-n // 8) * 8                                             # noqa: E731
    assert kv.bytes_per_page() == 128 * sum(pad8(m.record) if hasattr(m, "kv_rank") else m.k_channels + m.v_channels for m in runs)
    assert kv.state.shape[1] * 4 >= cfg.state_bytes == 4 * sum((m.conv - 1) * (m.q_channels + m.k_channels) for m in runs if getattr(m, "conv", 0))
    with pytest.raises(ValueError, match="shape"):
        HybridWeights.build(snap.cfg.replace(vocab_size=cfg.vocab_size + 1), snap.catalog.read, cpu)


def test_plan_places_it_on_one_gpu(tmp_path):
    from cuteafd_b200.planner import plan as P
    rep = P.plan(write_random_snapshot(joined_config(), str(tmp_path / "m")), layout=True, gpus=8)
    assert rep.placement.ok and rep.placement.engine == "single"
    used = rep.placement.devices[0].by_category()
    assert any(c == "recurrent state" for c in used)
    assert "values out of keys" in P.render(rep) and "looped" in P.render(rep) and "shared" in P.render(rep)


def test_benchmark_sizes_match():
    for size in ("small", "base", "large"):
        a, b = rofapel_bench(size), rofapel_bench_gqa(size)
        assert len(a.layer_runs) == b.num_layers and (a.hidden, a.num_experts, a.expert_ffn, a.top_k) == (b.hidden, b.num_experts, b.expert_ffn, b.top_k)
        for n, r in enumerate(a.layer_runs):
            m = a.layer_specs[r.layer].mixer
            assert m.heads == b.num_heads and a.window_of(r.layer) == b.window_of(n)
            assert hasattr(m, "kv_rank") or (m.q_channels, m.k_channels, m.v_channels) == (b.num_heads * 128, b.num_kv_heads * 128, b.num_kv_heads * 128)


# ---- the oracle against direct statements ------------------------------------------------------------------------------
def test_yarn_frequencies():
    """Eight pairs at base 10000: pair x makes 1000 / 2 pi * 10^(-x / 2) turns over 1000 positions.  50 turns lie at x = 1.006, 2 turns at
    x = 3.80: the blend runs over pairs 1 to 4."""
    r = RopeSpec(16, 1e4, 10.0, 2.0, 50.0, 1000, "yarn")
    plain = [10 ** (-i / 2) for i in range(8)]
    want = [f * ((1 - t) + t / 10) for f, t in zip(plain, (0, 0, 1 / 3, 2 / 3, 1, 1, 1, 1))]
    assert R.scaled_frequencies(r) == pytest.approx(want)
    assert r.magnitude == pytest.approx(0.1 * math.log(10) + 1) and RopeSpec(16, 1e4, 10.0, 2.0, 50.0, 1000).magnitude == 1
    # both ends beyond the pairs there are: from 0 to dims - 1
    wide = RopeSpec(8, 10.0, 4.0, 1e-9, 1e9, 100, "yarn")
    assert R.scaled_frequencies(wide) == pytest.approx([10 ** (-i / 4) * ((1 - i / 7) + i / 28) for i in range(4)])
    # both ends at one pair: a step
    step = RopeSpec(8, 1e4, 4.0, 1.0, 1.0, 2 * math.pi * 100.0, "yarn")                   # one turn lies at pair 2 exactly
    assert R.scaled_frequencies(step)[0] == 1.0 and R.scaled_frequencies(step)[3] == pytest.approx(0.001 / 4)
    assert R.scaled_frequencies(RopeSpec(4, 100.0, 5.0, kind="linear")) == pytest.approx([0.2, 0.02])


def test_engine_frequencies_agree():
    from cuteafd_b200.models.hybrid import rope_frequencies
    for rr in (RopeSpec(16, 1e4, 10.0, 2.0, 50.0, 1000, "yarn"), RopeSpec(64, 1e6, 8.0, 1.0, 32.0, 4096, "yarn"), RopeSpec(8, 10.0, 4.0, 1e-9, 1e9, 100, "yarn"),
               RopeSpec(30, 5e5, 8.0, kind="linear", halves=True), RopeSpec(12, 300.0, 1.0, 1.0, 32.0, 50, "yarn"), RopeSpec(0, 10.0, 2.0, kind="linear"),
               RopeSpec(6, 20.0, 3.0, 0.5, 0.5, 9, "yarn")):
        assert rope_frequencies(rr).tolist() == pytest.approx(R.scaled_frequencies(rr), rel=1e-6)


def test_rotation_of_halves_and_neighbours():
    x = torch.tensor([[1.0, 2.0, 3.0, 4.0, 5.0]], dtype=torch.float64)
    c0, s0, c1, s1 = math.cos(3), math.sin(3), math.cos(0.3), math.sin(0.3)
    y = R.rotate(x, torch.tensor([3]), RopeSpec(4, 100.0, halves=True))
    assert y[0].tolist() == pytest.approx([1 * c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + 1 * s0, 4 * c1 + 2 * s1, 5.0])
    y = R.rotate(x, torch.tensor([3]), RopeSpec(4, 100.0))
    assert y[0].tolist() == pytest.approx([1 * c0 - 2 * s0, 2 * c0 + 1 * s0, 3 * c1 - 4 * s1, 4 * c1 + 3 * s1, 5.0])
    m = 0.1 * math.log(8) + 1
    y = R.rotate(x, torch.tensor([0]), RopeSpec(4, 100.0, 8.0, 1.0, 32.0, 64, "yarn"))
    assert y[0].tolist() == pytest.approx([m, 2 * m, 3 * m, 4 * m, 5.0])


def _mixer_state(m):
    st = {"k": torch.zeros(0, m.kv_heads, 1, m.dim), "v": torch.zeros(0, m.kv_heads, m.vdim)}
    for n, c in (("q", m.q_channels), ("k", m.k_channels), ("v", m.v_channels)):
        st["conv." + n] = torch.zeros(max(0, m.conv - 1), c)
    return st


def test_norms_over_heads_and_over_the_projection():
    """Two heads, one ten times louder: per head the two scores come out alike, over the projection the loud one keeps its lead."""
    for kind, lead in (("head", 1.0), ("all", 10.0)):
        m = dataclasses.replace(normed(2, 2, 2, 1, RopeSpec(0, 1.0, halves=True), scale=1.0), qk_norm=kind, gate=False)
        base = torch.tensor([[1.0, 0.0], [0.0, 1.0]])
        p = {"q": torch.cat([base, 10 * base]), "k": torch.cat([base, base]), "v": torch.tensor([[1.0, 0.0]] * 2), "o": torch.eye(2)}
        n = 2 if kind == "head" else 4
        p["q.norm"], p["k.norm"] = torch.full((n,), 0.5), torch.ones(n)
        st, h = _mixer_state(m), torch.tensor([[2.0, 0.0], [0.0, 3.0]])
        y = R.attention_mixer(h, p, "", m, 0.0, 0, st)[1]                  # second token: keys e0, e1; values 2 and 0
        w = y / 2                                                          # weight of the first key per head
        score = -torch.log(1 / w - 1)                                      # its score less the other's: minus the query's second channel . k
        assert float(score[1] / score[0]) == pytest.approx(lead, rel=1e-5) and score[0] < 0


def test_values_are_the_convolved_keys_before_norm_and_rotation():
    m = dataclasses.replace(key_valued(1, 1, 2, 1, RopeSpec(2, 10.0, halves=True), 2), sink=False, gate=False)
    p = {"q": torch.eye(2), "k": torch.eye(2), "q.conv": torch.tensor([[0.0, 1.0]] * 2), "k.conv": torch.tensor([[0.5, 2.0], [0.25, 1.0]]),
         "q.norm": torch.ones(2), "k.norm": torch.tensor([7.0, 9.0]), "o": torch.eye(2)}
    st = _mixer_state(m)
    h = torch.tensor([[4.0, 8.0], [1.0, 3.0]])
    y = R.attention_mixer(h, p, "", m, 0.0, 0, st)                            # a window of one: the token's own value
    assert y[0].tolist() == pytest.approx([8.0, 8.0]) and y[1].tolist() == pytest.approx([0.5 * 4 + 2, 0.25 * 8 + 3])
    assert st["conv.k"].tolist() == [[1.0, 3.0]] and st["v"].shape == (2, 1, 2)


def test_sink_takes_its_share_whatever_the_scale():
    q, k, v = torch.zeros(1, 2, 1), torch.zeros(3, 2, 1), torch.ones(3, 2, 1)
    sink = torch.tensor([math.log(5.0), -40.0])
    y = R.sink_attention(q, k, v, 2, 0, 0, 100.0, sink)
    assert y[0, :, 0].tolist() == pytest.approx([3 / 8, 1.0])
    y = R.sink_attention(q, k, v, 2, 2, 0, 100.0, sink)
    assert y[0, :, 0].tolist() == pytest.approx([2 / 7, 1.0])


def test_gate_is_one_number_per_head():
    m = dataclasses.replace(normed(2, 1, 2, 2, RopeSpec(0, 1.0, halves=True)), qk_norm="")
    p = {"q": torch.zeros(4, 2), "k": torch.zeros(2, 2), "v": torch.eye(2), "o": torch.eye(4), "g": torch.tensor([[1.0, 0.0], [0.0, -1.0]])}
    y = R.attention_mixer(torch.tensor([[2.0, 3.0]]), p, "", m, 0.0, 0, _mixer_state(m))[0]
    s = lambda z: 1 / (1 + math.exp(-z))                                   # noqa: E731
    assert y.tolist() == pytest.approx([2 * s(2), 3 * s(2), 2 * s(-3), 3 * s(-3)])


def test_bias_is_part_of_the_router_logits():
    h, w = torch.tensor([[1.0, 0.0]]), torch.tensor([[1.0, 0], [2.0, 0], [0.5, 0], [0.0, 0]])
    ids, wt = R.route_by_logits(h, w, torch.tensor([0.0, -3.0, 0.0, 2.0]), 2)        # logits 1, -1, 0.5, 2
    assert ids.tolist() == [[3, 0]] and wt[0].tolist() == pytest.approx([1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])


def test_both_halves_read_the_same_residual_under_their_own_norms():
    cfg = lone_config().replace(layer_specs=(two_norms(normed(1, 1, 4, 3, RopeSpec(4, 50.0, halves=True)), 5, 2, 1, 6),), num_layers=1, loop=())
    p, x = params(cfg), torch.randn(4, cfg.hidden, generator=torch.Generator().manual_seed(1))
    m = R.HybridRefDecoder(cfg, p)
    norm = lambda n: R.rms(x, cfg.rms_eps) * (1 + p[n])                        # noqa: E731
    s = cfg.layer_specs[0]
    mix = R.attention_mixer(norm("l0.norm1"), p, "l0.mix.", s.mixer, cfg.rms_eps, 0, m.new_state().layers[0])
    h = norm("l0.norm2")
    ff = R.routed_ffn(h, p, "l0.mlp.", s.router) + R.dense_ffn(h, p, "l0.mlp.shared.")
    assert torch.allclose(m._layer(0, x, 0, m.new_state().layers[0]), x + mix + ff, atol=1e-5)


def test_every_pass_starts_with_a_product_of_both_halves():
    cfg = joined_config()
    p = params(cfg)
    for k in p:
        if k.endswith((".mix.o", ".down")):
            p[k].zero_()                                         # layers add nothing
    H = cfg.hidden
    p["loop.in"] = torch.cat([0.5 * torch.eye(H), 2.0 * torch.eye(H)], 1)
    p["loop.step"] = torch.tensor([1.0, 10.0, 100.0])[:, None].expand(3, H).contiguous()
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    m.trace, ids = [], torch.tensor([4, 9])
    m.forward(ids, m.new_state())
    e = p["embed"][ids] * 5.0
    x1 = 2.5 * e + 1
    x2 = 0.5 * x1 + 2 * e + 10
    x3 = 0.5 * x2 + 2 * e + 100
    for got, want in zip(m.trace, [e] + [x1] * 3 + [x2] * 3 + [x3] * 3 + [x3] * 2):
        assert torch.allclose(got, want, atol=1e-4)
    assert len(m.trace) == 12


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_oracle_prefill_equals_token_by_token(cfg):
    p, toks = params(cfg), tokens(70, cfg.vocab_size)
    want = oracle_logits(cfg, p, toks, torch.float64)
    m = R.HybridRefDecoder(cfg, {k: v.double() for k, v in p.items()})
    st = m.new_state()
    with torch.no_grad():
        a = m.forward(torch.tensor(toks[:43]), st)
        b = torch.cat([m.forward(torch.tensor([t]), st) for t in toks[43:]])
    assert err(torch.cat([a, b]), want).max() < 1e-6
    with torch.no_grad():
        m.forward(torch.tensor([1, 2, 3]), st)
        st.truncate(70)
    with pytest.raises(ValueError):
        st.truncate(3)


CHANGES = [(0, dict(window=36)), (0, dict(window=38)), (0, dict(conv=2)), (0, dict(scale=0.33)), (0, dict(rope=RopeSpec(12, 5000.0, halves=True))),
           (0, dict(rope=RopeSpec(12, 5000.0, 3.0, kind="linear"))), (0, dict(rope=RopeSpec(10, 5000.0, 3.0, kind="linear", halves=True))), (0, dict(sink=False)),
           (0, dict(gate=False)), (0, dict(qk_norm="")), (1, dict(window=64)), (1, dict(rope=RopeSpec(12, 300.0))),
           (1, dict(rope=RopeSpec(12, 300.0, 5.0, 1.5, 24.0, 700, "yarn", halves=True))), (1, dict(rope=RopeSpec(12, 300.0, 5.0, 1.5, 24.0, 700))),
           (3, dict(gate=False)), (3, dict(qk_norm="")), (3, dict(rope=RopeSpec(14, 1e4, halves=True)))]


@pytest.mark.parametrize("layer,change", CHANGES, ids=str)
def test_every_constant_shows_in_the_logits(layer, change):
    """The tests' weights are such that a constant that is slightly off moves the logits by more than the GPU tests allow."""
    cfg = joined_config()
    p, toks = params(cfg), tokens(90, cfg.vocab_size)
    want = oracle_logits(cfg, p, toks)
    s = cfg.layer_specs[layer]
    bad = dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, **change))
    q = {k: v[:, 1:] if change.get("conv") and k.startswith("l0.") and k.endswith(".conv") else v for k, v in p.items()}
    assert err(oracle_logits(cfg.replace(layer_specs=cfg.layer_specs[:layer] + (bad,) + cfg.layer_specs[layer + 1:]), q, toks), want).max() > 5e-3


@pytest.mark.parametrize("change", [dict(embed_scale=4.9), dict(loop=(1, 4, 2)), dict(loop=(1, 3, 3)), dict(loop_join=False), dict(norm_offset=0.9),
                                    dict(rms_eps=1e-2)], ids=str)
def test_every_model_constant_shows_in_the_logits(change):
    cfg = joined_config()
    p, toks = params(cfg), tokens(40, cfg.vocab_size)
    assert err(oracle_logits(cfg.replace(**change), p, toks), oracle_logits(cfg, p, toks)).max() > 2e-3


# ---- scheduler over the oracle backend -----------------------------------------------------------------------------------
@pytest.mark.parametrize("draft", [False, True])
def test_scheduler_generates_like_the_oracle(draft):
    from cuteafd_b200.runtime.backends import OracleBackend
    from cuteafd_b200.runtime.scheduler import Request, Scheduler, collect
    from cuteafd_b200.runtime.speculation import NgramDrafter
    cfg = joined_config()
    p = params(cfg)
    be = OracleBackend(cfg, p, total_pages=64, prefill_chunk=24)
    sched = Scheduler(be, drafter=NgramDrafter(block=3) if draft else None)
    prompts = [tokens(50, cfg.vocab_size, 1), tokens(5, cfg.vocab_size, 2), (tokens(7, cfg.vocab_size, 3) * 5)[:31]]
    reqs = [sched.submit(Request(list(q), max_tokens=8)) for q in prompts]
    for _ in range(400):
        sched.step()
    for q, r in zip(prompts, reqs):
        assert collect(r, 1.0)["tokens"] == greedy(cfg, p, q, 8)


def test_serve_builds_over_a_snapshot(tmp_path):
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    cfg = joined_config().replace(vocab_size=271)            # the byte tokenizer takes 260
    path = write_random_snapshot(cfg, str(tmp_path / "m"), seed=3)
    st = build_state(build_parser().parse_args(["serve", "--fake-engine", "--snapshot", path, "--speculator", "off"]))
    r = st.sched.submit(Request([5, 6, 7], max_tokens=4))
    for _ in range(20):
        st.sched.step()
    _, p = load_params(path)
    assert collect(r, 1.0)["tokens"] == greedy(cfg, p, [5, 6, 7], 4)
