"""Stacks of parallel layers (differential attention beside a dense feed-forward, looped layers) on the CPU: configuration and
loading, the oracle's mechanisms by hand and against itself, planning, scheduler and serving over the oracle backend."""
import json
import math

import pytest
import torch

from cuteafd_b200.config import ModelConfig, RopeSpec, guberax_bench, guberax_bench_gqa, scaled_down
from cuteafd_b200.loader.load import load_params, open_snapshot
from cuteafd_b200.loader.snapshot import from_hf_config, to_hf_config, write_random_snapshot
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import attention, bare_config, err, looped_config, oracle_logits, paired_config, params, tokens

CFGS = [looped_config(), bare_config(), paired_config()]


@pytest.mark.parametrize("cfg", CFGS + [guberax_bench("base")], ids=lambda c: c.name)
def test_config_round_trips(cfg):
    d = json.loads(json.dumps(to_hf_config(cfg)))
    assert from_hf_config(d) == cfg
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg
    small = scaled_down(cfg, 2, 64)
    assert small.layer_specs == cfg.layer_specs[:2] and small.norm_offset == 1.0 and small.logit_softcap == cfg.logit_softcap
    assert all(r.layer < 2 for r in small.layer_runs)


def test_config_keys():
    """The reader against a configuration written out by hand."""
    d = {"architecture": "Guberax", "vocab": 99, "width": 48, "logit_softcap": 7.5, "norm": {"eps": 1e-4}, "loop": {"start": 0, "stop": 1, "times": 4},
         "layers": [{"type": "attention", "mlp": {"kind": "dense", "ff": 31}, "mixer": {
             "heads": 6, "kv_heads": 3, "dim": 14, "vdim": 9, "conv": 2, "diff": 0.25, "scale": 0.3, "mask": {"size": 11, "keep_first": 4},
             "rot": {"base": 123.0, "dims": 6, "scaling": {"factor": 2.0, "low": 1.5, "high": 3.0, "original": 77}}}},
             {"type": "attention", "mlp": None, "mixer": {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 5, "conv": 1, "diff": 0.5, "scale": 1.0,
                                                          "mask": {"size": 3, "keep_first": 0}, "rot": {"base": 10.0, "dims": 4}}}]}
    c = from_hf_config(d)
    m = c.layer_specs[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.conv, m.diff, m.scale, m.window, m.keep_first) == (6, 3, 14, 9, 2, 0.25, 0.3, 11, 4)
    assert m.rope == RopeSpec(6, 123.0, 2.0, 1.5, 3.0, 77) and c.layer_specs[1].mixer.rope == RopeSpec(4, 10.0)
    assert c.layer_specs[0].dense.ffn == 31 and c.layer_specs[1].dense is None
    assert (c.vocab_size, c.hidden, c.rms_eps, c.logit_softcap, c.loop) == (99, 48, 1e-4, 7.5, (0, 1, 4))
    assert [(r.layer, r.add_embedding) for r in c.layer_runs] == [(0, False), (0, True), (0, True), (0, True), (1, False)]
    for k in ("logit_softcap", "loop"):
        d.pop(k)
    d["layers"][0]["mixer"].pop("mask")
    c = from_hf_config(d)
    assert c.logit_softcap == 0 and [r.layer for r in c.layer_runs] == [0, 1] and c.layer_specs[0].mixer.window == 0


def test_unknown_parts_are_refused():
    d = to_hf_config(looped_config())
    for change in (lambda e: e.update(type="delta"), lambda e: e["mlp"].update(kind="moe"), lambda e: e["mixer"]["rot"].update(dims=14),
                   lambda e: e["mixer"].update(kv_heads=4)):
        bad = json.loads(json.dumps(d))
        change(bad["layers"][0])
        with pytest.raises(ValueError):
            from_hf_config(bad)
    with pytest.raises(ValueError):
        from_hf_config(dict(d, loop={"start": 2, "stop": 9, "times": 2}))


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_snapshot_is_recognised_and_sized(cfg, tmp_path):
    from cuteafd_b200.models.hybrid import HybridCache, HybridWeights, tensor_shapes
    path = write_random_snapshot(cfg, str(tmp_path / "m"))
    snap = open_snapshot(path)
    assert snap.family.id == "guberax" and not snap.hints() and snap.cfg.layer_specs == cfg.layer_specs
    shapes = tensor_shapes(cfg)
    assert {n: tuple(e.shape) for n, e in snap.catalog.entries.items()} == shapes
    assert cfg.total_params() == sum(e.numel for e in snap.catalog.entries.values())
    assert snap.model.classify("l0.mlp.up") == ("dense_ffn", 0, None)
    assert {snap.model.classify(n)[0] for n in shapes} <= {"embedding", "head", "final_norm", "norm", "attention", "dense_ffn"}
    cpu = torch.device("cpu")
    W = HybridWeights.build(snap.cfg, snap.catalog.read, cpu)
    assert len(W.layers) == cfg.num_layers
    _, p = load_params(path)
    assert set(p) == set(shapes)
    for i, L in enumerate(W.layers):
        assert L.lam == pytest.approx(float(R.difference_weight({k: v.double() for k, v in p.items()}, f"l{i}.mix.", cfg.layer_specs[i].mixer.diff)), rel=1e-6)
    kv = HybridCache(cfg, 3, cpu, 4)
    runs = [cfg.layer_specs[r.layer].mixer for r in cfg.layer_runs]
    assert len(kv.k) == len(kv.v) == len(runs) and kv.bytes_per_page() == 128 * sum(cfg.kv_elems_of(r.layer) for r in cfg.layer_runs)
    assert kv.state.shape[1] * 4 >= cfg.state_bytes == 4 * sum((m.conv - 1) * m.conv_channels for m in runs)
    with pytest.raises(ValueError, match="shape"):
        HybridWeights.build(snap.cfg.replace(vocab_size=cfg.vocab_size + 1), snap.catalog.read, cpu)


def test_plan_places_it_on_one_gpu(tmp_path):
    from cuteafd_b200.planner import plan as P
    rep = P.plan(write_random_snapshot(looped_config(), str(tmp_path / "m")), layout=True, gpus=8)
    assert rep.placement.ok and rep.placement.engine == "single"
    assert any(c == "recurrent state" for c in rep.placement.devices[0].by_category())
    assert "differential attention" in P.render(rep) and "looped" in P.render(rep)


def test_benchmark_sizes_match():
    for size in ("small", "base", "large"):
        a, b = guberax_bench(size), guberax_bench_gqa(size)
        assert len(a.layer_runs) == b.num_layers and (a.hidden, a.dense_ffn) == (b.hidden, b.dense_ffn)
        m = a.layer_specs[0].mixer
        assert (m.q_channels, m.k_channels, m.v_channels) == (b.num_heads * 128, b.num_kv_heads * 128, b.num_kv_heads * 128)


# ---- the oracle against direct statements ------------------------------------------------------------------------------
def test_frequencies_are_kept_stretched_and_blended():
    r = RopeSpec(8, 10000.0, 4.0, 1.0, 4.0, 64)
    f = R.scaled_frequencies(r)                                   # wavelengths 6.28, 62.8, 628, 6283 against 64 / 4 and 64 / 1
    s = (64 * 0.1 / (2 * math.pi) - 1) / 3
    assert f == pytest.approx([1.0, (1 - s) * 0.1 / 4 + s * 0.1, 0.01 / 4, 0.001 / 4])
    assert R.scaled_frequencies(RopeSpec(8, 10000.0)) == pytest.approx([1.0, 0.1, 0.01, 0.001])
    from cuteafd_b200.models.hybrid import rope_frequencies
    for rr in (r, RopeSpec(8, 1e4), RopeSpec(0, 1e4), RopeSpec(30, 5e5, 8.0, 0.7, 3.3, 1000)):
        assert rope_frequencies(rr).tolist() == pytest.approx(R.scaled_frequencies(rr), rel=1e-6)


def test_rotation_pairs_neighbours_and_leaves_the_rest():
    x = torch.tensor([[1.0, 0.0, 0.0, 1.0, 5.0]], dtype=torch.float64)
    y = R.rotate(x, torch.tensor([3]), RopeSpec(4, 100.0))
    assert y[0].tolist() == pytest.approx([math.cos(3), math.sin(3), -math.sin(0.3), math.cos(0.3), 5.0])


def test_window_edges_and_kept_tokens():
    q, k = torch.zeros(1, 1, 2), torch.zeros(9, 1, 2)
    v = (2.0 ** torch.arange(9.0)).view(9, 1, 1)
    see = lambda window, keep: R.sink_attention(q, k, v, 8, window, keep, 1.0).item()     # noqa: E731
    assert see(3, 0) == pytest.approx((64 + 128 + 256) / 3)
    assert see(3, 2) == pytest.approx((64 + 128 + 256 + 1 + 2) / 5)
    assert see(3, 8) == pytest.approx(511 / 9) and see(0, 0) == pytest.approx(511 / 9) and see(1, 0) == pytest.approx(256)
    assert R.sink_attention(q, k, v, 1, 1, 5, 1.0).item() == pytest.approx(1.5)           # kept tokens ahead are not seen


def test_maps_are_subtracted_and_normed():
    m = attention(1, 1, 2, 2, 0, 0, RopeSpec(0, 1.0), 0, 0.25, scale=1.0)
    p = {"q": torch.zeros(4, 2), "k": torch.zeros(4, 2), "v": torch.eye(2), "o": torch.eye(2),
         **{n: torch.zeros(2) for n in ("lq1", "lk1", "lq2", "lk2")}}
    p["q"][0, 0] = p["k"][0, 0] = 1.0                            # map 1 attends by channel 0, map 2 evenly
    st = {"k": torch.zeros(0, 1, 2, 2), "v": torch.zeros(0, 1, 2)}
    h = torch.tensor([[0.0, 4.0], [8.0, 0.0]])
    y = R.attention_mixer(h, p, "", m, 0.0, 0, st)[1]
    w = math.exp(64) / (1 + math.exp(64))
    a1, a2 = torch.tensor([8 * w, 4 * (1 - w)]), torch.tensor([4.0, 2.0])
    o = a1 - 0.25 * a2                                           # lambda = 1 - 1 + 0.25
    assert torch.allclose(y, 0.75 * o / o.pow(2).mean().sqrt(), atol=1e-5)
    p["lq1"], p["lk1"] = torch.tensor([1.0, 2.0]), torch.tensor([0.5, 0.25])
    assert R.difference_weight(p, "", 0.25).item() == pytest.approx(math.e - 1 + 0.25, rel=1e-6)


def test_loop_adds_the_embedding_before_every_later_pass():
    cfg = looped_config()
    p = params(cfg)
    for k in p:
        if k.endswith((".mix.o", ".mlp.down")):
            p[k].zero_()                                         # layers add nothing
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    m.trace, ids = [], torch.tensor([4, 9])
    m.forward(ids, m.new_state())
    got = [float((t / p["embed"][ids]).mean()) for t in m.trace]
    assert got == pytest.approx([1, 1, 1, 2, 2, 3, 3, 3])        # layers 0, 1 2, 1 2, 1 2, 3


def test_cap_bounds_the_logits():
    assert R.softcap(torch.tensor([0.0, 1e-3, 1e6, -1e6]), 5.0).tolist() == pytest.approx([0.0, 1e-3, 5.0, -5.0], rel=1e-5)


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_oracle_prefill_equals_token_by_token(cfg):
    p, toks = params(cfg), tokens(90, cfg.vocab_size)
    want = oracle_logits(cfg, p, toks, torch.float64)
    m = R.HybridRefDecoder(cfg, {k: v.double() for k, v in p.items()})
    st = m.new_state()
    with torch.no_grad():
        a = m.forward(torch.tensor(toks[:53]), st)
        b = torch.cat([m.forward(torch.tensor([t]), st) for t in toks[53:]])
    assert err(torch.cat([a, b]), want).max() < 1e-6
    with torch.no_grad():
        m.forward(torch.tensor([1, 2, 3]), st)
        st.truncate(90)
        st.truncate(90)
    with pytest.raises(ValueError):
        st.truncate(3)


@pytest.mark.parametrize("change", [
    dict(window=36), dict(window=38), dict(keep_first=4), dict(keep_first=6), dict(conv=2), dict(diff=0.31),
    dict(rope=RopeSpec(8, 5000.0)), dict(rope=RopeSpec(6, 5000.0, 3.0, 1.0, 4.0, 100)), dict(scale=0.4)], ids=str)
def test_every_constant_shows_in_the_logits(change):
    """The tests' weights are such that a constant that is slightly off moves the logits by more than the GPU tests allow."""
    import dataclasses
    cfg = looped_config()
    p, toks = params(cfg), tokens(120, cfg.vocab_size)
    want = oracle_logits(cfg, p, toks)
    s = cfg.layer_specs[0]
    bad = dataclasses.replace(s, mixer=dataclasses.replace(s.mixer, **change))
    q = {k: v[:, 1:] if change.get("conv") and k.startswith("l0.") and k.endswith(".conv") else v for k, v in p.items()}
    assert err(oracle_logits(cfg.replace(layer_specs=(bad,) + cfg.layer_specs[1:]), q, toks), want).max() > 5e-3


# ---- scheduler over the oracle backend -----------------------------------------------------------------------------------
def greedy(cfg, p, prompt, n):
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    st, out = m.new_state(), []
    with torch.no_grad():
        lg = m.forward(torch.tensor(prompt), st)[-1]
        for _ in range(n):
            out.append(int(lg.argmax()))
            lg = m.forward(torch.tensor(out[-1:]), st)[-1]
    return out


@pytest.mark.parametrize("draft", [False, True])
def test_scheduler_generates_like_the_oracle(draft):
    from cuteafd_b200.runtime.backends import OracleBackend
    from cuteafd_b200.runtime.scheduler import Request, Scheduler, collect
    from cuteafd_b200.runtime.speculation import NgramDrafter
    cfg = looped_config()
    p = params(cfg)
    be = OracleBackend(cfg, p, total_pages=64, prefill_chunk=24)
    sched = Scheduler(be, drafter=NgramDrafter(block=3) if draft else None)
    prompts = [tokens(70, cfg.vocab_size, 1), tokens(5, cfg.vocab_size, 2), (tokens(7, cfg.vocab_size, 3) * 5)[:31]]
    reqs = [sched.submit(Request(list(q), max_tokens=12)) for q in prompts]
    for _ in range(400):
        sched.step()
    for q, r in zip(prompts, reqs):
        assert collect(r, 1.0)["tokens"] == greedy(cfg, p, q, 12)


def test_serve_builds_over_a_snapshot(tmp_path):
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    cfg = looped_config().replace(vocab_size=271)            # the byte tokenizer takes 260
    path = write_random_snapshot(cfg, str(tmp_path / "m"), seed=3)
    st = build_state(build_parser().parse_args(["serve", "--fake-engine", "--snapshot", path, "--speculator", "off"]))
    r = st.sched.submit(Request([5, 6, 7], max_tokens=4))
    for _ in range(20):
        st.sched.step()
    _, p = load_params(path)
    assert collect(r, 1.0)["tokens"] == greedy(cfg, p, [5, 6, 7], 4)
