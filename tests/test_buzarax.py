"""Layers normed after their sublayers (gated linear recurrences, attention beside linear attention, averages over depth) without a GPU:
configuration reader, registry, loading, the oracle's mechanisms by hand and against itself, planning, scheduler and serving over the
oracle backend."""
import dataclasses
import json
import math

import pytest
import torch

from cuteafd_b200.config import DenseSpec, ModelConfig, RopeSpec, RouterSpec, buzarax_bench, buzarax_bench_gqa, scaled_down
from cuteafd_b200.loader.load import load_params, open_snapshot
from cuteafd_b200.loader.snapshot import from_hf_config, to_hf_config, write_random_snapshot
from cuteafd_b200.ref import hybrid as R

from tests.hybrid_common import averaged_config, dual_config, err, faint_config, fading, oracle_logits, params, tokens, turned
from tests.test_rofapel import greedy

CFGS = [averaged_config(), faint_config(), dual_config()]


# ---- configuration -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cfg", CFGS + [buzarax_bench("small"), scaled_down(buzarax_bench(), 3)], ids=lambda c: c.name)
def test_config_round_trip(cfg):
    d = json.loads(json.dumps(to_hf_config(cfg)))
    back = from_hf_config(d)
    assert back.layer_specs == cfg.layer_specs and back == cfg
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg


def test_config_keys():
    """The reader against a configuration written out by hand."""
    d = {"architecture": "Buzarax", "vocab": 99, "width": 48, "norm": {"eps": 1e-4}, "logit_softcap": 12.0,
         "embedding": {"bigram": {"buckets": 53, "mul_prev": 11, "mul_cur": 3}},
         "layers": [
             {"type": "rglru", "mixer": {"width": 30, "blocks": 6, "conv": 2}, "mlp": {"kind": "dense", "ff": 31, "limit": 0.9}},
             {"type": "parallel", "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 2}}, "mixer": {
                 "left": {"heads": 6, "kv_heads": 3, "dim": 14, "vdim": 10, "scale": 0.4, "softcap": 7.0,
                          "rot": {"base": 123.0, "dims": 8, "scaling": {"factor": 2.0, "original": 77, "fast": 9.0, "slow": 1.5}}},
                 "right": {"heads": 2, "dim": 5, "vdim": 9, "decay": [0.5, 0.75]}, "left_scale": 0.3, "right_scale": 1.7}},
             {"type": "rglru", "mixer": {"width": 8, "blocks": 1, "conv": 1}, "mlp": None}]}
    c = from_hf_config(d)
    a, b, e = c.layer_specs
    assert (a.mixer.width, a.mixer.blocks, a.mixer.block, a.mixer.conv, a.mixer.c) == (30, 6, 5, 2, 8.0)
    assert a.dense == DenseSpec(31, 0.9, 1.702, 1.0) and a.router is None
    m = b.mixer
    assert (m.left_scale, m.right_scale, m.left.heads, m.left.kv_heads, m.left.dim, m.left.vdim, m.left.scale) == (0.3, 1.7, 6, 3, 14, 10, 0.4)
    assert m.left.rope == RopeSpec(8, 123.0, 2.0, 1.5, 9.0, 77, "yarn", halves=True) and m.left.v_rope == RopeSpec(10, 123.0, halves=True)
    assert (m.left.softcap, m.left.unit_sink, m.left.qk_norm, m.left.window, m.left.conv, m.left.sink, m.left.gate) == (7.0, True, "rotated", 0, 0, False, False)
    assert (m.right.heads, m.right.dim, m.right.vdim, m.right.decay) == (2, 5, 9, (0.5, 0.75))
    assert b.router == RouterSpec(5, 12, 2, scoring="sigmoid") and b.dense is None and not b.router.normalize
    assert not e.has_ffn and all(s.post_norm and not s.parallel for s in c.layer_specs)
    assert (c.vocab_size, c.hidden, c.rms_eps, c.bigram, c.logit_softcap, c.depth_average, c.norm_scalar) == (99, 48, 1e-4, (53, 11, 3), 12.0, True, True)
    assert from_hf_config(dict(d, embedding={})).bigram == ()


def test_unknown_parts_are_refused():
    d = to_hf_config(averaged_config())
    left = lambda e: e["mixer"]["left"]                                         # noqa: E731
    for i, change in ((0, lambda e: e.update(type="delta")), (1, lambda e: e["mlp"].update(kind="other")), (0, lambda e: left(e)["rot"].update(dims=22)),
                      (0, lambda e: left(e).update(kv_heads=4)), (0, lambda e: left(e).update(vdim=13)), (1, lambda e: e["mixer"].update(blocks=5)),
                      (0, lambda e: left(e)["rot"].update(scaling={"factor": 2.0, "low": 1.0})), (1, lambda e: e["mlp"]["expert"].update(act="gelu")),
                      (1, lambda e: e["mlp"]["router"].update(top=7)), (0, lambda e: e["mixer"]["right"].update(decay=[0.5]))):
        bad = json.loads(json.dumps(d))
        change(bad["layers"][i])
        with pytest.raises(ValueError):
            from_hf_config(bad)


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_snapshot_is_recognised_and_sized(cfg, tmp_path):
    from cuteafd_b200.models.hybrid import HybridCache, HybridWeights, tensor_shapes
    path = write_random_snapshot(cfg, str(tmp_path / "m"))
    snap = open_snapshot(path)
    assert snap.family.id == "buzarax" and not snap.hints() and snap.cfg.layer_specs == cfg.layer_specs
    shapes = tensor_shapes(cfg)
    assert {n: tuple(e.shape) for n, e in snap.catalog.entries.items()} == shapes
    assert cfg.total_params() == sum(e.numel for e in snap.catalog.entries.values())
    assert snap.model.classify("bigram")[0] == "embedding" and snap.model.classify("l1.dwa") == ("norm", 1, None)
    assert {snap.model.classify(n)[0] for n in shapes} <= {"embedding", "head", "final_norm", "norm", "attention", "dense_ffn", "router", "routed_expert"}
    cpu = torch.device("cpu")
    W = HybridWeights.build(snap.cfg, snap.catalog.read, cpu)
    assert len(W.layers) == cfg.num_layers and W.bigram.shape[0] == cfg.bigram[0] + 1
    kv = HybridCache(cfg, 3, cpu, 4)
    pairs = [s.mixer for s in cfg.layer_specs if hasattr(s.mixer, "right")]
    recs = [s.mixer for s in cfg.layer_specs if hasattr(s.mixer, "blocks")]
    assert kv.bytes_per_page() == 128 * sum(m.left.k_channels + m.left.v_channels for m in pairs)
    floats = sum(m.right.heads * m.right.dim * m.right.vdim for m in pairs) + sum(m.conv * m.width for m in recs) + 1
    assert kv.state.shape[1] * 4 >= cfg.state_bytes == 4 * floats
    with pytest.raises(ValueError, match="shape"):
        HybridWeights.build(snap.cfg.replace(vocab_size=cfg.vocab_size + 1), snap.catalog.read, cpu)


def test_plan_places_it_on_one_gpu(tmp_path):
    from cuteafd_b200.planner import plan as P
    from cuteafd_b200.planner.capacity import workspace_bytes
    rep = P.plan(write_random_snapshot(averaged_config(), str(tmp_path / "m")), layout=True, gpus=8)
    assert rep.placement.ok and rep.placement.engine == "single"
    assert any(c == "recurrent state" for c in rep.placement.devices[0].by_category())
    assert "rg-lru" in P.render(rep) and "beside linear attention" in P.render(rep)
    c = buzarax_bench()
    assert workspace_bytes(c, 100) > 100 * 4 * c.hidden * len(c.layer_runs)     # every layer's result of a step is kept


def test_benchmark_sizes_match():
    for size in ("small", "base", "large"):
        a, b = buzarax_bench(size), buzarax_bench_gqa(size)
        assert a.num_layers == b.num_layers and (a.hidden, a.num_experts, a.expert_ffn, a.top_k) == (b.hidden, b.num_experts, b.expert_ffn, b.top_k)
        assert a.layer_specs[0].dense.ffn == b.dense_ffn and b.first_dense_layers == 1
        m = a.layer_specs[0].mixer.left
        assert (m.q_channels, m.k_channels, m.v_channels) == (b.num_heads * 128, b.num_kv_heads * 128, b.num_kv_heads * 128)


# ---- the oracle against direct statements ------------------------------------------------------------------------------
def test_scores_are_capped_and_the_unit_sink_takes_its_share():
    """One key: weight e^s / (1 + e^s) with s = cap tanh(q k scale / cap)."""
    q, k, v = torch.tensor([[[3.0, 0.0]]]), torch.tensor([[[2.0, 1.0]]]), torch.tensor([[[5.0, 7.0]]])
    s = 4 * math.tanh(6 * 0.5 / 4)
    w = math.exp(s) / (1 + math.exp(s))
    got = R.sink_attention(q, k, v, 0, 0, 0, 0.5, torch.zeros(1), 4.0)
    assert torch.allclose(got, w * v, atol=1e-6)


def test_rotated_norm_and_turned_values():
    """A norm after a rotation that scales; values as the cache holds them; a head that sees one key gets its value as it was, one at
    distance n turned by n."""
    m = turned(1, 1, 4, 2, RopeSpec(2, 10.0, 3.0, 1.0, 8.0, 50, "yarn", halves=True))
    eye = torch.eye(4)
    p = {"m.q": eye, "m.k": eye, "m.v": eye[:2], "m.o": torch.eye(2)}
    st = {"k": torch.zeros(0, 1, 1, 4), "v": torch.zeros(0, 1, 2)}
    h = torch.tensor([[1.0, 2.0, 3.0, 4.0], [4.0, -1.0, 0.5, 2.0], [0.0, 1.0, 2.0, 0.0]])
    o = R.attention_mixer(h, p, "m.", m, 1e-5, 0, st)
    mag = 0.1 * math.log(3.0) + 1
    norm2 = [float((mag * mag * x[:2].square().sum() + x[2:].square().sum()) / 4) for x in h]
    for t in range(3):
        assert abs(float(st["k"][t].square().mean()) - 1) < 1e-4 and torch.allclose(st["k"][t, 0, 0, 2:], h[t, 2:] / math.sqrt(norm2[t] + 1e-5), atol=1e-6)
        c, s = math.cos(t), math.sin(t)
        want = torch.tensor([h[t, 0] * c - h[t, 1] * s, h[t, 1] * c + h[t, 0] * s])
        assert torch.allclose(st["v"][t, 0], want, atol=1e-5)
    w = R.softcap(st["k"][0, 0, 0].square().sum() * m.scale, m.softcap).exp()
    assert torch.allclose(o[0], w / (1 + w) * h[0, :2], atol=1e-5)              # its own value: turned there and back


def test_linear_attention_by_hand():
    """o_t = sum over j <= t of decay^(t - j) (q_t . k_j) v_j."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(6, 2, d, generator=g, dtype=torch.float64) for d in (3, 3, 4))
    decay = (0.5, 0.9)
    o, S = R.decayed_products(q, k, v, decay, torch.zeros(2, 3, 4, dtype=torch.float64))
    for h in range(2):
        for t in range(6):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)
        assert torch.allclose(S[h], sum(decay[h] ** (5 - j) * torch.outer(k[j, h], v[j, h]) for j in range(6)))


def test_gated_recurrence_by_hand():
    lam, u, r, i = torch.tensor([0.3, -2.0]), torch.tensor([[1.0, -2.0], [0.5, 3.0]]), torch.tensor([[0.2, 0.9], [0.7, 0.1]]), torch.tensor([[0.6, 0.4], [0.5, 1.0]])
    s, last = R.gated_recurrence(u, r, i, lam, 8.0, torch.zeros(2))
    for c in range(2):
        S = 0.0
        for t in range(2):
            a = math.exp(-8 * float(r[t, c]) * math.log(1 + math.exp(float(lam[c]))))
            S = a * S + math.sqrt(1 - a * a) * float(i[t, c] * u[t, c])          # the first token is no special case
            assert abs(float(s[t, c]) - S) < 1e-6
    assert torch.equal(last, s[-1])
    w, b = torch.arange(8.0).view(2, 2, 2), torch.tensor([[1.0, 2.0], [3.0, 4.0]])
    got = R.block_products(torch.tensor([[1.0, 10.0, 100.0, 1000.0]]), w, b)
    assert got.tolist() == [[11.0, 34.0, 5403.0, 7604.0]]


def test_convolution_starts_from_zeros_not_from_the_bias():
    cfg = averaged_config()
    m = cfg.layer_specs[1].mixer
    p = params(cfg)
    st = {"S": torch.zeros(m.width), "conv": torch.zeros(m.conv - 1, m.width)}
    h = torch.zeros(1, cfg.hidden)
    R.rglru_mixer(h, p, "l1.mix.", m, st)
    u = p["l1.mix.conv"][:, -1] * p["l1.mix.x.b"] + p["l1.mix.conv.b"]
    gate = lambda n: torch.sigmoid(R.block_products(u[None], p["l1.mix." + n], p[f"l1.mix.{n}.b"]))[0]           # noqa: E731
    a = torch.exp(-8 * gate("ra") * torch.nn.functional.softplus(p["l1.mix.lam"]))
    assert torch.allclose(st["S"], torch.sqrt(1 - a * a) * gate("ri") * u, atol=1e-5)
    assert torch.equal(st["conv"][-1], p["l1.mix.x.b"]) and not st["conv"][0].any()


def test_clipped_feed_forward_by_hand():
    eye = torch.eye(3)
    p = {"f.gate": eye, "f.up": 2 * eye, "f.down": eye}
    h = torch.tensor([[0.5, 4.0, -3.0]])
    sig = lambda z: 1 / (1 + math.exp(-z))                                      # noqa: E731
    want = [0.5 * sig(0.851) * 2.0, 1.5 * sig(1.702 * 1.5) * 2.5, -3.0 * sig(-1.702 * 3) * -0.5]     # the gate is cut above only, up on both sides
    assert torch.allclose(R.dense_ffn(h, p, "f.", DenseSpec(3, 1.5, 1.702, 1.0)), torch.tensor([want]), atol=1e-6)


def test_sigmoid_routing_by_hand():
    """The correction chooses, the plain scores weigh, nothing is renormalised."""
    ids, w = R.route_by_sigmoid(torch.tensor([[1.0]]), torch.tensor([[2.0], [1.0], [0.0], [-1.0]]), torch.tensor([0.0, 0.0, 0.5, 0.4]), 2)
    assert ids.tolist() == [[2, 0]]
    assert torch.allclose(w, torch.sigmoid(torch.tensor([[0.0, 2.0]])))


def test_bigram_rows():
    assert R.bigram_rows([5, 7, 0], -1, 10, 3, 2) == [10, (15 + 14) % 10, 21 % 10]
    assert R.bigram_rows([65535], 65534, 65521, 1000003, 7919) == [(65534 * 1000003 + 65535 * 7919) % 65521]     # past 32 bits
    assert R.bigram_rows([3], 0, 10, 3, 2) == [6]                                # token 0 is a token before it


def test_average_over_depth():
    """Layers that add nothing: every result is the average before it, and X_0 is what the embedding gives."""
    cfg = averaged_config()
    p = params(cfg)
    for k in p:
        if k.endswith((".norm1", ".norm2")) and k.startswith("l"):
            p[k] = p[k] * 0
    m = R.HybridRefDecoder(cfg, p, mark_rows=0)
    m.trace, ids = [], torch.tensor([4, 9])
    m.forward(ids, m.new_state())
    e = p["embed"][ids] + p["bigram"][[97, (4 * 31 + 9 * 5) % 97]]
    sums = []
    for i in range(cfg.num_layers):
        w = p[f"l{i}.dwa"].tolist()
        results = [1.0, *([1.0] + sums)[:i + 1]]                                # X_0, X_1 = X_0's average so far, ...
        sums.append(sum(a * x for a, x in zip(w, results, strict=True)))
    for got, s in zip(m.trace, sums, strict=True):
        assert torch.allclose(got, s * e, atol=1e-4)


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
        st.truncate(71)
        again = m.forward(torch.tensor([2]), st)
        st.truncate(71)
        assert err(m.forward(torch.tensor([2]), st), again).max() < 1e-9 and st.last_token == 2
    with pytest.raises(ValueError):
        st.truncate(3)


def _pair(**kw):
    def change(m):
        left = {k: v for k, v in kw.items() if hasattr(m.left, k)}
        right = {k: v for k, v in kw.items() if k == "decay"}
        own = {k: v for k, v in kw.items() if k.endswith("_scale")}
        return dataclasses.replace(m, left=dataclasses.replace(m.left, **left), right=dataclasses.replace(m.right, **right), **own)
    return change


A = averaged_config().layer_specs[0].mixer
CHANGES = [(0, _pair(softcap=3.8)), (0, _pair(softcap=0.0)), (0, _pair(unit_sink=False)), (0, _pair(v_rope=None)), (0, _pair(qk_norm="")),
           (0, _pair(v_rope=RopeSpec(12, 290.0, halves=True))), (0, _pair(v_rope=RopeSpec(12, 300.0))), (0, _pair(scale=A.left.scale * 1.05)),
           (0, _pair(v_rope=dataclasses.replace(A.left.rope, dims=12))), (0, _pair(rope=dataclasses.replace(A.left.rope, halves=False))),
           (0, _pair(rope=dataclasses.replace(A.left.rope, factor=1.0))), (0, _pair(rope=dataclasses.replace(A.left.rope, original=2000))),
           (0, _pair(rope=dataclasses.replace(A.left.rope, high=12.0))), (0, _pair(rope=dataclasses.replace(A.left.rope, low=4.0))),
           (0, _pair(left_scale=0.72)), (0, _pair(right_scale=0.42)), (0, _pair(decay=fading(5, lo=0.5).decay)), (0, _pair(decay=A.right.decay[::-1])),
           (1, lambda m: dataclasses.replace(m, c=7.5))]


@pytest.mark.parametrize("n", range(len(CHANGES)))
def test_every_constant_shows_in_the_logits(n):
    """The tests' weights are such that a constant that is slightly off moves the logits by more than the 32-bit GPU tests allow."""
    layer, change = CHANGES[n]
    cfg = averaged_config()
    p, toks = params(cfg), tokens(90, cfg.vocab_size)
    s = cfg.layer_specs[layer]
    bad = cfg.replace(layer_specs=cfg.layer_specs[:layer] + (dataclasses.replace(s, mixer=change(s.mixer)),) + cfg.layer_specs[layer + 1:])
    assert err(oracle_logits(bad, p, toks), oracle_logits(cfg, p, toks)).max() > 2e-3


@pytest.mark.parametrize("change", [dict(bigram=(97, 31, 6)), dict(bigram=(97, 30, 5)), dict(bigram=()), dict(depth_average=False), dict(rms_eps=1e-2),
                                    dict(logit_softcap=8.0)], ids=str)
def test_every_model_constant_shows_in_the_logits(change):
    cfg = averaged_config()
    p, toks = params(cfg), tokens(40, cfg.vocab_size)
    assert err(oracle_logits(cfg.replace(**change), p, toks), oracle_logits(cfg, p, toks)).max() > 2e-3


# ---- scheduler over the oracle backend -----------------------------------------------------------------------------------
@pytest.mark.parametrize("draft", [False, True])
def test_scheduler_generates_like_the_oracle(draft):
    from cuteafd_b200.runtime.backends import OracleBackend
    from cuteafd_b200.runtime.scheduler import Request, Scheduler, collect
    from cuteafd_b200.runtime.speculation import NgramDrafter
    cfg = averaged_config()
    p = params(cfg)
    be = OracleBackend(cfg, p, total_pages=64, prefill_chunk=24)
    sched = Scheduler(be, drafter=NgramDrafter(block=3) if draft else None)
    prompts = [tokens(50, cfg.vocab_size, 1), tokens(5, cfg.vocab_size, 2), (tokens(7, cfg.vocab_size, 3) * 5)[:31]]
    reqs = [sched.submit(Request(list(q), max_tokens=8)) for q in prompts]
    for _ in range(400):
        if not sched.step() and not sched.pending and sched.waiting.empty():
            break
    for q, r in zip(prompts, reqs):
        assert collect(r, 1.0)["tokens"] == greedy(cfg, p, q, 8)


def test_serve_builds_over_a_snapshot(tmp_path):
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    cfg = averaged_config().replace(vocab_size=271)          # the byte tokenizer takes 260
    path = write_random_snapshot(cfg, str(tmp_path / "m"), seed=3)
    st = build_state(build_parser().parse_args(["serve", "--fake-engine", "--snapshot", path, "--speculator", "off"]))
    r = st.sched.submit(Request([5, 6, 7], max_tokens=4))
    for _ in range(20):
        st.sched.step()
    _, p = load_params(path)
    assert collect(r, 1.0)["tokens"] == greedy(cfg, p, [5, 6, 7], 4)
