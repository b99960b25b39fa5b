"""Per-layer hybrid decoders on the CPU: configuration and loading, the oracle's mechanisms, state slots, prefix cache and
scheduler over recurrent state."""
import json

import pytest
import torch

from cuteafd_b200.config import DeltaSpec, ModelConfig, RouterSpec, scaled_down
from cuteafd_b200.loader.load import load_params, open_snapshot
from cuteafd_b200.loader.snapshot import from_hf_config, to_hf_config, write_random_snapshot
from cuteafd_b200.ref import hybrid as R
from cuteafd_b200.runtime.paged import PagePool, SequenceTable
from cuteafd_b200.runtime.state import FIRST_SLOT, OutOfSlots, StatePool

from tests.hybrid_common import err, odd_config, oracle_logits, params, plain_config, tokens

CFGS = [odd_config(), plain_config()]


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_config_round_trips(cfg):
    d = json.loads(json.dumps(to_hf_config(cfg)))
    assert from_hf_config(d) == cfg
    assert ModelConfig.from_dict(json.loads(cfg.to_json())) == cfg
    assert scaled_down(cfg, 1, 64).layer_specs == cfg.layer_specs[:1]


def test_unknown_parts_are_refused():
    d = to_hf_config(odd_config())
    for change in (lambda e: e.update(type="something"), lambda e: e["mlp"].update(kind="dense"),
                   lambda e: e["mixer"]["rot"].update(dims=4), lambda e: e["mlp"]["router"]["groups"].update(count=3)):
        bad = json.loads(json.dumps(d))
        change(bad["layers"][0])
        with pytest.raises(ValueError):
            from_hf_config(bad)


def test_absent_router_options_mean_none():
    d = to_hf_config(plain_config())
    r = d["layers"][1]["mlp"]["router"]
    r.pop("groups"), r.pop("identity")
    assert from_hf_config(d).layer_specs[1].router == RouterSpec(2, 40, 2)


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_snapshot_is_recognised_and_sized(cfg, tmp_path):
    from cuteafd_b200.models.hybrid import HybridWeights, tensor_shapes
    path = write_random_snapshot(cfg, str(tmp_path / "m"))
    snap = open_snapshot(path)
    assert snap.family.id == "karusun" and not snap.hints() and snap.cfg.layer_specs == cfg.layer_specs
    shapes = tensor_shapes(cfg)
    assert {n: tuple(e.shape) for n, e in snap.catalog.entries.items()} == shapes
    assert cfg.total_params() == sum(e.numel for e in snap.catalog.entries.values())
    assert snap.model.classify("l0.mlp.e1.up") == ("routed_expert", 0, 1)
    assert {snap.model.classify(n)[0] for n in shapes} <= {"embedding", "head", "final_norm", "norm", "attention", "router", "routed_expert"}
    W = HybridWeights.build(snap.cfg, snap.catalog.read, torch.device("cpu"))
    assert len(W.layers) == cfg.num_layers
    _, p = load_params(path)
    assert set(p) == set(shapes)
    with pytest.raises(ValueError, match="shape"):
        HybridWeights.build(snap.cfg.replace(vocab_size=cfg.vocab_size + 1), snap.catalog.read, torch.device("cpu"))


def test_plan_places_a_hybrid_on_one_gpu(tmp_path):
    from cuteafd_b200.planner import plan as P
    rep = P.plan(write_random_snapshot(odd_config(), str(tmp_path / "m")), layout=True, gpus=8)
    assert rep.placement.ok and rep.placement.engine == "single"
    assert any(c == "recurrent state" for c in rep.placement.devices[0].by_category())
    assert "latent" in P.render(rep) and "delta" in P.render(rep)


# ---- the oracle against direct statements ------------------------------------------------------------------------------
def test_group_norm_and_convolution_by_hand():
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=torch.float64)
    y = R.group_rms(x, torch.tensor([1.0, 1.0, 1.0, 10.0], dtype=torch.float64), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[3 / 12.5 ** .5, 4 / 12.5 ** .5, 0.0, 10 * 2 / 2 ** .5]], dtype=torch.float64))
    w = torch.tensor([[0.5, 2.0, 1.0]])
    y, past = R.causal_conv(torch.tensor([[1.0], [10.0], [100.0]]), w, torch.zeros(2, 1))
    assert y.flatten().tolist() == [1.0, 12.0, 120.5] and past.flatten().tolist() == [10.0, 100.0]


def test_delta_rule_replaces_what_a_key_holds():
    k = torch.tensor([[[0.6, 0.8]]]).expand(2, 1, 2)
    v = torch.tensor([[[5.0]], [[7.0]]])
    one = torch.ones(2, 1)
    o, S = R.delta_recurrence(k, k, v, one, one, torch.zeros(1, 2, 1))
    assert torch.allclose(o.flatten(), torch.tensor([5.0, 7.0]))          # beta 1: the second write replaces the first
    o, _ = R.delta_recurrence(k, k, v, one * 0.5, one * 0.5, torch.zeros(1, 2, 1))
    assert torch.allclose(o.flatten(), torch.tensor([2.5, 1.25 + 0.5 * (7 - 1.25)]))


def test_route_groups_with_negative_choice_scores():
    r = RouterSpec(experts=4, ffn=1, top=2, identity=2, groups=3, groups_kept=1)
    h, w = torch.ones(1, 1), torch.tensor([[0.0], [1.0], [2.0], [0.0], [1.0], [0.5]])
    c = torch.tensor([-9.0, -2.0, -9.0, -3.0, -1.5, -8.0])
    ids, wts = R.route(h, w, c, r)
    assert ids.tolist() == [[4, 5]]                                       # the group of the best member, poor neighbour included
    s = torch.softmax(w[:, 0], -1)
    assert torch.allclose(wts[0], s[[4, 5]])


def test_identity_output_hands_the_input_through():
    r = RouterSpec(experts=1, ffn=3, top=1, identity=1)
    p = {"router": torch.zeros(2, 4), "correction": torch.tensor([0.0, 5.0])}
    h = torch.randn(3, 4)
    assert torch.allclose(R.routed_ffn(h, p, "", r), 0.5 * h)


def test_window_edges():
    q, k = torch.zeros(1, 1, 2), torch.zeros(9, 1, 2)
    v = torch.arange(9.0).view(9, 1, 1)
    assert R.window_attention(q, k, v, 8, 3, 1.0).item() == pytest.approx(7.0)        # 6, 7, 8
    assert R.window_attention(q, k, v, 8, 100, 1.0).item() == pytest.approx(4.0)


@pytest.mark.parametrize("cfg", CFGS, ids=lambda c: c.name)
def test_oracle_prefill_equals_token_by_token(cfg):
    p, toks = params(cfg), tokens(60, cfg.vocab_size)
    want = oracle_logits(cfg, p, toks, torch.float64)
    m = R.HybridRefDecoder(cfg, {k: v.double() for k, v in p.items()})
    st = m.new_state()
    with torch.no_grad():
        a = m.forward(torch.tensor(toks[:33]), st)
        b = torch.cat([m.forward(torch.tensor([t]), st) for t in toks[33:]])
    assert err(torch.cat([a, b]), want).max() < 1e-6


def test_oracle_state_returns_to_an_earlier_token():
    cfg = odd_config()
    p, toks = params(cfg), tokens(24, cfg.vocab_size)
    m = R.HybridRefDecoder(cfg, p)
    with torch.no_grad():
        st = m.new_state()
        m.forward(torch.tensor(toks[:20]), st)
        m.forward(torch.tensor([1, 2, 3, 4]), st)
        st.truncate(20)
        got = m.forward(torch.tensor(toks[20:]), st)
    assert err(got, oracle_logits(cfg, p, toks)[20:]).max() < 1e-5
    with pytest.raises(ValueError):
        st.truncate(3)


# ---- slots -------------------------------------------------------------------------------------------------------------
def test_state_slots_step_settle_and_free():
    sp = StatePool(FIRST_SLOT + 4)
    table = SequenceTable(PagePool(16), sp)
    a, b = table.new(), table.new()
    for s in (a, b):
        table.reserve(s, 5)
    ins, outs = sp.begin([a, b])
    assert ins == [0, 0] and len(set(outs)) == 2 and not set(outs) & {0, 1}
    for s in (a, b):
        s.kv_len = 5
    sp.commit([a, b], outs)
    assert (a.state, b.state) == tuple(outs) and sp.free_slots == 2 and a.lag == 0
    ins, o2 = sp.begin([a])                        # a speculative step of 4 rows, 2 of them kept
    a.kv_len = 9
    sp.commit([a], o2, keep_old=True)
    a.kv_len = 7
    sp.settle(a, 7)
    assert a.state == outs[0] and a.state_len == 5 and a.lag == 2 and sp.free_slots == 2
    ins, o3 = sp.begin([a])
    a.kv_len = 8
    sp.commit([a], o3, keep_old=True)
    sp.settle(a, 8)
    assert a.state == o3[0] and a.lag == 0 and a.old_state is None and sp.free_slots == 2
    c = table.fork(a)
    assert sp.refs[a.state] == 2
    with pytest.raises(ValueError):
        table.fork(a, 3)
    for s in (a, b, c):
        table.free(s)
    assert sp.free_slots == 4
    x = [table.new() for _ in range(5)]
    with pytest.raises(OutOfSlots):
        sp.begin(x)
    assert sp.free_slots == 4                      # a refused step leaves nothing taken


# ---- scheduler over the oracle backend -----------------------------------------------------------------------------------
def _greedy(cfg, p, prompt, n):
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
    cfg = odd_config()
    p = params(cfg)
    be = OracleBackend(cfg, p, total_pages=64, prefill_chunk=24)
    sched = Scheduler(be, drafter=NgramDrafter(block=3) if draft else None)
    prompts = [tokens(70, cfg.vocab_size, 1), tokens(5, cfg.vocab_size, 2), (tokens(7, cfg.vocab_size, 3) * 5)[:31]]
    reqs = [sched.submit(Request(list(q), max_tokens=12)) for q in prompts]
    for _ in range(400):
        sched.step()
    for q, r in zip(prompts, reqs):
        assert collect(r, 1.0)["tokens"] == _greedy(cfg, p, q, 12)
    again = prompts[0] + _greedy(cfg, p, prompts[0], 12)[:11] + [3, 4]     # resumes from the turn's snapshot
    r = sched.submit(Request(list(again), max_tokens=6))
    for _ in range(100):
        sched.step()
    got = collect(r, 1.0)
    assert got["tokens"] == _greedy(cfg, p, again, 6) and got["usage"]["cached_tokens"] in (70, 81)


def test_serve_builds_over_a_snapshot(tmp_path):
    from cuteafd_b200.cli import build_parser
    from cuteafd_b200.runtime.scheduler import Request, collect
    from cuteafd_b200.serve.server import build_state
    cfg = odd_config().replace(vocab_size=271)            # the byte tokenizer takes 260
    path = write_random_snapshot(cfg, str(tmp_path / "m"), seed=3)
    st = build_state(build_parser().parse_args(["serve", "--fake-engine", "--snapshot", path, "--speculator", "off"]))
    r = st.sched.submit(Request([5, 6, 7], max_tokens=4))
    for _ in range(20):
        st.sched.step()
    _, p = load_params(path)
    assert collect(r, 1.0)["tokens"] == _greedy(cfg, p, [5, 6, 7], 4)


def test_delta_channels():
    assert DeltaSpec(6, 2, 20, 36, 3).conv_channels == 2 * 40 + 216
