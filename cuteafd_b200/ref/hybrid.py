"""CPU oracle of the per-layer hybrid decoders (``ModelConfig.layer_specs``): windowed latent attention layers and gated
delta-rule layers in any order, each behind grouped RMS norms, input convolutions and a routed feed-forward; parallel
layers of plain or differential or latent attention beside a dense or routed feed-forward, some of them looped; layers normed
after their sublayers (gated linear recurrences, attention beside linear attention) with averages over depth.

One function per mechanism, written as the equations read: no chunking, no absorbed products, one token at a time where a
recurrence runs.  ``HybridRefDecoder`` strings them together over a parameter dictionary in the checkpoint's own tensor
names and plugs into the same places as ``RefDecoder``.  All arithmetic is in the dtype the parameters are given in
(fp32 or fp64); nothing here is shared with the CUDA path.
"""
from __future__ import annotations

import math

import torch

from ..config import AttentionSpec, DeltaSpec, DenseSpec, LatentSpec, LightningSpec, ModelConfig, PairSpec, RglruSpec, RopeSpec, RouterSpec

Params = dict[str, torch.Tensor]


# ---- mechanisms -----------------------------------------------------------------------------------------------------
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_rms(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """RMS norm in ``groups`` equal runs of channels, each with its own root mean square; one weight per channel."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * w


def causal_conv(x: torch.Tensor, w: torch.Tensor, past: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """Per-channel causal convolution over time.  x [T, C], w [C, taps] (last column = the current token), ``past``
    [taps - 1, C] the inputs just before x.  Returns (y [T, C], the new past)."""
    taps, T = w.shape[1], x.shape[0]
    full = torch.cat([past, x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + w[:, j] * full[j:j + T]
    return y, full[T:]


def scaled_frequencies(r: RopeSpec) -> list[float]:
    """Turns per position (in radians) of every rotated pair.

    bands: short wavelengths as they are, long ones stretched by the factor, a linear blend (in turns over the original length)
    between.  linear: all stretched.  yarn: pair number x makes ``turns`` turns over the original length at
    x = dims * ln(original / (2 pi turns)) / (2 ln base); from the x of ``high`` turns (rounded down) to that of ``low`` turns
    (rounded up) the blend is linear in the pair's number."""
    f = [r.base ** (-2.0 * i / r.dims) for i in range(r.dims // 2)]
    if r.factor == 1.0:
        return f
    if r.kind == "linear":
        return [x / r.factor for x in f]
    out = []
    if r.kind == "yarn":
        number = lambda turns: r.dims * math.log(r.original / (2.0 * math.pi * turns)) / (2.0 * math.log(r.base))      # noqa: E731
        lo, hi = max(math.floor(number(r.high)), 0), min(math.ceil(number(r.low)), r.dims - 1)
        for i, x in enumerate(f):
            ramp = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
            out.append(x / r.factor * ramp + x * (1.0 - ramp))
        return out
    for x in f:
        turns = r.original * x / (2.0 * math.pi)                  # original length over wavelength
        if turns < r.low:
            x = x / r.factor
        elif turns <= r.high:
            s = (turns - r.low) / (r.high - r.low)
            x = (1.0 - s) * x / r.factor + s * x
        out.append(x)
    return out


def rotate(x: torch.Tensor, positions: torch.Tensor, r: RopeSpec) -> torch.Tensor:
    """x [T, ..., d]: the pairs of the first ``r.dims`` dimensions, neighbours (2i, 2i + 1) or halves (i, i + dims / 2), are turned by
    position * frequency; cosines and sines carry the scaling's magnitude."""
    h = r.dims // 2
    mag = 0.1 * math.log(r.factor) + 1.0 if r.kind == "yarn" else 1.0
    a = positions.to(x.dtype)[:, None] * torch.tensor(scaled_frequencies(r), dtype=x.dtype)
    a = a.reshape(a.shape[0], *([1] * (x.dim() - 2)), h)
    c, s = mag * a.cos(), mag * a.sin()
    first, second = (slice(0, h), slice(h, r.dims)) if r.halves else (slice(0, r.dims, 2), slice(1, r.dims, 2))
    out = x.clone()
    u, v = x[..., first], x[..., second]
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, start: int, window: int, keep: int, scale: float,
                   sink: torch.Tensor | None = None, cap: float = 0.0) -> torch.Tensor:
    """Softmax attention of q [T, H, Dk] (positions start, start + 1, ...) over k [L, H, Dk], v [L, H, Dv] (positions 0, 1, ...):
    the query at position i reads the keys j <= i that lie among the last ``window`` positions (0: anywhere) or the first
    ``keep``.  ``sink`` [H]: a further logit per head that takes a share of the softmax and hands nothing through.  ``cap``: scores
    are cap * tanh(score / cap)."""
    i = torch.arange(start, start + q.shape[0])[:, None]
    j = torch.arange(k.shape[0])[None]
    seen = (j <= i) & ((i - j < window) | (j < keep)) if window else j <= i
    s = torch.einsum("thd,jhd->htj", q, k) * scale
    if cap:
        s = softcap(s, cap)
    s = s.masked_fill(~seen, -math.inf)
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, q.shape[0], 1)], -1)
    return torch.einsum("htj,jhd->thd", torch.softmax(s, -1)[..., :k.shape[0]], v)


def difference_weight(p: Params, pre: str, diff: float) -> torch.Tensor:
    """lambda: the weight of the second map, one number per layer."""
    return torch.exp((p[pre + "lq1"] * p[pre + "lk1"]).sum()) - torch.exp((p[pre + "lq2"] * p[pre + "lk2"]).sum()) + diff


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(x / cap)


def window_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, start: int, window: int, scale: float) -> torch.Tensor:
    """Softmax attention of q [T, H, Dk] (positions start, start + 1, ...) over k [L, H, Dk], v [L, H, Dv] (positions 0, 1, ...);
    the query at position i reads keys i - window + 1 .. i (window 0: 0 .. i)."""
    out = []
    for t in range(q.shape[0]):
        i = start + t
        lo = max(0, i - window + 1) if window else 0
        s = torch.einsum("hd,jhd->hj", q[t], k[lo:i + 1]) * scale
        out.append(torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[lo:i + 1]))
    return torch.stack(out)


def delta_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: torch.Tensor, g: torch.Tensor,
                     S: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """Gated delta rule.  q, k [T, H, D], v [T, H, Dv], beta, g [T, H], S [H, D, Dv].  Per token: decay the state, move
    what it holds under k towards v by beta, read with q (the read sees this token's write)."""
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + torch.einsum("hd,hv->hdv", k[t], u)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def decayed_products(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay, S: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """Linear attention.  q, k [T, H, D], v [T, H, Dv], S [H, D, Dv]: per token the state of head h fades by decay[h], takes k v^T
    and is read with q (the read sees this token's write)."""
    d = torch.tensor(decay, dtype=S.dtype)[:, None, None]
    out = []
    for t in range(q.shape[0]):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def block_products(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C] in equal parts, part n through the square matrix w[n] [out, in] with the offsets b[n]."""
    parts = u.view(u.shape[0], w.shape[0], -1)
    return torch.stack([parts[:, n] @ w[n].T + b[n] for n in range(w.shape[0])], 1).reshape(u.shape)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def gated_recurrence(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor, c: float, S: torch.Tensor):
    """u, r, i [T, C] (r and i in (0, 1)), S [C]: log a = -c r softplus(lam), S <- a S + sqrt(1 - a^2) i u.  Returns (all S, the last)."""
    out = []
    for t in range(u.shape[0]):
        log_a = -c * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out), S


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def bigram_rows(tokens: list[int], previous: int, buckets: int, mul_prev: int, mul_cur: int) -> list[int]:
    """Row of the second embedding table for each token; ``previous``: the token before them, -1 at a sequence's start."""
    out = []
    for t in tokens:
        out.append(buckets if previous < 0 else (previous * mul_prev + t * mul_cur) % buckets)
        previous = t
    return out


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def route(h: torch.Tensor, w: torch.Tensor, correction: torch.Tensor, r: RouterSpec) -> tuple[torch.Tensor, torch.Tensor]:
    """Softmax scores over experts and identity experts; the choice goes by score + correction inside the best groups
    (a group counts by its best member); the weights are the plain scores.  Returns (ids [T, top], weights [T, top])."""
    s = torch.softmax(h @ w.T, -1)
    ids, wts = [], []
    n = s.shape[1]
    for t in range(s.shape[0]):
        choice = s[t] + correction
        per = n // r.groups
        best = [(max(choice[g * per:(g + 1) * per].tolist()), -g) for g in range(r.groups)]
        kept = {-g for _, g in sorted(best, reverse=True)[:r.groups_kept]}
        order = sorted((e for e in range(n) if e // per in kept), key=lambda e: (-float(choice[e]), e))[:r.top]
        ids.append(order)
        wts.append(s[t][order])
    return torch.tensor(ids), torch.stack(wts)


def route_by_logits(h: torch.Tensor, w: torch.Tensor, bias: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """The ``top`` largest of the biased logits; the weights are the softmax over those alone."""
    z = h @ w.T + bias
    ids = torch.tensor([sorted(range(z.shape[1]), key=lambda e: (-float(row[e]), e))[:top] for row in z])
    return ids, torch.softmax(z.gather(1, ids), -1)


def route_by_sigmoid(h: torch.Tensor, w: torch.Tensor, correction: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Sigmoid scores; the ``top`` largest of score + correction are chosen and weigh in with their plain scores."""
    s = torch.sigmoid(h @ w.T)
    ids = torch.tensor([sorted(range(s.shape[1]), key=lambda e: (-float(row[e]), e))[:top] for row in s + correction])
    return ids, s.gather(1, ids)


def routed_ffn(h: torch.Tensor, p: Params, pre: str, r: RouterSpec) -> torch.Tensor:
    if r.logit_bias:
        ids, wts = route_by_logits(h, p[pre + "router"], p[pre + "router.b"], r.top)
    elif r.scoring == "sigmoid":
        ids, wts = route_by_sigmoid(h, p[pre + "router"], p[pre + "correction"], r.top)
    else:
        ids, wts = route(h, p[pre + "router"], p[pre + "correction"], r)
    y = torch.zeros_like(h)
    for e in ids.unique().tolist():
        t, slot = (ids == e).nonzero(as_tuple=True)
        x = h[t]
        if e < r.experts:
            x = (silu(x @ p[f"{pre}e{e}.gate"].T) * (x @ p[f"{pre}e{e}.up"].T)) @ p[f"{pre}e{e}.down"].T
        y[t] += wts[t, slot][:, None] * x
    return y


# ---- mixers ---------------------------------------------------------------------------------------------------------
def latent_mixer(h: torch.Tensor, p: Params, pre: str, m: LatentSpec, eps: float, start: int, st: dict) -> torch.Tensor:
    """Latent attention: keys and values of every head come out of one normed latent per token; a shared rotated key part."""
    T = h.shape[0]
    pos = torch.arange(start, start + T)
    q = (h @ p[pre + "q"].T).view(T, m.heads, m.dim + m.rot_dim)
    q = torch.cat([q[..., :m.dim], rotate(q[..., m.dim:], pos, m.rope)], -1)
    d = h @ p[pre + "dkv"].T
    c = rms(d[:, :m.kv_rank], eps) * p[pre + "dkv.norm"]
    kr = rotate(d[:, m.kv_rank:], pos, m.rope)
    st["c"] = torch.cat([st["c"], c])
    st["kr"] = torch.cat([st["kr"], kr])
    L = st["c"].shape[0]
    k = (st["c"] @ p[pre + "uk"].T).view(L, m.heads, m.dim)
    k = torch.cat([k, st["kr"][:, None].expand(L, m.heads, m.rot_dim)], -1)
    v = (st["c"] @ p[pre + "uv"].T).view(L, m.heads, m.vdim)
    o = window_attention(q, k, v, start, m.window, m.scale).reshape(T, m.heads * m.vdim)
    if m.gate:
        o = o * torch.sigmoid(h @ p[pre + "g"].T)
    return o @ p[pre + "o"].T


def delta_mixer(h: torch.Tensor, p: Params, pre: str, m: DeltaSpec, eps: float, st: dict) -> torch.Tensor:
    T = h.shape[0]
    x = {}
    for n in ("q", "k", "v"):
        y, st["conv." + n] = causal_conv(h @ p[pre + n].T, p[pre + n + ".conv"], st["conv." + n])
        x[n] = silu(y)
    rep = m.heads // m.kv_heads
    q = unit(x["q"].view(T, m.kv_heads, m.dim)).repeat_interleave(rep, 1) * m.dim ** -0.5
    k = unit(x["k"].view(T, m.kv_heads, m.dim)).repeat_interleave(rep, 1)
    v = x["v"].view(T, m.heads, m.vdim)
    beta = torch.sigmoid(h @ p[pre + "b"].T)
    a = h @ p[pre + "a"].T + p[pre + "dt_bias"]
    g = torch.exp(-torch.exp(p[pre + "A_log"]) * torch.log1p(torch.exp(-a.abs())).add(a.clamp_min(0)))
    o, st["S"] = delta_recurrence(q, k, v, beta, g, st["S"])
    o = rms(o, eps) * p[pre + "norm"]
    o = o.reshape(T, m.heads * m.vdim) * silu(h @ p[pre + "g"].T)
    return o @ p[pre + "o"].T


def attention_mixer(h: torch.Tensor, p: Params, pre: str, m: AttentionSpec, eps: float, start: int, st: dict) -> torch.Tensor:
    """Attention with convolved, normed and rotated queries and keys; with two maps per head their difference, normed per head."""
    T, rep = h.shape[0], m.heads // m.kv_heads
    pos = torch.arange(start, start + T)
    x = {}
    for n in ("q", "k") if m.v_from_k else ("q", "k", "v"):
        x[n] = h @ p[pre + n].T
        if m.conv:
            x[n], st["conv." + n] = causal_conv(x[n], p[pre + n + ".conv"], st["conv." + n])
    v = x["k" if m.v_from_k else "v"].view(T, m.kv_heads, m.vdim)
    st["v"] = torch.cat([st["v"], rotate(v, pos, m.v_rope) if m.v_rope else v])
    for n in ("q", "k"):
        if m.qk_norm == "all":
            x[n] = rms(x[n], eps) * p[f"{pre}{n}.norm"]
        elif m.qk_norm == "head":
            x[n] = (rms(x[n].view(T, -1, m.dim), eps) * p[f"{pre}{n}.norm"]).view(T, -1)
    q, k = rotate(x["q"].view(T, m.heads, m.maps, m.dim), pos, m.rope), rotate(x["k"].view(T, m.kv_heads, m.maps, m.dim), pos, m.rope)
    if m.qk_norm == "rotated":
        q, k = rms(q, eps), rms(k, eps)
    st["k"] = torch.cat([st["k"], k])
    k, v = st["k"].repeat_interleave(rep, 1), st["v"].repeat_interleave(rep, 1)
    sink = p[pre + "sink"] if m.sink else torch.zeros(m.heads, dtype=h.dtype) if m.unit_sink else None
    a = [sink_attention(q[:, :, j], k[:, :, j], v, start, m.window, m.keep_first, m.scale, sink, m.softcap) for j in range(m.maps)]
    if m.v_rope:
        a = [rotate(o, -pos, m.v_rope) for o in a]
    o = a[0] if m.maps == 1 else rms(a[0] - difference_weight(p, pre, m.diff) * a[1], eps) * (1 - m.diff)
    if m.gate:
        o = o * torch.sigmoid(h @ p[pre + "g"].T)[..., None]
    return o.reshape(T, m.heads * m.vdim) @ p[pre + "o"].T


def lightning_mixer(h: torch.Tensor, p: Params, pre: str, m: LightningSpec, eps: float, st: dict) -> torch.Tensor:
    T = h.shape[0]
    q, k = (silu(h @ p[pre + n].T).view(T, m.heads, m.dim) for n in "qk")
    o, st["S"] = decayed_products(q, k, silu(h @ p[pre + "v"].T).view(T, m.heads, m.vdim), m.decay, st["S"])
    o = rms(o.reshape(T, m.heads * m.vdim), eps) * p[pre + "norm"] * torch.sigmoid(h @ p[pre + "g"].T)
    return o @ p[pre + "o"].T


def pair_mixer(h: torch.Tensor, p: Params, pre: str, m: PairSpec, eps: float, start: int, st: dict) -> torch.Tensor:
    return (m.left_scale * attention_mixer(h, p, pre + "left.", m.left, eps, start, st)
            + m.right_scale * lightning_mixer(h, p, pre + "right.", m.right, eps, st))


def rglru_mixer(h: torch.Tensor, p: Params, pre: str, m: RglruSpec, st: dict) -> torch.Tensor:
    """Gated linear recurrence on one branch, gelu on the other, multiplied."""
    y = gelu_tanh(h @ p[pre + "y"].T + p[pre + "y.b"])
    u, st["conv"] = causal_conv(h @ p[pre + "x"].T + p[pre + "x.b"], p[pre + "conv"], st["conv"])
    u = u + p[pre + "conv.b"]
    r, i = (torch.sigmoid(block_products(u, p[pre + n], p[pre + n + ".b"])) for n in ("ra", "ri"))
    s, st["S"] = gated_recurrence(u, r, i, p[pre + "lam"], m.c, st["S"])
    return (s * y) @ p[pre + "o"].T


def dense_ffn(h: torch.Tensor, p: Params, pre: str, d: DenseSpec = DenseSpec(0)) -> torch.Tensor:
    g, u = h @ p[pre + "gate"].T, h @ p[pre + "up"].T
    if d.limit:
        g, u = g.clamp_max(d.limit), u.clamp(-d.limit, d.limit)
    return (g * torch.sigmoid(d.alpha * g) * (u + d.up_bias)) @ p[pre + "down"].T


def feed_forward(h: torch.Tensor, p: Params, pre: str, spec) -> torch.Tensor:
    """Dense, or the routed experts with the shared one beside them."""
    if spec.router is None:
        return dense_ffn(h, p, pre, spec.dense)
    y = routed_ffn(h, p, pre, spec.router)
    return y if spec.dense is None else y + dense_ffn(h, p, pre + "shared.", spec.dense)


def depth_average(w: torch.Tensor, results: list[torch.Tensor]) -> torch.Tensor:
    """The embedding rows and the layers' results so far, each times its weight."""
    x = torch.zeros_like(results[0])
    for a, y in zip(w, results, strict=True):
        x = x + a * y
    return x


def join_embedding(x: torch.Tensor, x0: torch.Tensor, p: Params, t: int) -> torch.Tensor:
    """Start of pass t of a loop: a product of [x; embedding row] and the pass's own vector."""
    return torch.cat([x, x0], -1) @ p["loop.in"].T + p["loop.step"][t]


# ---- state ----------------------------------------------------------------------------------------------------------
class HybridState:
    """What one sequence carries: latent records per position, and the recurrent parts.  The recurrent parts cannot be
    cut back, so the state keeps a copy per token of the last call; ``truncate`` returns to one of them."""

    def __init__(self, cfg: ModelConfig, dtype: torch.dtype = torch.float32):
        self.length_ = 0
        self.last_token = -1
        self.layers: list[dict] = []
        self.marks: dict[int, tuple] = {}
        for spec in (cfg.layer_specs[r.layer] for r in cfg.layer_runs):
            z = lambda *s: torch.zeros(*s, dtype=dtype)               # noqa: E731
            st = {} if spec.parallel or spec.post_norm else {"canon1": z(cfg.canon_taps - 1, cfg.hidden), "canon2": z(cfg.canon_taps - 1, cfg.hidden)}
            m = spec.mixer
            if isinstance(m, RglruSpec):
                st.update(S=z(m.width), conv=z(m.conv - 1, m.width))
                self.layers.append(st)
                continue
            if isinstance(m, PairSpec):
                st.update(S=z(m.right.heads, m.right.dim, m.right.vdim))
                m = m.left
            if isinstance(m, AttentionSpec):
                st.update(k=z(0, m.kv_heads, m.maps, m.dim), v=z(0, m.kv_heads, m.vdim))
                for n, c in (("q", m.q_channels), ("k", m.k_channels), ("v", m.v_channels)):
                    if m.conv and not (n == "v" and m.v_from_k):
                        st["conv." + n] = z(m.conv - 1, c)
            elif isinstance(m, LatentSpec):
                st.update(c=z(0, m.kv_rank), kr=z(0, m.rot_dim))
            else:
                st.update(S=z(m.heads, m.dim, m.vdim))
                for n, c in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                    st["conv." + n] = z(m.conv - 1, c)
            self.layers.append(st)

    def length(self, layer: int = 0) -> int:
        return self.length_

    @property
    def rows(self) -> list[list[torch.Tensor]]:
        """Every tensor of the state, per layer (state hashes)."""
        return [[st[k] for k in sorted(st)] for st in self.layers]

    def truncate(self, length: int) -> None:
        if length == self.length_:
            return
        if length not in self.marks:
            raise ValueError(f"recurrent state at {self.length_} tokens cannot return to {length}")
        layers, self.last_token = self.marks[length]
        self.layers = [dict(st) for st in layers]
        self.length_ = length

    def mark(self) -> None:
        self.marks[self.length_] = ([dict(st) for st in self.layers], self.last_token)


# ---- whole model ----------------------------------------------------------------------------------------------------
class HybridRefDecoder:
    def __init__(self, cfg: ModelConfig, params: Params, mark_rows: int = 16):
        self.cfg, self.p = cfg, params
        self.usage = None
        self.moe_fn = None
        self.mark_rows = mark_rows        # calls of at most this many tokens keep a state per token (``truncate``)
        self.trace: list | None = None    # residual after every layer, when set to a list

    def new_state(self) -> HybridState:
        return HybridState(self.cfg, self.p["embed"].dtype)

    def _layer(self, i: int, x: torch.Tensor, start: int, st: dict) -> torch.Tensor:
        cfg, p, spec, pre = self.cfg, self.p, self.cfg.layer_specs[i], f"l{i}."

        if spec.parallel:
            norm = lambda n: group_rms(x, p[pre + n] + cfg.norm_offset, cfg.norm_groups, cfg.rms_eps)      # noqa: E731
            mixer = latent_mixer if isinstance(spec.mixer, LatentSpec) else attention_mixer
            h = norm("norm1")
            y = mixer(h, p, pre + "mix.", spec.mixer, cfg.rms_eps, start, st)
            if spec.dense is None and spec.router is None:
                return x + y
            return x + (y + feed_forward(norm("norm2") if spec.two_norms else h, p, pre + "mlp.", spec))

        if spec.post_norm:
            m, norm = spec.mixer, lambda y, n: rms(y, cfg.rms_eps) * p[pre + n]                                   # noqa: E731
            y = pair_mixer(x, p, pre + "mix.", m, cfg.rms_eps, start, st) if isinstance(m, PairSpec) else rglru_mixer(x, p, pre + "mix.", m, st)
            x = x + norm(y, "norm1")
            return x + norm(feed_forward(x, p, pre + "mlp.", spec), "norm2") if spec.has_ffn else x

        def sublayer(x, n, fn):
            h = group_rms(x, p[f"{pre}norm{n}"], cfg.norm_groups, cfg.rms_eps)
            y, st[f"canon{n}"] = causal_conv(h, p[f"{pre}canon{n}"], st[f"canon{n}"])
            return x + group_rms(fn(h + y), p[f"{pre}norm{n}b"], cfg.norm_groups, cfg.rms_eps)

        m = spec.mixer
        if isinstance(m, LatentSpec):
            x = sublayer(x, 1, lambda h: latent_mixer(h, p, pre + "mix.", m, cfg.rms_eps, start, st))
        else:
            x = sublayer(x, 1, lambda h: delta_mixer(h, p, pre + "mix.", m, cfg.rms_eps, st))
        if spec.router is not None:
            x = sublayer(x, 2, lambda h: routed_ffn(h, p, pre + "mlp.", spec.router))
        return x

    def _run(self, tokens: torch.Tensor, kv: HybridState) -> torch.Tensor:
        e, start = self.p["embed"][tokens] * self.cfg.embed_scale, kv.length_
        if self.cfg.bigram:
            ids = tokens.tolist()
            e = e + self.p["bigram"][bigram_rows(ids, kv.last_token, *self.cfg.bigram)]
            kv.last_token = ids[-1] if ids else kv.last_token
        x, results = e, [e]
        for n, r in enumerate(self.cfg.layer_runs):
            if r.join >= 0:
                x = join_embedding(x, e, self.p, r.join)
            x = self._layer(r.layer, x + e if r.add_embedding else x, start, kv.layers[n])
            if self.cfg.depth_average:
                results.append(x)
                x = depth_average(self.p[f"l{r.layer}.dwa"], results)
            if self.trace is not None:
                self.trace.append(x)
        kv.length_ = start + tokens.shape[0]
        return x

    def hidden_states(self, tokens: torch.Tensor, kv: HybridState, embeds: tuple | None = None) -> torch.Tensor:
        if embeds is not None:
            raise ValueError("media rows are not part of this family")
        kv.marks = {}
        kv.mark()
        if tokens.shape[0] > self.mark_rows:
            return self._run(tokens, kv)
        out = []
        for t in range(tokens.shape[0]):
            out.append(self._run(tokens[t:t + 1], kv))
            kv.mark()
        return torch.cat(out)

    def head(self, x: torch.Tensor) -> torch.Tensor:
        cfg = self.cfg
        z = group_rms(x, self.p["final.norm"] + cfg.norm_offset, cfg.norm_groups, cfg.rms_eps) @ self.p["head"].T
        return softcap(z, cfg.logit_softcap) if cfg.logit_softcap else z

    def forward(self, tokens: torch.Tensor, kv: HybridState, embeds: tuple | None = None) -> torch.Tensor:
        return self.head(self.hidden_states(tokens, kv, embeds))


def init_hybrid_weights(cfg: ModelConfig, seed: int = 0, dtype: torch.dtype = torch.float32, std: float | None = None) -> Params:
    """Random parameters under the checkpoint's tensor names, scaled so that every branch matters."""
    g = torch.Generator().manual_seed(seed)

    def w(*shape: int, s: float | None = None) -> torch.Tensor:
        return (torch.randn(*shape, generator=g) * (s if s is not None else std if std is not None else shape[-1] ** -0.5)).to(dtype)

    def near_one(n: int) -> torch.Tensor:
        return (1 - cfg.norm_offset + 0.2 * torch.randn(n, generator=g)).to(dtype)

    def latent_weights(x: str, m: LatentSpec) -> None:
        p.update({x + "q": w(m.heads * (m.dim + m.rot_dim), H), x + "dkv": w(m.kv_rank + m.rot_dim, H),
                  x + "dkv.norm": 1 + 0.2 * w(m.kv_rank, s=1.0), x + "uk": w(m.heads * m.dim, m.kv_rank), x + "uv": w(m.heads * m.vdim, m.kv_rank)})
        if m.gate:
            p[x + "g"] = w(m.heads * m.vdim, H)

    def routed_weights(x: str, r: RouterSpec) -> None:
        p[x + "router"] = w(r.outputs, H)
        p[x + ("router.b" if r.logit_bias else "correction")] = w(r.outputs, s=0.7 if r.logit_bias else 0.1)
        for e in range(r.experts):
            p[f"{x}e{e}.gate"], p[f"{x}e{e}.up"], p[f"{x}e{e}.down"] = w(r.ffn, H), w(r.ffn, H), w(H, r.ffn)

    H = cfg.hidden
    p: Params = {"embed": w(cfg.vocab_size, H, s=1.0 / cfg.embed_scale), "final.norm": near_one(1)[0] if cfg.norm_scalar else near_one(H), "head": w(cfg.vocab_size, H)}
    if cfg.loop and cfg.loop_join:
        p["loop.in"], p["loop.step"] = w(H, 2 * H), w(cfg.loop[2], H, s=0.3)
    if cfg.bigram:
        p["bigram"] = w(cfg.bigram[0] + 1, H, s=0.7)
    for i, spec in enumerate(cfg.layer_specs):
        pre, m, r = f"l{i}.", spec.mixer, spec.router
        if spec.post_norm:
            x = pre + "mix."
            for n in ("norm1", "norm2")[:1 + spec.has_ffn]:
                p[pre + n] = 0.8 * near_one(1)[0] if cfg.norm_scalar else near_one(H)
            if cfg.depth_average:
                p[pre + "dwa"] = torch.cat([w(i + 1, s=0.3), near_one(1)])
            if isinstance(m, PairSpec):
                a, b = m.left, m.right
                for n, c in (("q", a.q_channels), ("k", a.k_channels), ("v", a.v_channels)):
                    p[f"{x}left.{n}"] = w(c, H)
                p[x + "left.o"] = w(H, a.heads * a.vdim)
                for n, c in (("q", b.heads * b.dim), ("k", b.heads * b.dim), ("v", b.heads * b.vdim), ("g", b.heads * b.vdim)):
                    p[f"{x}right.{n}"] = w(c, H)
                p[x + "right.o"], p[x + "right.norm"] = w(H, b.heads * b.vdim), near_one(b.heads * b.vdim)
            else:
                c = m.width
                for n in "yx":
                    p[x + n], p[f"{x}{n}.b"] = w(c, H), w(c, s=0.5)
                p[x + "conv"], p[x + "conv.b"], p[x + "lam"] = w(c, m.conv), w(c, s=0.3), w(c, s=1.5) - 3
                for n in ("ra", "ri"):
                    p[x + n], p[f"{x}{n}.b"] = w(m.blocks, m.block, m.block), w(m.blocks, m.block, s=0.5)
                p[x + "o"] = w(H, c)
            if r is not None:
                routed_weights(pre + "mlp.", r)
            elif spec.dense is not None:
                d, x = spec.dense, pre + "mlp."
                p[x + "gate"], p[x + "up"], p[x + "down"] = w(d.ffn, H), w(d.ffn, H), w(H, d.ffn)
            continue
        if spec.parallel:
            x, d = pre + "mix.", spec.dense
            p[pre + "norm1"] = near_one(H)
            if isinstance(m, LatentSpec):
                latent_weights(x, m)
            else:
                for n, c in (("q", m.q_channels), ("k", m.k_channels), ("v", m.v_channels)):
                    if n == "v" and m.v_from_k:
                        continue
                    p[x + n] = w(c, H)
                    if m.conv:
                        p[x + n + ".conv"] = w(c, m.conv)
                    if m.qk_norm and n != "v":
                        p[f"{x}{n}.norm"] = 1 + 0.2 * w(m.dim if m.qk_norm == "head" else c, s=1.0)
                if m.sink:
                    p[x + "sink"] = w(m.heads, s=1.5)
                if m.gate:
                    p[x + "g"] = w(m.heads, H)
                if m.maps == 2:
                    p.update({x + n: w(m.dim, s=0.5 * m.dim ** -0.5) for n in ("lq1", "lk1", "lq2", "lk2")})
            p[x + "o"] = w(H, m.heads * m.vdim)
            if spec.two_norms and (r is not None or d is not None):
                p[pre + "norm2"] = near_one(H)
            if r is not None:
                routed_weights(pre + "mlp.", r)
            if d is not None:
                x = pre + ("mlp.shared." if r is not None else "mlp.")
                p[x + "gate"], p[x + "up"], p[x + "down"] = w(d.ffn, H), w(d.ffn, H), w(H, d.ffn)
            continue
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if r is not None else ()):
            p[pre + n] = near_one(H)
        for n in ("canon1",) + (("canon2",) if r is not None else ()):
            p[pre + n] = w(H, cfg.canon_taps, s=0.3)
        x = pre + "mix."
        if isinstance(m, LatentSpec):
            latent_weights(x, m)
        else:
            kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
            p.update({x + "q": w(kd, H), x + "k": w(kd, H), x + "v": w(vd, H), x + "g": w(vd, H), x + "b": w(m.heads, H),
                      x + "a": w(m.heads, H), x + "A_log": w(m.heads, s=0.5), x + "dt_bias": w(m.heads, s=1.0) - 2,
                      x + "norm": near_one(m.vdim), x + "q.conv": w(kd, m.conv), x + "k.conv": w(kd, m.conv), x + "v.conv": w(vd, m.conv)})
        p[x + "o"] = w(H, m.heads * m.vdim)
        if r is not None:
            routed_weights(pre + "mlp.", r)
    return p


def bf16_params(p: Params, dtype: torch.dtype = torch.float32) -> Params:
    """The parameters as a bfloat16 checkpoint holds them."""
    return {k: v.to(torch.bfloat16).to(dtype) for k, v in p.items()}


__all__ = ["HybridRefDecoder", "HybridState", "init_hybrid_weights", "bf16_params", "group_rms", "causal_conv", "rotate",
           "scaled_frequencies", "sink_attention", "difference_weight", "softcap", "attention_mixer", "dense_ffn", "feed_forward",
           "join_embedding", "window_attention", "delta_recurrence", "route", "route_by_logits", "routed_ffn", "latent_mixer", "delta_mixer",
           "rms", "unit", "decayed_products", "block_products", "softplus", "gated_recurrence", "gelu_tanh", "bigram_rows", "route_by_sigmoid",
           "lightning_mixer", "pair_mixer", "rglru_mixer", "depth_average"]
