"""Per-layer hybrid decoders (``ModelConfig.layer_specs``): windowed latent attention and gated delta-rule layers in any
order, grouped RMS norms before and after every sublayer, a causal convolution on every sublayer's input, routed
feed-forwards with identity outputs; and stacks of parallel layers (plain, differential or latent attention beside a dense or routed
feed-forward, under one norm or one each), some of them looped; and layers whose sublayers read the residual itself and are normed
after they ran (a gated linear recurrence, or attention beside linear attention), with averages over depth.

A layer is a fixed launch sequence over preallocated workspaces:

    norm_conv -> fused projection -> mixer kernels -> o projection -> norm_conv -> routes -> plan / dispatch -> fc1 -> fc2
    parallel:  norm_conv -> fused q / k / v -> conv_rope_kv -> attention -> gate / up -> [o | down] as one product
               (routed: the shared expert's gate / up and down there, routes -> plan / dispatch -> fc1 -> fc2 beside it)
    normed after: norm_conv -> fused projection -> [conv_rope_kv -> attention, linear attention -> norm + gate] or [convolution ->
               gates' product -> recurrence] -> o -> norm_conv -> feed-forward

``norm_conv`` is everything between two sublayers (the routed rows' weighted sum, the norm after the sublayer, the fp32
residual, the norm before the next one, its convolution).  What a sequence carries besides latent records lives in slots
of one fp32 pool; a step reads one slot per sequence and writes another (``Batch.state_in`` / ``state_out``), so a step
can be repeated and a slot can be shared with a cached prefix.  ``compute_dtype`` "f32" runs the same sequence with every
product and activation in 32-bit.  A looped layer runs several times with the same weights; cache and state belong to the run
(``ModelConfig.layer_runs``), not to the layer.  With averages over depth the layers' results of a step stay in fp32 buffers
until its last layer has read them.  Where a pass starts with a product of [x; embedding row], both halves lie in one
buffer whose second half is written once per step.
"""
from __future__ import annotations

import math

import torch

from ..config import AttentionSpec, DeltaSpec, DenseSpec, LatentSpec, ModelConfig, PairSpec, RglruSpec, RopeSpec, RouterSpec, attention_part
from ..ops import kernels as K
from ..parallel.moe_exchange import ExchangeGeometry, LocalExchange
from .gqa_moe import PAGE, Batch
from .mla_moe import _HeadTiles


def pad8(n: int) -> int:
    return -(-n // 8) * 8


def engine_dtype(cfg: ModelConfig) -> torch.dtype:
    return torch.float32 if cfg.compute_dtype == "f32" else torch.bfloat16


def record_pitch(m: LatentSpec) -> int:
    """Elements of one cached record: latent, rotated key part, padding to whole 16-byte pieces."""
    return pad8(m.record)


def rope_frequencies(r: RopeSpec) -> torch.Tensor:
    """fp32 [dims / 2] radians per position, worked out in fp64."""
    f = r.base ** (-torch.arange(0, r.dims, 2, dtype=torch.float64) / max(1, r.dims))
    if r.factor == 1.0 or not r.dims:
        return f.float()
    if r.kind == "linear":
        f = f / r.factor
    elif r.kind == "yarn":
        log_base = math.log(r.base)
        edge = [r.dims * math.log(r.original / (2 * math.pi * turns)) / (2 * log_base) for turns in (r.high, r.low)]
        lo, hi = max(math.floor(edge[0]), 0), min(math.ceil(edge[1]), r.dims - 1)
        ramp = ((torch.arange(r.dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        f = torch.lerp(f, f / r.factor, ramp)
    else:
        wave = 2 * torch.pi / f
        s = (r.original / wave - r.low) / (r.high - r.low) if r.high != r.low else torch.zeros_like(f)
        f = torch.where(wave < r.original / r.high, f, torch.where(wave > r.original / r.low, f / r.factor, (1 - s) * f / r.factor + s * f))
    return f.float()


def out_columns(m, d) -> tuple[int, int]:
    """Columns of a parallel layer's second product: (the heads' values, the dense activations after them).  Latent heads are
    written by a product whose rows are heads, so a row is then a whole number of heads long."""
    vp = pad8(m.vdim)
    f = pad8(d.ffn) if d is not None else 0
    return m.heads * vp, -(-f // vp) * vp if isinstance(m, LatentSpec) else f


class HybridLayer:
    """One layer's weights in the layout the kernels stream: the projections that read the same input are one matrix
    (``offs`` names its sections, each padded to a multiple of 8 rows), experts are stacked."""
    __slots__ = ("norm1", "norm1b", "norm2", "norm2b", "canon1", "canon2", "w_in", "offs", "w_o",
                 "kv_norm", "w_uk", "w_uv", "w_kb", "conv_w", "A_log", "dt_bias", "out_norm",
                 "router", "correction", "w_gate", "w_up", "w_down", "d_gate", "d_up", "d_down", "w_out", "lam", "q_norm", "k_norm",
                 "sink", "decay", "x_bias", "y_bias", "conv_b", "w_gates", "gate_bias", "dwa")

    def __init__(self) -> None:
        for s in self.__slots__:
            setattr(self, s, None)


class HybridWeights:
    def __init__(self, cfg: ModelConfig):
        self.cfg = cfg
        self.embed = self.bigram = self.final_norm = self.lm_head = self.loop_in = self.loop_step = None
        self.layers: list[HybridLayer] = []

    @staticmethod
    def build(cfg: ModelConfig, get, device: torch.device) -> "HybridWeights":
        """``get(name) -> tensor`` under the checkpoint's names (any float dtype, any device)."""
        dt = engine_dtype(cfg)
        H, Hp = cfg.hidden, pad8(cfg.hidden)

        def t(name: str, shape: tuple | None = None) -> torch.Tensor:
            x = get(name).to(device=device, dtype=dt)
            if shape is not None and tuple(x.shape) != shape:
                raise ValueError(f"{name}: shape {tuple(x.shape)}, the configuration says {shape}")
            return x.contiguous()

        def reads(x: torch.Tensor) -> torch.Tensor:
            """A matrix that reads the layer input: columns up to whole 16-byte rows."""
            return x if Hp == H else torch.nn.functional.pad(x, (0, Hp - H)).contiguous()

        def f(name: str, shape: tuple | None = None) -> torch.Tensor:
            x = get(name).to(device=device, dtype=torch.float32).contiguous()
            if shape is not None and tuple(x.shape) != shape:
                raise ValueError(f"{name}: shape {tuple(x.shape)}, the configuration says {shape}")
            return x

        def fuse(parts: list[tuple[str, torch.Tensor]]) -> tuple[torch.Tensor, dict]:
            rows = sum(pad8(x.shape[0]) for _, x in parts)
            out = torch.zeros(rows, Hp, dtype=dt, device=device)
            offs, o = {}, 0
            for n, x in parts:
                out[o:o + x.shape[0], :H] = x
                offs[n] = o
                o += pad8(x.shape[0])
            return out, offs

        def norm_weight(name: str) -> torch.Tensor:
            """A weight per channel, also where the checkpoint has one number for all of them."""
            return t(name, ()).expand(H).contiguous() if cfg.norm_scalar else t(name, (H,))

        def heads_o(name: str, heads: int, vdim: int) -> torch.Tensor:
            """o projection with every head's columns padded to the row layout the mixers write."""
            w = t(name, (H, heads * vdim)).view(H, heads, vdim)
            out = torch.zeros(Hp, heads, pad8(vdim), dtype=dt, device=device)
            out[:H, :, :vdim] = w
            return out.view(Hp, heads * pad8(vdim))

        W = HybridWeights(cfg)
        def attention(m: AttentionSpec, x: str, L: HybridLayer) -> None:
            own = ("q", "k") if m.v_from_k else ("q", "k", "v")
            rows = dict(q=m.q_channels, k=m.k_channels, v=m.v_channels)
            L.w_in, L.offs = fuse([(n, t(x + n, (rows[n], H))) for n in own] + ([("g", t(x + "g", (m.heads, H)))] if m.gate else []))
            if m.conv:
                L.conv_w = torch.cat([f(x + n + ".conv") for n in own])
                if tuple(L.conv_w.shape) != (m.conv_channels, m.conv):
                    raise ValueError(f"{x}*.conv: {tuple(L.conv_w.shape)}, the configuration says {(m.conv_channels, m.conv)}")
                L.conv_w = L.conv_w.T.contiguous()
            if m.qk_norm in ("head", "all"):
                L.q_norm, L.k_norm = (f(x + n + ".norm", (m.dim if m.qk_norm == "head" else rows[n],)) for n in ("q", "k"))
            if m.sink or m.unit_sink:
                L.sink = f(x + "sink", (m.heads,)) if m.sink else torch.zeros(m.heads, dtype=torch.float32, device=device)
            L.lam = 0.0
            if m.maps == 2:
                q1, k1, q2, k2 = (get(x + n).double() for n in ("lq1", "lk1", "lq2", "lk2"))
                L.lam = float((q1 * k1).sum().exp() - (q2 * k2).sum().exp()) + m.diff

        def latent(m: LatentSpec, x: str, L: HybridLayer) -> None:
            L.w_in, L.offs = fuse([("q", t(x + "q", (m.heads * (m.dim + m.rot_dim), H))), ("kv", t(x + "dkv", (m.record, H)))]
                                  + ([("g", t(x + "g", (m.heads * m.vdim, H)))] if m.gate else []))
            L.kv_norm = f(x + "dkv.norm", (m.kv_rank,))
            uk = t(x + "uk", (m.heads * m.dim, m.kv_rank)).view(m.heads, m.dim, m.kv_rank)
            L.w_uk = torch.zeros(m.heads, m.kv_rank, pad8(m.dim), dtype=dt, device=device)
            L.w_uk[..., :m.dim] = uk.transpose(1, 2)
            L.w_uv = torch.zeros(m.heads, m.vdim, pad8(m.kv_rank), dtype=dt, device=device)
            L.w_uv[..., :m.kv_rank] = t(x + "uv", (m.heads * m.vdim, m.kv_rank)).view(m.heads, m.vdim, m.kv_rank)
            if tensor_core_latent(cfg, m):
                L.w_kb = uk.reshape(m.heads * m.dim, m.kv_rank).contiguous()

        def routed(r: RouterSpec, y: str, L: HybridLayer) -> None:
            L.router, L.correction = reads(t(y + "router", (r.outputs, H))), f(y + ("router.b" if r.logit_bias else "correction"), (r.outputs,))
            F = pad8(r.ffn)
            L.w_gate, L.w_up = (torch.zeros(r.experts, F, Hp, dtype=dt, device=device) for _ in range(2))
            L.w_down = torch.zeros(r.experts, Hp, F, dtype=dt, device=device)
            for e in range(r.experts):
                L.w_gate[e, :r.ffn, :H] = t(f"{y}e{e}.gate", (r.ffn, H))
                L.w_up[e, :r.ffn, :H] = t(f"{y}e{e}.up", (r.ffn, H))
                L.w_down[e, :H, :r.ffn] = t(f"{y}e{e}.down", (H, r.ffn))

        def dense(d: DenseSpec, y: str, L: HybridLayer, F: int) -> torch.Tensor:
            """Gate and up into the layer; returns down [H padded, F]."""
            L.d_gate, L.d_up = (torch.zeros(F, Hp, dtype=dt, device=device) for _ in range(2))
            L.d_gate[:d.ffn, :H], L.d_up[:d.ffn, :H] = t(y + "gate", (d.ffn, H)), t(y + "up", (d.ffn, H))
            down = torch.zeros(Hp, F, dtype=dt, device=device)
            down[:H, :d.ffn] = t(y + "down", (H, d.ffn))
            return down

        def pair(m: PairSpec, x: str, L: HybridLayer) -> None:
            a, b = m.left, m.right
            if a.conv or a.gate or a.sink or a.maps != 1 or a.qk_norm not in ("", "rotated"):
                raise ValueError("attention with weights beyond its projections is not supported in a pair")
            attention(a, x + "left.", L)
            rows = dict(q=b.heads * b.dim, k=b.heads * b.dim, v=b.heads * b.vdim, g=b.heads * b.vdim)
            w, offs = fuse([(n, t(f"{x}right.{n}", (rows[n], H))) for n in rows])
            L.offs.update({"right." + n: o + L.w_in.shape[0] for n, o in offs.items()})
            L.w_in = torch.cat([L.w_in, w])
            L.w_out = torch.cat([heads_o(x + "left.o", a.heads, a.vdim), heads_o(x + "right.o", b.heads, b.vdim)], 1).contiguous()
            # the right half's factor rides on its norm's weights; the left half's on what its attention hands out
            L.out_norm = f(x + "right.norm", (b.heads * b.vdim,)) * m.right_scale
            L.decay = torch.tensor(b.decay, dtype=torch.float32, device=device)

        def rglru(m: RglruSpec, x: str, L: HybridLayer) -> None:
            c, n, bs, bp = m.width, m.blocks, m.block, pad8(m.block)
            L.w_in, L.offs = fuse([(k, t(x + k, (c, H))) for k in "xy"])
            L.x_bias, L.y_bias, L.conv_b, L.lam = (f(x + k, (c,)) for k in ("x.b", "y.b", "conv.b", "lam"))
            L.conv_w = f(x + "conv", (c, m.conv)).T.contiguous()
            L.w_gates = torch.zeros(n, 2, bp, bp, dtype=dt, device=device)
            L.gate_bias = torch.zeros(n, 2, bp, dtype=torch.float32, device=device)
            for j, k in enumerate(("ra", "ri")):
                L.w_gates[:, j, :bs, :bs] = t(x + k, (n, bs, bs))
                L.gate_bias[:, j, :bs] = f(f"{x}{k}.b", (n, bs))
            L.w_gates, L.gate_bias = L.w_gates.view(n, 2 * bp, bp), L.gate_bias.view(n, 2 * bp)
            L.w_out = torch.zeros(Hp, pad8(c), dtype=dt, device=device)
            L.w_out[:H, :c] = t(x + "o", (H, c))

        W.embed, W.final_norm, W.lm_head = t("embed", (cfg.vocab_size, H)), norm_weight("final.norm"), reads(t("head", (cfg.vocab_size, H)))
        if cfg.bigram:
            W.bigram = t("bigram", (cfg.bigram[0] + 1, H))
        if cfg.loop and cfg.loop_join:
            w = t("loop.in", (H, 2 * H))
            W.loop_in = torch.cat([reads(w[:, :H]), reads(w[:, H:])], 1).contiguous()
            W.loop_step = t("loop.step", (cfg.loop[2], H))
        for i, spec in enumerate(cfg.layer_specs):
            pre, m, r, L = f"l{i}.", spec.mixer, spec.router, HybridLayer()
            x = pre + "mix."
            if spec.post_norm:
                y = pre + "mlp."
                L.norm1b = norm_weight(pre + "norm1")
                (pair if isinstance(m, PairSpec) else rglru)(m, x, L)
                if spec.has_ffn:
                    L.norm2b = norm_weight(pre + "norm2")
                if r is not None:
                    routed(r, y, L)
                elif spec.dense is not None:
                    L.d_down = dense(spec.dense, y, L, pad8(spec.dense.ffn))
                if cfg.depth_average:
                    L.dwa = f(pre + "dwa", (i + 2,))
                W.layers.append(L)
                continue
            if spec.parallel:
                d, y = spec.dense, pre + "mlp."
                L.norm1 = t(pre + "norm1", (H,))
                if spec.two_norms and (d is not None or r is not None):
                    L.norm2 = t(pre + "norm2", (H,))
                if isinstance(m, LatentSpec):
                    if m.gate:
                        raise ValueError(f"layer {i}: gated latent attention beside a feed-forward is not supported")
                    latent(m, x, L)
                else:
                    attention(m, x, L)
                if r is not None:
                    routed(r, y, L)
                    y += "shared."
                L.w_out = heads_o(x + "o", m.heads, m.vdim)
                if d is not None:
                    L.w_out = torch.cat([L.w_out, dense(d, y, L, out_columns(m, d)[1])], 1).contiguous()
                W.layers.append(L)
                continue
            L.norm1, L.norm1b = t(pre + "norm1", (H,)), t(pre + "norm1b", (H,))
            L.canon1 = t(pre + "canon1", (H, cfg.canon_taps)).T.contiguous()
            if isinstance(m, LatentSpec):
                latent(m, x, L)
            else:
                kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
                L.w_in, L.offs = fuse([(n, t(x + n, (rows, H))) for n, rows in
                                       (("q", kd), ("k", kd), ("v", vd), ("g", vd), ("b", m.heads), ("a", m.heads))])
                L.conv_w = torch.cat([f(x + n + ".conv") for n in ("q", "k", "v")]).contiguous()
                if tuple(L.conv_w.shape) != (m.conv_channels, m.conv):
                    raise ValueError(f"{x}*.conv: {tuple(L.conv_w.shape)}, the configuration says {(m.conv_channels, m.conv)}")
                L.A_log, L.dt_bias, L.out_norm = f(x + "A_log"), f(x + "dt_bias"), f(x + "norm")
            L.w_o = heads_o(x + "o", m.heads, m.vdim)
            if r is not None:
                y = pre + "mlp."
                L.norm2, L.norm2b = t(pre + "norm2", (H,)), t(pre + "norm2b", (H,))
                L.canon2 = t(pre + "canon2", (H, cfg.canon_taps)).T.contiguous()
                routed(r, y, L)
            W.layers.append(L)
        return W

    @staticmethod
    def from_params(cfg: ModelConfig, p: dict[str, torch.Tensor], device: torch.device) -> "HybridWeights":
        return HybridWeights.build(cfg, p.__getitem__, device)

    @staticmethod
    def random_init(cfg: ModelConfig, device: torch.device, seed: int = 0, std: float = 0.02) -> "HybridWeights":
        """Random weights made on the device tensor by tensor: N(0, std) matrices, norm weights one, mild decays."""
        g = torch.Generator(device=device).manual_seed(seed)
        shapes = tensor_shapes(cfg)

        def get(name: str) -> torch.Tensor:
            shape = shapes[name]
            if name.rsplit(".", 1)[-1].startswith("norm"):
                return torch.full(shape, 1.0 if ".mix." in name else 1.0 - cfg.norm_offset, device=device)
            if name.endswith(".dwa"):
                return torch.full(shape, 1.0 / shape[0], device=device)
            s = 0.3 if "conv" in name or "canon" in name else std
            x = torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, s, generator=g)
            return x - 3.0 if name.endswith("dt_bias") else x
        return HybridWeights.build(cfg, get, device)


def tensor_shapes(cfg: ModelConfig) -> dict[str, tuple]:
    """Every tensor of the checkpoint and its shape."""
    H = cfg.hidden
    one = () if cfg.norm_scalar else (H,)
    out: dict[str, tuple] = {"embed": (cfg.vocab_size, H), "final.norm": one, "head": (cfg.vocab_size, H)}
    if cfg.bigram:
        out["bigram"] = (cfg.bigram[0] + 1, H)
    if cfg.loop and cfg.loop_join:
        out.update({"loop.in": (H, 2 * H), "loop.step": (cfg.loop[2], H)})
    for i, spec in enumerate(cfg.layer_specs):
        pre, m, r = f"l{i}.", spec.mixer, spec.router
        x = pre + "mix."
        if spec.post_norm:
            out[pre + "norm1"] = one
            out.update(_pair_shapes(x, m, H) if isinstance(m, PairSpec) else _rglru_shapes(x, m, H))
            if spec.has_ffn:
                out[pre + "norm2"] = one
            if r is not None:
                out.update(_routed_shapes(pre + "mlp.", r, H))
            elif spec.dense is not None:
                d = spec.dense.ffn
                out.update({pre + "mlp.gate": (d, H), pre + "mlp.up": (d, H), pre + "mlp.down": (H, d)})
            if cfg.depth_average:
                out[pre + "dwa"] = (i + 2,)
            continue
        if spec.parallel:
            out[pre + "norm1"], out[x + "o"] = (H,), (H, m.heads * m.vdim)
            if spec.two_norms and (spec.dense is not None or r is not None):
                out[pre + "norm2"] = (H,)
            if isinstance(m, LatentSpec):
                out.update(_latent_shapes(x, m, H))
            else:
                for n, c in (("q", m.q_channels), ("k", m.k_channels)) + (() if m.v_from_k else (("v", m.v_channels),)):
                    out[x + n] = (c, H)
                    if m.conv:
                        out[x + n + ".conv"] = (c, m.conv)
                    if m.qk_norm and n != "v":
                        out[f"{x}{n}.norm"] = (m.dim if m.qk_norm == "head" else c,)
                if m.sink:
                    out[x + "sink"] = (m.heads,)
                if m.gate:
                    out[x + "g"] = (m.heads, H)
                if m.maps == 2:
                    out.update({x + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
            y = pre + "mlp."
            if r is not None:
                out.update(_routed_shapes(y, r, H))
                y += "shared."
            if spec.dense is not None:
                d = spec.dense.ffn
                out.update({y + "gate": (d, H), y + "up": (d, H), y + "down": (H, d)})
            continue
        out.update({pre + "norm1": (H,), pre + "norm1b": (H,), pre + "canon1": (H, cfg.canon_taps), x + "o": (H, m.heads * m.vdim)})
        if isinstance(m, LatentSpec):
            out.update(_latent_shapes(x, m, H))
        else:
            kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
            for n, c in (("q", kd), ("k", kd), ("v", vd)):
                out[x + n], out[x + n + ".conv"] = (c, H), (c, m.conv)
            out.update({x + "g": (vd, H), x + "b": (m.heads, H), x + "a": (m.heads, H), x + "A_log": (m.heads,), x + "dt_bias": (m.heads,),
                        x + "norm": (m.vdim,)})
        if r is not None:
            out.update({pre + "norm2": (H,), pre + "norm2b": (H,), pre + "canon2": (H, cfg.canon_taps)})
            out.update(_routed_shapes(pre + "mlp.", r, H))
    return out


def _latent_shapes(x: str, m: LatentSpec, H: int) -> dict[str, tuple]:
    out = {x + "q": (m.heads * (m.dim + m.rot_dim), H), x + "dkv": (m.record, H), x + "dkv.norm": (m.kv_rank,),
           x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (m.heads * m.vdim, m.kv_rank)}
    if m.gate:
        out[x + "g"] = (m.heads * m.vdim, H)
    return out


def _pair_shapes(x: str, m: PairSpec, H: int) -> dict[str, tuple]:
    a, b = m.left, m.right
    out = {f"{x}left.{n}": (c, H) for n, c in (("q", a.q_channels), ("k", a.k_channels), ("v", a.v_channels))}
    out.update({f"{x}right.{n}": (c, H) for n, c in (("q", b.heads * b.dim), ("k", b.heads * b.dim), ("v", b.heads * b.vdim), ("g", b.heads * b.vdim))})
    return out | {x + "left.o": (H, a.heads * a.vdim), x + "right.o": (H, b.heads * b.vdim), x + "right.norm": (b.heads * b.vdim,)}


def _rglru_shapes(x: str, m: RglruSpec, H: int) -> dict[str, tuple]:
    c, out = m.width, {x + "o": (H, m.width), x + "conv": (m.width, m.conv)}
    out.update({x + n: (c,) for n in ("x.b", "y.b", "conv.b", "lam")})
    for n in ("ra", "ri"):
        out.update({x + n: (m.blocks, m.block, m.block), f"{x}{n}.b": (m.blocks, m.block)})
    return out | {x + "x": (c, H), x + "y": (c, H)}


def _routed_shapes(y: str, r: RouterSpec, H: int) -> dict[str, tuple]:
    out = {y + "router": (r.outputs, H), y + ("router.b" if r.logit_bias else "correction"): (r.outputs,)}
    for e in range(r.experts):
        out.update({f"{y}e{e}.gate": (r.ffn, H), f"{y}e{e}.up": (r.ffn, H), f"{y}e{e}.down": (H, r.ffn)})
    return out


def tensor_core_latent(cfg: ModelConfig, m: LatentSpec) -> bool:
    """Whether the tcgen05 latent attention kernels take this layer (their record and head sizes are fixed)."""
    return (engine_dtype(cfg) == torch.bfloat16 and (m.kv_rank, m.rot_dim, m.dim, m.vdim) == (512, 64, 128, 128)
            and 128 % m.heads == 0)


def tensor_core_attention(cfg: ModelConfig, m: AttentionSpec) -> bool:
    """Whether the tensor-core attention kernels take this layer: key rows (all maps) and values of 128."""
    rows = m.maps * (m.heads // m.kv_heads)
    return engine_dtype(cfg) == torch.bfloat16 and m.maps * m.dim == 128 and m.vdim == 128 and rows <= 16 and 16 % rows == 0


class HybridCache:
    """Paged records of the attention layers and the slot pool of everything recurrent, per layer run.

    ``c``: one pool [pages, 64, record] per run of a latent layer; ``k`` / ``v``: [pages, kv heads, 64, width] per run of an
    attention layer (page 0 stays zero).  ``of_run``: a run's pool or (K, V) pools.  ``state`` [slots, floats] fp32: slot 0 is
    the zero state every sequence starts from, slot 1 takes the writes of dummy steps; ``offsets`` names a run's parts."""

    def __init__(self, cfg: ModelConfig, num_pages: int, device: torch.device, state_slots: int = 34):
        dt = engine_dtype(cfg)
        self.num_pages = num_pages
        self.c: list[torch.Tensor] = []
        self.k: list[torch.Tensor] = []
        self.v: list[torch.Tensor] = []
        self.of_run: dict = {}
        self.offsets: list[dict[str, int]] = []
        n = 0
        for i, run in enumerate(cfg.layer_runs):
            m, off = cfg.layer_specs[run.layer].mixer, {}
            att = attention_part(m)
            if att is not None:
                kv = [torch.zeros(num_pages, att.kv_heads, PAGE, w, dtype=dt, device=device) for w in (att.maps * att.dim, att.vdim)]
                self.of_run[i] = tuple(kv)
                self.k.append(kv[0])
                self.v.append(kv[1])
            elif isinstance(m, LatentSpec):
                self.of_run[i] = torch.zeros(num_pages, PAGE, record_pitch(m), dtype=dt, device=device)
                self.c.append(self.of_run[i])
            for name, size in cfg.state_parts(run.layer):
                off[name] = n
                n += -(-size // 32) * 32
            self.offsets.append(off)
        self.token_off = n               # a sequence's last token (models with a bigram table)
        n += 32 * bool(cfg.bigram)
        self.state = torch.zeros(max(3, state_slots), max(n, 32), dtype=torch.float32, device=device)

    @property
    def state_slots(self) -> int:
        return self.state.shape[0]

    def bytes_per_page(self) -> int:
        return sum(t[0].numel() * t.element_size() for t in self.c + self.k + self.v)

    def copy_page(self, src: int, dst: int) -> None:
        for c in self.c + self.k + self.v:
            c[dst].copy_(c[src])


class _LatentWs:
    """Workspaces shared by the latent layers of one shape."""

    def __init__(self, cfg: ModelConfig, m: LatentSpec, max_tokens: int, device: torch.device):
        kw = dict(dtype=engine_dtype(cfg), device=device)
        rows = -(-max_tokens // 128) * 128
        self.q_slab = torch.zeros(m.heads * rows * pad8(m.dim), **kw)
        self.o_slab = torch.zeros(m.heads * rows * pad8(m.kv_rank), **kw)
        self.q_abs = torch.zeros(max_tokens, m.heads, record_pitch(m), **kw)
        self.attn = torch.zeros(max_tokens, m.heads, pad8(m.vdim), **kw)
        self.inv_freq = rope_frequencies(m.rope).to(device)
        self.lat = self.k_exp = self.v_exp = None      # expanded-form prompts: made on first use


class _AttnWs:
    """Workspaces of the attention layers of one shape; ``table`` is shared by all that rotate alike."""

    def __init__(self, cfg: ModelConfig, m: AttentionSpec, max_tokens: int, device: torch.device, tables: dict):
        self.q = torch.zeros(max_tokens, m.q_channels, dtype=engine_dtype(cfg), device=device)
        if m.rope not in tables:
            tables[m.rope] = (rope_frequencies(m.rope).to(device), torch.zeros(max_tokens, max(1, m.rope.dims // 2), 2, device=device))
        if m.v_rope is not None and m.v_rope not in tables:
            tables[m.v_rope] = (rope_frequencies(m.v_rope).to(device), torch.zeros(max_tokens, max(1, m.v_rope.dims // 2), 2, device=device))
        self.table, self.v_table = tables[m.rope][1], tables[m.v_rope][1] if m.v_rope is not None else None
        self.tensor_core = tensor_core_attention(cfg, m)


class _RglruWs:
    """Workspaces shared by the gated linear recurrences of one shape (rows of a block are whole 16-byte pieces; the padding stays zero)."""

    def __init__(self, cfg: ModelConfig, m: RglruSpec, max_tokens: int, device: torch.device):
        rows, bp, dt = -(-max_tokens // 128) * 128, pad8(m.block), engine_dtype(cfg)
        self.u = torch.zeros(m.blocks * rows * bp, dtype=dt, device=device)
        self.gates = torch.empty(m.blocks * rows * 2 * bp, dtype=torch.float32, device=device)
        self.out = torch.zeros(max_tokens, pad8(m.width), dtype=dt, device=device)


class HybridEngine:
    """Single-GPU engine of the per-layer hybrids behind the same calls as the other engines (``forward`` on a ``Batch``)."""
    embed_rows = None
    EXPANDED_PREFILL_TOKENS = 64     # fresh prompt chunks of at least this many tokens use the expanded-form attention
    CHUNKED_DELTA_TOKENS = 32        # steps with a portion of at least this many tokens take the chunked delta rule
    CHUNKED_LIGHTNING_TOKENS = 32    # likewise linear attention
    CHUNK_SCRATCH_BYTES = 128 << 20  # its operands of one slab of chunks (about an L2's worth)
    FUSED_ROUTE_TOKENS = 64          # steps up to this many tokens run router scores + selection as one launch

    def __init__(self, cfg: ModelConfig, weights: HybridWeights, kv: HybridCache, max_tokens: int, max_seqs: int = 64):
        assert cfg.is_hybrid
        self.cfg, self.W, self.kv = cfg, weights, kv
        self.device = dev = weights.embed.device
        self.dtype = dt = engine_dtype(cfg)
        # a decode step may carry as many rows again: accepted rows the recurrent state has yet to see
        max_seqs *= 2
        self.max_tokens = max_tokens = max(max_tokens, max_seqs)
        H = cfg.hidden

        class _Ws:
            pass
        ws = self.ws = _Ws()
        ws.x = [torch.empty(max_tokens, H, dtype=torch.float32, device=dev) for _ in range(2)]
        # averages over depth: the embedding rows and every layer run's result but the last one's
        runs = len(cfg.layer_runs)
        ws.past = torch.empty(runs, max_tokens, H, dtype=torch.float32, device=dev) if cfg.depth_average else None
        ws.rows2 = torch.zeros(max_tokens, dtype=torch.int32, device=dev) if cfg.bigram else None
        Hp = pad8(H)                     # rows the matrix products read are whole 16-byte pieces; the padding stays zero
        ws.h = [torch.zeros(max_tokens, Hp, dtype=dt, device=dev) for _ in range(2)]
        ws.y = torch.zeros(max_tokens, Hp, dtype=dt, device=dev)
        ws.h2 = torch.zeros(max_tokens, Hp, dtype=dt, device=dev) if any(L.norm2 is not None and L.norm2b is None for L in weights.layers) else None
        if weights.loop_in is not None:  # [x | embedding row] of a pass's joining product, and what comes out of it
            ws.join = torch.zeros(max_tokens, 2 * Hp, dtype=dt, device=dev)
            ws.joined = torch.empty(max_tokens, H, dtype=torch.float32, device=dev)
        ws.proj = torch.empty(max_tokens * max(L.w_in.shape[0] for L in weights.layers), dtype=dt, device=dev)
        outs = max((s.router.outputs for s in cfg.layer_specs if s.router), default=1)
        ws.router = torch.empty(max_tokens * outs, dtype=torch.float32, device=dev)
        self._lat: dict[LatentSpec, _LatentWs] = {}
        self._attn: dict[AttentionSpec, _AttnWs] = {}
        self._rope: dict[RopeSpec, tuple] = {}       # frequencies, the step's table
        self._delta: dict[DeltaSpec, torch.Tensor] = {}
        self._rglru: dict[RglruSpec, _RglruWs] = {}
        self._moe: dict = {}
        raw = scratch = 0
        for spec in cfg.layer_specs:
            m, r = spec.mixer, spec.router
            if isinstance(m, LatentSpec):
                if m not in self._lat:
                    self._lat[m] = _LatentWs(cfg, m, max_tokens, dev)
            elif isinstance(m, RglruSpec):
                if m not in self._rglru:
                    self._rglru[m] = _RglruWs(cfg, m, max_tokens, dev)
            elif (a := attention_part(m)) is not None:
                if a not in self._attn:
                    self._attn[a] = _AttnWs(cfg, a, max_tokens, dev, self._rope)
                if isinstance(m, PairSpec):
                    raw = max(raw, m.right.heads * m.right.vdim)
            else:
                if m not in self._delta:
                    self._delta[m] = torch.zeros(max_tokens, m.heads, pad8(m.vdim), dtype=dt, device=dev)
                chunked = K.delta_chunk_ok(m, dt)
                if m.vdim > 128 or chunked:
                    raw = max(raw, m.heads * m.vdim)
                if chunked:
                    per = K.delta_chunk_bytes(m)
                    chunks = max(max(1, self.CHUNK_SCRATCH_BYTES // per), 1)
                    scratch = max(scratch, per * min(chunks, max_tokens // 64 + max_seqs))
            if r is not None and r not in self._moe:
                self._moe[r] = LocalExchange(ExchangeGeometry(Hp, pad8(r.ffn), r.experts, r.top, max_tokens, 1), dev, dtype=dt)
        # rows of a parallel layer's second product: the heads' values, then the feed-forward's activations
        act = max((w.shape[1] for L in weights.layers for w in (L.w_out, L.d_down) if w is not None), default=0)
        ws.act = torch.zeros(max_tokens * act, dtype=dt, device=dev) if act else None
        ws.raw = torch.empty(max_tokens * raw, dtype=torch.float32, device=dev) if raw else None
        ws.chunk = torch.empty(scratch, dtype=torch.uint8, device=dev) if scratch else None
        self.moe = None
        rows = max_seqs
        self._logits = torch.empty(rows, pad8(cfg.vocab_size), dtype=torch.float32, device=dev)
        self.logits = self._logits[:, :cfg.vocab_size]
        self.next_tokens = torch.empty(rows, dtype=torch.int32, device=dev)
        self._tiles: dict[tuple[int, int, int], _HeadTiles] = {}
        self._blocks: dict = {}
        self._zero1 = torch.zeros(1, dtype=torch.int32, device=dev)
        self._scratch: torch.Tensor | None = None
        self._outgrown: list = []
        self.fixed_kv_split = K.batch_invariant_from_env()
        self.layer_hook = None           # callable(layer, residual [T, H]) for tests and traces (eager mode only)
        self.launches = 0
        self._pending: dict = {}

    # ---- between sublayers ------------------------------------------------------------------------------------------
    def _source(self, b: Batch, add_embedding: bool = False) -> dict:
        """Where a launch between sublayers takes the residual from."""
        src = {} if self._x is None else dict(x_in=self._x)
        if self._x is None or add_embedding:
            src.update(tokens=b.tokens, embed=self.W.embed, embed_scale=self.cfg.embed_scale)
            if self.W.bigram is not None:
                src.update(second=(self.ws.rows2[:b.tokens.shape[0]], self.W.bigram))
        return src

    def _between(self, b: Batch, T: int, w: torch.Tensor | None, conv: torch.Tensor | None, off: int = 0, add_embedding: bool = False,
                 step: torch.Tensor | None = None, w2: torch.Tensor | None = None) -> torch.Tensor:
        """Residual, norms and input convolution up to the next sublayer; returns its input rows (``w2``: the same norm's rows under
        other weights go to ``ws.h2``)."""
        ws, p = self.ws, self._pending
        h = ws.h[self._hi][:T]
        if self._x is None and ws.past is not None:
            xo = ws.past[0, :T]
        else:
            xo = ws.x[0 if self._x is None or self._x.data_ptr() != ws.x[0].data_ptr() else 1][:T]
        K.norm_conv(h, w, self.cfg.norm_groups, self.cfg.rms_eps, conv=conv, x_out=xo, state=self.kv.state, state_off=off,
                    state_in=b.state_in, state_out=b.state_out, q_start=b.q_start, w_offset=self.cfg.norm_offset, step=step,
                    w2=w2, h2_out=ws.h2[:T] if w2 is not None else None, **self._source(b, add_embedding), **p)
        self._x, self._hi = xo, self._hi ^ 1
        self.launches += 1
        return h

    def _join(self, b: Batch, T: int) -> None:
        """Start of a pass: the residual becomes a product of [x; embedding row] (the embedding's half is there already)."""
        ws, cfg = self.ws, self.cfg
        K.norm_conv(ws.join[:T], None, cfg.norm_groups, cfg.rms_eps, **self._source(b), **self._pending)
        K.linear(ws.join[:T], self.W.loop_in, out=ws.joined[:T], out_f32=True, swap=True if cfg.hidden % 4 else None)
        self._x, self._pending = ws.joined[:T], {}
        self.launches += 2

    def residual(self, T: int) -> torch.Tensor:
        """The residual stream [T, H] after everything launched so far (tests and traces)."""
        x = self._x.clone()
        p = self._pending
        if p:
            H = self.cfg.hidden
            y, G = p["y"][:, :H].float(), self.cfg.norm_groups
            if "slots" in p:
                w, idx, n, ident = p["slots"]
                rows = torch.where((idx >= n)[..., None], ident[:, :H].float()[:, None], y[:T * w.shape[1]].view(T, w.shape[1], -1))
                y = (w[..., None] * rows).sum(1)
                if p.get("base") is not None:
                    y = y + p["base"][:, :H].float()
            if p.get("w_b") is None:
                return x + y
            g = y.view(T, G, -1)
            x = x + (g / torch.sqrt((g * g).mean(-1, keepdim=True) + self.cfg.rms_eps)).view(T, -1) * p["w_b"]
            if p.get("past") is not None:
                results, w, _ = p["past"]
                x = (w[:-1, None, None] * results[:, :T]).sum(0) + w[-1] * x
        return x

    # ---- mixers -----------------------------------------------------------------------------------------------------
    def _project(self, i: int, h: torch.Tensor, T: int) -> torch.Tensor:
        w = self.W.layers[i].w_in
        a = self.ws.proj[:T * w.shape[0]].view(T, w.shape[0])
        self.launches += 1
        return K.linear(h, w, out=a)

    def _partials(self, floats: int) -> torch.Tensor:
        """Scratch for the partial sums of split attention.  An outgrown buffer is kept: a captured graph may still write it."""
        if self._scratch is None or self._scratch.numel() < floats:
            self._outgrown.append(self._scratch)
            self._scratch = torch.empty(floats, dtype=torch.float32, device=self.device)
        return self._scratch

    def _block_table(self, S: int, max_q_len: int, per: int):
        key = (S, max_q_len, per)
        if key not in self._blocks:
            nb = (max_q_len + per - 1) // per
            i32 = dict(dtype=torch.int32, device=self.device)
            self._blocks[key] = (torch.arange(S, **i32).repeat_interleave(nb).contiguous(), (torch.arange(nb, **i32) * per).repeat(S).contiguous())
        return self._blocks[key]

    def _latent(self, n: int, i: int, m: LatentSpec, h: torch.Tensor, T: int, b: Batch, out: torch.Tensor | None = None) -> None:
        """Latent attention of layer run n and its o projection into ``ws.y``; with ``out`` the heads' values go to that buffer's
        first columns instead, without gate and projection."""
        L, ws, lw = self.W.layers[i], self.ws, self._lat[m]
        a = self._project(i, h, T)
        cache = self.kv.of_run[n]
        dp, rp, vp, rec = pad8(m.dim), pad8(m.kv_rank), pad8(m.vdim), record_pitch(m)
        attn = lw.attn[:T] if out is None else out
        key = (T, m.heads, attn.stride(0) // vp)
        if key not in self._tiles:
            self._tiles[key] = _HeadTiles(T, m.heads, self.device, out_heads=key[2])
        ht = self._tiles[key]
        fast = L.w_kb is not None
        expanded = fast and b.prefill and b.fresh and T >= self.EXPANDED_PREFILL_TOKENS
        if expanded and lw.lat is None:
            rows, kw = -(-self.max_tokens // 64) * 64, dict(dtype=self.dtype, device=self.device)
            lw.lat = torch.zeros(self.max_tokens, m.kv_rank, **kw)
            lw.k_exp, lw.v_exp = torch.zeros(rows, m.heads * 128, **kw), torch.zeros(rows, m.heads * 128, **kw)
        slab = lw.q_slab[:m.heads * ht.t_pad * dp].view(m.heads, ht.t_pad, dp)
        o_slab = lw.o_slab[:m.heads * ht.t_pad * rp].view(m.heads, ht.t_pad, rp)
        q = a[:, L.offs["q"]:L.offs["q"] + m.heads * (m.dim + m.rot_dim)]
        # (the batch-invariant form keeps one absorb / un-absorb route for every decode width: the grouped GEMMs)
        small = fast and T <= K.MLA_SMALL_ROWS and not self.fixed_kv_split
        K.latent_prep(a, L.offs["q"], L.offs["kv"], m.heads, m.dim, m.rot_dim, L.kv_norm, lw.inv_freq, b.positions, b.slots, cache,
                      None if expanded or small else slab, None if small else lw.q_abs[:T], self.cfg.rms_eps,
                      lat_out=lw.lat[:T] if expanded else None, halves=m.rope.halves, magnitude=m.rope.magnitude)
        self.launches += 1
        if small:
            # decode-sized step: rotation and absorb in one launch, un-absorb and output gate in another
            K.mla_absorb_small(q, L.w_uk, lw.inv_freq, b.positions, lw.q_abs[:T], m.heads, not m.rope.halves, m.rope.magnitude)
            self._attend_tensor_core(m, lw, T, b, cache, o_slab, ht.t_pad)
            K.mla_unabsorb_small(o_slab, L.w_uv, attn, T, gate=a[:, L.offs["g"]:L.offs["g"] + m.heads * m.vdim] if m.gate else None)
            self.launches += 3
            if out is None:
                K.linear(attn.view(T, -1), L.w_o, out=ws.y[:T])
                self.launches += 1
            return
        if expanded:
            rows = -(-T // 64) * 64
            K.linear(lw.lat[:T], L.w_kb, out=lw.k_exp[:T])
            K.linear(lw.lat[:T], L.w_uv.view(m.heads * m.vdim, m.kv_rank), out=lw.v_exp[:T])
            K.attn_prefill_mla(q, lw.q_abs[:T], lw.k_exp[:rows], lw.v_exp[:rows], self._zero1, cache, b.page_table, b.seq_lens, b.q_start,
                               attn, b.max_q_len, m.heads, m.scale, window=m.window)
            self.launches += 3
        else:
            K.grouped_linear(slab.view(-1, dp), L.w_uk, lw.q_abs, ht.tile_expert, ht.tile_row0, ht.num_tiles, ht.max_tiles, ht.tile_rows,
                             row_dst=ht.row_dst, ldo=rec, split_k=False)
            if fast:
                self._attend_tensor_core(m, lw, T, b, cache, o_slab, ht.t_pad)
            else:
                K.latent_attn(lw.q_abs[:T], cache, m.kv_rank, m.rot_dim, b.page_table, b.positions, b.q_start, o_slab, m.scale, m.window)
            K.grouped_linear(o_slab.view(-1, rp), L.w_uv, attn, ht.tile_expert, ht.tile_row0, ht.num_tiles, ht.max_tiles, ht.tile_rows,
                             row_dst=ht.row_out, ldo=vp, split_k=False)
            self.launches += 3
        if out is not None:
            return
        if m.gate:
            K.latent_gate(attn, a, L.offs["g"], m.heads, m.vdim)
        K.linear(attn.view(T, -1), L.w_o, out=ws.y[:T])
        self.launches += 2

    def _attend_tensor_core(self, m: LatentSpec, lw: _LatentWs, T: int, b: Batch, cache: torch.Tensor, o_slab: torch.Tensor, t_pad: int) -> None:
        S, max_pages = b.page_table.shape
        bseq, btok = self._block_table(S, b.max_q_len, 128 // m.heads)
        nb = bseq.numel()
        tiles = max_pages * 2
        if m.window > 0:
            tiles = min(tiles, (m.window + b.max_q_len + 31) // 32 + 1)
        splits = 1 if b.prefill else max(1, min(K.num_sms() // max(1, nb * 2), max(1, tiles // 8), 32))
        if self.fixed_kv_split and not b.prefill:
            splits = K.kv_splits_fixed(max_pages, cap=64)
        if splits > 1:
            need = K.mla_scratch_floats(nb, splits)
            self._partials(need)
        K.mla_attention(lw.q_abs[:T], cache, b.page_table, b.seq_lens, b.q_start, bseq, btok, o_slab, m.scale, splits,
                        self._scratch if splits > 1 else None, out_tpad=t_pad, window=m.window)
        self.launches += 1 if splits > 1 else 0

    def _attention(self, n: int, i: int, m: AttentionSpec, h: torch.Tensor, T: int, b: Batch, out: torch.Tensor,
                   a: torch.Tensor | None = None, out_scale: float = 1.0) -> None:
        """Attention of layer run n; head h's values, times ``out_scale``, go to columns [h * pad8(vdim), + vdim) of ``out``.  ``a``: the
        projected rows, if they are there already."""
        L, aw = self.W.layers[i], self._attn[m]
        if a is None:
            a = self._project(i, h, T)
        (k, v), q = self.kv.of_run[n], aw.q[:T]
        K.conv_rope_kv(a, L.offs, m, L.conv_w, aw.table, b.slots, q, k, v, state=self.kv.state, state_off=self.kv.offsets[n]["conv"],
                       state_in=b.state_in, state_out=b.state_out, q_start=b.q_start, q_norm=L.q_norm, k_norm=L.k_norm, eps=self.cfg.rms_eps,
                       v_table=aw.v_table)
        self.launches += 2
        gate = a[:, L.offs["g"]:L.offs["g"] + m.heads] if m.gate else None
        if not aw.tensor_core:
            K.paged_attn(q, k, v, m, b.page_table, b.positions, b.q_start, out, pad8(m.vdim), L.lam, self.cfg.rms_eps, sink=L.sink, gate=gate,
                         v_table=aw.v_table, out_scale=out_scale)
            return
        kw = dict(scale=m.scale, window=m.window, keep=m.keep_first, maps=m.maps, lam=L.lam, out_scale=(1.0 - m.diff) * out_scale,
                  eps=self.cfg.rms_eps, sink=L.sink, gate=gate, cap=m.softcap, v_table=aw.v_table)
        q = q.view(T, m.heads, 128)
        if b.prefill:
            K.attn_prefill(q, k, v, b.page_table, b.seq_lens, b.q_start, out, b.max_q_len, **kw)
            return
        S, max_pages = b.page_table.shape
        q_per_tile = 16 // (m.maps * (m.heads // m.kv_heads))
        tiles = (b.max_q_len + q_per_tile - 1) // q_per_tile
        splits = (K.kv_splits_fixed(max_pages) if self.fixed_kv_split else
                  K.attn_decode_splits(S, tiles, m.kv_heads, max_pages, m.window, m.keep_first))
        need = K.attn_decode_scratch_floats(S, b.max_q_len, m.maps * m.heads, m.kv_heads, splits)
        K.attn_decode(q, k, v, b.page_table, b.seq_lens, b.q_start, out, self._partials(need) if splits > 1 else None, b.max_q_len, splits, **kw)
        self.launches += 1 if splits > 1 else 0

    def _parallel(self, n: int, i: int, spec, h: torch.Tensor, T: int, b: Batch) -> None:
        """Mixer and feed-forward on rows of the same residual; one product over both reads the mixer's values and the dense (or
        shared expert's) activations side by side, the routed experts' rows are summed by the next launch between layers."""
        L, m, r = self.W.layers[i], spec.mixer, spec.router
        act = self.ws.act[:T * L.w_out.shape[1]].view(T, L.w_out.shape[1])
        (self._latent if isinstance(m, LatentSpec) else self._attention)(n, i, m, h, T, b, act)
        f = self.ws.h2[:T] if L.norm2 is not None else h
        if spec.dense is not None:
            K.linear(f, L.d_gate, out=act[:, m.heads * pad8(m.vdim):], w_up=L.d_up)
            self.launches += 1
        K.linear(act, L.w_out, out=self.ws.y[:T])
        self.launches += 1
        self._pending = dict(y=self.ws.y[:T])
        if r is not None:
            self._pending = dict(slots=self._experts(i, r, f, T), y=self._moe[r].att.combine, base=self.ws.y[:T])

    def _pair(self, n: int, i: int, m: PairSpec, h: torch.Tensor, T: int, b: Batch) -> None:
        """Attention and linear attention on the same rows; one product over both reads their values side by side."""
        L, ws = self.W.layers[i], self.ws
        a = self._project(i, h, T)
        act = ws.act[:T * L.w_out.shape[1]].view(T, L.w_out.shape[1])
        self._attention(n, i, m.left, h, T, b, act, a=a, out_scale=m.left_scale)
        r = m.right
        args = (a, {k: L.offs["right." + k] for k in "qkvg"}, r, L, self.kv.state, self.kv.offsets[n]["S"], b.state_in, b.state_out,
                b.q_start, ws.raw, act[:, m.left.heads * pad8(m.left.vdim):], pad8(r.vdim), self.cfg.rms_eps)
        if b.prefill and b.max_q_len >= self.CHUNKED_LIGHTNING_TOKENS and K.lightning_chunk_ok(r, self.dtype):
            K.lightning_chunked(*args, self._partials(K.lightning_scratch_bytes(r, T, b.q_start.shape[0] - 1) // 4))
            self.launches += 2
        else:
            K.lightning_step(*args)
        K.linear(act, L.w_out, out=ws.y[:T])
        self.launches += 3

    def _rglru_mixer(self, n: int, i: int, m: RglruSpec, h: torch.Tensor, T: int, b: Batch) -> None:
        L, rw, off = self.W.layers[i], self._rglru[m], self.kv.offsets[n]
        a = self._project(i, h, T)
        bp = pad8(m.block)
        key = (T, m.blocks, 0)
        if key not in self._tiles:
            self._tiles[key] = _HeadTiles(T, m.blocks, self.device)
        ht = self._tiles[key]
        u = rw.u[:m.blocks * ht.t_pad * bp].view(m.blocks, ht.t_pad, bp)
        gates = rw.gates[:m.blocks * ht.t_pad * 2 * bp].view(m.blocks, ht.t_pad, 2 * bp)
        out = rw.out[:T]
        args = (a, L.offs, m, L, u, gates, self.kv.state, off["S"], off["conv"], b.state_in, b.state_out, b.q_start, out, b.max_q_len)
        if K.rglru_step_ok(m, self.dtype, max(T, b.q_start.shape[0] - 1)):
            K.rglru_step(*args)
            K.linear(out, L.w_out, out=self.ws.y[:T])
            self.launches += 2
            return
        K.rglru_conv(*args)
        K.grouped_linear(u.view(-1, bp), L.w_gates, gates.view(-1, 2 * bp), ht.tile_expert, ht.tile_row0, ht.num_tiles, ht.max_tiles, ht.tile_rows,
                         split_k=False)
        K.rglru_scan(*args)
        K.linear(out, L.w_out, out=self.ws.y[:T])
        self.launches += 4

    def _dense(self, i: int, d: DenseSpec, h: torch.Tensor, T: int) -> None:
        L, F = self.W.layers[i], pad8(d.ffn)
        act = self.ws.act[:T * F].view(T, F)
        K.linear(h, L.d_gate, out=act, w_up=L.d_up, glu=None if d == DenseSpec(d.ffn) else (d.limit or math.inf, d.alpha, d.up_bias))
        K.linear(act, L.d_down, out=self.ws.y[:T])
        self.launches += 2

    def _post_norm(self, n: int, i: int, spec, T: int, b: Batch) -> None:
        """Sublayers that read the residual and are normed after they ran; then the average over depth, in the launch that takes the
        last sublayer's rows."""
        L, m, r = self.W.layers[i], spec.mixer, spec.router
        h = self._between(b, T, None, None)
        (self._pair if isinstance(m, PairSpec) else self._rglru_mixer)(n, i, m, h, T, b)
        self._pending = dict(y=self.ws.y[:T], w_b=L.norm1b)
        if spec.has_ffn:
            h = self._between(b, T, None, None)
            self._pending = dict(y=self.ws.y[:T], w_b=L.norm2b)
            if r is not None:
                self._pending.update(slots=self._experts(i, r, h, T), y=self._moe[r].att.combine)
            else:
                self._dense(i, spec.dense, h, T)
        if L.dwa is not None:
            past = self.ws.past
            self._pending["past"] = (past[:n + 1], L.dwa, past[n + 1, :T] if n + 1 < past.shape[0] else None)

    def _delta_mixer(self, n: int, i: int, m: DeltaSpec, h: torch.Tensor, T: int, b: Batch) -> None:
        L, ws = self.W.layers[i], self.ws
        a = self._project(i, h, T)
        off, out = self.kv.offsets[n], self._delta[m][:T]
        args = (a, L.offs, m, L, self.kv.state, off["S"], off["conv"], b.state_in, b.state_out, b.q_start, out, ws.raw, self.cfg.rms_eps)
        if b.prefill and b.max_q_len >= self.CHUNKED_DELTA_TOKENS and K.delta_chunk_ok(m, self.dtype):
            K.delta_chunked(ws.chunk, *args)
            slabs = -(-((T + 63 * (b.q_start.shape[0] - 1)) // 64) * K.delta_chunk_bytes(m) // ws.chunk.numel())
            self.launches += 2 * slabs + 1
        else:
            K.delta_step(*args)
            self.launches += 1 if m.vdim <= 128 else 2
        K.linear(out.view(T, -1), L.w_o, out=ws.y[:T])
        self.launches += 1

    # ---- routed feed-forward ----------------------------------------------------------------------------------------
    def _experts(self, i: int, r, h: torch.Tensor, T: int) -> tuple:
        L, moe = self.W.layers[i], self._moe[r]
        kw = dict(scoring="softmax_bias" if r.logit_bias else r.scoring, bias=L.correction, num_groups=r.groups, topk_groups=r.groups_kept,
                  normalize=r.normalize, routed_scale=1.0, group_score="max")
        logits = None
        idx, w = moe.att.idx[:T], moe.att.w[:T]
        if self.dtype == torch.bfloat16 and T <= self.FUSED_ROUTE_TOKENS and h.shape[1] <= 8192:
            K.norm_route(h, None, 0.0, L.router, None, idx, w, r.top, **kw)
            self.launches += 1
        else:
            logits = K.linear(h, L.router, out=self.ws.router[:T * r.outputs].view(T, r.outputs), out_f32=True,
                              swap=True if r.outputs % 4 else None)
            self.launches += 2
        moe.experts(h, logits, kw, L.w_gate, L.w_up, L.w_down)
        self.launches += 4
        return w, idx, r.experts, h

    # ---- whole step -------------------------------------------------------------------------------------------------
    def layers(self, b: Batch) -> int:
        T = b.tokens.shape[0]
        assert T <= self.max_tokens
        if b.embeds is not None:
            raise ValueError("media rows are not part of this family")
        self._x, self._hi, self._pending = None, 0, {}
        for r, (freq, table) in self._rope.items():
            if r.dims:
                K.rope_table(b.positions, freq, table.view(-1)[:T * r.dims], r.magnitude)
                self.launches += 1
        if self.W.bigram is not None:
            K.bigram_rows(b.tokens, self.cfg.bigram, self.kv.state, self.kv.token_off, b.state_in, b.state_out, b.q_start, self.ws.rows2[:T])
            self.launches += 1
        if self.W.loop_in is not None:
            K.norm_conv(self.ws.join[:T, pad8(self.cfg.hidden):], None, self.cfg.norm_groups, self.cfg.rms_eps, **self._source(b))
            self.launches += 1
        for n, run in enumerate(self.cfg.layer_runs):
            i, spec = run.layer, self.cfg.layer_specs[run.layer]
            L, off, m, r = self.W.layers[i], self.kv.offsets[n], spec.mixer, spec.router
            if spec.post_norm:
                self._post_norm(n, i, spec, T, b)
                if self.layer_hook is not None:
                    self.layer_hook(n, self.residual(T))
                continue
            if spec.parallel:
                step = None
                if run.join >= 0:
                    self._join(b, T)
                    step = self.W.loop_step[run.join]
                self._parallel(n, i, spec, self._between(b, T, L.norm1, None, add_embedding=run.add_embedding, step=step, w2=L.norm2), T, b)
                if self.layer_hook is not None:
                    self.layer_hook(n, self.residual(T))
                continue
            h = self._between(b, T, L.norm1, L.canon1, off["canon1"])
            if isinstance(m, LatentSpec):
                self._latent(n, i, m, h, T, b)
            else:
                self._delta_mixer(n, i, m, h, T, b)
            self._pending = dict(y=self.ws.y[:T], w_b=L.norm1b)
            if r is not None:
                h = self._between(b, T, L.norm2, L.canon2, off["canon2"])
                slots = self._experts(i, r, h, T)
                self._pending = dict(y=self._moe[r].att.combine, w_b=L.norm2b, slots=slots)
            if self.layer_hook is not None:
                self.layer_hook(n, self.residual(T))
        return T

    def head(self, T: int, rows: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 logits of ``rows`` (None = all) of the step ``layers`` just ran."""
        n = T if rows is None else rows.shape[0]
        xn = self.ws.h[self._hi][:n]
        if rows is not None and rows.dtype != torch.int32:
            rows = rows.to(torch.int32)
        K.norm_conv(xn, self.W.final_norm, self.cfg.norm_groups, self.cfg.rms_eps, x_in=self._x, rows=rows, w_offset=self.cfg.norm_offset,
                    **self._pending)
        self.launches += 2
        out = K.linear(xn, self.W.lm_head, out=self.logits[:n], out_f32=True)
        if self.cfg.logit_softcap:
            K.softcap(out, self.cfg.logit_softcap)
            self.launches += 1
        return out

    def forward(self, b: Batch) -> torch.Tensor:
        return self.head(self.layers(b), b.last_rows)

    def greedy(self, logits: torch.Tensor) -> torch.Tensor:
        self.launches += 1
        return K.argmax(logits, out=self.next_tokens[:logits.shape[0]])

    def decode_step(self, b: Batch, advance: bool = False) -> torch.Tensor:
        out = self.greedy(self.forward(b))
        if advance:
            K.decode_advance(b.tokens, out, b.positions, b.seq_lens, b.slots, b.page_table)
            K.swap_ids(b.state_in, b.state_out)
            self.launches += 2
        return out
