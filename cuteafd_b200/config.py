"""Model geometry shared by the CPU oracle, the planner, the loader and the CUDA engine.

One dataclass describes every decoder family the engine serves: GQA or MLA attention,
dense or routed-MoE feed-forward layers, optional shared expert, optional multi-token
prediction (MTP) layers and the optional sparse-attention "lightning indexer".  The
reference keeps the same facts in ``ModelSpec/LayerSpec/AttentionKind/MoeSpec/
SpeculatorSpec`` (rust/crates/cuteafd-loader/src/plan/spec.rs:7-190).
"""
from __future__ import annotations

import dataclasses
import json
import math
from dataclasses import dataclass, field
from typing import Any


@dataclass(frozen=True)
class RopeSpec:
    """Rotary positions on the first ``dims`` dimensions of a head: pairs (2i, 2i + 1), or (i, i + dims / 2) with ``halves``.
    ``factor`` other than 1 stretches the frequencies as ``kind`` says:

    bands    wavelengths above ``original / low`` are divided by it, those below ``original / high`` are kept, the band between is
             blended linearly in the number of turns over ``original`` positions
    linear   every frequency is divided by it
    yarn     between the pairs that make ``high`` and ``low`` turns over ``original`` positions the blend is linear in the pair's
             index, and cosines and sines carry a ``magnitude``"""
    dims: int
    base: float
    factor: float = 1.0
    low: float = 1.0
    high: float = 4.0
    original: int = 0
    kind: str = "bands"
    halves: bool = False

    @property
    def magnitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0 if self.kind == "yarn" else 1.0


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention of one layer: all heads' keys and values come out of a normed latent of ``kv_rank`` values plus one
    shared rotated key part of ``rot_dim``; a query at position i sees the last ``window`` positions (0 = all of them).  ``gate``:
    every output value is multiplied by the sigmoid of a projected one."""
    heads: int
    dim: int                             # unrotated query / key dims per head
    rot_dim: int
    vdim: int
    kv_rank: int
    window: int
    scale: float
    rope: RopeSpec
    gate: bool = True

    @property
    def record(self) -> int:
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule of one layer: per head a [dim, vdim] state; q / k heads are shared by ``heads // kv_heads`` heads;
    q, k and v pass a causal convolution of ``conv`` taps."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def conv_channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention of one layer over paged keys and values, with a causal convolution of ``conv`` taps on the channels of
    q, k and v (0 = none).  A query at position i sees the last ``window`` positions (0 = all of them) and the first
    ``keep_first`` ones.  ``maps`` 2 is differential attention: two score maps per head over the same values, combined as
    map 1 - lambda * map 2, the difference normed per head and scaled by 1 - ``diff`` (lambda's constant part).

    ``qk_norm``: RMS norm of queries and keys before their rotation, per head ("head", one weight vector for all heads) or over the
    whole projection ("all"), or after it, per head and without a weight ("rotated").  ``v_from_k``: the values are the convolved keys
    before norm and rotation.  ``sink``: a trained logit per head that takes a share of the softmax and hands nothing through;
    ``unit_sink``: the same with logit 0 for every head.  ``gate``: a head's output is multiplied by the sigmoid of one projected
    number.  ``softcap``: scores pass cap * tanh(score / cap) (0 = they do not).  ``v_rope``: a value is rotated by its position
    before it is cached, and a head's output is turned back by the query's."""
    heads: int
    kv_heads: int
    dim: int                             # query / key dims per map and head
    vdim: int
    window: int
    keep_first: int
    scale: float
    rope: RopeSpec
    conv: int = 0
    maps: int = 1
    diff: float = 0.0
    qk_norm: str = ""                    # "" | "head" | "all" | "rotated"
    v_from_k: bool = False
    sink: bool = False
    gate: bool = False
    softcap: float = 0.0
    unit_sink: bool = False
    v_rope: RopeSpec | None = None

    @property
    def q_channels(self) -> int:
        return self.heads * self.maps * self.dim

    @property
    def k_channels(self) -> int:
        return self.kv_heads * self.maps * self.dim

    @property
    def v_channels(self) -> int:
        return self.kv_heads * self.vdim

    @property
    def conv_channels(self) -> int:
        """Projected channels of q, k and v (those the convolution runs over)."""
        return self.q_channels + self.k_channels + (0 if self.v_from_k else self.v_channels)


@dataclass(frozen=True)
class RglruSpec:
    """Gated linear recurrence of ``width`` channels beside a gelu branch of the same width: a causal convolution of ``conv`` taps, then
    per channel S <- a S + sqrt(1 - a^2) i u with a = exp(-``c`` r softplus(lam)); r and i are sigmoids of block-diagonal products
    (``blocks`` square matrices each)."""
    width: int
    blocks: int
    conv: int
    c: float = 8.0

    @property
    def block(self) -> int:
        return self.width // self.blocks


@dataclass(frozen=True)
class LightningSpec:
    """Linear attention with one constant decay per head: S <- decay S + k v^T, o = S^T q on silu'd projections; all heads' outputs are
    normed together under one weight vector and multiplied by the sigmoid of a projection as wide as they are."""
    heads: int
    dim: int
    vdim: int
    decay: tuple

    @property
    def channels(self) -> int:
        """Projected channels of q, k, v and the gate."""
        return 2 * self.heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class PairSpec:
    """Two mixers on the same rows: left_scale * left + right_scale * right."""
    left: AttentionSpec
    right: LightningSpec
    left_scale: float = 1.0
    right_scale: float = 1.0

    @property
    def heads(self) -> int:
        return max(self.left.heads, self.right.heads)


def attention_part(m: Any) -> AttentionSpec | None:
    """The attention of a mixer that caches keys and values per position (one half of a pair, or the mixer itself)."""
    m = m.left if isinstance(m, PairSpec) else m
    return m if isinstance(m, AttentionSpec) else None


@dataclass(frozen=True)
class DenseSpec:
    """Gated feed-forward of width ``ffn``: with g and u the two projections, g sigmoid(``alpha`` g) (u + ``up_bias``).  ``limit`` other
    than 0: g is cut off above it and u on both sides first."""
    ffn: int
    limit: float = 0.0
    alpha: float = 1.0
    up_bias: float = 0.0


@dataclass(frozen=True)
class RouterSpec:
    """Routed feed-forward of one layer: ``experts`` SwiGLU experts of width ``ffn`` and ``identity`` outputs that hand the
    input through; ``top`` of them per token out of the best ``groups_kept`` of ``groups``.  The router's bias takes part in the
    selection alone, or with ``logit_bias`` is part of the logits; the weights are the chosen scores, with ``normalize`` divided by
    their sum."""
    experts: int
    ffn: int
    top: int
    identity: int = 0
    groups: int = 1
    groups_kept: int = 1
    logit_bias: bool = False
    normalize: bool = False
    scoring: str = "softmax"             # "softmax" | "sigmoid"

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                           # LatentSpec | DeltaSpec | AttentionSpec | RglruSpec | PairSpec
    router: RouterSpec | None = None     # None = the layer has no routed feed-forward
    dense: DenseSpec | None = None       # dense feed-forward (parallel layers); beside a router: the shared expert
    # parallel: mixer and feed-forward read one norm and are added together, nothing is normed after them; otherwise the
    # sublayers follow one another, each with a norm before and after it and a convolution on its input
    parallel: bool = False
    two_norms: bool = False              # parallel: the feed-forward reads a norm of its own
    # the sublayers follow one another and read the residual itself; what each gives is normed before it is added
    post_norm: bool = False

    @staticmethod
    def from_dict(d: dict[str, Any]) -> "LayerSpec":
        def mixer(m: dict[str, Any]) -> Any:
            if "left" in m:
                return PairSpec(**dict(m, left=mixer(m["left"]), right=mixer(m["right"])))
            m = {k: RopeSpec(**v) if k in ("rope", "v_rope") and v else tuple(v) if k == "decay" else v for k, v in m.items()}
            kind = (LatentSpec if "kv_rank" in m else AttentionSpec if "rope" in m else RglruSpec if "blocks" in m else
                    LightningSpec if "decay" in m else DeltaSpec)
            return kind(**m)
        return LayerSpec(mixer(d["mixer"]), RouterSpec(**d["router"]) if d.get("router") else None,
                         DenseSpec(**d["dense"]) if d.get("dense") else None, bool(d.get("parallel", False)), bool(d.get("two_norms", False)),
                         bool(d.get("post_norm", False)))

    @property
    def has_ffn(self) -> bool:
        return self.router is not None or self.dense is not None


@dataclass(frozen=True)
class LayerRun:
    """One run of a layer: looped layers run several times with the same weights, each run with its own cache and state."""
    layer: int
    add_embedding: bool = False          # the embedding row is added to the residual right before this run
    join: int = -1                       # pass t >= 0 starts here: x = W [x; embedding row] + step vector t


@dataclass(frozen=True)
class ModelConfig:
    name: str = "tiny-moe"
    family: str = "deepseek_v3"          # deepseek_v3 | deepseek_v32 | qwen3_moe | glm4_moe | qwen2 | llama | tiny_moe
    vocab_size: int = 1024
    num_layers: int = 2
    hidden: int = 256
    # attention
    attention: str = "mla"               # "mla" | "gqa"
    num_heads: int = 4
    num_kv_heads: int = 4                # gqa only
    head_dim: int = 64                   # gqa only
    qk_norm: bool = False                # Qwen3: RMSNorm over head_dim on q and k
    rotary_dim: int = 0                  # gqa: leading dims of a head that are rotated (0 = all; GLM-4.5: half the head)
    attention_bias: bool = False         # gqa: q / k / v projections carry a bias (GLM-4.5, Qwen2)
    sliding_window: int = 0              # gqa: a query at position t sees keys (t - window, t] on the windowed layers (0 = none)
    window_layers: tuple = ()            # per layer, 1 = windowed; empty = every layer when sliding_window is set
    q_lora_rank: int = 128               # mla (0 = direct q projection)
    kv_lora_rank: int = 64
    qk_nope_dim: int = 32
    qk_rope_dim: int = 32
    v_head_dim: int = 32
    rope_theta: float = 10000.0
    rope_interleaved: bool = True        # pairs (2i, 2i+1); False = rotate-half (neox)
    # long-context frequency scaling of the checkpoint (config.json "rope_scaling"); see ref/ops.py::rope_inv_freq
    rope_scaling: str = "none"           # none | linear | llama3 | yarn
    rope_factor: float = 1.0
    rope_original_max: int = 4096        # positions the base frequencies were trained for (yarn, llama3)
    rope_beta_fast: float = 32.0         # yarn correction range
    rope_beta_slow: float = 1.0
    rope_mscale: float = 1.0             # yarn magnitude terms (DeepSeek: softmax scale *= mscale(all_dim)^2)
    rope_mscale_all_dim: float = 0.0
    rope_low_freq_factor: float = 1.0    # llama3
    rope_high_freq_factor: float = 4.0
    rms_eps: float = 1e-6
    # feed forward
    dense_ffn: int = 512                 # intermediate size of the dense SwiGLU layers
    first_dense_layers: int = 1          # layers [0, first_dense_layers) are dense
    num_experts: int = 8
    expert_ffn: int = 128
    top_k: int = 2
    scoring: str = "softmax"             # "softmax" | "sigmoid"
    num_groups: int = 1                  # group-limited routing (DeepSeek-V3: 8)
    topk_groups: int = 1                 # groups kept (DeepSeek-V3: 4)
    num_shared_experts: int = 1
    routed_scale: float = 1.0
    norm_topk_prob: bool = True
    router_bias: bool = False            # selection-only correction bias
    # speculation / sparse attention
    mtp_layers: int = 0
    indexer_heads: int = 0               # 0 = dense attention
    indexer_dim: int = 128
    indexer_topk: int = 2048
    # storage
    weight_format: str = "bf16"          # bf16 | fp8_block128 | nvfp4 | mxfp4 | exl3
    tie_embeddings: bool = False
    kv_format: str = "bf16"              # MLA cache record: bf16 (1152 bytes) | fp8_ds_mla (656 bytes; sparse attention only)
    # per-layer designs (attention == "hybrid"): one LayerSpec per layer; the flat fields above then only summarise it
    layer_specs: tuple = ()
    canon_taps: int = 0                  # taps of the convolution every sublayer's input passes (0 = none)
    norm_groups: int = 1                 # channel groups of the RMS norms
    norm_offset: float = 0.0             # added to the stored norm weights (1: they are stored around zero)
    norm_scalar: bool = False            # a norm's weight is one number for all channels
    loop: tuple = ()                     # (start, stop, times): layers [start, stop) run ``times`` times in a row
    loop_join: bool = False              # every pass starts with a product of [x; embedding row] and adds a vector of its own
    embed_scale: float = 1.0             # the embedding's rows are multiplied by it
    # (buckets, mul_prev, mul_cur): row (previous token * mul_prev + token * mul_cur) mod buckets of a second table is added to the
    # embedding row, for a sequence's first token the row after the last bucket
    bigram: tuple = ()
    # after every layer the residual becomes a weighted sum of the embedding rows and all layers' results so far
    depth_average: bool = False
    logit_softcap: float = 0.0           # logits = cap * tanh(logits / cap); 0 = none
    compute_dtype: str = "bf16"          # bf16 | f32 (every product and activation in 32-bit; hybrid engine only)

    # ---- derived -----------------------------------------------------------------
    @property
    def is_mla(self) -> bool:
        return self.attention == "mla"

    @property
    def qk_head_dim(self) -> int:
        return self.qk_nope_dim + self.qk_rope_dim if self.is_mla else self.head_dim

    @property
    def is_hybrid(self) -> bool:
        return self.attention == "hybrid"

    @property
    def layer_runs(self) -> tuple:
        """The layers in the order they run (``LayerRun``), loops unrolled."""
        start, stop, times = self.loop or (0, 0, 1)
        passes = [LayerRun(i, not self.loop_join and t > 0 and i == start, t if self.loop_join and i == start else -1)
                  for t in range(times) for i in range(start, stop)]
        return tuple([LayerRun(i) for i in range(start)] + passes + [LayerRun(i) for i in range(stop, self.num_layers)])

    def state_parts(self, layer: int) -> list[tuple[str, int]]:
        """(name, floats) of everything recurrent one run of ``layer`` carries per sequence."""
        spec = self.layer_specs[layer]
        m, out = spec.mixer, []
        if not spec.parallel and not spec.post_norm:
            out.append(("canon1", (self.canon_taps - 1) * self.hidden))
            if spec.router is not None:
                out.append(("canon2", (self.canon_taps - 1) * self.hidden))
        if isinstance(m, DeltaSpec):
            out += [("S", m.heads * m.dim * m.vdim), ("conv", (m.conv - 1) * m.conv_channels)]
        elif isinstance(m, RglruSpec):
            out += [("S", m.width), ("conv", (m.conv - 1) * m.width)]
        elif isinstance(m, PairSpec):
            out.append(("S", m.right.heads * m.right.dim * m.right.vdim))
        a = attention_part(m)
        if a is not None:
            out.append(("conv", max(0, a.conv - 1) * a.conv_channels))
        return out

    @property
    def state_bytes(self) -> int:
        """Recurrent state of one sequence (fp32): the mixers' states, the last inputs of every causal convolution, the last token."""
        return 4 * (sum(n for r in self.layer_runs for _, n in self.state_parts(r.layer)) + bool(self.bigram))

    def kv_elems_of(self, layer: int) -> int:
        """Elements one run of ``layer`` caches per token."""
        if self.is_hybrid:
            m = self.layer_specs[layer].mixer
            a = attention_part(m)
            if a is not None:
                return a.k_channels + a.v_channels
            return m.record if isinstance(m, LatentSpec) else 0
        return self.kv_record_elems

    @property
    def kv_record_elems(self) -> int:
        """Elements cached per token per layer (latent+rope for MLA, K and V for GQA; a hybrid's layer runs averaged over its layers)."""
        if self.is_hybrid:
            return -(-sum(self.kv_elems_of(r.layer) for r in self.layer_runs) // max(1, self.num_layers))
        if self.is_mla:
            return self.kv_lora_rank + self.qk_rope_dim
        return 2 * self.num_kv_heads * self.head_dim

    @property
    def rope_dim(self) -> int:
        """Dims of a head that RoPE rotates."""
        if self.is_mla:
            return self.qk_rope_dim
        return self.rotary_dim or self.head_dim

    def window_of(self, layer: int) -> int:
        """Sliding window of ``layer`` in tokens; 0 = full causal attention."""
        if self.is_hybrid:
            m = self.layer_specs[layer].mixer
            return getattr(attention_part(m) or m, "window", 0)
        if not self.sliding_window or self.is_mla:
            return 0
        if self.window_layers:
            return self.sliding_window if layer < len(self.window_layers) and self.window_layers[layer] else 0
        return self.sliding_window

    def is_moe_layer(self, layer: int) -> bool:
        if self.is_hybrid:
            return self.layer_specs[layer].router is not None
        return self.num_experts > 0 and layer >= self.first_dense_layers

    def mixer_params(self, layer: int) -> int:
        return self._mixer_params(self.layer_specs[layer].mixer)

    def _mixer_params(self, m: Any) -> int:
        h = self.hidden
        if isinstance(m, PairSpec):
            return self._mixer_params(m.left) + self._mixer_params(m.right)
        if isinstance(m, LightningSpec):
            return h * (m.channels + m.heads * m.vdim) + m.heads * m.vdim
        if isinstance(m, RglruSpec):
            return m.width * (3 * h + m.conv + 2 * m.block + 6)
        if isinstance(m, AttentionSpec):
            norms = {"": 0, "head": 2 * m.dim, "all": m.q_channels + m.k_channels, "rotated": 0}[m.qk_norm]
            return (h * (m.conv_channels + m.heads * m.vdim + m.heads * m.gate) + m.conv * m.conv_channels + norms + m.heads * m.sink
                    + (4 * m.dim if m.maps == 2 else 0))
        if isinstance(m, LatentSpec):
            return (h * (m.heads * (m.dim + m.rot_dim) + m.record + (1 + m.gate) * m.heads * m.vdim)
                    + m.kv_rank * (1 + m.heads * (m.dim + m.vdim)))
        return h * (m.conv_channels + 2 * m.heads + 2 * m.heads * m.vdim) + m.conv * m.conv_channels + 2 * m.heads + m.vdim

    def attention_params(self) -> int:
        h = self.hidden
        if self.is_hybrid:
            return sum(self.mixer_params(i) for i in range(self.num_layers)) // max(1, self.num_layers)
        if self.is_mla:
            q = (h * self.q_lora_rank + self.q_lora_rank * self.num_heads * self.qk_head_dim
                 if self.q_lora_rank else h * self.num_heads * self.qk_head_dim)
            kv = h * (self.kv_lora_rank + self.qk_rope_dim)
            kvb = self.kv_lora_rank * self.num_heads * (self.qk_nope_dim + self.v_head_dim)
            o = self.num_heads * self.v_head_dim * h
            return q + kv + kvb + o
        return h * (self.num_heads + 2 * self.num_kv_heads) * self.head_dim + self.num_heads * self.head_dim * h

    def expert_params(self) -> int:
        return 3 * self.hidden * self.expert_ffn

    def layer_params(self, layer: int) -> int:
        if self.is_hybrid:
            spec = self.layer_specs[layer]
            r, d = spec.router, spec.dense
            routed = r.outputs * (self.hidden + 1) + 3 * r.experts * self.hidden * r.ffn if r is not None else 0
            if spec.post_norm:
                norm = 1 if self.norm_scalar else self.hidden
                return (self.mixer_params(layer) + routed + (3 * self.hidden * d.ffn if d is not None else 0) + norm * (1 + spec.has_ffn)
                        + (layer + 2 if self.depth_average else 0))
            if spec.parallel:
                norms = 2 if spec.two_norms and (r is not None or d is not None) else 1
                return self.mixer_params(layer) + norms * self.hidden + routed + (3 * self.hidden * d.ffn if d is not None else 0)
            p = self.mixer_params(layer) + (2 + self.canon_taps) * self.hidden + routed
            if r is not None:
                p += (2 + self.canon_taps) * self.hidden
            return p
        p = self.attention_params() + 2 * self.hidden
        if self.is_moe_layer(layer):
            p += self.num_experts * self.expert_params() + self.hidden * self.num_experts
            p += self.num_shared_experts * self.expert_params()
        else:
            p += 3 * self.hidden * self.dense_ffn
        return p

    def total_params(self) -> int:
        p = self.vocab_size * self.hidden * (1 if self.tie_embeddings else 2) + (1 if self.norm_scalar else self.hidden)
        if self.bigram:
            p += (self.bigram[0] + 1) * self.hidden
        if self.loop and self.loop_join:
            p += (2 * self.hidden + self.loop[2]) * self.hidden
        return p + sum(self.layer_params(i) for i in range(self.num_layers))

    def to_json(self) -> str:
        return json.dumps(dataclasses.asdict(self), indent=1, sort_keys=True)

    @staticmethod
    def from_dict(d: dict[str, Any]) -> "ModelConfig":
        names = {f.name for f in dataclasses.fields(ModelConfig)}
        d = {k: v for k, v in d.items() if k in names}
        if "window_layers" in d:
            d["window_layers"] = tuple(d["window_layers"])
        for k in ("loop", "bigram"):
            if k in d:
                d[k] = tuple(d[k])
        if d.get("layer_specs"):
            d["layer_specs"] = tuple(v if isinstance(v, LayerSpec) else LayerSpec.from_dict(v) for v in d["layer_specs"])
        return ModelConfig(**d)

    def replace(self, **kw: Any) -> "ModelConfig":
        return dataclasses.replace(self, **kw)


def tiny_moe() -> ModelConfig:
    """The CPU correctness config: 2 layers, MLA, layer 0 dense, layer 1 MoE 8x top-2 + shared."""
    return ModelConfig()


def qwen3_30b_a3b() -> ModelConfig:
    """Qwen3-30B-A3B geometry (48 layers, GQA 32/4, 128 experts top-8, no shared expert)."""
    return ModelConfig(
        name="qwen3-30b-a3b", family="qwen3_moe", vocab_size=151936, num_layers=48, hidden=2048,
        attention="gqa", num_heads=32, num_kv_heads=4, head_dim=128, qk_norm=True,
        rope_theta=1.0e6, rope_interleaved=False, rms_eps=1e-6,
        dense_ffn=6144, first_dense_layers=0, num_experts=128, expert_ffn=768, top_k=8,
        scoring="softmax", num_shared_experts=0, norm_topk_prob=True, weight_format="bf16")


def deepseek_v3() -> ModelConfig:
    """DeepSeek-V3 geometry (61 layers, MLA 128 heads, 256 experts sigmoid group-limited top-8)."""
    return ModelConfig(
        name="deepseek-v3", family="deepseek_v3", vocab_size=129280, num_layers=61, hidden=7168,
        attention="mla", num_heads=128, q_lora_rank=1536, kv_lora_rank=512, qk_nope_dim=128,
        qk_rope_dim=64, v_head_dim=128, rope_theta=10000.0, rope_interleaved=True, rms_eps=1e-6,
        dense_ffn=18432, first_dense_layers=3, num_experts=256, expert_ffn=2048, top_k=8,
        scoring="sigmoid", num_groups=8, topk_groups=4, num_shared_experts=1, routed_scale=2.5,
        norm_topk_prob=True, router_bias=True, mtp_layers=1, weight_format="fp8_block128",
        # the shipped long-context setting: YaRN x40 over 4096 trained positions, mscale on the softmax scale
        rope_scaling="yarn", rope_factor=40.0, rope_original_max=4096, rope_beta_fast=32.0, rope_beta_slow=1.0,
        rope_mscale=1.0, rope_mscale_all_dim=1.0)


def deepseek_v32() -> ModelConfig:
    """DeepSeek-V3.2 geometry: V3 plus the lightning indexer and NVFP4 routed experts."""
    return deepseek_v3().replace(name="deepseek-v3.2", family="deepseek_v32", indexer_heads=64,
                                 indexer_dim=128, indexer_topk=2048, weight_format="nvfp4")


def mixtral_8x7b() -> ModelConfig:
    """Mixtral-8x7B geometry (32 layers, GQA 32/8, 8 experts top-2, softmax over the selected pair); served by the
    GQA engine, tensor names canonicalised by ``loader.families.canonical_name``."""
    return ModelConfig(
        name="mixtral-8x7b", family="qwen3_moe", vocab_size=32000, num_layers=32, hidden=4096,
        attention="gqa", num_heads=32, num_kv_heads=8, head_dim=128, qk_norm=False,
        rope_theta=1.0e6, rope_interleaved=False, rms_eps=1e-5,
        dense_ffn=14336, first_dense_layers=0, num_experts=8, expert_ffn=14336, top_k=2,
        scoring="softmax", num_shared_experts=0, norm_topk_prob=True, weight_format="bf16")


def mistral_7b() -> ModelConfig:
    """Mistral-7B-v0.1 geometry: a dense GQA 32 / 8 decoder whose every layer attends through a 4096-token sliding
    window; served by the GQA engine's dense path."""
    return ModelConfig(name="mistral-7b", family="llama", vocab_size=32000, num_layers=32, hidden=4096, attention="gqa",
                       num_heads=32, num_kv_heads=8, head_dim=128, qk_norm=False, sliding_window=4096, rope_theta=10000.0,
                       rope_interleaved=False, rms_eps=1e-5, dense_ffn=14336, first_dense_layers=32, num_experts=0,
                       expert_ffn=0, top_k=0, num_shared_experts=0)


def glm45_air() -> ModelConfig:
    """GLM-4.5-Air geometry (glm4_moe): 46 layers with one dense layer first, GQA 96 / 8 heads of 128 with biased q / k / v
    projections and RoPE on the first half of every head, 128 routed experts (FFN 1408) with sigmoid top-8 selection under a
    correction bias, one shared expert, one MTP depth."""
    return ModelConfig(name="glm-4.5-air", family="glm4_moe", vocab_size=151552, num_layers=46, hidden=4096, attention="gqa",
                       num_heads=96, num_kv_heads=8, head_dim=128, qk_norm=False, rotary_dim=64, attention_bias=True,
                       rope_theta=1.0e6, rope_interleaved=False, dense_ffn=10944, first_dense_layers=1, num_experts=128,
                       expert_ffn=1408, top_k=8, scoring="sigmoid", num_groups=1, topk_groups=1, num_shared_experts=1,
                       routed_scale=1.0, norm_topk_prob=True, router_bias=True, mtp_layers=1, rms_eps=1e-5)


def kimi_k2() -> ModelConfig:
    """Kimi-K2 geometry: the DeepSeek-V3 architecture with 64 heads and 384 routed experts (one dense layer, one
    routing group); served by the MLA engine."""
    return deepseek_v3().replace(name="kimi-k2", vocab_size=163840, num_heads=64, first_dense_layers=1, num_experts=384,
                                 num_groups=1, topk_groups=1, routed_scale=2.827, mtp_layers=0, rope_theta=50000.0,
                                 rope_factor=32.0, rope_beta_fast=1.0, rope_beta_slow=1.0)


def hybrid_config(name: str, vocab: int, hidden: int, specs, canon_taps: int, norm_groups: int, eps: float,
                  family: str = "karusun", **kw: Any) -> ModelConfig:
    """ModelConfig of a per-layer design.  The flat fields carry the widest layer's values for code that only sizes
    things (planner, reports); the engine reads the specs.  ``kw``: further fields (norm_offset, loop, logit_softcap)."""
    specs = tuple(specs)
    lat = [s.mixer for s in specs if isinstance(s.mixer, LatentSpec)]
    att = [a for a in (attention_part(s.mixer) for s in specs) if a is not None]
    routers = [s.router for s in specs if s.router is not None]
    big = max(lat, key=lambda m: m.heads * (m.dim + m.rot_dim), default=None)
    wide = max(routers, key=lambda r: r.experts * r.ffn, default=None)
    top = max(att, key=lambda m: m.conv_channels, default=None)
    rope = big.rope if big else top.rope if top else RopeSpec(0, 10000.0, halves=True)
    head_dim = (big.dim + big.rot_dim) if big else (top.maps * top.dim) if top else getattr(specs[0].mixer, "dim", 0)
    vdim = big.vdim if big else top.vdim if top else getattr(specs[0].mixer, "vdim", 0)
    return ModelConfig(
        name=name, family=family, vocab_size=vocab, num_layers=len(specs), hidden=hidden, attention="hybrid", layer_specs=specs,
        canon_taps=canon_taps, norm_groups=norm_groups, rms_eps=eps, rope_interleaved=not rope.halves,
        num_heads=max(getattr(s.mixer, "heads", 1) for s in specs), num_kv_heads=top.kv_heads if top else 1, head_dim=head_dim,
        q_lora_rank=0, kv_lora_rank=big.kv_rank if big else 0, qk_nope_dim=big.dim if big else 0, qk_rope_dim=big.rot_dim if big else 0,
        v_head_dim=vdim, rope_theta=rope.base,
        sliding_window=max((m.window for m in lat + att), default=0), dense_ffn=max((s.dense.ffn for s in specs if s.dense and not s.router), default=0),
        first_dense_layers=0, num_experts=wide.experts if wide else 0, expert_ffn=wide.ffn if wide else 0, top_k=wide.top if wide else 0,
        num_groups=wide.groups if wide else 1, topk_groups=wide.groups_kept if wide else 1, num_shared_experts=int(any(s.router and s.dense for s in specs)),
        norm_topk_prob=bool(wide and wide.normalize), router_bias=bool(routers), scoring=wide.scoring if wide else "softmax", **kw)


def parallel_config(name: str, vocab: int, hidden: int, specs, eps: float, loop: tuple = (), logit_softcap: float = 0.0,
                    family: str = "guberax", **kw: Any) -> ModelConfig:
    """ModelConfig of a stack of parallel layers: norm weights stored around zero, an optional loop, capped logits.  ``kw``: further
    fields (loop_join, embed_scale)."""
    return hybrid_config(name, vocab, hidden, specs, canon_taps=1, norm_groups=1, eps=eps, family=family, norm_offset=1.0,
                         loop=tuple(loop), logit_softcap=logit_softcap, **kw)


def post_norm_config(name: str, vocab: int, hidden: int, specs, eps: float, bigram: tuple = (), logit_softcap: float = 0.0,
                     family: str = "buzarax", **kw: Any) -> ModelConfig:
    """ModelConfig of a stack whose sublayers are normed after they ran, under one number per norm, with averages over depth."""
    return hybrid_config(name, vocab, hidden, specs, canon_taps=1, norm_groups=1, eps=eps, family=family, norm_scalar=True,
                         bigram=tuple(bigram), depth_average=True, logit_softcap=logit_softcap, **kw)


# Benchmark sizes: width, layers, heads, expert width (latent 512 + 64 and heads of 128 throughout, as real models have them)
KARUSUN_SIZES = {"small": (1024, 24, 16, 512), "base": (2048, 24, 32, 1024), "large": (4096, 12, 64, 1536)}


def karusun_bench(size: str = "base") -> ModelConfig:
    """A Karusun-shaped stack at the sizes of a real model's layers (latent 512 + 64, heads of 128, 64 router outputs top-6 of
    which the last eight hand their input through): three delta-rule layers to one latent attention layer."""
    width, layers, heads, ffn = KARUSUN_SIZES[size]
    r = RouterSpec(experts=56, ffn=ffn, top=6, identity=8, groups=8, groups_kept=4)
    lat = LatentSpec(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=2048, scale=192 ** -0.5,
                     rope=RopeSpec(64, 1.0e6, halves=True))
    delta = DeltaSpec(heads=heads, kv_heads=heads // 2, dim=128, vdim=128, conv=4)
    specs = [LayerSpec(lat if i % 4 == 3 else delta, r) for i in range(layers)]
    return hybrid_config(f"karusun-{size}", 65536, width, specs, canon_taps=4, norm_groups=4, eps=1e-5)


def karusun_bench_mla(size: str = "base") -> ModelConfig:
    """The MLA decoder at the size of ``karusun_bench``: same width, depth, heads, latent, experts and vocabulary."""
    width, layers, heads, ffn = KARUSUN_SIZES[size]
    return ModelConfig(name=f"mla-{size}", family="deepseek_v3", vocab_size=65536, num_layers=layers, hidden=width, attention="mla",
                       num_heads=heads, q_lora_rank=0, kv_lora_rank=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128, rope_theta=1.0e6,
                       rope_interleaved=False, rms_eps=1e-5, dense_ffn=0, first_dense_layers=0, num_experts=56, expert_ffn=ffn, top_k=6,
                       scoring="softmax", num_groups=8, topk_groups=4, num_shared_experts=0, norm_topk_prob=False, router_bias=True)


# Benchmark sizes: width, layers, heads, key / value heads, feed-forward width (two 64-wide maps and 128-wide values per head)
GUBERAX_SIZES = {"small": (1024, 24, 8, 4, 2816), "base": (2048, 24, 16, 8, 5632), "large": (4096, 16, 32, 8, 11008)}


def guberax_bench(size: str = "base") -> ModelConfig:
    """A Guberax-shaped stack at the sizes of a real model's layers: differential attention with a 2048-token window and 128
    kept tokens, four-tap convolutions, the middle third of the layers run twice."""
    width, layers, heads, kv_heads, ffn = GUBERAX_SIZES[size]
    m = AttentionSpec(heads=heads, kv_heads=kv_heads, dim=64, vdim=128, window=2048, keep_first=128, scale=64 ** -0.5,
                      rope=RopeSpec(64, 5.0e5, 8.0, 1.0, 4.0, 8192), conv=4, maps=2, diff=0.5)
    once = layers - layers // 4
    start = (once - layers // 4) // 2
    return parallel_config(f"guberax-{size}", 65536, width, [LayerSpec(m, dense=DenseSpec(ffn), parallel=True)] * once, eps=1e-6,
                           loop=(start, start + layers // 4, 2), logit_softcap=30.0)


def guberax_bench_gqa(size: str = "base") -> ModelConfig:
    """The dense GQA decoder at the size of ``guberax_bench``: as many layer runs of the same width, heads, window and
    feed-forward."""
    width, layers, heads, kv_heads, ffn = GUBERAX_SIZES[size]
    return ModelConfig(name=f"gqa-{size}", family="llama", vocab_size=65536, num_layers=layers, hidden=width, attention="gqa",
                       num_heads=heads, num_kv_heads=kv_heads, head_dim=128, qk_norm=False, sliding_window=2048, rope_theta=5.0e5,
                       rope_interleaved=False, rms_eps=1e-6, dense_ffn=ffn, first_dense_layers=layers, num_experts=0, expert_ffn=0,
                       top_k=0, num_shared_experts=0)


# Benchmark sizes: width, layer runs, heads, key / value heads, expert width (heads of 128, latent 512 + 64)
ROFAPEL_SIZES = {"small": (1024, 24, 8, 4, 512), "base": (2048, 24, 16, 8, 1024), "large": (4096, 12, 32, 8, 1536)}


def rofapel_bench(size: str = "base") -> ModelConfig:
    """A Rofapel-shaped stack at the sizes of a real model's layers: latent, windowed (values out of keys) and plain attention in
    turn, each beside 64 routed experts (top 6) and a shared one; a quarter of the layer runs are second passes."""
    width, runs, heads, kv_heads, ffn = ROFAPEL_SIZES[size]
    lat = LatentSpec(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=0, scale=192 ** -0.5,
                     rope=RopeSpec(64, 1.0e6, 8.0, 1.0, 32.0, 4096, "yarn"), gate=False)
    att = AttentionSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, window=0, keep_first=0, scale=128 ** -0.5,
                        rope=RopeSpec(128, 1.0e6, halves=True), qk_norm="all", gate=True)
    win = AttentionSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, window=2048, keep_first=0, scale=128 ** -0.5,
                        rope=RopeSpec(64, 1.0e4, 4.0, kind="linear", halves=True), conv=4, qk_norm="head", v_from_k=True, sink=True, gate=True)
    r = RouterSpec(experts=64, ffn=ffn, top=6, logit_bias=True, normalize=True)
    once = runs - runs // 4
    start = (once - runs // 4) // 2
    specs = [LayerSpec((lat, win, att)[i % 3], r, DenseSpec(ffn), parallel=True, two_norms=True) for i in range(once)]
    return parallel_config(f"rofapel-{size}", 65536, width, specs, eps=1e-5, loop=(start, start + runs // 4, 2), family="rofapel",
                           loop_join=True, embed_scale=width ** 0.5)


def rofapel_bench_gqa(size: str = "base") -> ModelConfig:
    """The GQA + MoE decoder at the size of ``rofapel_bench``: as many layer runs of the same width, heads, experts and shared
    expert, per-head norms of queries and keys, the same window on the layers that have one there."""
    width, runs, heads, kv_heads, ffn = ROFAPEL_SIZES[size]
    a = rofapel_bench(size)
    return ModelConfig(name=f"gqa-moe-{size}", family="qwen3_moe", vocab_size=65536, num_layers=runs, hidden=width, attention="gqa",
                       num_heads=heads, num_kv_heads=kv_heads, head_dim=128, qk_norm=True, sliding_window=2048,
                       window_layers=tuple(int(a.window_of(r.layer) > 0) for r in a.layer_runs), rope_theta=1.0e6, rope_interleaved=False,
                       rms_eps=1e-5, dense_ffn=0, first_dense_layers=0, num_experts=64, expert_ffn=ffn, top_k=6, scoring="softmax",
                       num_shared_experts=1, norm_topk_prob=True)


# Benchmark sizes: width, layers, heads, key / value heads, expert width (heads of 128 in both halves of a pair, recurrences as wide as
# the model in blocks of 128)
BUZARAX_SIZES = {"small": (1024, 24, 8, 4, 512), "base": (2048, 24, 16, 8, 1024), "large": (4096, 12, 32, 8, 1536)}


def buzarax_bench(size: str = "base") -> ModelConfig:
    """A Buzarax-shaped stack at the sizes of a real model's layers: attention beside linear attention and gated linear recurrences in
    turn, a dense feed-forward in the first layer, 64 routed experts (top 6) in the others."""
    width, layers, heads, kv_heads, ffn = BUZARAX_SIZES[size]
    att = AttentionSpec(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, window=0, keep_first=0, scale=128 ** -0.5,
                        rope=RopeSpec(64, 1.0e6, 4.0, 1.0, 32.0, 8192, "yarn", halves=True), qk_norm="rotated", softcap=30.0, unit_sink=True,
                        v_rope=RopeSpec(128, 1.0e6, halves=True))
    lin = LightningSpec(heads=heads, dim=128, vdim=128, decay=tuple(1.0 - 2.0 ** (-1 - 8.0 * h / heads) for h in range(heads)))
    pair, rec = PairSpec(att, lin, 0.75, 0.6), RglruSpec(width=width, blocks=width // 128, conv=4)
    r = RouterSpec(experts=64, ffn=ffn, top=6, scoring="sigmoid")
    specs = [LayerSpec(rec if i % 2 else pair, r if i else None, None if i else DenseSpec(6 * ffn, 7.0, 1.702, 1.0), post_norm=True) for i in range(layers)]
    return post_norm_config(f"buzarax-{size}", 65536, width, specs, eps=1e-5, bigram=(65521, 31, 7), logit_softcap=30.0)


def buzarax_bench_gqa(size: str = "base") -> ModelConfig:
    """The GQA + MoE decoder at the size of ``buzarax_bench``: same width, depth, heads, experts and vocabulary."""
    width, layers, heads, kv_heads, ffn = BUZARAX_SIZES[size]
    return ModelConfig(name=f"gqa-moe-{size}", family="qwen3_moe", vocab_size=65536, num_layers=layers, hidden=width, attention="gqa",
                       num_heads=heads, num_kv_heads=kv_heads, head_dim=128, qk_norm=True, rope_theta=1.0e6, rope_interleaved=False, rms_eps=1e-5,
                       dense_ffn=6 * ffn, first_dense_layers=1, num_experts=64, expert_ffn=ffn, top_k=6, scoring="softmax",
                       num_shared_experts=0, norm_topk_prob=True)


PRESETS = {
    "buzarax-base": buzarax_bench,
    "karusun-base": karusun_bench,
    "guberax-base": guberax_bench,
    "rofapel-base": rofapel_bench,
    "tiny-moe": tiny_moe,
    "mixtral-8x7b": mixtral_8x7b,
    "mistral-7b": mistral_7b,
    "kimi-k2": kimi_k2,
    "glm-4.5-air": glm45_air,
    "qwen3-30b-a3b": qwen3_30b_a3b,
    "deepseek-v3": deepseek_v3,
    "deepseek-v3.2": deepseek_v32,
}


def scaled_down(cfg: ModelConfig, layers: int = 2, vocab: int = 2048) -> ModelConfig:
    """Same per-layer geometry with fewer layers and a small vocabulary (tests, smoke)."""
    if cfg.is_hybrid:
        start, stop, times = cfg.loop or (0, 0, 1)
        return hybrid_config(cfg.name + "-mini", vocab, cfg.hidden, cfg.layer_specs[:layers], cfg.canon_taps, cfg.norm_groups,
                             cfg.rms_eps, cfg.family, norm_offset=cfg.norm_offset, logit_softcap=cfg.logit_softcap,
                             loop_join=cfg.loop_join, embed_scale=cfg.embed_scale, norm_scalar=cfg.norm_scalar, bigram=cfg.bigram,
                             depth_average=cfg.depth_average,
                             loop=(start, min(stop, layers), times) if start < layers and cfg.loop else ())
    first_dense = min(cfg.first_dense_layers, max(layers - 1, 0)) if cfg.first_dense_layers else 0
    return cfg.replace(name=cfg.name + "-mini", num_layers=layers, vocab_size=vocab,
                       first_dense_layers=first_dense)
