"""Hugging Face snapshot layout: ``config.json`` <-> ``ModelConfig``, snapshot resolution, and
writers of random-init snapshots in each shipped weight format.

A snapshot is a directory with config.json, model.safetensors.index.json and shards; runs load it
"as shipped", nothing is repacked on disk.  Counterpart: rust/crates/cuteafd-loader/src/snapshot.rs
(resolve), plan/testing.rs (snapshot writers for tests).
"""
from __future__ import annotations

import json
import os

import torch

from ..config import (AttentionSpec, DeltaSpec, DenseSpec, LatentSpec, LayerSpec, LightningSpec, ModelConfig, PairSpec, RglruSpec, RopeSpec,
                      RouterSpec, hybrid_config, parallel_config, post_norm_config)
from ..ref.model import init_weights
from . import formats
from .safetensors_io import write_sharded

ARCH = {"llama": "LlamaForCausalLM", "qwen3_moe": "Qwen3MoeForCausalLM", "deepseek_v3": "DeepseekV3ForCausalLM",
        "deepseek_v32": "DeepseekV32ForCausalLM", "tiny_moe": "DeepseekV3ForCausalLM", "glm4_moe": "Glm4MoeForCausalLM",
        "qwen2": "Qwen2ForCausalLM"}


def _layer_list_to_json(cfg: ModelConfig) -> dict:
    """config.json of a per-layer design (the ``layers`` list form)."""
    if cfg.family == "guberax":
        return _parallel_layers_to_json(cfg)
    if cfg.family == "rofapel":
        return _two_norm_layers_to_json(cfg)
    if cfg.family == "buzarax":
        return _post_norm_layers_to_json(cfg)
    layers = []
    for s in cfg.layer_specs:
        m, r = s.mixer, s.router
        if isinstance(m, LatentSpec):
            e = {"type": "latent_attention", "mixer": {
                "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale,
                "mask": {"size": m.window}, "rot": {"base": m.rope.base, "dims": m.rot_dim}}}
        else:
            e = {"type": "delta", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}}
        e["mlp"] = None if r is None else {"kind": "moe", "expert": {"ff": r.ffn}, "router": {
            "experts": r.experts, "identity": r.identity, "top": r.top, "groups": {"count": r.groups, "keep": r.groups_kept}}}
        layers.append(e)
    return {"architecture": "Karusun", "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden, "layers": layers,
            "canon": {"taps": cfg.canon_taps}, "norm": {"eps": cfg.rms_eps, "groups": cfg.norm_groups}}


def _parallel_layers_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m, r = s.mixer, s.mixer.rope
        rot = {"base": r.base, "dims": r.dims}
        if r.factor != 1.0:
            rot["scaling"] = {"factor": r.factor, "low": r.low, "high": r.high, "original": r.original}
        e = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv, "diff": m.diff, "scale": m.scale, "rot": rot}
        if m.window:
            e["mask"] = {"size": m.window, "keep_first": m.keep_first}
        layers.append({"type": "attention", "mixer": e, "mlp": None if s.dense is None else {"kind": "dense", "ff": s.dense.ffn}})
    d = {"architecture": "Guberax", "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden, "layers": layers, "norm": {"eps": cfg.rms_eps}}
    if cfg.loop:
        d["loop"] = dict(zip(("start", "stop", "times"), cfg.loop))
    if cfg.logit_softcap:
        d["logit_softcap"] = cfg.logit_softcap
    return d


def _loop_of(d: dict, layers: int) -> tuple:
    lp = d.get("loop")
    loop = (lp["start"], lp["stop"], lp["times"]) if lp and lp["stop"] != lp["start"] else ()
    if loop and not (0 <= loop[0] < loop[1] <= layers and loop[2] >= 1):
        raise ValueError(f"loop {loop} over {layers} layers")
    return loop


def _silu_only(i: int, *parts: dict) -> None:
    for e in parts:
        if (e.get("act") or "silu") != "silu":
            raise ValueError(f"layer {i}: unsupported feed-forward activation {e['act']!r}")


# How the two attention mixers of Rofapel treat queries, keys and values; everything else about them is in the configuration.
_TWO_NORM_ATTENTION = {"attention": dict(qk_norm="all", gate=True),
                       "attention_2": dict(qk_norm="head", v_from_k=True, sink=True, gate=True)}


def _rope_from_json(i: int, rot: dict, dims: int, halves: bool) -> RopeSpec:
    """``rot`` of a mixer whose rotated vectors are ``dims`` wide."""
    sc, n = rot.get("scaling") or {}, rot.get("dims", dims)
    if n % 2 or n > dims:
        raise ValueError(f"layer {i}: {n} rotated dims of {dims}")
    if not sc:
        return RopeSpec(n, float(rot["base"]), halves=halves)
    if set(sc) == {"factor"}:
        return RopeSpec(n, float(rot["base"]), float(sc["factor"]), kind="linear", halves=halves)
    if set(sc) == {"factor", "original", "fast", "slow"}:
        return RopeSpec(n, float(rot["base"]), float(sc["factor"]), float(sc["slow"]), float(sc["fast"]), sc["original"], "yarn", halves)
    raise ValueError(f"layer {i}: unsupported rotary scaling {sorted(sc)}")


def _rope_to_json(r: RopeSpec) -> dict:
    rot = {"base": r.base, "dims": r.dims}
    if r.kind == "linear":
        rot["scaling"] = {"factor": r.factor}
    elif r.kind == "yarn":
        rot["scaling"] = {"factor": r.factor, "original": r.original, "fast": r.high, "slow": r.low}
    return rot


def _two_norm_layers_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m, r = s.mixer, s.router
        e = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": _rope_to_json(m.rope)}
        if isinstance(m, LatentSpec):
            kind = "latent_attention"
            e.update(rot_dim=m.rot_dim, kv_rank=m.kv_rank)
        else:
            kind = "attention_2" if m.v_from_k else "attention"
            e["kv_heads"] = m.kv_heads
            if m.conv:
                e["conv"] = m.conv
        if m.window:
            e["mask"] = {"size": m.window}
        mlp = None
        if r is not None:
            mlp = {"kind": "moe", "expert": {"ff": r.ffn}, "router": {"experts": r.experts, "top": r.top}}
            if s.dense is not None:
                mlp["shared"] = {"ff": s.dense.ffn}
        elif s.dense is not None:
            mlp = {"kind": "dense", "ff": s.dense.ffn}
        layers.append({"type": kind, "mixer": e, "mlp": mlp})
    d = {"architecture": "Rofapel", "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden, "layers": layers,
         "norm": {"eps": cfg.rms_eps}, "embedding": {"scale": cfg.embed_scale}}
    if cfg.loop:
        d["loop"] = dict(zip(("start", "stop", "times"), cfg.loop))
    return d


def _two_norm_layers_from_json(d: dict) -> ModelConfig:
    """Parallel layers with a norm for each half: latent attention or one of two attention mixers beside a dense or routed
    feed-forward (``architecture`` Rofapel)."""
    specs = []
    for i, e in enumerate(d["layers"]):
        m, mlp, kind = e["mixer"], e.get("mlp"), e["type"]
        window = (m.get("mask") or {}).get("size") or 0
        if kind == "latent_attention":
            rope = _rope_from_json(i, m["rot"], m["rot_dim"], halves=False)
            if rope.dims != m["rot_dim"]:
                raise ValueError(f"layer {i}: {rope.dims} rotated dims of a rotated part of {m['rot_dim']} are not supported")
            mixer = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], window=window,
                               scale=float(m["scale"]), rope=rope, gate=False)
        elif kind in _TWO_NORM_ATTENTION:
            mixer = AttentionSpec(heads=m["heads"], kv_heads=m.get("kv_heads") or m["heads"], dim=m["dim"], vdim=m.get("vdim") or m["dim"],
                                  window=window, keep_first=0, scale=float(m["scale"]), rope=_rope_from_json(i, m["rot"], m["dim"], halves=True),
                                  conv=m.get("conv") or 0, **_TWO_NORM_ATTENTION[kind])
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key heads")
            if mixer.v_from_k and mixer.vdim != mixer.dim:
                raise ValueError(f"layer {i}: values of {mixer.vdim} out of keys of {mixer.dim}")
        else:
            raise ValueError(f"layer {i}: unsupported mixer {kind!r}")
        router = dense = None
        if mlp is not None and mlp.get("kind") == "dense":
            _silu_only(i, mlp)
            dense = DenseSpec(mlp["ff"])
        elif mlp is not None and mlp.get("kind") == "moe":
            r, shared = mlp["router"], mlp.get("shared")
            _silu_only(i, mlp["expert"], shared or {})
            router = RouterSpec(experts=r["experts"], ffn=mlp["expert"]["ff"], top=r["top"], logit_bias=True, normalize=True)
            if not 1 <= router.top <= router.experts:
                raise ValueError(f"layer {i}: {router.top} of {router.experts} experts")
            dense = DenseSpec(shared["ff"]) if shared else None
        elif mlp is not None:
            raise ValueError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
        specs.append(LayerSpec(mixer, router, dense, parallel=True, two_norms=True))
    return parallel_config(d.get("name", d["architecture"].lower()), d["vocab"], d["width"], specs, float(d["norm"]["eps"]),
                           _loop_of(d, len(specs)), family="rofapel", loop_join=True,
                           embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)))


# Constants of Buzarax's feed-forward that its configuration does not carry.
_CLIPPED_ALPHA, _CLIPPED_UP_BIAS = 1.702, 1.0


def _post_norm_layers_to_json(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m, r, mlp = s.mixer, s.router, None
        if isinstance(m, PairSpec):
            a, b = m.left, m.right
            e = {"type": "parallel", "mixer": {
                "left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "softcap": a.softcap or None,
                         "rot": _rope_to_json(a.rope)},
                "right": {"heads": b.heads, "dim": b.dim, "vdim": b.vdim, "decay": list(b.decay)},
                "left_scale": m.left_scale, "right_scale": m.right_scale}}
        else:
            e = {"type": "rglru", "mixer": {"width": m.width, "blocks": m.blocks, "conv": m.conv}}
        if r is not None:
            mlp = {"kind": "moe", "expert": {"ff": r.ffn}, "router": {"experts": r.experts, "top": r.top}}
        elif s.dense is not None:
            mlp = {"kind": "dense", "ff": s.dense.ffn, "limit": s.dense.limit}
        layers.append(dict(e, mlp=mlp))
    d = {"architecture": "Buzarax", "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden, "layers": layers, "norm": {"eps": cfg.rms_eps},
         "embedding": {}}
    if cfg.bigram:
        d["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), cfg.bigram))
    if cfg.logit_softcap:
        d["logit_softcap"] = cfg.logit_softcap
    return d


def _post_norm_layers_from_json(d: dict) -> ModelConfig:
    """Layers whose sublayers are normed after they ran: a gated linear recurrence, or attention beside linear attention, then a dense
    or routed feed-forward or none (``architecture`` Buzarax)."""
    specs = []
    for i, e in enumerate(d["layers"]):
        m, mlp, kind = e["mixer"], e.get("mlp"), e["type"]
        if kind == "rglru":
            mixer = RglruSpec(width=m["width"], blocks=m["blocks"], conv=m["conv"])
            if mixer.width % mixer.blocks:
                raise ValueError(f"layer {i}: {mixer.width} channels in {mixer.blocks} blocks")
        elif kind == "parallel":
            a, b = m["left"], m["right"]
            rope, vdim = _rope_from_json(i, a["rot"], a["dim"], halves=True), a.get("vdim") or a["dim"]
            if vdim % 2:
                raise ValueError(f"layer {i}: values of {vdim} are rotated in pairs")
            left = AttentionSpec(heads=a["heads"], kv_heads=a.get("kv_heads") or a["heads"], dim=a["dim"], vdim=vdim, window=0, keep_first=0,
                                 scale=float(a["scale"]), rope=rope, qk_norm="rotated", softcap=float(a.get("softcap") or 0.0), unit_sink=True,
                                 v_rope=RopeSpec(vdim, rope.base, halves=True))
            right = LightningSpec(heads=b["heads"], dim=b["dim"], vdim=b.get("vdim") or b["dim"], decay=tuple(float(x) for x in b["decay"]))
            mixer = PairSpec(left, right, float(m.get("left_scale", 1.0)), float(m.get("right_scale", 1.0)))
            if left.heads % left.kv_heads:
                raise ValueError(f"layer {i}: {left.heads} heads over {left.kv_heads} key heads")
            if len(right.decay) != right.heads:
                raise ValueError(f"layer {i}: {len(right.decay)} decays for {right.heads} heads")
        else:
            raise ValueError(f"layer {i}: unsupported mixer {kind!r}")
        router = dense = None
        if mlp is not None and mlp.get("kind") == "dense":
            dense = DenseSpec(mlp["ff"], limit=float(mlp.get("limit") or 0.0), alpha=_CLIPPED_ALPHA, up_bias=_CLIPPED_UP_BIAS)
        elif mlp is not None and mlp.get("kind") == "moe":
            _silu_only(i, mlp["expert"])
            r = mlp["router"]
            router = RouterSpec(experts=r["experts"], ffn=mlp["expert"]["ff"], top=r["top"], scoring="sigmoid")
            if not 1 <= router.top <= router.experts:
                raise ValueError(f"layer {i}: {router.top} of {router.experts} experts")
        elif mlp is not None:
            raise ValueError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
        specs.append(LayerSpec(mixer, router, dense, post_norm=True))
    g = (d.get("embedding") or {}).get("bigram")
    return post_norm_config(d.get("name", d["architecture"].lower()), d["vocab"], d["width"], specs, float(d["norm"]["eps"]),
                            bigram=(g["buckets"], g["mul_prev"], g["mul_cur"]) if g else (), logit_softcap=float(d.get("logit_softcap") or 0.0))


def _parallel_layers_from_json(d: dict) -> ModelConfig:
    """Parallel layers of differential attention and a dense feed-forward (``architecture`` Guberax)."""
    specs = []
    for i, e in enumerate(d["layers"]):
        m, mlp = e["mixer"], e.get("mlp")
        if e["type"] != "attention":
            raise ValueError(f"layer {i}: unsupported mixer {e['type']!r}")
        rot, mask = m["rot"], m.get("mask") or {}
        sc = rot.get("scaling") or {}
        rope = RopeSpec(dims=rot.get("dims", m["dim"]), base=float(rot["base"]))
        if float(sc.get("factor", 1.0)) != 1.0:
            rope = RopeSpec(rope.dims, rope.base, float(sc["factor"]), float(sc["low"]), float(sc["high"]), int(sc["original"]))
        mixer = AttentionSpec(heads=m["heads"], kv_heads=m.get("kv_heads") or m["heads"], dim=m["dim"], vdim=m.get("vdim") or m["dim"],
                              window=mask.get("size") or 0, keep_first=(mask.get("keep_first") or 0) if mask.get("size") else 0,
                              scale=float(m["scale"]), rope=rope, conv=m.get("conv") or 0, maps=2, diff=float(m["diff"]))
        if mixer.heads % mixer.kv_heads:
            raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key heads")
        if rope.dims % 2 or rope.dims > mixer.dim:
            raise ValueError(f"layer {i}: {rope.dims} rotated dims of {mixer.dim}")
        dense = None
        if mlp is not None:
            if mlp.get("kind") != "dense" or (mlp.get("act") or "silu") != "silu":
                raise ValueError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r} {mlp.get('act') or ''}")
            dense = DenseSpec(mlp["ff"])
        specs.append(LayerSpec(mixer, dense=dense, parallel=True))
    loop = _loop_of(d, len(specs))
    return parallel_config(d.get("name", d["architecture"].lower()), d["vocab"], d["width"], specs, float(d["norm"]["eps"]), loop,
                           float(d.get("logit_softcap") or 0.0))


def _layer_list_from_json(d: dict) -> ModelConfig:
    """The ``layers`` list form of config.json.  Every layer carries its own sizes; a type or kind that is not built is
    refused by name."""
    if d["architecture"] == "Guberax":
        return _parallel_layers_from_json(d)
    if d["architecture"] == "Rofapel":
        return _two_norm_layers_from_json(d)
    if d["architecture"] == "Buzarax":
        return _post_norm_layers_from_json(d)
    specs = []
    for i, e in enumerate(d["layers"]):
        m, mlp = e["mixer"], e.get("mlp")
        if e["type"] == "latent_attention":
            rot = m["rot"]
            if rot.get("dims", m["rot_dim"]) != m["rot_dim"]:
                raise ValueError(f"layer {i}: {rot['dims']} rotated dims of a rotated part of {m['rot_dim']} are not supported")
            mixer = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                               window=m["mask"]["size"], scale=float(m["scale"]),
                               rope=RopeSpec(m["rot_dim"], float(rot["base"]), halves=True))
        elif e["type"] == "delta":
            mixer = DeltaSpec(heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"], vdim=m["vdim"], conv=m["conv"])
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key heads")
        else:
            raise ValueError(f"layer {i}: unsupported mixer {e['type']!r}")
        router = None
        if mlp is not None:
            if mlp.get("kind") != "moe":
                raise ValueError(f"layer {i}: unsupported feed-forward {mlp.get('kind')!r}")
            r = mlp["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            router = RouterSpec(experts=r["experts"], ffn=mlp["expert"]["ff"], top=r["top"], identity=r.get("identity", 0) or 0,
                                groups=g["count"], groups_kept=g["keep"])
            if router.outputs % router.groups:
                raise ValueError(f"layer {i}: {router.outputs} router outputs in {router.groups} groups")
        specs.append(LayerSpec(mixer, router))
    return hybrid_config(d.get("name", d["architecture"].lower()), d["vocab"], d["width"], specs, d["canon"]["taps"],
                         d["norm"].get("groups", 1), float(d["norm"]["eps"]))


def to_hf_config(cfg: ModelConfig) -> dict:
    if cfg.is_hybrid:
        return _layer_list_to_json(cfg)
    d = {"architectures": [ARCH.get(cfg.family, "DeepseekV3ForCausalLM")], "model_type": cfg.family,
         "vocab_size": cfg.vocab_size, "hidden_size": cfg.hidden, "num_hidden_layers": cfg.num_layers,
         "num_attention_heads": cfg.num_heads, "rms_norm_eps": cfg.rms_eps, "rope_theta": cfg.rope_theta,
         "tie_word_embeddings": cfg.tie_embeddings, "torch_dtype": "bfloat16",
         "intermediate_size": cfg.dense_ffn, "moe_intermediate_size": cfg.expert_ffn,
         "num_experts_per_tok": cfg.top_k, "norm_topk_prob": cfg.norm_topk_prob,
         "cuteafd": {"name": cfg.name, "rope_interleaved": cfg.rope_interleaved, "family": cfg.family}}
    if cfg.is_mla:
        d.update(q_lora_rank=cfg.q_lora_rank or None, kv_lora_rank=cfg.kv_lora_rank, qk_nope_head_dim=cfg.qk_nope_dim,
                 qk_rope_head_dim=cfg.qk_rope_dim, v_head_dim=cfg.v_head_dim, n_routed_experts=cfg.num_experts,
                 n_shared_experts=cfg.num_shared_experts, first_k_dense_replace=cfg.first_dense_layers,
                 scoring_func=cfg.scoring, n_group=cfg.num_groups, topk_group=cfg.topk_groups,
                 routed_scaling_factor=cfg.routed_scale, num_nextn_predict_layers=cfg.mtp_layers,
                 topk_method="noaux_tc" if cfg.router_bias else "greedy")
        if cfg.indexer_heads:
            d.update(index_n_heads=cfg.indexer_heads, index_head_dim=cfg.indexer_dim, index_topk=cfg.indexer_topk)
    elif cfg.family == "glm4_moe":
        d.update(num_key_value_heads=cfg.num_kv_heads, head_dim=cfg.head_dim, n_routed_experts=cfg.num_experts,
                 n_shared_experts=cfg.num_shared_experts, first_k_dense_replace=cfg.first_dense_layers, n_group=cfg.num_groups,
                 topk_group=cfg.topk_groups, routed_scaling_factor=cfg.routed_scale, use_qk_norm=cfg.qk_norm,
                 attention_bias=cfg.attention_bias, partial_rotary_factor=cfg.rope_dim / cfg.head_dim,
                 num_nextn_predict_layers=cfg.mtp_layers)
    else:
        d.update(num_key_value_heads=cfg.num_kv_heads, head_dim=cfg.head_dim, num_experts=cfg.num_experts,
                 decoder_sparse_step=1, mlp_only_layers=list(range(cfg.first_dense_layers)), qk_norm=cfg.qk_norm)
        if cfg.attention_bias:
            d["attention_bias"] = True
    if cfg.sliding_window and not cfg.is_mla:
        d.update(sliding_window=cfg.sliding_window, use_sliding_window=True,
                 layer_types=["sliding_attention" if cfg.window_of(i) else "full_attention" for i in range(cfg.num_layers)])
    if cfg.rope_scaling != "none":
        rs = {"type": cfg.rope_scaling, "rope_type": cfg.rope_scaling, "factor": cfg.rope_factor,
              "original_max_position_embeddings": cfg.rope_original_max}
        if cfg.rope_scaling == "yarn":
            rs.update(beta_fast=cfg.rope_beta_fast, beta_slow=cfg.rope_beta_slow, mscale=cfg.rope_mscale,
                      mscale_all_dim=cfg.rope_mscale_all_dim)
        if cfg.rope_scaling == "llama3":
            rs.update(low_freq_factor=cfg.rope_low_freq_factor, high_freq_factor=cfg.rope_high_freq_factor)
        d["rope_scaling"] = rs
    if cfg.weight_format == "fp8_block128":
        d["quantization_config"] = {"quant_method": "fp8", "fmt": "e4m3", "weight_block_size": [128, 128],
                                    "activation_scheme": "dynamic"}
    elif cfg.weight_format == "nvfp4":
        d["quantization_config"] = {"quant_method": "modelopt", "quant_algo": "NVFP4", "group_size": 16}
    elif cfg.weight_format == "mxfp4":
        d["quantization_config"] = {"quant_method": "mxfp4", "group_size": 32}
    elif cfg.weight_format.startswith("exl3"):
        d["quantization_config"] = {"quant_method": "exl3", "bits": 4}
    return d


def _windows(d: dict) -> dict:
    """config.json sliding-window fields -> ModelConfig fields.  ``layer_types`` names the windowed layers where it is
    present; the Qwen2 / Qwen3 form (``use_sliding_window`` with ``max_window_layers``) windows the layers from that
    index on; a bare ``sliding_window`` (Mistral, Mixtral) windows every layer."""
    w, n = d.get("sliding_window"), d["num_hidden_layers"]
    kinds = d.get("layer_types")
    if kinds:
        unknown = set(kinds) - {"sliding_attention", "full_attention"}
        if unknown or len(kinds) != n:
            raise ValueError(f"layer_types {sorted(unknown)} / {len(kinds)} entries for {n} layers is not supported")
        flags = tuple(1 if k == "sliding_attention" else 0 for k in kinds)
    elif str(d.get("model_type", "")).startswith("qwen"):
        first = d.get("max_window_layers", n) if d.get("use_sliding_window") else n
        flags = tuple(1 if i >= first else 0 for i in range(n))
    else:
        flags = (1,) * n
    if not w or not any(flags):
        return {}
    return {"sliding_window": int(w), "window_layers": () if all(flags) else flags}


def _rope_scaling(d: dict) -> dict:
    """config.json ``rope_scaling`` / ``rope_parameters`` -> ModelConfig fields.  Unknown kinds are refused: serving a
    long-context checkpoint with the wrong frequencies gives fluent nonsense, not an error."""
    rs = d.get("rope_scaling") or d.get("rope_parameters") or {}
    kind = rs.get("rope_type") or rs.get("type") or "none"
    if kind in ("none", "default") or not rs:
        return {}
    if kind not in ("linear", "llama3", "yarn"):
        raise ValueError(f"unsupported rope scaling {kind!r}")
    out = dict(rope_scaling=kind, rope_factor=float(rs.get("factor", 1.0)),
               rope_original_max=int(rs.get("original_max_position_embeddings") or d.get("max_position_embeddings") or 4096))
    if kind == "yarn":
        out.update(rope_beta_fast=float(rs.get("beta_fast") or 32.0), rope_beta_slow=float(rs.get("beta_slow") or 1.0),
                   rope_mscale=float(rs.get("mscale") or 1.0), rope_mscale_all_dim=float(rs.get("mscale_all_dim") or 0.0))
    if kind == "llama3":
        out.update(rope_low_freq_factor=float(rs.get("low_freq_factor", 1.0)), rope_high_freq_factor=float(rs.get("high_freq_factor", 4.0)))
    return out


def from_hf_config(d: dict) -> ModelConfig:
    """Map a config.json onto the engine's geometry.  Unknown architectures raise ValueError."""
    if d.get("architecture") in ("Karusun", "Guberax", "Rofapel", "Buzarax"):
        return _layer_list_from_json(d)
    mt = d.get("model_type", "")
    extra = d.get("cuteafd", {})
    q = d.get("quantization_config") or {}
    fmt = {"fp8": "fp8_block128", "modelopt": "nvfp4", "mxfp4": "mxfp4", "exl3": "exl3"}.get(q.get("quant_method", ""), "bf16")
    common = dict(name=extra.get("name", d.get("_name_or_path", mt) or mt), vocab_size=d["vocab_size"],
                  num_layers=d["num_hidden_layers"], hidden=d["hidden_size"], num_heads=d["num_attention_heads"],
                  rms_eps=d.get("rms_norm_eps", 1e-6), rope_theta=float(d.get("rope_theta") or (d.get("rope_parameters") or {}).get("rope_theta") or 10000.0),
                  tie_embeddings=bool(d.get("tie_word_embeddings", False)), dense_ffn=d.get("intermediate_size", 0),
                  expert_ffn=d.get("moe_intermediate_size", 0), top_k=d.get("num_experts_per_tok", 0),
                  norm_topk_prob=bool(d.get("norm_topk_prob", True)), weight_format=fmt, **_rope_scaling(d))
    if mt in ("deepseek_v3", "deepseek_v32", "deepseek_v2", "tiny_moe", "glm_moe_dsa", "kimi_k2"):
        return ModelConfig(
            family=extra.get("family", "deepseek_v32" if d.get("index_n_heads") else "deepseek_v3"), attention="mla",
            q_lora_rank=d.get("q_lora_rank") or 0, kv_lora_rank=d["kv_lora_rank"], qk_nope_dim=d["qk_nope_head_dim"],
            qk_rope_dim=d["qk_rope_head_dim"], v_head_dim=d["v_head_dim"],
            rope_interleaved=extra.get("rope_interleaved", True), first_dense_layers=d.get("first_k_dense_replace", 0),
            num_experts=d.get("n_routed_experts", 0), scoring=d.get("scoring_func", "softmax"),
            num_groups=d.get("n_group", 1) or 1, topk_groups=d.get("topk_group", 1) or 1,
            num_shared_experts=d.get("n_shared_experts", 0) or 0, routed_scale=d.get("routed_scaling_factor", 1.0),
            router_bias=d.get("topk_method") == "noaux_tc", mtp_layers=d.get("num_nextn_predict_layers", 0) or 0,
            indexer_heads=d.get("index_n_heads", 0) or 0, indexer_dim=d.get("index_head_dim", 128),
            indexer_topk=d.get("index_topk", 2048), **common)
    if mt in ("qwen3_moe", "qwen3", "qwen2_moe", "mixtral"):
        # refuse what the engines would silently compute differently
        if d.get("shared_expert_intermediate_size"):
            raise ValueError("a gated shared expert (shared_expert_intermediate_size) is not supported")
        if d.get("decoder_sparse_step", 1) not in (0, 1):
            raise ValueError("interleaved dense / sparse layers (decoder_sparse_step > 1) are not supported")
        dense_layers = sorted(d.get("mlp_only_layers", []) or [])
        if dense_layers != list(range(len(dense_layers))):
            raise ValueError("dense layers must be the first layers of the stack")
        if d.get("attention_bias"):
            raise ValueError("projection biases are not supported for this model type")
        return ModelConfig(
            family="qwen3_moe", attention="gqa", num_kv_heads=d.get("num_key_value_heads", d["num_attention_heads"]),
            head_dim=d.get("head_dim", d["hidden_size"] // d["num_attention_heads"]), qk_norm=bool(d.get("qk_norm", mt.startswith("qwen3"))),
            rope_interleaved=extra.get("rope_interleaved", False), first_dense_layers=len(d.get("mlp_only_layers", []) or []),
            num_experts=d.get("num_experts", d.get("num_local_experts", 0)), scoring="softmax", num_shared_experts=0, **_windows(d), **common)
    if mt == "glm4_moe":
        # GLM-4.5 / 4.6: GQA with biased q / k / v projections and RoPE on part of every head, sigmoid routing under a
        # correction bias (noaux_tc), one shared expert, dense layers first, optional MTP depth
        hd = d.get("head_dim") or d["hidden_size"] // d["num_attention_heads"]
        rot = int(round(hd * float(d.get("partial_rotary_factor", 1.0))))
        if hd != 128 or rot not in (64, 128):
            raise ValueError(f"glm4_moe with head_dim {hd} and {rot} rotated dims is not supported (128 with 64 or 128)")
        return ModelConfig(
            family="glm4_moe", attention="gqa", num_kv_heads=d.get("num_key_value_heads", d["num_attention_heads"]), head_dim=hd,
            qk_norm=bool(d.get("use_qk_norm", False)), rotary_dim=0 if rot == hd else rot, attention_bias=bool(d.get("attention_bias", False)),
            rope_interleaved=extra.get("rope_interleaved", False), first_dense_layers=d.get("first_k_dense_replace", 0),
            num_experts=d.get("n_routed_experts", 0), scoring="sigmoid", num_groups=d.get("n_group", 1) or 1,
            topk_groups=d.get("topk_group", 1) or 1, num_shared_experts=d.get("n_shared_experts", 0) or 0,
            routed_scale=d.get("routed_scaling_factor", 1.0), router_bias=True, mtp_layers=d.get("num_nextn_predict_layers", 0) or 0,
            **common)
    if mt == "qwen2":
        # dense Qwen2 / Qwen2.5: a Llama-shaped stack whose q / k / v projections carry a bias
        return ModelConfig(
            family="qwen2", attention="gqa", num_kv_heads=d.get("num_key_value_heads", d["num_attention_heads"]),
            head_dim=d.get("head_dim") or d["hidden_size"] // d["num_attention_heads"], qk_norm=False, attention_bias=True,
            rope_interleaved=extra.get("rope_interleaved", False), first_dense_layers=d["num_hidden_layers"], num_experts=0,
            num_shared_experts=0, **_windows(d), **dict(common, top_k=0, expert_ffn=0))
    if mt in ("llama", "mistral"):
        # dense GQA decoders without projection biases: every layer takes the dense SwiGLU path
        if d.get("attention_bias") or d.get("mlp_bias"):
            raise ValueError("projection biases are not supported")
        return ModelConfig(
            family="llama", attention="gqa", num_kv_heads=d.get("num_key_value_heads", d["num_attention_heads"]),
            head_dim=d.get("head_dim") or d["hidden_size"] // d["num_attention_heads"], qk_norm=False,
            rope_interleaved=extra.get("rope_interleaved", False), first_dense_layers=d["num_hidden_layers"], num_experts=0,
            num_shared_experts=0, **_windows(d), **dict(common, top_k=0, expert_ffn=0))
    raise ValueError(f"unsupported model_type {mt!r}")


def resolve(path: str) -> str:
    """Accept a snapshot directory or a hub cache root (models--org--name/snapshots/<rev>)."""
    if os.path.isfile(os.path.join(path, "config.json")):
        return path
    snaps = os.path.join(path, "snapshots")
    if os.path.isdir(snaps):
        revs = sorted(os.listdir(snaps))
        if revs:
            return os.path.join(snaps, revs[-1])
    raise FileNotFoundError(f"{path}: no config.json and no snapshots/ directory")


def core_view(path: str, view: str | None = None):
    """The verified core view of a multi-core repository (``loader/mc.py``), or None for a plain checkpoint served as
    it is.  ``view`` None reads ``$CUTEAFD_CORE_VIEW`` (what ``serve --core-view`` sets), default ``original``."""
    from . import mc
    view = view or os.environ.get("CUTEAFD_CORE_VIEW", "") or "original"
    return mc.select(mc.discover(resolve(path)), view)


def view_weight_map(path: str, view: str | None = None) -> dict[str, str] | None:
    """tensor name -> shard of the selected view; None when the directory is a plain checkpoint (every shard belongs)."""
    sel = core_view(path, view)
    if sel is None:
        return None
    with open(os.path.join(resolve(path), sel.view.index)) as f:
        return json.load(f)["weight_map"]


def read_config(path: str, view: str | None = None) -> tuple[ModelConfig, dict]:
    sel = core_view(path, view)
    with open(os.path.join(resolve(path), sel.view.config if sel is not None else "config.json")) as f:
        d = json.load(f)
    return from_hf_config(d), d


def _quantised(name: str, cfg: ModelConfig, scope: str) -> bool:
    if not name.endswith(".weight") or "norm" in name or "embed_tokens" in name or name.startswith("lm_head"):
        return False
    if ".mlp.gate.weight" in name:
        return False
    if scope == "experts":
        return ".mlp.experts." in name
    return ".mlp." in name or ".self_attn." in name


def write_random_snapshot(cfg: ModelConfig, directory: str, fmt: str | None = None, seed: int = 0,
                          scope: str = "experts", shard_bytes: int = 1 << 30) -> str:
    """Random-init snapshot of ``cfg`` in format ``fmt`` (bf16 | fp8_block128 | nvfp4 | mxfp4 | exl3_k4).

    ``scope`` = "experts": only routed experts carry the quantised format (the usual shipped
    mix); "linear": every projection does (DeepSeek FP8 style)."""
    fmt = fmt or cfg.weight_format
    if cfg.is_hybrid:
        if fmt != "bf16":
            raise ValueError(f"per-layer designs are stored in bf16, not {fmt}")
        from ..ref.hybrid import init_hybrid_weights
        os.makedirs(directory, exist_ok=True)
        with open(os.path.join(directory, "config.json"), "w") as f:
            json.dump(to_hf_config(cfg), f, indent=1, sort_keys=True)
        write_sharded(directory, {k: v.to(torch.bfloat16) for k, v in init_hybrid_weights(cfg, seed).items()}, shard_bytes)
        return directory
    cfg = cfg.replace(weight_format=fmt if not fmt.startswith("exl3") else "exl3")
    params = init_weights(cfg, seed=seed)
    gen = torch.Generator().manual_seed(seed + 17)
    out: dict[str, torch.Tensor] = {}
    for name, t in params.items():
        if fmt != "bf16" and _quantised(name, cfg, scope) and t.shape[-1] % 128 == 0 and t.shape[0] % 16 == 0:
            out.update(formats.encode(t, fmt, name[: -len(".weight")], gen))
        elif name.endswith("e_score_correction_bias"):
            out[name] = t.float()
        else:
            out[name] = t.to(torch.bfloat16)
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(to_hf_config(cfg), f, indent=1, sort_keys=True)
    write_sharded(directory, out, shard_bytes)
    return directory
