"""Small per-layer hybrid configurations and helpers shared by the hybrid tests."""
import dataclasses

import torch

from cuteafd_b200.config import (AttentionSpec, DeltaSpec, DenseSpec, LatentSpec, LayerSpec, LightningSpec, PairSpec, RglruSpec, RopeSpec,
                                 RouterSpec, hybrid_config, parallel_config, post_norm_config)
from cuteafd_b200.ref import hybrid as R


def latent(heads=3, dim=24, rot_dim=8, vdim=20, kv_rank=40, window=37, scale=None, base=5000.0):
    return LatentSpec(heads, dim, rot_dim, vdim, kv_rank, window, scale if scale is not None else 1.7 * (dim + rot_dim) ** -0.5,
                      RopeSpec(rot_dim, base, halves=True))


def delta(heads=6, kv_heads=2, dim=20, vdim=36, conv=3):
    return DeltaSpec(heads, kv_heads, dim, vdim, conv)


def odd_config():
    """Nothing is a power of two, every layer differs: layers without a feed-forward, routers with and without identity
    outputs and groups, a value size above one block's columns."""
    return hybrid_config("odd", 203, 96, [
        LayerSpec(latent(), RouterSpec(6, 28, 3, 2, 4, 2)),
        LayerSpec(delta()),
        LayerSpec(delta(2, 2, 40, 136, 5), RouterSpec(5, 24, 2)),
        LayerSpec(latent(5, 16, 12, 24, 64, 130, base=300.0), RouterSpec(7, 16, 4, 5, 3, 1)),
        LayerSpec(latent(1, 8, 4, 8, 12, 1))], canon_taps=3, norm_groups=3, eps=2e-5)


def plain_config():
    """Values that make a mechanism vanish: one norm group, one-tap convolutions, one head, one group of experts."""
    return hybrid_config("plain", 130, 64, [
        LayerSpec(delta(1, 1, 16, 16, 1), RouterSpec(4, 8, 1, 1, 5, 5)),
        LayerSpec(latent(1, 16, 2, 16, 24, 500), RouterSpec(2, 40, 2)),
        LayerSpec(delta(4, 1, 64, 24, 4))], canon_taps=1, norm_groups=1, eps=1e-3)


def narrow_config():
    """A width that is no multiple of 8, so that rows are padded between the kernels, and longer convolutions."""
    return hybrid_config("narrow", 77, 90, [
        LayerSpec(latent(2, 12, 4, 10, 18, 21), RouterSpec(3, 10, 2, 1, 2, 1)),
        LayerSpec(delta(3, 3, 10, 6, 6), RouterSpec(4, 9, 2, 0, 2, 2))], canon_taps=6, norm_groups=3, eps=1e-4)


def wide_config(window=100):
    """The sizes the tensor-core kernels take."""
    return hybrid_config("wide", 500, 256, [
        LayerSpec(latent(8, 128, 64, 128, 512, window, base=1e5), RouterSpec(8, 128, 2, 2, 5, 3)),
        LayerSpec(delta(4, 2, 128, 128, 4), RouterSpec(6, 64, 3, 3, 3, 2)),
        LayerSpec(latent(16, 128, 64, 128, 512, 2 * window + 3, base=1e4))], canon_taps=4, norm_groups=4, eps=1e-5)


def attention(heads=6, kv_heads=2, dim=12, vdim=20, window=37, keep=5, rope=RopeSpec(8, 5000.0, 3.0, 1.0, 4.0, 100), conv=3, diff=0.3, scale=None):
    return AttentionSpec(heads, kv_heads, dim, vdim, window, keep, scale if scale is not None else 1.6 * dim ** -0.5, rope, conv, 2, diff)


def parallel(m, ffn=None):
    return LayerSpec(m, dense=DenseSpec(ffn) if ffn else None, parallel=True)


def looped_config():
    """Every layer differs: head sizes that are no multiples of 8, odd ones among them, layers without a feed-forward, a window
    of one token, one that starts inside the kept tokens, none at all; the middle runs three times."""
    return parallel_config("looped", 203, 104, [
        parallel(attention(), 72),
        parallel(attention(3, 3, 8, 8, 1, 2, RopeSpec(8, 300.0), 1, 0.0)),
        parallel(attention(5, 1, 15, 7, 130, 70, RopeSpec(10, 1e4, 8.0, 0.5, 2.0, 64), 5, 0.8), 33),
        parallel(attention(4, 4, 16, 24, 0, 0, RopeSpec(16, 700.0), 4, 0.45), 40)], 2e-5, loop=(1, 3, 3), logit_softcap=9.0)


def bare_config():
    """Values that make a mechanism vanish: one head, no kept tokens, no loop, no cap, no rotation, a width that is no multiple
    of 8."""
    return parallel_config("bare", 77, 90, [
        parallel(attention(1, 1, 10, 6, 21, 0, RopeSpec(10, 1e3), 2), 11),
        parallel(attention(8, 2, 8, 16, 64, 64, RopeSpec(0, 1e3), 3, 0.2), 24)], 1e-3)


def paired_config(window=100, keep=70):
    """The sizes the tensor-core attention kernels take; everything runs twice."""
    return parallel_config("paired", 500, 256, [
        parallel(attention(4, 2, 64, 128, window, keep, RopeSpec(64, 1e5, 4.0, 1.0, 4.0, 256), 4, 0.6), 192),
        parallel(attention(8, 1, 64, 128, 2 * window + 3, 3, RopeSpec(32, 1e4), 3, 0.2), 136)], 1e-5, loop=(0, 2, 2), logit_softcap=30.0)


def single_map_config():
    """Plain attention (one map per head) in the same layers, at sizes of both kinds of kernels."""
    one = lambda m: dataclasses.replace(m, maps=1, diff=0.0)                    # noqa: E731
    return parallel_config("single", 300, 192, [
        parallel(one(attention(4, 2, 128, 128, 90, 10, RopeSpec(64, 1e5), 3)), 88),
        parallel(one(attention(3, 1, 20, 12, 50, 66, RopeSpec(20, 1e3), 2)), 40)], 1e-5, loop=(1, 2, 2))


def normed(heads=5, kv_heads=1, dim=14, vdim=7, rope=RopeSpec(10, 1e4, halves=True), window=0, scale=None):
    """Attention with norms over the whole projections and a gate per head."""
    return AttentionSpec(heads, kv_heads, dim, vdim, window, 0, scale if scale is not None else 1.6 * dim ** -0.5, rope, qk_norm="all", gate=True)


def key_valued(heads=6, kv_heads=2, dim=20, window=37, rope=RopeSpec(12, 5000.0, 3.0, kind="linear", halves=True), conv=3, scale=None):
    """Attention whose values are the convolved keys, norms per head, sinks and a gate per head."""
    return AttentionSpec(heads, kv_heads, dim, dim, window, 0, scale if scale is not None else 1.3 * dim ** -0.5, rope, conv, qk_norm="head",
                         v_from_k=True, sink=True, gate=True)


def open_latent(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=40, rope=None, window=0, scale=None):
    """Latent attention without a window or a gate, neighbouring pairs, YaRN scaling."""
    return LatentSpec(heads, dim, rot_dim, vdim, kv_rank, window, scale if scale is not None else 1.7 * (dim + rot_dim) ** -0.5,
                      rope or RopeSpec(rot_dim, 300.0, 5.0, 1.5, 24.0, 700, "yarn"), gate=False)


def two_norms(m, ffn=None, experts=0, top=0, expert_ffn=0):
    r = RouterSpec(experts, expert_ffn, top, logit_bias=True, normalize=True) if experts else None
    return LayerSpec(m, r, DenseSpec(ffn) if ffn else None, parallel=True, two_norms=True)


def joined_config():
    """Every layer differs: routed with a shared expert and without, dense, none; odd head sizes, a window of one token; three
    passes that each start with a product of [x; embedding row]."""
    return parallel_config("joined", 203, 104, [
        two_norms(key_valued(), 26, 6, 3, 28),
        two_norms(open_latent(), 72),
        two_norms(key_valued(3, 3, 8, 1, RopeSpec(8, 300.0, halves=True), 1), 0, 5, 1, 16),
        two_norms(normed()),
        two_norms(open_latent(5, 16, 8, 24, 64, RopeSpec(8, 1e4, 2.0, 0.5, 8.0, 100, "yarn")), 33, 9, 9, 8),
        two_norms(normed(4, 4, 16, 24, RopeSpec(16, 700.0, halves=True)), 40)], 2e-5, loop=(1, 4, 3), family="rofapel", loop_join=True, embed_scale=5.0)


def lone_config():
    """Values that make a mechanism vanish: one head, one expert, one tap, one pass (over everything), no rotation, scales of one, a
    width that is no multiple of 8."""
    return parallel_config("lone", 77, 90, [
        two_norms(key_valued(1, 1, 10, 64, RopeSpec(0, 1e3, kind="linear", halves=True), 1, 1.0), 11, 1, 1, 9),
        two_norms(open_latent(1, 8, 4, 8, 12, RopeSpec(4, 1e3)), 24),
        two_norms(normed(1, 1, 6, 5, RopeSpec(6, 1e2, halves=True), 65), 7, 3, 2, 10)], 1e-3, loop=(0, 3, 1), family="rofapel", loop_join=True)


def joint_config(window=100):
    """The sizes the tensor-core kernels take; the first two layers run twice."""
    return parallel_config("joint", 500, 256, [
        two_norms(open_latent(8, 128, 64, 128, 512, RopeSpec(64, 1e5, 4.0, 1.0, 32.0, 256, "yarn"), scale=0.1), 192, 8, 2, 128),
        two_norms(key_valued(4, 2, 128, window, RopeSpec(64, 1e4, 2.0, kind="linear", halves=True), 4), 136),
        two_norms(normed(8, 1, 128, 128, RopeSpec(128, 1e5, halves=True)), 128, 6, 3, 64)], 1e-5, loop=(0, 2, 2), family="rofapel", loop_join=True,
        embed_scale=16.0)


def turned(heads=6, kv_heads=2, dim=20, vdim=12, rope=RopeSpec(12, 300.0, 3.0, 1.5, 24.0, 200, "yarn", halves=True), scale=None, cap=4.0):
    """Attention with queries and keys normed after their rotation, rotated values, capped scores and a sink of logit 0."""
    return AttentionSpec(heads, kv_heads, dim, vdim, 0, 0, scale if scale is not None else 1.6 * dim ** -0.5, rope, qk_norm="rotated", softcap=cap,
                         unit_sink=True, v_rope=RopeSpec(vdim, rope.base, halves=True))


def fading(heads=5, dim=12, vdim=20, lo=0.55, hi=0.995):
    """Linear attention whose heads forget at different rates."""
    return LightningSpec(heads, dim, vdim, tuple(round(lo + (hi - lo) * h / max(1, heads - 1), 6) for h in range(heads)))


def post(m, ffn=None, limit=1.1, experts=0, top=0, expert_ffn=0):
    r = RouterSpec(experts, expert_ffn, top, scoring="sigmoid") if experts else None
    return LayerSpec(m, r, DenseSpec(ffn, limit, 1.702, 1.0) if ffn else None, post_norm=True)


def averaged_config():
    """Every layer differs: pairs and recurrences of odd sizes, dense and routed feed-forwards and none, one expert of several, blocks of
    five channels, one to five taps, values wider than one block's columns."""
    return post_norm_config("averaged", 203, 104, [
        post(PairSpec(turned(), fading(), 0.7, 0.4), 72),
        post(RglruSpec(72, 3, 3), experts=6, top=3, expert_ffn=28),
        post(RglruSpec(60, 5, 5)),
        post(PairSpec(turned(3, 3, 8, 24, RopeSpec(8, 300.0, halves=True), cap=2.0), fading(2, 40, 136, 0.8), 0.9, 1.3), experts=5, top=1, expert_ffn=16),
        post(RglruSpec(35, 7, 1), 33, 0.6)], 2e-5, bigram=(97, 31, 5), logit_softcap=9.0)


def faint_config():
    """Values that make a mechanism vanish: one head, one expert, one block, one tap, one bucket, no decay, scales of one, no caps, a
    width that is no multiple of 8."""
    return post_norm_config("faint", 77, 90, [
        post(PairSpec(turned(1, 1, 6, 2, RopeSpec(6, 100.0, halves=True), cap=0.0), LightningSpec(1, 1, 4, (1.0,))), experts=1, top=1, expert_ffn=9),
        post(RglruSpec(10, 1, 1), 24, 50.0),
        post(PairSpec(turned(4, 1, 10, 6, RopeSpec(4, 50.0, halves=True)), fading(3, 7, 5, 0.0), 1.0, 0.3))], 1e-3, bigram=(1, 3, 1))


def dual_config():
    """The sizes the tensor-core kernels take, and recurrences in blocks of 128."""
    return post_norm_config("dual", 500, 256, [
        post(PairSpec(turned(4, 2, 128, 128, RopeSpec(64, 1e4, 4.0, 1.0, 32.0, 256, "yarn", halves=True), cap=6.0), fading(4, 128, 128, 0.7), 0.9, 0.6), 192),
        post(RglruSpec(256, 2, 4), experts=8, top=2, expert_ffn=128),
        post(PairSpec(turned(8, 1, 128, 128, RopeSpec(128, 1e5, halves=True), cap=30.0), fading(2, 64, 64, 0.9, 0.999), 1.2, 0.7), experts=6, top=3, expert_ffn=64),
        post(RglruSpec(384, 3, 2), 136, 2.0)], 1e-5, bigram=(211, 113, 9), logit_softcap=20.0)


def params(cfg, seed=0, spread=0.4):
    """Random bf16-representable weights.  The selection correction is spread out by ``spread``: above 1 the choice is the
    correction's alone, so that 16-bit rounding cannot flip a close one; a bias that is part of the logits likewise."""
    p = R.init_hybrid_weights(cfg, seed)
    g = torch.Generator().manual_seed(seed + 99)
    for k in p:
        if k.endswith(".correction"):
            p[k] = (torch.randperm(p[k].numel(), generator=g).float() - p[k].numel() / 2) * spread
        elif k.endswith(".router.b") and spread > 1:
            p[k] = (torch.randperm(p[k].numel(), generator=g).float() - p[k].numel() / 2) * 0.3
            p[k[:-2]] = p[k[:-2]] * 0.02
        elif k.endswith(".A_log"):
            p[k] = p[k] - 1.0
    return R.bf16_params(p)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(cfg, p, toks, dtype=torch.float32):
    m = R.HybridRefDecoder(cfg, {k: v.to(dtype) for k, v in p.items()}, mark_rows=0)
    with torch.no_grad():
        return m.forward(torch.tensor(toks), m.new_state()).float()


def err(got, want):
    """Per row: rms of the difference over the rms of the wanted logits, means taken off."""
    d = got.float() - want.float()
    d, w = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def write_model(cfg, p, directory):
    """config.json and model.safetensors (bfloat16) of ``cfg`` with parameters ``p``; returns the path."""
    import json
    import os

    from cuteafd_b200.loader.safetensors_io import write_file
    from cuteafd_b200.loader.snapshot import to_hf_config
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(to_hf_config(cfg), f)
    write_file(os.path.join(directory, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in p.items()})
    return str(directory)
