"""ctypes bindings of libcuteafd_b200.so (CUDA kernels) and libcuteafd_rt.so (host runtime)."""
from __future__ import annotations

import ctypes as C
import os
import threading

from . import build

_lock = threading.Lock()
_cuda = None
_rt = None

c_void_p, c_int, c_float, c_u32p = C.c_void_p, C.c_int, C.c_float, C.c_void_p


class GemmArgs(C.Structure):
    _fields_ = [
        ("w0", C.c_void_p), ("w1", C.c_void_p), ("x", C.c_void_p), ("out", C.c_void_p),
        ("residual", C.c_void_p), ("row_scale", C.c_void_p), ("row_dst", C.c_void_p),
        ("tile_expert", C.c_void_p), ("tile_row0", C.c_void_p), ("num_x_tiles", C.c_void_p),
        ("w_scale", C.c_void_p), ("x_scale", C.c_void_p), ("w_scale1", C.c_void_p),
        ("wait_flag", C.c_void_p), ("epoch", C.c_void_p), ("done_counter", C.c_void_p),
        ("signal_flag", C.c_void_p), ("status", C.c_void_p),
        ("splitk_scratch", C.c_void_p), ("splitk_tickets", C.c_void_p),
        ("splitk_scratch_floats", C.c_longlong), ("splitk_ticket_count", C.c_int),
        ("w_rows_total", C.c_longlong), ("x_rows_total", C.c_longlong),
        ("k", C.c_int), ("n_features", C.c_int), ("x_rows", C.c_int), ("ldo", C.c_int),
        ("w_rows_per_expert", C.c_int), ("w1_row_offset", C.c_int), ("max_x_tiles", C.c_int),
        ("swap", C.c_int), ("dual", C.c_int), ("bx", C.c_int), ("out_f32", C.c_int), ("fp8", C.c_int),
        ("num_sms", C.c_int),
        ("rs_ranks", C.c_int), ("rs_rows_per_rank", C.c_int), ("rs_my_rank", C.c_int), ("n_signal_flags", C.c_int),
        ("n_wait_flags", C.c_int), ("reserved0", C.c_int),
        ("rs_out", C.c_void_p * 8), ("signal_flags", C.c_void_p * 8),
        ("glu", C.c_int), ("glu_limit", C.c_float), ("glu_alpha", C.c_float), ("glu_bias", C.c_float),
    ]


MAX_RANKS = 8
# one setter per translation unit that waits (each holds its own copy of the limit)
WAIT_LIMIT_SETTERS = ("cafd_gemm_set_wait_limit_ns", "cafd_moe_set_wait_limit_ns", "cafd_attn_set_wait_limit_ns",
                      "cafd_gemm_fp8_set_wait_limit_ns", "cafd_tp_set_wait_limit_ns", "cafd_mla_set_wait_limit_ns",
                      "cafd_indexer_set_wait_limit_ns", "cafd_gemm_w4_set_wait_limit_ns", "cafd_gemm_exl3_set_wait_limit_ns",
                      "cafd_decode_step_set_wait_limit_ns")


BOUNDS_UNITS = ("cafd_moe", "cafd_tp")        # translation units with checked peer-store sites
BOUNDS_SITES = {1: "plan+dispatch: slab row", 2: "plan+dispatch: owner rank", 3: "dispatch: slab row", 4: "dispatch: owner rank",
                6: "head exchange: table row", 7: "head exchange: rank"}


def bounds_check_enabled() -> bool:
    lib = cuda_lib()
    return all(getattr(lib, f"{tu}_bounds_check_enabled")() == 1 for tu in BOUNDS_UNITS)


def take_bad_indices() -> list[tuple[str, int]]:
    """Records the bounds-check build left since the last call: (site, offending index).  Synchronises the device."""
    lib, out = cuda_lib(), []
    for tu in BOUNDS_UNITS:
        v = C.c_ulonglong(0)
        check(getattr(lib, f"{tu}_take_bad_index")(C.byref(v)), f"{tu}_take_bad_index")
        if v.value:
            idx = v.value & 0xffffffffffff
            if idx >= 1 << 47:
                idx -= 1 << 48
            out.append((BOUNDS_SITES.get((v.value >> 48) & 0x7fff, "?"), idx))
    return out


class MoeLayout(C.Structure):
    _fields_ = [
        ("n_ranks", C.c_int), ("expert_lo", C.c_int * (MAX_RANKS + 1)),
        ("slab", C.c_void_p * MAX_RANKS), ("meta", C.c_void_p * MAX_RANKS), ("flag", C.c_void_p * MAX_RANKS),
        ("max_tiles", C.c_int), ("max_rows", C.c_int),
        ("fp8", C.c_int), ("slab_q", C.c_void_p * MAX_RANKS), ("slab_s", C.c_void_p * MAX_RANKS),
    ]


class NormArgs(C.Structure):
    """cafd_norm_conv (csrc/hybrid_norm.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("tokens", "embed", "x_in", "y", "slot_w", "slot_idx", "ident", "w_b", "w", "base", "step",
                                          "w2", "h2_out", "conv", "x_out", "h_out", "row_idx", "state", "state_in", "state_out", "q_start",
                                          "rows2", "embed2", "past", "past_w", "past_out")]
    _fields_ += [(n, C.c_longlong) for n in ("slot_stride", "state_off", "past_stride")]
    _fields_ += [(n, C.c_int) for n in ("T", "H", "S", "ldy", "ldh", "ldb", "ldi", "groups", "taps", "top_k", "n_experts", "vocab", "run", "vocab2",
                                        "n_past")]
    _fields_ += [(n, C.c_float) for n in ("eps", "w_off", "e_scale")]


class BigramArgs(C.Structure):
    """cafd_bigram_rows (csrc/hybrid_norm.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("tokens", "q_start", "state_in", "state_out", "state", "rows")]
    _fields_ += [(n, C.c_longlong) for n in ("slot_stride", "state_off", "mul_prev", "mul_cur", "buckets")]
    _fields_ += [(n, C.c_int) for n in ("T", "S")]


class RglruArgs(C.Structure):
    """cafd_rglru_* (csrc/rglru.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("proj", "y_bias", "x_bias", "conv_w", "conv_b", "lam", "w", "gate_bias", "u", "gates", "out",
                                          "state", "state_in", "state_out", "q_start")]
    _fields_ += [(n, C.c_longlong) for n in ("slot_stride", "s_off", "c_off")]
    _fields_ += [(n, C.c_int) for n in ("T", "S", "ld", "x_off", "y_off", "width", "blocks", "taps", "u_pitch", "t_pad", "ldo", "max_q")]
    _fields_ += [("c", C.c_float)]


class LightningArgs(C.Structure):
    """cafd_lightning_* (csrc/lightning.cuh)."""
    _fields_ = [(n, C.c_void_p) for n in ("proj", "decay", "norm_w", "raw", "out", "scratch", "state", "state_in", "state_out", "q_start")]
    _fields_ += [(n, C.c_longlong) for n in ("slot_stride", "s_off", "scratch_bytes")]
    _fields_ += [(n, C.c_int) for n in ("T", "S", "ld", "q_off", "k_off", "v_off", "g_off", "heads", "dim", "vdim", "ldo", "out_vd", "max_q")]
    _fields_ += [("eps", C.c_float)]


class ConvRope(C.Structure):
    """cafd_conv_rope_kv (csrc/conv_rope.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("proj", "conv_w", "table", "slots", "q_start", "state_in", "state_out", "state", "q_out",
                                          "k_cache", "v_cache", "q_norm", "k_norm", "v_table")]
    _fields_ += [("slot_stride", C.c_longlong), ("state_off", C.c_longlong)]
    _fields_ += [(n, C.c_int) for n in ("T", "S", "ld", "q_off", "k_off", "v_off", "nq", "nk", "nv", "maps_dim", "dim", "vdim", "kv_heads",
                                        "rot", "taps", "run", "norm", "halves", "v_from_k", "units")]
    _fields_ += [("eps", C.c_float), ("rot_sq", C.c_float)]


class PagedAttn(C.Structure):
    """cafd_paged_attn (csrc/attention_any.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("q", "k_cache", "v_cache", "page_table", "positions", "q_start", "out", "sink", "gate", "v_table")]
    _fields_ += [(n, C.c_int) for n in ("T", "S", "heads", "kv_heads", "maps", "dim", "vdim", "window", "keep", "max_pages", "ldo",
                                        "head_pitch", "heads_per_block", "gate_ld")]
    _fields_ += [(n, C.c_float) for n in ("scale", "lam", "out_scale", "eps", "cap")]


class LatentPrep(C.Structure):
    """cafd_latent_prep (csrc/latent.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("a", "norm_w", "inv_freq", "positions", "slots", "cache", "slab", "q_abs", "lat_out")]
    _fields_ += [(n, C.c_int) for n in ("lda", "q_off", "kv_off", "heads", "dim", "rot", "rank", "rec", "dim_pad", "t_pad", "T", "halves")]
    _fields_ += [("eps", C.c_float), ("mag", C.c_float)]


class LatentAttn(C.Structure):
    """cafd_latent_attn (csrc/latent.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("q_abs", "cache", "page_table", "positions", "q_start", "out")]
    _fields_ += [(n, C.c_int) for n in ("T", "S", "heads", "rank", "rot", "rec", "max_pages", "window", "t_pad", "out_ld",
                                        "heads_per_block")]
    _fields_ += [("scale", C.c_float)]


class DeltaArgs(C.Structure):
    """cafd_delta_step (csrc/delta.cu)."""
    _fields_ = [(n, C.c_void_p) for n in ("proj", "conv_w", "A_log", "dt_bias", "norm_w", "state", "state_in", "state_out", "q_start",
                                          "out", "raw")]
    _fields_ += [(n, C.c_longlong) for n in ("slot_stride", "s_off", "c_off")]
    _fields_ += [(n, C.c_int) for n in ("ld", "q_off", "k_off", "v_off", "g_off", "b_off", "a_off", "T", "S", "heads", "kv_heads", "dim",
                                        "vdim", "taps", "out_vd")]
    _fields_ += [("eps", C.c_float)]


class TpReduceArgs(C.Structure):
    _fields_ = [
        ("partials", C.c_void_p), ("residual", C.c_void_p), ("norm_w", C.c_void_p), ("x_out", C.c_void_p * 8),
        ("rs_flags", C.c_void_p), ("ag_flags", C.c_void_p * 8), ("epoch", C.c_void_p), ("done_counter", C.c_void_p),
        ("status", C.c_void_p), ("ranks", C.c_int), ("my_rank", C.c_int), ("rows_per_rank", C.c_int),
        ("rows_valid", C.c_int), ("N", C.c_int), ("eps", C.c_float), ("n_sum", C.c_int), ("n_wait", C.c_int),
    ]


class TpHeadArgs(C.Structure):
    _fields_ = [
        ("cand_v", C.c_void_p), ("cand_i", C.c_void_p), ("table_out", C.c_void_p * 8), ("table_in", C.c_void_p),
        ("flags_out", C.c_void_p * 8), ("flags_in", C.c_void_p), ("epoch", C.c_void_p), ("done_counter", C.c_void_p),
        ("status", C.c_void_p), ("out", C.c_void_p), ("ranks", C.c_int), ("my_rank", C.c_int), ("max_rows", C.c_int),
        ("T", C.c_int), ("slices", C.c_int), ("lo", C.c_int),
    ]


def _sig(lib, name, argtypes, restype=C.c_int):
    fn = getattr(lib, name)
    fn.argtypes = argtypes
    fn.restype = restype
    return fn


def cuda_lib():
    """Load (building first when the shared object is absent) the CUDA kernel library."""
    global _cuda
    with _lock:
        if _cuda is not None:
            return _cuda
        # CAFD_BOUNDS_CHECK=1: the library whose peer-store paths check every index before the access
        checked = os.environ.get("CAFD_BOUNDS_CHECK", "") == "1"
        path = build.CHECK_LIB if checked else build.CUDA_LIB
        if not os.path.exists(path):
            build.build_check() if checked else build.build_cuda()
        lib = C.CDLL(path)
        P, I, F = C.c_void_p, C.c_int, C.c_float
        _sig(lib, "cafd_gemm", [C.POINTER(GemmArgs), P])
        _sig(lib, "cafd_gemm_fp8", [C.POINTER(GemmArgs), P])
        _sig(lib, "cafd_quant_rows_fp8", [P, P, P, I, I, I, P])
        for n in WAIT_LIMIT_SETTERS:
            _sig(lib, n, [C.c_ulonglong])
        _sig(lib, "cafd_embed", [P, P, P, I, I, I, P])
        _sig(lib, "cafd_rmsnorm", [P, P, P, P, I, I, F, P])
        _sig(lib, "cafd_qk_rope_kv", [P, P, P, P, P, P, P, P, P, I, I, I, I, F, I, P, I, P])
        _sig(lib, "cafd_argmax", [P, P, P, I, I, I, P])
        _sig(lib, "cafd_argmax_slices", [])
        _sig(lib, "cafd_bump_epoch", [P, P])
        _sig(lib, "cafd_decode_advance", [P, P, P, P, P, P, I, I, I, P])
        _sig(lib, "cafd_route_topk", [P, P, P, P, I, I, I, I, I, I, I, F, I, P])
        _sig(lib, "cafd_moe_meta_ints", [I, I])
        _sig(lib, "cafd_wait_flag", [P, P, P, P])
        _sig(lib, "cafd_tp_reduce_norm_gather", [C.POINTER(TpReduceArgs), P])
        _sig(lib, "cafd_tp_signal", [P, I, P, P])
        _sig(lib, "cafd_tp_head_pick", [C.POINTER(TpHeadArgs), P])
        for tu in BOUNDS_UNITS:
            _sig(lib, f"{tu}_bounds_check_enabled", [])
            _sig(lib, f"{tu}_take_bad_index", [P])
        _sig(lib, "cafd_argmax_candidates", [P, P, P, I, I, I, P])
        _sig(lib, "cafd_moe_plan", [P, I, I, I, I, C.POINTER(MoeLayout), P, P, P, P])
        _sig(lib, "cafd_moe_plan_wide", [P, I, I, I, I, C.POINTER(MoeLayout), P, P, P, P, P])
        _sig(lib, "cafd_moe_plan_wide_ints", [I, I])
        _sig(lib, "cafd_moe_plan_dispatch", [P, I, I, I, I, C.POINTER(MoeLayout), P, P, P, P, I, P, P])
        _sig(lib, "cafd_norm_route", [P, P, F, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, P])
        _sig(lib, "cafd_moe_combine_norm", [P, P, P, P, P, I, I, I, P, I, P, P, P, F, P, P])
        _sig(lib, "cafd_moe_dispatch", [P, P, P, I, I, I, C.POINTER(MoeLayout), P, P, P])
        _sig(lib, "cafd_moe_combine", [P, P, P, P, P, I, I, I, P, I, P, P, P])
        _sig(lib, "cafd_attn_decode_scratch_floats", [I, I, I, I], C.c_longlong)
        _sig(lib, "cafd_attn_decode", [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, I, I, I, F, F, F, P, P, I, F, P, P])
        _sig(lib, "cafd_attn_decode_partial", [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, P])
        _sig(lib, "cafd_attn_merge", [P, P, P, I, I, I, I, I, P])
        _sig(lib, "cafd_set_fixed_kv_split", [I])
        _sig(lib, "cafd_fixed_kv_split", [])
        _sig(lib, "cafd_attn_prefill", [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, I, I, F, F, F, P, P, I, F, P, P])
        _sig(lib, "cafd_mla_scratch_floats", [I, I], C.c_longlong)
        _sig(lib, "cafd_mla_attention", [P, P, P, P, P, P, P, P, P, P, C.c_longlong, I, I, I, I, I, I, F, P, I, I, P])
        _sig(lib, "cafd_indexer_scores", [P, P, P, I, F, P, P, P, P, P, P, P, C.c_longlong, I, I, I, I, I, I, P])
        _sig(lib, "cafd_index_topk", [P, I, P, P, P, I, I, I, P, P])
        _sig(lib, "cafd_index_k_store", [P, I, P, P, I, P])
        _sig(lib, "cafd_mla_prep_a", [P, I, I, P, P, P, P, P, P, P, I, F, I, P, P])
        _sig(lib, "cafd_mla_prep_a_fp8", [P, I, I, P, P, P, P, P, P, P, I, F, I, P, P])
        _sig(lib, "cafd_mla_fp8_gather", [P, P, I, P, I, P, P, P, P, I, P, P])
        _sig(lib, "cafd_mla_attention_partial", [P, P, P, P, P, P, P, P, P, I, I, P, C.c_longlong, I, I, I, I, I, F, P])
        _sig(lib, "cafd_mla_merge", [P, P, P, P, P, I, I, I, I, P])
        _sig(lib, "cafd_mla_attention_gathered", [P, P, P, P, P, P, P, P, P, P, C.c_longlong, I, I, I, I, I, F, P, I, P])
        _sig(lib, "cafd_attn_prefill_mla", [P, I, I, P, I, I, P, P, C.c_longlong, P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, I, P])
        _sig(lib, "cafd_gemm_w4", [C.POINTER(GemmArgs), I, P, P, P])
        _sig(lib, "cafd_w4_dequant", [P, P, P, P, C.c_longlong, I, I, I, P])
        _sig(lib, "cafd_fp8_dequant_block128", [P, P, P, C.c_longlong, I, P])
        _sig(lib, "cafd_gemm_exl3", [P, I, P, P, P, P, P, I, P, P, P, I, I, I, I, I, I, P])
        _sig(lib, "cafd_sample_rows", [P, I, I, P, P, I, P, P, P])
        _sig(lib, "cafd_accept_prefix", [P, P, P, I, P, P, P])
        _sig(lib, "cafd_norm_conv", [C.POINTER(NormArgs), I, P])
        _sig(lib, "cafd_bigram_rows", [C.POINTER(BigramArgs), P])
        _sig(lib, "cafd_rglru_step_ok", [I, I, I])
        _sig(lib, "cafd_lightning_chunked", [C.POINTER(LightningArgs), P])
        for n in ("cafd_rglru_conv", "cafd_rglru_scan", "cafd_rglru_step"):
            _sig(lib, n, [C.POINTER(RglruArgs), I, P])
        _sig(lib, "cafd_lightning_step", [C.POINTER(LightningArgs), I, P])
        _sig(lib, "cafd_rope_table", [P, P, P, I, I, F, P])
        _sig(lib, "cafd_conv_rope_kv", [C.POINTER(ConvRope), I, P])
        _sig(lib, "cafd_softcap", [P, I, I, C.c_longlong, F, P])
        _sig(lib, "cafd_paged_attn", [C.POINTER(PagedAttn), I, P])
        _sig(lib, "cafd_delta_chunked", [C.POINTER(DeltaArgs), P, C.c_longlong, P])
        _sig(lib, "cafd_delta_chunk_bytes", [I, I, I], C.c_longlong)
        _sig(lib, "cafd_swap_ids", [P, P, I, P])
        _sig(lib, "cafd_gemm_f32", [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, F, F, P])
        _sig(lib, "cafd_latent_prep", [C.POINTER(LatentPrep), I, P])
        _sig(lib, "cafd_latent_attn", [C.POINTER(LatentAttn), I, P])
        _sig(lib, "cafd_latent_gate", [P, P, I, I, I, I, I, I, I, P])
        _sig(lib, "cafd_delta_step", [C.POINTER(DeltaArgs), I, P])
        _sig(lib, "cafd_mla_q_split", [P, I, P, P, P, P, I, I, I, I, P])
        _sig(lib, "cafd_mla_small_rows", [])
        _sig(lib, "cafd_mla_absorb_small", [P, I, P, P, P, P, I, I, I, F, P])
        _sig(lib, "cafd_mla_unabsorb_small", [P, I, P, P, I, I, P, I, I, P])
        _cuda = lib
        return lib


def rt_lib():
    """Load the host runtime library (C++; no CUDA needed)."""
    global _rt
    with _lock:
        if _rt is not None:
            return _rt
        path = build.RT_LIB
        if not os.path.exists(path):
            build.build_rt()
        _rt = C.CDLL(path)
        return _rt


def loaded_libraries() -> list[str]:
    return [p for p, l in ((build.CUDA_LIB, _cuda), (build.RT_LIB, _rt)) if l is not None]


class NativeError(RuntimeError):
    pass


def check(rc: int, what: str) -> None:
    if rc != 0:
        raise NativeError(f"{what} failed with code {rc}")
