// Shared by the linear attention kernels: arguments, and the norm and gate after them.
#pragma once

#include "cafd_api.h"
#include "common.cuh"

namespace cafd {

struct LightningArgs {
  const void* proj;           // [T, ld] E: q | k | v | gate sections at the offsets below
  const float* decay;         // [heads]
  const float* norm_w;        // [heads * vdim]
  float* raw;                 // [T, heads * vdim]: what the state gives, before norm and gate
  void* out;                  // [T, ldo] E: head h's values at h * out_vd
  void* scratch;              // chunked form
  float* state;               // pool, slot_stride floats per slot; [heads, dim, vdim] at s_off
  const int* state_in;        // [S]
  const int* state_out;       // [S]
  const int* q_start;         // [S + 1]
  long long slot_stride, s_off, scratch_bytes;
  int T, S, ld, q_off, k_off, v_off, g_off, heads, dim, vdim, ldo, out_vd, max_q;
  float eps;
};

inline bool lightning_args_ok(const LightningArgs& p) {
  return p.S >= 1 && p.heads >= 1 && p.dim >= 1 && p.dim <= 256 && p.vdim >= 1 && p.out_vd >= p.vdim && p.ldo >= (p.heads - 1) * p.out_vd + p.vdim &&
         p.proj && p.decay && p.norm_w && p.raw && p.out && p.state && p.state_in && p.state_out && p.q_start;
}

template <typename E> int launch_lightning_out(const LightningArgs& p, cudaStream_t st);

}  // namespace cafd
