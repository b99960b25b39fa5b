// Shared by the gated delta-rule kernels: arguments, scalar maths and the output norm.
#pragma once

#include "common.cuh"

namespace cafd {

template <typename E> __device__ __forceinline__ float de_f(E v);
template <> __device__ __forceinline__ float de_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float de_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename E> __device__ __forceinline__ E de_e(float v);
template <> __device__ __forceinline__ float de_e<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 de_e<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct DeltaArgs {
  const void* proj;           // [T, ld] E: q | k | v | gate | b | a sections at the offsets below
  const float* conv_w;        // [channels, taps] (q heads, k heads, v heads)
  const float* A_log;         // [heads]
  const float* dt_bias;       // [heads]
  const float* norm_w;        // [vdim]
  float* state;               // pool, slot_stride floats per slot
  const int* state_in;        // [S]
  const int* state_out;       // [S]
  const int* q_start;         // [S + 1]
  void* out;                  // [T, heads * out_vd] E: normed and gated rows (head h at h * out_vd)
  float* raw;                 // [T, heads * vdim] fp32: o before the norm, when a head's columns span several blocks
  long long slot_stride, s_off, c_off;   // the layer's state and convolution inputs inside a slot
  int ld, q_off, k_off, v_off, g_off, b_off, a_off;
  int T, S, heads, kv_heads, dim, vdim, taps, out_vd;
  float eps;
};

__device__ __forceinline__ float softplus(float a) { return fmaxf(a, 0.f) + log1pf(expf(-fabsf(a))); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ void de_load4(const float* p, float (&v)[4]) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void de_load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  v[0] = bf16_lo(q.x); v[1] = bf16_hi(q.x); v[2] = bf16_lo(q.y); v[3] = bf16_hi(q.y);
}
__device__ __forceinline__ void de_store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void de_store4(__nv_bfloat16* p, const float (&v)[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
}

// out[t, h] = raw[t, h] / rms(raw[t, h]) * norm_w * silu(gate): one warp per (token, head), several in flight where a head
// is at most 128 columns of whole pieces of four
constexpr int kOutRows = 4;
template <typename E>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaArgs p) {
  pdl_wait();
  pdl_trigger();
  const long long n = static_cast<long long>(p.T) * p.heads, stride = static_cast<long long>(gridDim.x) * 8;
  const int lane = threadIdx.x & 31;
  long long i = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (n < (1ll << 30) && p.vdim <= 128 && p.vdim % 4 == 0 && p.out_vd % 4 == 0 && p.ld % 4 == 0 && p.g_off % 4 == 0) {
    const bool on = 4 * lane < p.vdim;
    float nw[4] = {};
    if (on) de_load4(p.norm_w + 4 * lane, nw);
    const uint32_t rows = static_cast<uint32_t>(n), step = static_cast<uint32_t>(stride), heads = static_cast<uint32_t>(p.heads);
    for (uint32_t r0 = static_cast<uint32_t>(i); r0 < rows; r0 += kOutRows * step) {
      float o[kOutRows][4] = {}, g[kOutRows][4] = {};
#pragma unroll
      for (int j = 0; j < kOutRows; ++j) {
        const uint32_t r = r0 + j * step;
        if (r < rows && on) {
          const uint32_t t = r / heads, h = r - t * heads;
          de_load4(p.raw + static_cast<size_t>(r) * p.vdim + 4 * lane, o[j]);
          de_load4(static_cast<const E*>(p.proj) + static_cast<size_t>(t) * p.ld + p.g_off + h * p.vdim + 4 * lane, g[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < kOutRows; ++j) {
        const uint32_t r = r0 + j * step;
        const float ss = warp_sum(o[j][0] * o[j][0] + o[j][1] * o[j][1] + o[j][2] * o[j][2] + o[j][3] * o[j][3]);
        const float inv = 1.0f / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
        if (r < rows && on) {
          float v[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) v[e] = o[j][e] * inv * nw[e] * g[j][e] / (1.0f + __expf(fminf(-g[j][e], 80.f)));
          de_store4(static_cast<E*>(p.out) + static_cast<size_t>(r) * p.out_vd + 4 * lane, v);
        }
      }
    }
    return;
  }
  for (; i < n; i += stride) {
    const long long t = i / p.heads;
    const int h = static_cast<int>(i - t * p.heads);
    const float* o = p.raw + i * p.vdim;
    const E* gate = static_cast<const E*>(p.proj) + t * p.ld + p.g_off + h * p.vdim;
    float ss = 0.f;
    for (int v = lane; v < p.vdim; v += 32) ss = fmaf(o[v], o[v], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(p.vdim) + p.eps);
    E* dst = static_cast<E*>(p.out) + i * p.out_vd;
    for (int v = lane; v < p.vdim; v += 32) {
      const float g = de_f<E>(gate[v]);
      dst[v] = de_e<E>(o[v] * inv * p.norm_w[v] * g * sigmoid_f(g));
    }
  }
}

}  // namespace cafd
