// Linear attention with one constant decay per head: q, k and v pass silu, then
//     S <- decay S + k v^T;  o = S^T q
// and all heads' outputs are normed together under one weight vector and multiplied by a sigmoid gate.
//
// lightning_step runs any mix of portions token by token with the state in registers, at any sizes, bf16 or fp32 activations.
// Everything from the silu to the gate is fp32.  The state is read from one slot and written to another, as everywhere.
#include "cafd_api.h"
#include "common.cuh"
#include "delta.cuh"
#include "lightning.cuh"

namespace cafd {

constexpr int kLiCols = 128;       // state columns per block at most
constexpr int kLiCells = 64;       // state cells per thread
constexpr int kLiMinThreads = 128;
constexpr int kLiAhead = 5;        // channels of the next token per thread: 2 * 256 + 128 over at least 128 threads

// Block (head, sequence, run of columns).  A thread holds kLiCells / V state rows of V neighbouring columns.
template <typename E, int V>
__global__ void __launch_bounds__(512) lightning_step_kernel(const LightningArgs p) {
  constexpr int R = kLiCells / V;
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, seq = blockIdx.y, v0 = blockIdx.z * kLiCols;
  const int tid = threadIdx.x, nt = blockDim.x;
  const int vt = min(kLiCols, p.vdim - v0), nq = vt / V, groups = (p.dim + R - 1) / R;
  const int grp = tid / nq, col = (tid - grp * nq) * V, r0 = grp * R;
  const bool worker = grp < groups;
  const int n_ch = 2 * p.dim + vt;
  float* ch = sm;                                // [2][n_ch]: q, k, v
  float* red = ch + 2 * n_ch;                    // [2][groups][vt]
  const float* st_in = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.s_off;
  float* st_out = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.s_off;
  const size_t base = static_cast<size_t>(h) * p.dim * p.vdim + v0 + col;
  // the state of this step was written a whole step ago: its loads need not wait for the projection
  float S[R][V];
#pragma unroll
  for (int r = 0; r < R; ++r) {
#pragma unroll
    for (int e = 0; e < V; ++e) S[r][e] = 0.f;
    if (worker && r0 + r < p.dim) {
      const float* at = st_in + base + static_cast<size_t>(r0 + r) * p.vdim;
      if constexpr (V == 4) {
        const float4 q = __ldcg(reinterpret_cast<const float4*>(at));
        S[r][0] = q.x; S[r][1] = q.y; S[r][2] = q.z; S[r][3] = q.w;
      } else {
        S[r][0] = __ldcg(at);
      }
    }
  }
  const float decay = p.decay[h];
  pdl_wait();
  pdl_trigger();
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  const E* proj = static_cast<const E*>(p.proj);
  auto src = [&](int c) {
    return c < p.dim ? p.q_off + h * p.dim + c : c < 2 * p.dim ? p.k_off + h * p.dim + c - p.dim : p.v_off + h * p.vdim + v0 + c - 2 * p.dim;
  };
  float x[kLiAhead];
  auto fetch = [&](int t) {
#pragma unroll
    for (int n = 0; n < kLiAhead; ++n) {
      const int c = tid + n * nt;
      x[n] = c < n_ch ? de_f<E>(proj[static_cast<size_t>(t) * p.ld + src(c)]) : 0.f;
    }
  };
  if (t0 < t1) fetch(t0);
  for (int t = t0; t < t1; ++t) {
    float* c = ch + ((t - t0) & 1) * n_ch;
    float* rd = red + ((t - t0) & 1) * groups * vt;
#pragma unroll
    for (int n = 0; n < kLiAhead; ++n)
      if (tid + n * nt < n_ch) c[tid + n * nt] = x[n] * sigmoid_f(x[n]);
    __syncthreads();
    if (t + 1 < t1) fetch(t + 1);
    if (worker) {
      float o[V], v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) { o[e] = 0.f; v[e] = c[2 * p.dim + col + e]; }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        if (r0 + r < p.dim) {
          const float qv = c[r0 + r], kv = c[p.dim + r0 + r];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            S[r][e] = fmaf(kv, v[e], decay * S[r][e]);
            o[e] = fmaf(qv, S[r][e], o[e]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) rd[grp * vt + col + e] = o[e];
    }
    __syncthreads();
    for (int i = tid; i < vt; i += nt) {
      float o = 0.f;
      for (int g = 0; g < groups; ++g) o += rd[g * vt + i];
      p.raw[(static_cast<size_t>(t) * p.heads + h) * p.vdim + v0 + i] = o;
    }
  }
  if (t1 > t0 && worker) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (r0 + r < p.dim) {
        float* at = st_out + base + static_cast<size_t>(r0 + r) * p.vdim;
        if constexpr (V == 4) __stcg(reinterpret_cast<float4*>(at), make_float4(S[r][0], S[r][1], S[r][2], S[r][3]));
        else __stcg(at, S[r][0]);
      }
    }
  }
}

// out[t] = raw[t] / rms(raw[t]) * norm_w * sigmoid(gate): a block per token
template <typename E, int V>
__global__ void __launch_bounds__(256) lightning_out_kernel(const LightningArgs p) {
  __shared__ float part[8];
  const int C = p.heads * p.vdim, tid = threadIdx.x, nt = blockDim.x, t = blockIdx.x;
  pdl_wait();
  pdl_trigger();
  const float* o = p.raw + static_cast<size_t>(t) * C;
  float ss = 0.f;
  for (int i = tid * V; i < C; i += nt * V) {
    float v[V];
    if constexpr (V == 4) de_load4(o + i, v); else v[0] = o[i];
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) part[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nt / 32; ++w) ss += part[w];
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(C) + p.eps);
  const E* gate = static_cast<const E*>(p.proj) + static_cast<size_t>(t) * p.ld + p.g_off;
  E* dst = static_cast<E*>(p.out) + static_cast<size_t>(t) * p.ldo;
  for (int i = tid * V; i < C; i += nt * V) {
    const int h = i / p.vdim, d = i - h * p.vdim;
    float v[V], w[V], g[V];
    if constexpr (V == 4) {
      de_load4(o + i, v);
      de_load4(p.norm_w + i, w);
      de_load4(gate + i, g);
    } else {
      v[0] = o[i]; w[0] = p.norm_w[i]; g[0] = de_f<E>(gate[i]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = v[e] * inv * w[e] * sigmoid_f(g[e]);
    if constexpr (V == 4) de_store4(dst + h * p.out_vd + d, v); else dst[h * p.out_vd + d] = de_e<E>(v[0]);
  }
}

template <typename E>
int launch_lightning_out(const LightningArgs& p, cudaStream_t st) {
  const bool vec = p.vdim % 4 == 0 && p.ld % 4 == 0 && p.g_off % 4 == 0 && p.ldo % 4 == 0 && p.out_vd % 4 == 0;
  if (vec) launch_pdl(lightning_out_kernel<E, 4>, dim3(p.T), dim3(256), 0, st, p);
  else launch_pdl(lightning_out_kernel<E, 1>, dim3(p.T), dim3(256), 0, st, p);
  return static_cast<int>(cudaGetLastError());
}
template int launch_lightning_out<float>(const LightningArgs&, cudaStream_t);
template int launch_lightning_out<__nv_bfloat16>(const LightningArgs&, cudaStream_t);

template <typename E, int V>
static int launch_lightning_step(const LightningArgs& p, cudaStream_t st) {
  constexpr int R = kLiCells / V;
  const int vt = p.vdim < kLiCols ? p.vdim : kLiCols, groups = (p.dim + R - 1) / R;
  int threads = (vt / V * groups + 31) / 32 * 32;
  if (threads < kLiMinThreads) threads = kLiMinThreads;
  if (threads > 512) return -12;
  const size_t smem = static_cast<size_t>(2 * (2 * p.dim + vt) + 2 * groups * vt) * 4;
  launch_pdl(lightning_step_kernel<E, V>, dim3(p.heads, p.S, (p.vdim + kLiCols - 1) / kLiCols), dim3(threads), smem, st, p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_lightning_step(const LightningArgs* a, int is_f32, cafd_stream_t s) {
  if (a->T <= 0) return 0;
  const LightningArgs& p = *a;
  if (!lightning_args_ok(p)) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  // (a last run of columns that is shorter keeps whole vectors)
  const bool vec = p.vdim % 4 == 0 && p.s_off % 4 == 0 && p.slot_stride % 4 == 0;
  const int rc = is_f32 ? (vec ? launch_lightning_step<float, 4>(p, st) : launch_lightning_step<float, 1>(p, st))
                        : (vec ? launch_lightning_step<__nv_bfloat16, 4>(p, st) : launch_lightning_step<__nv_bfloat16, 1>(p, st));
  if (rc) return rc;
  return is_f32 ? launch_lightning_out<float>(p, st) : launch_lightning_out<__nv_bfloat16>(p, st);
}
