// Latent attention at any sizes over the paged latent cache, with a sliding window (the tcgen05 kernel of
// mla_attention.cu serves the 512 + 64 record; this file serves every other record and the fp32 engines).
//
//   latent_prep   one block per token: RMS norm of the latent, rotation of the shared key part and of every head's
//                 rotated query part (pairs of halves or of neighbours; cosines and sines times a constant), the cache record, and the unrotated query parts moved head-major for the absorb
//                 product q W_uk
//   latent_attn   absorbed attention: scores q_abs . record over the window, softmax in fp32, the weighted sum of latents
//   latent_gate   attn *= sigmoid(gate row)
//
// The cached record is [latent | rotated key part | padding]: `rec` elements per token, a multiple of 8.
#include "cafd_api.h"
#include "common.cuh"

namespace cafd {

template <typename E> __device__ __forceinline__ float to_f(E v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename E> __device__ __forceinline__ E from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct LatentPrep {
  const void* a;              // [T, lda] E: the fused projection's rows
  const float* norm_w;        // [rank]
  const float* inv_freq;      // [rot / 2]
  const int* positions;       // [T]
  const int* slots;           // [T] page * 64 + offset, < 0: nothing is cached
  void* cache;                // [pages * 64, rec] E
  void* slab;                 // [heads, t_pad, dim_pad] E
  void* q_abs;                // [T, heads, rec] E: the rotated part goes to [rank, rank + rot)
  void* lat_out;              // [T, rank] E or null: a contiguous copy of the normed latents
  int lda, q_off, kv_off, heads, dim, rot, rank, rec, dim_pad, t_pad, T, halves;
  float eps, mag;
};

template <typename E>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrep p) {
  extern __shared__ float cs[];               // cos [rot / 2], sin [rot / 2]
  __shared__ float red[8];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, tid = threadIdx.x, half = p.rot >> 1;
  const E* row = static_cast<const E*>(p.a) + static_cast<size_t>(t) * p.lda;
  const E* kv = row + p.kv_off;
  const float pos = static_cast<float>(p.positions[t]);
  for (int i = tid; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * p.inv_freq[i], &s, &c);
    cs[i] = c * p.mag;
    cs[half + i] = s * p.mag;
  }
  float ss = 0.f;
  for (int i = tid; i < p.rank; i += blockDim.x) { const float v = to_f<E>(kv[i]); ss += v * v; }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += red[i];
  const float inv = 1.0f / sqrtf(tot / static_cast<float>(p.rank) + p.eps);
  const int slot = p.slots[t];
  E* rec = static_cast<E*>(p.cache) + static_cast<size_t>(slot < 0 ? 0 : slot) * p.rec;
  for (int i = tid; i < p.rank; i += blockDim.x) {
    const E v = from_f<E>(to_f<E>(kv[i]) * inv * p.norm_w[i]);
    if (slot >= 0) rec[i] = v;
    if (p.lat_out) static_cast<E*>(p.lat_out)[static_cast<size_t>(t) * p.rank + i] = v;
  }
  for (int i = tid; i < half; i += blockDim.x) {
    const int e0 = p.rank + (p.halves ? i : 2 * i), e1 = p.halves ? e0 + half : e0 + 1;
    const float u = to_f<E>(kv[e0]), v = to_f<E>(kv[e1]);
    if (slot >= 0) {
      rec[e0] = from_f<E>(u * cs[i] - v * cs[half + i]);
      rec[e1] = from_f<E>(v * cs[i] + u * cs[half + i]);
    }
  }
  const E* q = row + p.q_off;
  const int qd = p.dim + p.rot;
  if (p.slab) {
    for (int i = tid; i < p.heads * p.dim; i += blockDim.x) {
      const int h = i / p.dim, d = i - h * p.dim;
      static_cast<E*>(p.slab)[(static_cast<size_t>(h) * p.t_pad + t) * p.dim_pad + d] = q[h * qd + d];
    }
  }
  for (int i = tid; i < p.heads * half; i += blockDim.x) {
    const int h = i / half, d = i - h * half;
    const int e0 = p.halves ? d : 2 * d, e1 = p.halves ? e0 + half : e0 + 1;
    const float u = to_f<E>(q[h * qd + p.dim + e0]), v = to_f<E>(q[h * qd + p.dim + e1]);
    E* o = static_cast<E*>(p.q_abs) + (static_cast<size_t>(t) * p.heads + h) * p.rec + p.rank;
    o[e0] = from_f<E>(u * cs[d] - v * cs[half + d]);
    o[e1] = from_f<E>(v * cs[d] + u * cs[half + d]);
  }
}

struct LatentAttn {
  const void* q_abs;          // [T, heads, rec] E
  const void* cache;          // [pages * 64, rec] E
  const int* page_table;      // [S, max_pages]
  const int* positions;       // [T]
  const int* q_start;         // [S + 1]
  void* out;                  // [heads, t_pad, out_ld] E: latent sums, head-major
  int T, S, heads, rank, rot, rec, max_pages, window, t_pad, out_ld, heads_per_block;
  float scale;
};

constexpr int kLatKeys = 32;        // keys per tile: tiles start at multiples of 32, whatever the window
constexpr int kLatThreads = 256;
constexpr int kLatAcc = 16;         // accumulator elements per thread: heads_per_block * rank <= 16 * 256

template <typename E>
__global__ void __launch_bounds__(kLatThreads) latent_attn_kernel(const LatentAttn p) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, h0 = blockIdx.y * p.heads_per_block, tid = threadIdx.x;
  const int nh = min(p.heads_per_block, p.heads - h0);
  const int dims = p.rank + p.rot, pitch = dims | 1;          // odd pitch: keys in different banks
  float* sq = sm;                                             // [nh][dims]
  float* sk = sq + p.heads_per_block * dims;                  // [32][pitch]
  float* sp = sk + kLatKeys * pitch;                          // [nh][32] scores, then weights
  float* sm_m = sp + p.heads_per_block * kLatKeys;            // running max, sum, correction per head
  float* sm_l = sm_m + p.heads_per_block;
  float* sm_c = sm_l + p.heads_per_block;
  int seq = 0, hi = p.S;
  while (hi - seq > 1) {
    const int mid = (seq + hi) >> 1;
    if (p.q_start[mid] <= t) seq = mid; else hi = mid;
  }
  const int pos = p.positions[t];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* pt = p.page_table + static_cast<size_t>(seq) * p.max_pages;
  for (int i = tid; i < nh * dims; i += kLatThreads) {
    const int h = i / dims, d = i - h * dims;
    sq[i] = to_f<E>(static_cast<const E*>(p.q_abs)[(static_cast<size_t>(t) * p.heads + h0 + h) * p.rec + d]);
  }
  for (int h = tid; h < nh; h += kLatThreads) { sm_m[h] = -INFINITY; sm_l[h] = 0.f; }
  float acc[kLatAcc];
#pragma unroll
  for (int i = 0; i < kLatAcc; ++i) acc[i] = 0.f;
  const int n_acc = nh * p.rank, warp = tid >> 5, lane = tid & 31;
  for (int k0 = lo & ~(kLatKeys - 1); k0 <= pos; k0 += kLatKeys) {
    __syncthreads();
    for (int i = tid; i < kLatKeys * dims; i += kLatThreads) {
      const int j = i / dims, d = i - j * dims, kp = k0 + j;
      float v = 0.f;
      if (kp >= lo && kp <= pos && (kp >> 6) < p.max_pages)
        v = to_f<E>(static_cast<const E*>(p.cache)[(static_cast<size_t>(pt[kp >> 6]) * 64 + (kp & 63)) * p.rec + d]);
      sk[j * pitch + d] = v;
    }
    __syncthreads();
    for (int i = tid; i < nh * kLatKeys; i += kLatThreads) {
      const int h = i >> 5, j = i & 31, kp = k0 + j;
      float s = 0.f;
      const float* a = sq + h * dims;
      const float* b = sk + j * pitch;
      for (int d = 0; d < dims; ++d) s = fmaf(a[d], b[d], s);
      sp[i] = (kp >= lo && kp <= pos) ? s * p.scale : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < nh; h += kLatThreads / 32) {
      const float s = sp[h * kLatKeys + lane];
      const float m_old = sm_m[h], m = fmaxf(m_old, warp_max(s));   // every tile of the loop holds at least one visible key
      const float w = expf(s - m);
      const float sum = warp_sum(w);
      sp[h * kLatKeys + lane] = w;
      __syncwarp();
      if (lane == 0) {
        const float c = expf(m_old - m);
        sm_c[h] = c;
        sm_l[h] = sm_l[h] * c + sum;
        sm_m[h] = m;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kLatAcc; ++i) {
      const int e = tid + i * kLatThreads;
      if (e < n_acc) {
        const int h = e / p.rank, d = e - h * p.rank;
        float v = acc[i] * sm_c[h];
        const float* w = sp + h * kLatKeys;
#pragma unroll 8
        for (int j = 0; j < kLatKeys; ++j) v = fmaf(w[j], sk[j * pitch + d], v);
        acc[i] = v;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kLatAcc; ++i) {
    const int e = tid + i * kLatThreads;
    if (e < n_acc) {
      const int h = e / p.rank, d = e - h * p.rank;
      static_cast<E*>(p.out)[(static_cast<size_t>(h0 + h) * p.t_pad + t) * p.out_ld + d] = from_f<E>(acc[i] / sm_l[h]);
    }
  }
}

// attn [T, heads, ld_head] E, gate rows [T, ldg] E with head h's values at g_off + h * vdim
template <typename E>
__global__ void __launch_bounds__(256) latent_gate_kernel(E* __restrict__ attn, const E* __restrict__ gate, int T, int heads, int vdim,
                                                          int ld_head, int ldg, int g_off) {
  pdl_wait();
  pdl_trigger();
  const int n = heads * vdim;
  if (sizeof(E) == 2 && ld_head == vdim && n % 8 == 0 && ldg % 8 == 0 && g_off % 8 == 0) {   // 16-byte pieces
    const int nv = n / 8;
    for (int t = blockIdx.x; t < T; t += gridDim.x) {
      uint4* o = reinterpret_cast<uint4*>(attn + static_cast<size_t>(t) * n);
      const uint4* gr = reinterpret_cast<const uint4*>(gate + static_cast<size_t>(t) * ldg + g_off);
#pragma unroll 2
      for (int i = threadIdx.x; i < nv; i += blockDim.x) {
        const uint4 a = o[i], g = gr[i];
        const uint32_t av[4] = {a.x, a.y, a.z, a.w}, gv[4] = {g.x, g.y, g.z, g.w};
        uint32_t r[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          r[e] = pack_bf16(bf16_lo(av[e]) / (1.0f + expf(-bf16_lo(gv[e]))), bf16_hi(av[e]) / (1.0f + expf(-bf16_hi(gv[e]))));
        o[i] = make_uint4(r[0], r[1], r[2], r[3]);
      }
    }
    return;
  }
  for (int t = blockIdx.x; t < T; t += gridDim.x)
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const int h = i / vdim, d = i - h * vdim;
      E* o = attn + (static_cast<size_t>(t) * heads + h) * ld_head + d;
      const float g = to_f<E>(gate[static_cast<size_t>(t) * ldg + g_off + i]);
      *o = from_f<E>(to_f<E>(*o) / (1.0f + expf(-g)));
    }
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_latent_prep(const LatentPrep* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (p->rot % 2 || p->rec < p->rank + p->rot || p->rot > 4096) return -10;
  const size_t smem = static_cast<size_t>(p->rot) * 4 + 8;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (is_f32) launch_pdl(latent_prep_kernel<float>, dim3(p->T), dim3(256), smem, st, *p);
  else launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(p->T), dim3(256), smem, st, *p);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int cafd_latent_attn(const LatentAttn* args, int is_f32, cafd_stream_t s) {
  LatentAttn p = *args;
  if (p.T <= 0) return 0;
  if (p.rank <= 0 || p.rank > kLatAcc * kLatThreads || p.rec < p.rank + p.rot || p.S < 1) return -10;
  const int dims = p.rank + p.rot;
  int hpb = kLatAcc * kLatThreads / p.rank;
  if (hpb > p.heads) hpb = p.heads;
  auto bytes = [&](int h) { return static_cast<size_t>(h * dims + kLatKeys * (dims | 1) + h * kLatKeys + 3 * h) * 4; };
  while (hpb > 1 && bytes(hpb) > 200 * 1024) --hpb;
  if (bytes(hpb) > 200 * 1024) return -12;
  p.heads_per_block = hpb;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  const dim3 grid(p.T, (p.heads + hpb - 1) / hpb);
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(latent_attn_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  if (is_f32) launch_pdl(latent_attn_kernel<float>, grid, dim3(kLatThreads), bytes(hpb), st, p);
  else launch_pdl(latent_attn_kernel<__nv_bfloat16>, grid, dim3(kLatThreads), bytes(hpb), st, p);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int cafd_latent_gate(void* attn, const void* gate, int T, int heads, int vdim, int ld_head, int ldg, int g_off, int is_f32,
                                cafd_stream_t s) {
  if (T <= 0) return 0;
  const dim3 grid(T < 4096 ? T : 4096);
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (is_f32)
    launch_pdl(latent_gate_kernel<float>, grid, dim3(256), 0, st, static_cast<float*>(attn), static_cast<const float*>(gate), T, heads,
               vdim, ld_head, ldg, g_off);
  else
    launch_pdl(latent_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<__nv_bfloat16*>(attn),
               static_cast<const __nv_bfloat16*>(gate), T, heads, vdim, ld_head, ldg, g_off);
  return static_cast<int>(cudaGetLastError());
}
