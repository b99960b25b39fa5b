// Softmax attention over paged keys and values at any head sizes, with a sliding window and kept first tokens, and with one or
// two score maps per head; scores may be capped, a head may have a sink, an output gate and an output that is turned back by its
// position (the tensor-core kernels of attention_prefill.cu and attention_decode.cu serve 128-wide key and value rows; this file
// serves every other size and the fp32 engines).
//
// One block per (token, kv head, run of its query heads).  Keys are walked in tiles that start at multiples of 32, first those
// of the kept tokens, then those of the window, so a row's arithmetic depends on its own position only.  Scores, softmax and
// the weighted sums are fp32.  With two maps per head the rows of both lie in one block: their difference, its norm over the
// head's values and the scale follow at the end.
#include "cafd_api.h"
#include "common.cuh"
#include "hybrid_norm.cuh"

namespace cafd {

struct PagedAttn {
  const void* q;              // [T, heads, maps * dim] E
  const void* k_cache;        // [pages, kv heads, 64, maps * dim] E
  const void* v_cache;        // [pages, kv heads, 64, vdim] E
  const int* page_table;      // [S, max_pages]
  const int* positions;       // [T]
  const int* q_start;         // [S + 1]
  void* out;                  // [T, ldo] E: head h's values at h * head_pitch
  const float* sink;          // [heads] or null: exp(sink) joins the denominator; one map only
  const void* gate;           // row t, head h: E gate[t * gate_ld + h], the head's values are multiplied by its sigmoid; or null; one map only
  const float2* v_table;      // [T, vdim / 2] cos, sin: a head's output is turned back by them, pairs (i, i + vdim / 2); or null; one map only
  int T, S, heads, kv_heads, maps, dim, vdim, window, keep, max_pages, ldo, head_pitch, heads_per_block, gate_ld;
  float scale, lambda, out_scale, eps;
  float cap;                  // scores are cap * tanh(score / cap); 0 = they are not
};

constexpr int kAnyKeys = 32;
constexpr int kAnyThreads = 256;
constexpr int kAnyAcc = 16;   // accumulators per thread: heads_per_block * maps * vdim <= 16 * 256

template <typename E>
__global__ void __launch_bounds__(kAnyThreads) paged_attn_kernel(const PagedAttn p) {
  extern __shared__ float sm[];
  pdl_wait();
  pdl_trigger();
  const int group = p.heads / p.kv_heads;
  const int t = blockIdx.x, kvh = blockIdx.y, h0 = kvh * group + blockIdx.z * p.heads_per_block, tid = threadIdx.x;
  const int nh = min(p.heads_per_block, (kvh + 1) * group - h0);
  const int rows = nh * p.maps, krow = p.maps * p.dim, kp = krow | 1;      // odd pitch: keys in different banks
  const int max_rows = p.heads_per_block * p.maps;
  float* sq = sm;                               // [rows][dim]
  float* sk = sq + max_rows * p.dim;            // [32][kp]
  float* sv = sk + kAnyKeys * kp;               // [32][vdim]
  float* sp = sv + kAnyKeys * p.vdim;           // [rows][32] scores, then weights
  float* sm_m = sp + max_rows * kAnyKeys;       // running maximum, sum and correction per row
  float* sm_l = sm_m + max_rows;
  float* sm_c = sm_l + max_rows;
  float* so = sm_c + max_rows;                  // [rows][vdim] (two maps, or outputs to turn back)
  const int seq = [&] {
    int s = 0, hi = p.S;
    while (hi - s > 1) {
      const int mid = (s + hi) >> 1;
      if (p.q_start[mid] <= t) s = mid; else hi = mid;
    }
    return s;
  }();
  const int pos = p.positions[t];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int keep = min(p.keep, lo);             // positions [0, keep) and [lo, pos] are visible
  const int* pt = p.page_table + static_cast<size_t>(seq) * p.max_pages;
  for (int i = tid; i < rows * p.dim; i += kAnyThreads)
    sq[i] = ld_e<E>(static_cast<const E*>(p.q) + (static_cast<size_t>(t) * p.heads + h0) * krow + i);
  for (int r = tid; r < rows; r += kAnyThreads) { sm_m[r] = -INFINITY; sm_l[r] = 0.f; }
  float acc[kAnyAcc];
#pragma unroll
  for (int i = 0; i < kAnyAcc; ++i) acc[i] = 0.f;
  const int n_acc = rows * p.vdim, warp = tid >> 5, lane = tid & 31;
  const int kept_tiles = (keep + kAnyKeys - 1) / kAnyKeys, first = lo / kAnyKeys, last = pos / kAnyKeys;
  const int skip = max(0, first - kept_tiles);  // tiles between the kept tokens and the window
  for (int i = 0; i <= last - skip; ++i) {
    const int k0 = (i < kept_tiles ? i : i + skip) * kAnyKeys;
    __syncthreads();
    for (int e = tid; e < kAnyKeys * (krow + p.vdim); e += kAnyThreads) {
      const bool is_v = e >= kAnyKeys * krow;
      const int per = is_v ? p.vdim : krow, ee = is_v ? e - kAnyKeys * krow : e;
      const int j = ee / per, d = ee - j * per, at = k0 + j;
      float v = 0.f;
      if (at <= pos && (at >= lo || at < keep) && (at >> 6) < p.max_pages)
        v = ld_e<E>(static_cast<const E*>(is_v ? p.v_cache : p.k_cache) +
                    ((static_cast<size_t>(pt[at >> 6]) * p.kv_heads + kvh) * 64 + (at & 63)) * per + d);
      if (is_v) sv[ee] = v; else sk[j * kp + d] = v;
    }
    __syncthreads();
    for (int e = tid; e < rows * kAnyKeys; e += kAnyThreads) {
      const int r = e >> 5, j = e & 31, at = k0 + j;
      const float* a = sq + r * p.dim;
      const float* b = sk + j * kp + (r % p.maps) * p.dim;
      float s = 0.f;
      for (int d = 0; d < p.dim; ++d) s = fmaf(a[d], b[d], s);
      s *= p.scale;
      if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
      sp[e] = (at <= pos && (at >= lo || at < keep)) ? s : -INFINITY;
    }
    __syncthreads();
    for (int r = warp; r < rows; r += kAnyThreads / 32) {
      const float s = sp[r * kAnyKeys + lane];
      const float m_old = sm_m[r], m = fmaxf(m_old, warp_max(s));      // every tile of the loop holds a visible key
      const float w = expf(s - m);
      const float sum = warp_sum(w);
      sp[r * kAnyKeys + lane] = w;
      __syncwarp();
      if (lane == 0) {
        const float c = expf(m_old - m);
        sm_c[r] = c;
        sm_l[r] = sm_l[r] * c + sum;
        sm_m[r] = m;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kAnyAcc; ++k) {
      const int e = tid + k * kAnyThreads;
      if (e < n_acc) {
        const int r = e / p.vdim, d = e - r * p.vdim;
        float v = acc[k] * sm_c[r];
        const float* w = sp + r * kAnyKeys;
#pragma unroll 8
        for (int j = 0; j < kAnyKeys; ++j) v = fmaf(w[j], sv[j * p.vdim + d], v);
        acc[k] = v;
      }
    }
  }
  E* out = static_cast<E*>(p.out) + static_cast<size_t>(t) * p.ldo;
#pragma unroll
  for (int k = 0; k < kAnyAcc; ++k) {
    const int e = tid + k * kAnyThreads;
    if (e < n_acc) {
      const int r = e / p.vdim, d = e - r * p.vdim;
      const float l = p.sink ? sm_l[r] + expf(p.sink[h0 + r] - sm_m[r]) : sm_l[r];
      float v[1] = {acc[k] / l * (p.maps == 1 ? p.out_scale : 1.f)};
      if (p.gate) v[0] /= 1.0f + expf(-ld_e<E>(static_cast<const E*>(p.gate) + static_cast<size_t>(t) * p.gate_ld + h0 + r));
      if (p.maps == 1 && !p.v_table) store_vec<E, 1>(out + (h0 + r) * p.head_pitch + d, v);
      else so[e] = v[0];
    }
  }
  if (p.maps == 1 && !p.v_table) return;
  __syncthreads();
  if (p.v_table) {
    const int vh = p.vdim >> 1;
    for (int e = tid; e < n_acc; e += kAnyThreads) {
      const int r = e / p.vdim, d = e - r * p.vdim;
      const bool first = d < vh;
      const float2 a = p.v_table[static_cast<size_t>(t) * vh + (first ? d : d - vh)];
      const float o = so[first ? e + vh : e - vh];
      float v[1] = {first ? so[e] * a.x + o * a.y : so[e] * a.x - o * a.y};
      store_vec<E, 1>(out + (h0 + r) * p.head_pitch + d, v);
    }
    return;
  }
  for (int h = warp; h < nh; h += kAnyThreads / 32) {
    float* a = so + 2 * h * p.vdim;
    const float* b = a + p.vdim;
    float ss = 0.f;
    for (int d = lane; d < p.vdim; d += 32) {
      const float o = a[d] - p.lambda * b[d];
      a[d] = o;
      ss += o * o;
    }
    const float inv = p.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(p.vdim) + p.eps);
    for (int d = lane; d < p.vdim; d += 32) {
      float v[1] = {a[d] * inv};
      store_vec<E, 1>(out + (h0 + h) * p.head_pitch + d, v);
    }
  }
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_paged_attn(const PagedAttn* args, int is_f32, cafd_stream_t s) {
  PagedAttn p = *args;
  if (p.T <= 0) return 0;
  if (p.S < 1 || p.kv_heads < 1 || p.heads % p.kv_heads || p.maps < 1 || p.maps > 2 || p.dim < 1 || p.vdim < 1 || p.window < 0 || p.keep < 0 ||
      p.maps * p.vdim > kAnyAcc * kAnyThreads || p.head_pitch < p.vdim || p.ldo < (p.heads - 1) * p.head_pitch + p.vdim ||
      (p.maps == 2 && (p.sink || p.gate || p.v_table)) || (p.v_table && p.vdim % 2) || (p.gate && p.gate_ld < p.heads))
    return -10;
  if (p.window == 0) p.keep = 0;
  const int group = p.heads / p.kv_heads;
  int hpb = kAnyAcc * kAnyThreads / (p.maps * p.vdim);
  if (hpb > group) hpb = group;
  auto bytes = [&](int h) {
    const int rows = h * p.maps;
    return static_cast<size_t>(rows * p.dim + kAnyKeys * ((p.maps * p.dim) | 1) + kAnyKeys * p.vdim + rows * kAnyKeys + 3 * rows +
                               (p.maps == 2 || p.v_table ? rows * p.vdim : 0)) * 4;
  };
  while (hpb > 1 && bytes(hpb) > 200 * 1024) --hpb;
  if (bytes(hpb) > 200 * 1024) return -12;
  p.heads_per_block = hpb;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(paged_attn_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(paged_attn_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  cudaStream_t st = static_cast<cudaStream_t>(s);
  const dim3 grid(p.T, p.kv_heads, (group + hpb - 1) / hpb);
  if (is_f32) launch_pdl(paged_attn_kernel<float>, grid, dim3(kAnyThreads), bytes(hpb), st, p);
  else launch_pdl(paged_attn_kernel<__nv_bfloat16>, grid, dim3(kAnyThreads), bytes(hpb), st, p);
  return static_cast<int>(cudaGetLastError());
}
