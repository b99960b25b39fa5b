// From a step's fused projection rows to queries and cached keys and values, in one launch: a causal convolution over time
// on every channel of q, k and v, an RMS norm of q and k, rotary positions on the leading dimensions of q and k, the paged K / V
// write and the convolution state of every sequence.
//
//   rope_table       cos / sin of position * frequency (times a constant) for every token of the step, once per step and kind of
//                    rotation: every layer that rotates alike reads it
//   conv_rope_kv     pairs (2i, 2i + 1), no norm: four channels per thread walking a run of tokens, the convolution's earlier
//                    inputs in registers
//   conv_rope_kv_any the same for any head sizes and any number of taps: one channel per thread and token
//   conv_norm_rope_kv  with norms (per head or over the whole projection), pairs of either kind, values of their own (rotated or
//                    not) or the convolved keys: a block walks a run of tokens, the projected rows in a ring in shared memory
//   conv_norm_rope_128 the same for bf16 heads of 128: a warp owns whole heads, four channels per lane, and walks a run of tokens
//                    with everything in registers; partners and square sums go by shuffles
//
// A sequence's last taps - 1 projected rows are fp32 in its state slot (oldest first, [taps - 1, channels]); a step reads one
// slot and writes another.  An output is a function of its own taps inputs in a fixed order, so it does not depend on where a
// portion of the sequence begins.
#include "cafd_api.h"
#include "common.cuh"
#include "hybrid_norm.cuh"

namespace cafd {

struct ConvRope {
  const void* proj;           // [T, ld] E
  const float* conv_w;        // [taps, channels], null = no convolution
  const float2* table;        // [T, rot / 2] cos, sin
  const int* slots;           // [T] page * 64 + offset, < 0: nothing is cached
  const int* q_start;         // [S + 1]
  const int* state_in;
  const int* state_out;
  float* state;
  void* q_out;                // [T, q channels] E
  void* k_cache;              // [pages, kv heads, 64, maps * dim] E
  void* v_cache;              // [pages, kv heads, 64, vdim] E
  const float* q_norm;        // [dim] (norm 1, null = no weights) or [nq] (norm 2)
  const float* k_norm;        // [dim] or [nk]
  const float2* v_table;      // [T, vdim / 2] cos, sin: values are rotated over their whole width, pairs (i, i + vdim / 2); null = not
  long long slot_stride, state_off;
  int T, S, ld, q_off, k_off, v_off, nq, nk, nv, maps_dim, dim, vdim, kv_heads, rot, taps, run;
  int norm;                   // 0 none, 1 per head (and map), 2 over all of q and all of k
  int halves;                 // rotated pairs are (i, i + rot / 2), else (2i, 2i + 1)
  int v_from_k;               // nv = 0: the values are the convolved keys before norm and rotation
  int units;                  // heads of q, k and v one block works on
  float eps;
  float rot_sq;               // norm 1: weight of the rotated dimensions' squares (a norm taken after a rotation that scales by its root)
};

__global__ void __launch_bounds__(256) rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ freq, float2* __restrict__ out,
                                                         int T, int half, float mag) {
  pdl_wait();
  pdl_trigger();
  const int n = T * half;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const int t = i / half;
    float s, c;
    sincosf(static_cast<float>(positions[t]) * freq[i - t * half], &s, &c);
    out[i] = make_float2(c * mag, s * mag);
  }
}

// Where channel c of the concatenated [q | k | v] channels goes for token t, whose K / V slot is `slot`; null = nowhere.
template <typename E>
__device__ __forceinline__ E* conv_rope_dest(const ConvRope& p, int t, int slot, int c) {
  if (c < p.nq) return static_cast<E*>(p.q_out) + static_cast<size_t>(t) * p.nq + c;
  if (slot < 0) return nullptr;
  const bool is_k = c < p.nq + p.nk;
  const int per = is_k ? p.maps_dim : p.vdim;
  const int cc = c - p.nq - (is_k ? 0 : p.nk);
  const int g = cc / per;
  E* base = static_cast<E*>(is_k ? p.k_cache : p.v_cache);
  return base + ((static_cast<size_t>(slot >> 6) * p.kv_heads + g) * 64 + (slot & 63)) * per + (cc - g * per);
}
__device__ __forceinline__ int conv_rope_col(const ConvRope& p, int c) {
  return c < p.nq ? p.q_off + c : c < p.nq + p.nk ? p.k_off + c - p.nq : p.v_off + c - p.nq - p.nk;
}
__device__ __forceinline__ int seq_of(const int* q_start, int S, int T, int t) {
  if (S == T && q_start[t] == t && q_start[t + 1] == t + 1) return t;     // decode: a token per sequence
  int s = 0, hi = S;
  while (hi - s > 1) {
    const int mid = (s + hi) >> 1;
    if (q_start[mid] <= t) s = mid; else hi = mid;
  }
  return s;
}

template <typename E, int MAXT>
__global__ void __launch_bounds__(128, MAXT <= 4 && sizeof(E) == 2 ? 7 : 2) conv_rope_kv_kernel(const ConvRope p) {
  constexpr int V = 4, W = MAXT - 1, kBatch = 4;
  extern __shared__ float4 sm4[];               // the run's angles [run][rot / 2] cos, sin, then its slots [run]
  float2* s_cs = reinterpret_cast<float2*>(sm4);
  int* s_slot = reinterpret_cast<int*>(s_cs + p.run * (p.rot >> 1));
  const int C = p.nq + p.nk + p.nv;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const int halo = p.conv_w ? p.taps - 1 : 0;
  float w[MAXT][V];                             // w[k]: weight of the input k tokens back (no kernel writes the weights)
#pragma unroll
  for (int k = 0; k < MAXT; ++k) {
#pragma unroll
    for (int e = 0; e < V; ++e) w[k][e] = !p.conv_w && k == 0 ? 1.f : 0.f;
    if (p.conv_w && k <= halo && c < C) load_vec<float, V>(p.conv_w + static_cast<size_t>(halo - k) * C + c, w[k]);
  }
  pdl_wait();
  pdl_trigger();
  const int r0 = blockIdx.x * p.run, r1 = min(p.T, r0 + p.run);
  const E* src = static_cast<const E*>(p.proj) + conv_rope_col(p, min(c, C - V));
  Packed<E, V> nx[kBatch];                      // the next batch's rows, on their way while one is worked on
#pragma unroll
  for (int j = 0; j < kBatch; ++j) nx[j] = load_packed<E, V>(src + static_cast<size_t>(min(r0 + j, p.T - 1)) * p.ld);
  int seq = 0, s_lo = 0, s_hi = p.T, s_in = 0;
  if (halo > 0) {
    seq = seq_of(p.q_start, p.S, p.T, r0);
    s_lo = p.q_start[seq];
    s_hi = p.q_start[seq + 1];
    s_in = p.state_in[seq];
  }
  for (int i = threadIdx.x; i < (r1 - r0) * (p.rot >> 1); i += blockDim.x) s_cs[i] = p.table[static_cast<size_t>(r0) * (p.rot >> 1) + i];
  for (int i = threadIdx.x; i < r1 - r0; i += blockDim.x) s_slot[i] = p.slots[r0 + i];
  __syncthreads();
  if (c >= C) return;
  const bool is_q = c < p.nq, is_v = c >= p.nq + p.nk;
  const int d0 = is_v ? p.rot : (is_q ? c : c - p.nq) % p.dim;   // first dimension inside its map; v: past the rotated ones
  const bool turns = d0 < p.rot;
  // K / V: where token (page 0, offset 0) would put these channels, elements per token of a head and per page
  E* const dst0 = is_q ? static_cast<E*>(p.q_out) + c : conv_rope_dest<E>(p, 0, 0, c);
  const int per = is_v ? p.vdim : p.maps_dim;
  const size_t page = static_cast<size_t>(p.kv_heads) * 64 * per;
  float x[W + kBatch][V];                       // a batch of kBatch tokens' inputs behind the W before it
#pragma unroll
  for (int i = 0; i < W; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) x[i][e] = 0.f;
  for (int t = r0; t < r1; t += kBatch) {
#pragma unroll
    for (int j = 0; j < kBatch; ++j) unpack(nx[j], x[W + j]);
    if (t + kBatch < r1) {
#pragma unroll
      for (int j = 0; j < kBatch; ++j) nx[j] = load_packed<E, V>(src + static_cast<size_t>(min(t + kBatch + j, p.T - 1)) * p.ld);
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const int row = t + j;
      if (row >= r1) break;
      if (halo > 0 && (row == r0 || row == s_hi)) {
        // The inputs before a run's or a sequence's first token: rows of this step, or the state where they lie before it.
        // (The slots held another sequence's last inputs, which are done with.)
        while (row == s_hi && seq + 1 < p.S) {  // (empty sequences are skipped)
          ++seq;
          s_lo = s_hi;
          s_hi = p.q_start[seq + 1];
          s_in = p.state_in[seq];
        }
        const float* st = p.state + static_cast<size_t>(s_in) * p.slot_stride + p.state_off + c;
#pragma unroll
        for (int k = 1; k < MAXT; ++k) {
          if (k <= halo) {
            if (row - k >= s_lo) load_vec<E, V>(src + static_cast<size_t>(row - k) * p.ld, x[W + j - k]);
            else load_vec<float, V>(st + static_cast<size_t>(halo + row - k - s_lo) * C, x[W + j - k]);
          }
        }
      }
      float y[V];
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = w[0][e] * x[W + j][e];
#pragma unroll
      for (int k = W; k > 0; --k) {
        if (k <= halo) {                        // (past the taps there may be another sequence's inputs)
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(w[k][e], x[W + j - k][e], y[e]);
        }
      }
      if (turns) {
        const float2* cs = s_cs + (row - r0) * (p.rot >> 1) + (d0 >> 1);
#pragma unroll
        for (int i = 0; i < V / 2; ++i) {
          if (d0 + 2 * i < p.rot) {
            const float2 a = cs[i];
            const float u = y[2 * i], v = y[2 * i + 1];
            y[2 * i] = u * a.x - v * a.y;
            y[2 * i + 1] = v * a.x + u * a.y;
          }
        }
      }
      const int slot = is_q ? 0 : s_slot[row - r0];
      const size_t off = is_q ? static_cast<size_t>(row) * p.nq : (slot >> 6) * page + (slot & 63) * per;
      if (slot >= 0) store_vec<E, V>(dst0 + off, y);
      if (halo > 0 && row == s_hi - 1) {        // the sequence's last halo inputs, oldest first
        float* st = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off + c;
#pragma unroll
        for (int k = 0; k < W; ++k)
          if (k < halo) store_vec<float, V>(st + static_cast<size_t>(halo - 1 - k) * C, x[W + j - k]);
      }
    }
#pragma unroll
    for (int i = 0; i < W; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = x[kBatch + i][e];
  }
}

// The same for every other shape: block = (token, 256 channels).
template <typename E>
__global__ void __launch_bounds__(256) conv_rope_kv_any_kernel(const ConvRope p) {
  pdl_wait();
  pdl_trigger();
  const int C = p.nq + p.nk + p.nv, t = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int halo = p.conv_w ? p.taps - 1 : 0;
  int seq = 0, s_lo = 0, s_hi = p.T;
  const float* st = nullptr;
  if (halo > 0) {
    seq = seq_of(p.q_start, p.S, p.T, t);
    s_lo = p.q_start[seq];
    s_hi = p.q_start[seq + 1];
    st = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.state_off;
  }
  auto input = [&](int row, int ch) {           // input of this step's token `row`, which may lie before the step
    return row >= s_lo ? ld_e<E>(static_cast<const E*>(p.proj) + static_cast<size_t>(row) * p.ld + conv_rope_col(p, ch))
                       : st[static_cast<size_t>(halo + row - s_lo) * C + ch];
  };
  auto conv = [&](int ch) {
    if (!p.conv_w) return input(t, ch);
    float y = p.conv_w[static_cast<size_t>(halo) * C + ch] * input(t, ch);
    for (int j = 0; j < halo; ++j) y = fmaf(p.conv_w[static_cast<size_t>(j) * C + ch], input(t - halo + j, ch), y);
    return y;
  };
  float y = conv(c);
  if (c < p.nq + p.nk) {
    const int d = (c < p.nq ? c : c - p.nq) % p.dim;
    if (d < p.rot) {
      const float2 k = p.table[static_cast<size_t>(t) * (p.rot >> 1) + (d >> 1)];
      const float o = conv(d & 1 ? c - 1 : c + 1);
      y = d & 1 ? y * k.x + o * k.y : y * k.x - o * k.y;
    }
  }
  E* dst = conv_rope_dest<E>(p, t, c < p.nq ? 0 : p.slots[t], c);
  if (dst) {
    float v[1] = {y};
    store_vec<E, 1>(dst, v);
  }
  if (halo > 0 && t == s_hi - 1) {
    float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off;
    for (int j = 0; j < halo; ++j) so[static_cast<size_t>(j) * C + c] = input(t - halo + 1 + j, c);
  }
}

__device__ __forceinline__ void cp_async_bytes(void* dst, const void* src, int bytes) {
  const uint32_t d = smem_u32(dst);
  if (bytes == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
  else if (bytes == 8) asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(d), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// Convolution, norm, rotation and the K / V write.  A block owns `units` consecutive heads of [q | k | v] and walks a run of
// tokens.  Per token: the thread that owns V channels convolves them (inputs from the ring, or from the state where they lie
// before the step) into shared memory, the heads' square sums are taken (by the lanes of a head where a head is a power of two
// of at most 32 vectors, else by a warp per head), then the channels are normed and rotated with their partners.
constexpr int kCnrThreads = 256, kCnrAhead = 2;

template <typename E, int V>
__global__ void __launch_bounds__(kCnrThreads) conv_norm_rope_kv_kernel(const ConvRope p) {
  extern __shared__ float4 sm4[];
  __shared__ float part[2][kCnrThreads / 32];
  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int uq = p.nq / p.dim, uk = p.nk / p.dim, uv = p.nv / p.vdim, kmaps = p.maps_dim / p.dim;
  const int u0 = blockIdx.y * p.units, u1 = min(uq + uk + uv, u0 + p.units);
  auto chan = [&](int u) { return u <= uq + uk ? u * p.dim : p.nq + p.nk + (u - uq - uk) * p.vdim; };
  const int c0 = chan(u0), c1 = chan(u1), n = c1 - c0, nvec = n / V, C = p.nq + p.nk + p.nv;
  const int halo = p.conv_w ? p.taps - 1 : 0, ring = halo + 1 + kCnrAhead;
  const int nqk = min(c1, p.nq + p.nk) - c0;    // channels of q and k among this block's (they come first); may be <= 0
  const int max_n = p.units * (p.dim > p.vdim ? p.dim : p.vdim);
  float* const y = reinterpret_cast<float*>(sm4);                        // [max_n] convolved channels of q and k
  float* const ss = y + ((max_n + 3) & ~3);                              // [units] square sums of the heads
  E* const rows = reinterpret_cast<E*>(ss + ((p.units + 3) & ~3));       // [ring][row_pitch]
  const int row_pitch = (max_n + 15) & ~15;
  const int vpu = p.dim / V;                                             // vectors of a head of q or k
  const bool lanes = p.norm && vpu <= 32 && (vpu & (vpu - 1)) == 0;
  const int half = p.rot >> 1;
  const int nrot = p.v_table ? n : nqk;                                  // channels that pass the second half of a token's work
  const int r0 = blockIdx.x * p.run, r1 = min(p.T, r0 + p.run);
  auto fetch = [&](int row) {
    if (row < r1) {
      const E* src = static_cast<const E*>(p.proj) + static_cast<size_t>(row) * p.ld;
      E* dst = rows + (row % ring) * row_pitch;
      for (int i = tid; i < nvec; i += kCnrThreads) {
        const E* a = src + conv_rope_col(p, c0 + i * V);
        if constexpr (V * sizeof(E) >= 16) {
#pragma unroll
          for (int b = 0; b < V; b += 16 / static_cast<int>(sizeof(E))) cp_async_bytes(dst + i * V + b, a + b, 16);
        } else if constexpr (V * sizeof(E) >= 4) {
          cp_async_bytes(dst + i * V, a, V * sizeof(E));
        } else {
          dst[i] = *a;
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (int row = max(0, r0 - halo); row < r0; ++row) fetch(row);
#pragma unroll
  for (int a = 0; a < kCnrAhead; ++a) fetch(r0 + a);
  int seq = 0, s_lo = 0, s_hi = p.T, s_in = 0;
  if (halo > 0) {
    seq = seq_of(p.q_start, p.S, p.T, r0);
    s_lo = p.q_start[seq];
    s_hi = p.q_start[seq + 1];
    s_in = p.state_in[seq];
  }
  for (int t = r0; t < r1; ++t) {
    fetch(t + kCnrAhead);
    asm volatile("cp.async.wait_group %0;" ::"n"(kCnrAhead) : "memory");
    __syncthreads();                            // row t is here; the last token's y and ss are done with
    while (halo > 0 && t == s_hi && seq + 1 < p.S) {                     // next sequence (empty ones are skipped)
      ++seq;
      s_lo = s_hi;
      s_hi = p.q_start[seq + 1];
      s_in = p.state_in[seq];
    }
    const float* st = halo > 0 ? p.state + static_cast<size_t>(s_in) * p.slot_stride + p.state_off : nullptr;
    const int slot = p.slots[t];
    for (int i = tid; i < (nvec + 31) / 32 * 32; i += kCnrThreads) {     // whole warps: the lanes of a head sum up together
      const int c = c0 + i * V;
      float v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
      if (i < nvec) {
        load_vec<E, V>(rows + (t % ring) * row_pitch + i * V, v);
        if (p.conv_w) {
          float w[V], x[V];
          load_vec<float, V>(p.conv_w + static_cast<size_t>(halo) * C + c, w);
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] *= w[e];
          for (int j = 0; j < halo; ++j) {
            const int row = t - halo + j;
            load_vec<float, V>(p.conv_w + static_cast<size_t>(j) * C + c, w);
            if (row >= s_lo) load_vec<E, V>(rows + (row % ring) * row_pitch + i * V, x);
            else load_vec<float, V>(st + static_cast<size_t>(halo + row - s_lo) * C + c, x);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = fmaf(w[e], x[e], v[e]);
          }
        }
        if (i * V < nrot) {
          store_vec<float, V>(y + i * V, v);
          if (p.v_from_k && c >= p.nq && slot >= 0) {
            const int cc = c - p.nq, g = cc / p.vdim;
            store_vec<E, V>(static_cast<E*>(p.v_cache) + ((static_cast<size_t>(slot >> 6) * p.kv_heads + g) * 64 + (slot & 63)) * p.vdim + (cc - g * p.vdim), v);
          }
        } else if (E* dst = conv_rope_dest<E>(p, t, slot, c)) {
          store_vec<E, V>(dst, v);
        }
        if (halo > 0 && t == s_hi - 1) {        // the sequence's last halo inputs, oldest first
          float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off + c;
          for (int j = 0; j < halo; ++j) {
            const int row = t - halo + 1 + j;
            float x[V];
            if (row >= s_lo) load_vec<E, V>(rows + (row % ring) * row_pitch + i * V, x);
            else load_vec<float, V>(st + static_cast<size_t>(halo + row - s_lo) * C + c, x);
            store_vec<float, V>(so + static_cast<size_t>(j) * C, x);
          }
        }
      }
      if (lanes) {
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) s += v[e] * v[e];
        if ((i % vpu) * V < p.rot) s *= p.rot_sq;                        // (a vector lies on one side of the rotated dimensions' end)
        for (int o = 1; o < vpu; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (i * V < nqk && i % vpu == 0) ss[i / vpu] = s;
      }
    }
    __syncthreads();
    if (nrot <= 0) continue;
    const int nu = max(0, nqk) / p.dim, nuq = max(0, min(u1, uq) - u0);          // heads of q and k here, of q among them
    if (p.norm && !lanes) {
      for (int u = warp; u < nu; u += kCnrThreads / 32) {
        float s = 0.f;
        for (int d = lane; d < p.dim; d += 32) s = fmaf(y[u * p.dim + d] * (d < p.rot ? p.rot_sq : 1.f), y[u * p.dim + d], s);
        s = warp_sum(s);
        if (lane == 0) ss[u] = s;
      }
      __syncthreads();
    }
    float inv_q = 1.f, inv_k = 1.f;
    if (p.norm == 2) {                          // (a block then owns all heads)
      float a = 0.f, b = 0.f;
      for (int u = tid; u < nu; u += kCnrThreads) (u < nuq ? a : b) += ss[u];
      a = warp_sum(a);
      b = warp_sum(b);
      if (lane == 0) { part[0][warp] = a; part[1][warp] = b; }
      __syncthreads();
      a = b = 0.f;
#pragma unroll
      for (int w = 0; w < kCnrThreads / 32; ++w) { a += part[0][w]; b += part[1][w]; }
      inv_q = 1.0f / sqrtf(a / static_cast<float>(p.nq) + p.eps);
      inv_k = 1.0f / sqrtf(b / static_cast<float>(p.nk) + p.eps);
    }
    const float2* cs = p.table + static_cast<size_t>(t) * half;
    for (int i = tid; i * V < nrot; i += kCnrThreads) {
      if (i * V >= nqk) {                       // a value (V divides vdim / 2)
        const int c = c0 + i * V, d = (c - p.nq - p.nk) % p.vdim, vh = p.vdim >> 1;
        const bool first = d < vh;
        const float2* a = p.v_table + static_cast<size_t>(t) * vh + (first ? d : d - vh);
        float v[V], o[V];
        load_vec<float, V>(y + i * V, v);
        load_vec<float, V>(y + i * V + (first ? vh : -vh), o);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = first ? v[e] * a[e].x - o[e] * a[e].y : v[e] * a[e].x + o[e] * a[e].y;
        if (E* dst = conv_rope_dest<E>(p, t, slot, c)) store_vec<E, V>(dst, v);
        continue;
      }
      const int c = c0 + i * V, u = i * V / p.dim, d = i * V - u * p.dim;
      const bool is_q = c < p.nq;
      const float* wn = !p.norm || !p.q_norm ? nullptr : p.norm == 1 ? (is_q ? p.q_norm : p.k_norm) + d : is_q ? p.q_norm + c : p.k_norm + c - p.nq;
      const float inv = p.norm == 1 ? 1.0f / sqrtf(ss[u] / static_cast<float>(p.dim) + p.eps) : is_q ? inv_q : inv_k;
      auto normed = [&](int at, float (&v)[V]) {                         // the normed channels `at` places from this thread's
        load_vec<float, V>(y + i * V + at, v);
        if (p.norm && !wn) {
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] *= inv;
        }
        if (wn) {
          float w[V];
          load_vec<float, V>(wn + at, w);
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] = v[e] * inv * w[e];
        }
      };
      float v[V];
      normed(0, v);
      if (d < p.rot) {
        if (p.halves) {                         // (V divides rot / 2)
          const bool first = d < half;
          float o[V];
          normed(first ? half : -half, o);
          const float2* a = cs + (first ? d : d - half);
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] = first ? v[e] * a[e].x - o[e] * a[e].y : v[e] * a[e].x + o[e] * a[e].y;
        } else if constexpr (V == 1) {
          float o[1];
          normed(d & 1 ? -1 : 1, o);
          const float2 a = cs[d >> 1];
          v[0] = d & 1 ? v[0] * a.x + o[0] * a.y : v[0] * a.x - o[0] * a.y;
        } else {                                // (V divides rot)
#pragma unroll
          for (int e = 0; e < V; e += 2) {
            const float2 a = cs[(d + e) >> 1];
            const float x0 = v[e], x1 = v[e + 1];
            v[e] = x0 * a.x - x1 * a.y;
            v[e + 1] = x1 * a.x + x0 * a.y;
          }
        }
      }
      E* dst;
      if (is_q) {
        dst = static_cast<E*>(p.q_out) + static_cast<size_t>(t) * p.nq + c;
      } else {
        const int uu = u0 + u - uq, g = uu / kmaps;                         // key head (with two maps: of map uu % kmaps)
        dst = slot < 0 ? nullptr : static_cast<E*>(p.k_cache) + ((static_cast<size_t>(slot >> 6) * p.kv_heads + g) * 64 + (slot & 63)) * p.maps_dim + (uu - g * kmaps) * p.dim + d;
      }
      if (dst) store_vec<E, V>(dst, v);
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

// bf16, heads of 128 and up to four taps.  A warp owns NH heads of one kind (q, k or v), a lane the same four channels of each, so
// weights, earlier inputs and the rows to come stay in registers.  kAll: norms over the projection (no convolution); a block
// then holds all heads, and the square sums of a batch of tokens meet in shared memory behind one barrier.
template <int NH, bool kConv, bool kAll>
__global__ void __launch_bounds__(kAll ? 512 : 128, kAll ? 1 : 4) conv_norm_rope_128_kernel(const ConvRope p) {
  constexpr int V = 4, W = 3, kBatch = kAll ? 2 : 4, kMaxWarps = kAll ? 16 : 1;
  using Row = Packed<__nv_bfloat16, V>;
  extern __shared__ float4 sm4[];               // the run's angles [run][rot / 2] cos, sin, then its slots [run]
  __shared__ float part[2][kBatch][kMaxWarps];
  const int half = p.rot >> 1, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float2* s_cs = reinterpret_cast<float2*>(sm4);
  int* s_slot = reinterpret_cast<int*>(s_cs + p.run * half);
  const int uq = p.nq >> 7, uk = p.nk >> 7, C = p.nq + p.nk + p.nv;
  const int u0 = (blockIdx.y * (blockDim.x >> 5) + warp) * NH;             // (the launch gives every warp its heads)
  const bool is_q = u0 < uq, is_k = !is_q && u0 < uq + uk;
  const int c = u0 * 128 + lane * V, d = lane * V;
  const int halo = kConv ? p.taps - 1 : 0;
  float w[kConv ? W + 1 : 1][NH][V];            // w[k]: weight of the input k tokens back
  float wn[kAll ? NH : 1][V];
  if constexpr (kConv) {
#pragma unroll
    for (int k = 0; k <= W; ++k)
#pragma unroll
      for (int h = 0; h < NH; ++h) {
#pragma unroll
        for (int e = 0; e < V; ++e) w[k][h][e] = 0.f;
        if (k <= halo) load_vec<float, V>(p.conv_w + static_cast<size_t>(halo - k) * C + c + h * 128, w[k][h]);
      }
  }
#pragma unroll
  for (int h = 0; h < (kAll ? NH : 1); ++h) {
#pragma unroll
    for (int e = 0; e < V; ++e) wn[h][e] = 1.f;
    if (p.norm && p.q_norm && (is_q || is_k)) load_vec<float, V>((is_q ? p.q_norm + (kAll ? c : d) : p.k_norm + (kAll ? c - p.nq : d)) + h * 128, wn[h]);
  }
  pdl_wait();
  pdl_trigger();
  const int r0 = blockIdx.x * p.run, r1 = min(p.T, r0 + p.run);
  const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.proj) + conv_rope_col(p, c);
  auto row_at = [&](int row, int h) { return load_packed<__nv_bfloat16, V>(src + static_cast<size_t>(row) * p.ld + h * 128); };
  Row nx[kBatch][NH];                           // the next batch's rows, on their way while one is worked on
#pragma unroll
  for (int j = 0; j < kBatch; ++j)
#pragma unroll
    for (int h = 0; h < NH; ++h) nx[j][h] = row_at(min(r0 + j, r1 - 1), h);
  int seq = 0, s_lo = 0, s_hi = p.T, s_in = 0;
  if (halo > 0) {
    seq = seq_of(p.q_start, p.S, p.T, r0);
    s_lo = p.q_start[seq];
    s_hi = p.q_start[seq + 1];
    s_in = p.state_in[seq];
  }
  for (int i = threadIdx.x; i < (r1 - r0) * half; i += blockDim.x) s_cs[i] = p.table[static_cast<size_t>(r0) * half + i];
  for (int i = threadIdx.x; i < r1 - r0; i += blockDim.x) s_slot[i] = p.slots[r0 + i];
  __syncthreads();
  Row x[W + kBatch][NH];                        // a batch of rows behind the W before it
#pragma unroll
  for (int i = 0; i < W; ++i)
#pragma unroll
    for (int h = 0; h < NH; ++h) x[i][h].q = make_uint2(0u, 0u);
  const bool turns = (is_q || is_k) && d < p.rot;
  const bool first = d < half;
  const int partner = !turns ? lane : first ? lane + half / V : lane - half / V;       // halves; neighbours lie in the same lane
  int flip = 0;
  for (int t = r0; t < r1; t += kBatch) {
#pragma unroll
    for (int j = 0; j < kBatch; ++j)
#pragma unroll
      for (int h = 0; h < NH; ++h) x[W + j][h] = nx[j][h];
    if (t + kBatch < r1) {
#pragma unroll
      for (int j = 0; j < kBatch; ++j)
#pragma unroll
        for (int h = 0; h < NH; ++h) nx[j][h] = row_at(min(t + kBatch + j, r1 - 1), h);
    }
    float inv_all[kBatch];
    if constexpr (kAll) {
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        float s = 0.f;
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          float v[V];
          unpack(x[W + j][h], v);
#pragma unroll
          for (int e = 0; e < V; ++e) s = fmaf(v[e], v[e], s);
        }
        s = warp_sum(s);
        if (lane == 0) part[flip][j][warp] = s;
      }
      __syncthreads();
      const int w0 = is_q ? 0 : uq / NH, w1 = is_q ? uq / NH : (uq + uk) / NH;
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        const float s = warp_sum(lane >= w0 && lane < w1 ? part[flip][j][lane & (kMaxWarps - 1)] : 0.f);
        inv_all[j] = 1.0f / sqrtf(s / static_cast<float>(is_q ? p.nq : p.nk) + p.eps);
      }
      flip ^= 1;
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const int row = t + j;
      if (row >= r1) break;
      if (halo > 0 && (row == r0 || row == s_hi)) {
        // The inputs before a run's or a sequence's first token: rows of this step, or the state where they lie before it.
        // (The slots held another sequence's last inputs, which are done with.)
        while (row == s_hi && seq + 1 < p.S) {  // (empty sequences are skipped)
          ++seq;
          s_lo = s_hi;
          s_hi = p.q_start[seq + 1];
          s_in = p.state_in[seq];
        }
        const float* st = p.state + static_cast<size_t>(s_in) * p.slot_stride + p.state_off + c;
#pragma unroll
        for (int k = 1; k <= W; ++k) {
          if (k <= halo) {
#pragma unroll
            for (int h = 0; h < NH; ++h) {
              if (row - k >= s_lo) {
                x[W + j - k][h] = row_at(row - k, h);
              } else {
                float v[V];
                load_vec<float, V>(st + static_cast<size_t>(halo + row - k - s_lo) * C + h * 128, v);
                x[W + j - k][h].q = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));      // what was stored were bf16 rows
              }
            }
          }
        }
      }
      const int slot = s_slot[row - r0];
      float2 cs[V];                             // neighbours use the first half of them
      if (turns) {
        const float2* a = s_cs + (row - r0) * half + (p.halves ? (first ? d : d - half) : d >> 1);
#pragma unroll
        for (int e = 0; e < V; ++e) cs[e] = p.halves || e < V / 2 ? a[e] : make_float2(1.f, 0.f);
      }
#pragma unroll
      for (int h = 0; h < NH; ++h) {
        float y[V];
        unpack(x[W + j][h], y);
        if constexpr (kConv) {
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] *= w[0][h][e];
#pragma unroll
          for (int k = W; k > 0; --k) {
            if (k <= halo) {                    // (past the taps there may be another sequence's inputs)
              float v[V];
              unpack(x[W + j - k][h], v);
#pragma unroll
              for (int e = 0; e < V; ++e) y[e] = fmaf(w[k][h][e], v[e], y[e]);
            }
          }
        }
        const size_t cell = slot < 0 ? 0 : (static_cast<size_t>(slot >> 6) * p.kv_heads) * 8192 + (slot & 63) * 128 + d;
        const int g = u0 + h - uq - (is_k ? 0 : uk);                       // key or value head
        if (!is_q && !is_k) {
          if (p.v_table) {                      // pairs (i, i + 64): lanes 16 apart
            const float2* a = p.v_table + static_cast<size_t>(row) * 64 + (lane & 15) * V;
#pragma unroll
            for (int e = 0; e < V; ++e) {
              const float o = __shfl_xor_sync(0xffffffffu, y[e], 16);
              y[e] = lane < 16 ? y[e] * a[e].x - o * a[e].y : y[e] * a[e].x + o * a[e].y;
            }
          }
          if (slot >= 0) store_vec<__nv_bfloat16, V>(static_cast<__nv_bfloat16*>(p.v_cache) + cell + static_cast<size_t>(g) * 8192, y);
          continue;
        }
        if (p.v_from_k && is_k && slot >= 0) store_vec<__nv_bfloat16, V>(static_cast<__nv_bfloat16*>(p.v_cache) + cell + static_cast<size_t>(g) * 8192, y);
        if (p.norm) {
          float inv;
          if constexpr (kAll) {
            inv = inv_all[j];
          } else {
            float s = 0.f;
#pragma unroll
            for (int e = 0; e < V; ++e) s = fmaf(y[e], y[e], s);
            if (d < p.rot) s *= p.rot_sq;
            inv = 1.0f / sqrtf(warp_sum(s) * (1.0f / 128.0f) + p.eps);
          }
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = y[e] * inv * wn[kAll ? h : 0][e];
        }
        if (p.halves) {
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const float o = __shfl_sync(0xffffffffu, y[e], partner);
            if (turns) y[e] = first ? y[e] * cs[e].x - o * cs[e].y : y[e] * cs[e].x + o * cs[e].y;
          }
        } else if (turns) {
#pragma unroll
          for (int e = 0; e < V; e += 2) {
            const float2 a = cs[e >> 1];
            const float x0 = y[e], x1 = y[e + 1];
            y[e] = x0 * a.x - x1 * a.y;
            y[e + 1] = x1 * a.x + x0 * a.y;
          }
        }
        if (is_q) store_vec<__nv_bfloat16, V>(static_cast<__nv_bfloat16*>(p.q_out) + static_cast<size_t>(row) * p.nq + c + h * 128, y);
        else if (slot >= 0) store_vec<__nv_bfloat16, V>(static_cast<__nv_bfloat16*>(p.k_cache) + cell + static_cast<size_t>(g) * 8192, y);
      }
      if (halo > 0 && row == s_hi - 1) {        // the sequence's last halo inputs, oldest first
        float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off + c;
#pragma unroll
        for (int k = 0; k < W; ++k) {
          if (k < halo) {
#pragma unroll
            for (int h = 0; h < NH; ++h) {
              float v[V];
              unpack(x[W + j - k][h], v);
              store_vec<float, V>(so + static_cast<size_t>(halo - 1 - k) * C + h * 128, v);
            }
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < W; ++i)
#pragma unroll
      for (int h = 0; h < NH; ++h) x[i][h] = x[kBatch + i][h];
  }
}

// logits = cap * tanh(logits / cap), rows of n values `ld` apart
__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, int n, long long ld, float cap) {
  pdl_wait();
  pdl_trigger();
  float* row = x + static_cast<size_t>(blockIdx.y) * ld;
  const float inv = 1.0f / cap;
  const int i0 = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i0 >= n) return;
  if ((ld & 3) == 0 && i0 + 4 <= n) {
    float4 v = *reinterpret_cast<float4*>(row + i0);
    v.x = cap * tanhf(v.x * inv); v.y = cap * tanhf(v.y * inv); v.z = cap * tanhf(v.z * inv); v.w = cap * tanhf(v.w * inv);
    *reinterpret_cast<float4*>(row + i0) = v;
  } else {
    for (int i = i0; i < min(n, i0 + 4); ++i) row[i] = cap * tanhf(row[i] * inv);
  }
}

template <typename E>
static int launch_conv_rope(ConvRope p, cudaStream_t st) {
  const int C = p.nq + p.nk + p.nv;
  const bool vec = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.ld % 4 == 0 && p.q_off % 4 == 0 && p.k_off % 4 == 0 && p.v_off % 4 == 0 &&
                   p.state_off % 4 == 0 && p.slot_stride % 4 == 0 && (!p.conv_w || p.taps <= 8);
  if (!vec) {
    launch_pdl(conv_rope_kv_any_kernel<E>, dim3(p.T, (C + 255) / 256), dim3(256), 0, st, p);
    return static_cast<int>(cudaGetLastError());
  }
  const int cols = (C / 4 + 127) / 128;
  // decode: one token per block; prompts: one wave of blocks, each with a run of tokens whose angles fit in shared memory
  const int want = 148 * 7;
  int run = (p.T * cols + want - 1) / want;
  run = p.T <= 64 ? 1 : run < 4 ? 4 : run > 64 ? 64 : run;
  const int row_bytes = p.rot * 4 + 4, fit = 40 * 1024 / row_bytes;
  if (fit < 1) return -12;
  p.run = run < fit ? run : fit;
  const dim3 grid((p.T + p.run - 1) / p.run, cols);
  const size_t smem = static_cast<size_t>(p.run) * row_bytes;
  if (!p.conv_w || p.taps <= 4) launch_pdl(conv_rope_kv_kernel<E, 4>, grid, dim3(128), smem, st, p);
  else launch_pdl(conv_rope_kv_kernel<E, 8>, grid, dim3(128), smem, st, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename E, int V>
static int launch_conv_norm_rope(ConvRope p, cudaStream_t st) {
  const int units = p.nq / p.dim + p.nk / p.dim + p.nv / p.vdim, wide = p.dim > p.vdim ? p.dim : p.vdim;
  const int ring = (p.conv_w ? p.taps : 1) + kCnrAhead;
  auto bytes = [&](int u) {
    return static_cast<size_t>((u * wide + 3) / 4 * 4 + (u + 3) / 4 * 4) * 4 + static_cast<size_t>(ring) * ((u * wide + 15) / 16 * 16) * sizeof(E);
  };
  // a norm over the whole projection needs all heads in one block; else few tokens are spread over more blocks by heads
  p.units = units;
  if (p.norm != 2) {
    const int want = (2 * 148 + p.T - 1) / p.T, room = 64 * 1024;
    int per = (units + want - 1) / want;
    const int least = (512 + wide - 1) / wide;                           // at least 512 channels a block
    if (per < least) per = least;
    if (per > units) per = units;
    while (per > 1 && bytes(per) > static_cast<size_t>(room)) --per;
    p.units = per;
  }
  const size_t smem = bytes(p.units);
  if (smem > 200 * 1024) return -12;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(conv_norm_rope_kv_kernel<E, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  const int cols = (units + p.units - 1) / p.units;
  const int resident = smem > 100 * 1024 ? 1 : smem > 50 * 1024 ? 3 : smem > 32 * 1024 ? 4 : 6;
  int run = (p.T * cols + 148 * resident - 1) / (148 * resident);        // one wave of blocks
  p.run = p.T <= 64 ? 1 : run < 1 ? 1 : run > 64 ? 64 : run;
  const dim3 grid((p.T + p.run - 1) / p.run, cols);
  launch_pdl(conv_norm_rope_kv_kernel<E, V>, grid, dim3(kCnrThreads), smem, st, p);
  return static_cast<int>(cudaGetLastError());
}

template <int NH, bool kConv, bool kAll>
static int launch_conv_norm_rope_128(ConvRope p, cudaStream_t st) {
  const int groups = (p.nq + p.nk + p.nv) / 128 / NH;
  int warps = groups;
  if (!kAll) {
    warps = 4;
    while (groups % warps) --warps;
  }
  const int cols = groups / warps, row_bytes = p.rot * 4 + 4;
  const int want = 148 * (warps < 16 ? 16 / warps : 1);                    // blocks of one wave: 16 warps of up to 128 registers a thread
  int run = (p.T * cols + want - 1) / want;
  run = p.T <= 64 ? 1 : run < 4 ? 4 : run > 128 ? 128 : run;
  const int fit = 40 * 1024 / row_bytes;
  p.run = run < fit ? run : fit;
  launch_pdl(conv_norm_rope_128_kernel<NH, kConv, kAll>, dim3((p.T + p.run - 1) / p.run, cols), dim3(warps * 32),
             static_cast<size_t>(p.run) * row_bytes, st, p);
  return static_cast<int>(cudaGetLastError());
}

// Whether the kernel for heads of 128 takes this shape; -1 = it does not.
static int dispatch_conv_norm_rope_128(const ConvRope& p, cudaStream_t st) {
  const int pair = p.halves ? p.rot / 2 : p.rot;
  if (p.dim != 128 || p.maps_dim != 128 || p.vdim != 128 || pair % 4 || p.ld % 4 || p.q_off % 4 || p.k_off % 4 || p.v_off % 4 || p.state_off % 4 ||
      p.slot_stride % 4 || (p.conv_w && p.taps > 4))
    return -1;
  const int q = p.nq / 128, k = p.nk / 128, units = q + k + p.nv / 128;
  if (p.norm == 2) {
    if (p.conv_w) return -1;
    if (q % 4 == 0 && k % 4 == 0 && units <= 64) return launch_conv_norm_rope_128<4, false, true>(p, st);
    if (q % 2 == 0 && k % 2 == 0 && units <= 32) return launch_conv_norm_rope_128<2, false, true>(p, st);
    return units <= 16 ? launch_conv_norm_rope_128<1, false, true>(p, st) : -1;
  }
  const bool two = q % 2 == 0 && k % 2 == 0;
  if (p.conv_w) return two ? launch_conv_norm_rope_128<2, true, false>(p, st) : launch_conv_norm_rope_128<1, true, false>(p, st);
  return two ? launch_conv_norm_rope_128<2, false, false>(p, st) : launch_conv_norm_rope_128<1, false, false>(p, st);
}

template <typename E>
static int dispatch_conv_norm_rope(const ConvRope& p, cudaStream_t st) {
  if (sizeof(E) == 2) {
    const int rc = dispatch_conv_norm_rope_128(p, st);
    if (rc != -1) return rc;
  }
  auto fits = [&](int v) {
    const int pair = p.halves ? p.rot / 2 : p.rot;
    return p.dim % v == 0 && p.vdim % v == 0 && p.ld % v == 0 && p.q_off % v == 0 && p.k_off % v == 0 && p.v_off % v == 0 && pair % v == 0 &&
           p.state_off % 4 == 0 && p.slot_stride % 4 == 0 && (!p.v_table || (p.vdim / 2) % v == 0);
  };
  return fits(8) ? launch_conv_norm_rope<E, 8>(p, st) : fits(4) ? launch_conv_norm_rope<E, 4>(p, st) : launch_conv_norm_rope<E, 1>(p, st);
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_rope_table(const int* positions, const float* freq, void* out, int T, int half, float mag, cafd_stream_t s) {
  if (T <= 0 || half <= 0) return 0;
  const int blocks = (T * half + 255) / 256;
  launch_pdl(rope_table_kernel, dim3(blocks < 1184 ? blocks : 1184), dim3(256), 0, static_cast<cudaStream_t>(s), positions, freq,
             static_cast<float2*>(out), T, half, mag);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int cafd_conv_rope_kv(const ConvRope* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (p->dim <= 0 || p->vdim <= 0 || p->rot < 0 || p->rot % 2 || p->rot > p->dim || p->maps_dim % p->dim || p->nk != p->kv_heads * p->maps_dim ||
      p->nv != (p->v_from_k ? 0 : p->kv_heads * p->vdim) || p->nq % p->dim || p->norm < 0 || p->norm > 2)
    return -10;
  if ((p->norm && (!p->q_norm != !p->k_norm || (p->norm == 2 && !p->q_norm))) || (p->v_table && (p->vdim % 2 || p->v_from_k)) || (p->v_from_k && (p->vdim != p->dim || p->maps_dim != p->dim))) return -10;
  if (p->conv_w && (p->taps < 1 || !p->q_start || p->S < 1 || (p->taps > 1 && (!p->state || !p->state_in || !p->state_out)))) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (p->norm || p->halves || p->v_from_k || p->v_table) return is_f32 ? dispatch_conv_norm_rope<float>(*p, st) : dispatch_conv_norm_rope<__nv_bfloat16>(*p, st);
  return is_f32 ? launch_conv_rope<float>(*p, st) : launch_conv_rope<__nv_bfloat16>(*p, st);
}

extern "C" int cafd_softcap(float* x, int rows, int n, long long ld, float cap, cafd_stream_t s) {
  if (rows <= 0 || n <= 0) return 0;
  if (!(cap > 0.f)) return -10;
  launch_pdl(softcap_kernel, dim3((n + 1023) / 1024, rows), dim3(256), 0, static_cast<cudaStream_t>(s), x, n, ld, cap);
  return static_cast<int>(cudaGetLastError());
}
