// From a step's fused projection rows to queries and cached keys and values, in one launch: a causal convolution over time
// on every channel of q, k and v, rotary positions on the leading dimensions of q and k (pairs 2i, 2i + 1), the paged K / V
// write and the convolution state of every sequence.
//
//   rope_table       cos / sin of position * frequency for every token of the step, once per step and kind of rotation:
//                    every layer that rotates alike reads it
//   conv_rope_kv     eight channels per thread walking a run of tokens, the convolution's earlier inputs in registers
//   conv_rope_kv_any any head sizes and any number of taps: one channel per thread and token
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
  long long slot_stride, state_off;
  int T, S, ld, q_off, k_off, v_off, nq, nk, nv, maps_dim, dim, vdim, kv_heads, rot, taps, run;
};

__global__ void __launch_bounds__(256) rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ freq, float2* __restrict__ out,
                                                         int T, int half) {
  pdl_wait();
  pdl_trigger();
  const int n = T * half;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    const int t = i / half;
    float s, c;
    sincosf(static_cast<float>(positions[t]) * freq[i - t * half], &s, &c);
    out[i] = make_float2(c, s);
  }
}

// Where channel c of the concatenated [q | k | v] channels goes for one token; null = nowhere.
template <typename E>
__device__ __forceinline__ E* conv_rope_dest(const ConvRope& p, int t, int c) {
  if (c < p.nq) return static_cast<E*>(p.q_out) + static_cast<size_t>(t) * p.nq + c;
  const int slot = p.slots[t];
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
__device__ __forceinline__ int seq_of(const int* q_start, int S, int t) {
  int s = 0, hi = S;
  while (hi - s > 1) {
    const int mid = (s + hi) >> 1;
    if (q_start[mid] <= t) s = mid; else hi = mid;
  }
  return s;
}

template <typename E, int MAXT>
__global__ void __launch_bounds__(128) conv_rope_kv_kernel(const ConvRope p) {
  constexpr int V = 8, W = MAXT > 1 ? MAXT - 1 : 1;
  const int C = p.nq + p.nk + p.nv;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const int halo = p.conv_w ? p.taps - 1 : 0;
  float w[MAXT][V];                             // taps, oldest first, at the array's end (weights: not written by any kernel)
#pragma unroll
  for (int j = 0; j < MAXT; ++j) {
    const int tap = j - (MAXT - 1 - halo);
#pragma unroll
    for (int e = 0; e < V; ++e) w[j][e] = 0.f;
    if (p.conv_w && tap >= 0 && c < C) load_vec<float, V>(p.conv_w + static_cast<size_t>(tap) * C + c, w[j]);
  }
  pdl_wait();
  pdl_trigger();
  if (c >= C) return;
  const int r0 = blockIdx.x * p.run, r1 = min(p.T, r0 + p.run);
  if (r0 >= r1) return;
  const int col = conv_rope_col(p, c);
  const E* src = static_cast<const E*>(p.proj) + col;
  const int d0 = c < p.nq + p.nk ? (c < p.nq ? c : c - p.nq) % p.dim : p.rot;   // first dimension inside its map; v: past the rotated ones
  const bool turns = d0 < p.rot;
  float win[W][V];                              // the last taps - 1 inputs, oldest first, at the array's end
#pragma unroll
  for (int j = 0; j < W; ++j)
#pragma unroll
    for (int e = 0; e < V; ++e) win[j][e] = 0.f;
  int seq = 0, s_lo = 0, s_hi = p.T;
  if (halo > 0) {
    seq = seq_of(p.q_start, p.S, r0);
    s_lo = p.q_start[seq];
    s_hi = p.q_start[seq + 1];
  }
  // inputs before token t0 of sequence seq: rows of this step, or the sequence's state where they lie before it
  auto fill = [&](int t0) {
    const float* st = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.state_off + c;
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const int back = W - j;                   // input of token t0 - back
      if (back <= halo) {
        const int row = t0 - back;
        if (row >= s_lo) load_vec<E, V>(src + static_cast<size_t>(row) * p.ld, win[j]);
        else load_vec<float, V>(st + static_cast<size_t>(halo + row - s_lo) * C, win[j]);
      }
    }
  };
  if (halo > 0) fill(r0);
  Packed<E, V> nx = load_packed<E, V>(src + static_cast<size_t>(r0) * p.ld);
  for (int t = r0; t < r1; ++t) {
    if (halo > 0 && t == s_hi) {                // next sequence (empty ones are skipped)
      do { ++seq; s_lo = s_hi; s_hi = p.q_start[seq + 1]; } while (s_hi == s_lo && seq + 1 < p.S);
      fill(t);
    }
    float x[V], y[V];
    unpack(nx, x);
    if (t + 1 < r1) nx = load_packed<E, V>(src + static_cast<size_t>(t + 1) * p.ld);
    if (p.conv_w) {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = w[MAXT - 1][e] * x[e];
#pragma unroll
      for (int j = 0; j < MAXT - 1; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w[j][e], win[j][e], y[e]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = x[e];
    }
    if (turns) {
      const float2* cs = p.table + static_cast<size_t>(t) * (p.rot >> 1) + (d0 >> 1);
#pragma unroll
      for (int i = 0; i < V / 2; ++i) {
        if (d0 + 2 * i < p.rot) {
          const float2 k = cs[i];
          const float u = y[2 * i], v = y[2 * i + 1];
          y[2 * i] = u * k.x - v * k.y;
          y[2 * i + 1] = v * k.x + u * k.y;
        }
      }
    }
    E* dst = conv_rope_dest<E>(p, t, c);
    if (dst) store_vec<E, V>(dst, y);
    if (halo > 0) {
#pragma unroll
      for (int j = 0; j + 1 < W; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) win[j][e] = win[j + 1][e];
#pragma unroll
      for (int e = 0; e < V; ++e) win[W - 1][e] = x[e];
      if (t == s_hi - 1) {
        float* st = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off + c;
#pragma unroll
        for (int j = 0; j < W; ++j) {
          const int dst_row = j - (W - halo);
          if (dst_row >= 0) store_vec<float, V>(st + static_cast<size_t>(dst_row) * C, win[j]);
        }
      }
    }
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
    seq = seq_of(p.q_start, p.S, t);
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
  E* dst = conv_rope_dest<E>(p, t, c);
  if (dst) {
    float v[1] = {y};
    store_vec<E, 1>(dst, v);
  }
  if (halo > 0 && t == s_hi - 1) {
    float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.state_off;
    for (int j = 0; j < halo; ++j) so[static_cast<size_t>(j) * C + c] = input(t - halo + 1 + j, c);
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
  const bool vec = p.dim % 8 == 0 && p.vdim % 8 == 0 && p.ld % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 && p.v_off % 8 == 0 &&
                   p.state_off % 4 == 0 && p.slot_stride % 4 == 0 && (!p.conv_w || p.taps <= 8);
  if (!vec) {
    launch_pdl(conv_rope_kv_any_kernel<E>, dim3(p.T, (C + 255) / 256), dim3(256), 0, st, p);
    return static_cast<int>(cudaGetLastError());
  }
  const int cols = (C / 8 + 127) / 128;
  // decode: one token per block; prompts: runs long enough that re-reading their halo is cheap, blocks enough for every SM
  const int want = 148 * 12;
  int run = (p.T * cols + want - 1) / want;
  run = p.T <= 64 ? 1 : run < 4 ? 4 : run > 64 ? 64 : run;
  p.run = run;
  const dim3 grid((p.T + run - 1) / run, cols);
  if (!p.conv_w || p.taps <= 4) launch_pdl(conv_rope_kv_kernel<E, 4>, grid, dim3(128), 0, st, p);
  else launch_pdl(conv_rope_kv_kernel<E, 8>, grid, dim3(128), 0, st, p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_rope_table(const int* positions, const float* freq, void* out, int T, int half, cafd_stream_t s) {
  if (T <= 0 || half <= 0) return 0;
  const int blocks = (T * half + 255) / 256;
  launch_pdl(rope_table_kernel, dim3(blocks < 1184 ? blocks : 1184), dim3(256), 0, static_cast<cudaStream_t>(s), positions, freq,
             static_cast<float2*>(out), T, half);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int cafd_conv_rope_kv(const ConvRope* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (p->dim <= 0 || p->rot < 0 || p->rot % 2 || p->rot > p->dim || p->maps_dim % p->dim || p->nk != p->kv_heads * p->maps_dim ||
      p->nv != p->kv_heads * p->vdim || p->nq % p->dim)
    return -10;
  if (p->conv_w && (p->taps < 1 || !p->q_start || p->S < 1 || (p->taps > 1 && (!p->state || !p->state_in || !p->state_out)))) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return is_f32 ? launch_conv_rope<float>(*p, st) : launch_conv_rope<__nv_bfloat16>(*p, st);
}

extern "C" int cafd_softcap(float* x, int rows, int n, long long ld, float cap, cafd_stream_t s) {
  if (rows <= 0 || n <= 0) return 0;
  if (!(cap > 0.f)) return -10;
  launch_pdl(softcap_kernel, dim3((n + 1023) / 1024, rows), dim3(256), 0, static_cast<cudaStream_t>(s), x, n, ld, cap);
  return static_cast<int>(cudaGetLastError());
}
