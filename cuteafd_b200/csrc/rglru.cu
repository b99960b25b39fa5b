// Gated linear recurrence: u = conv(x + x_bias) + conv_bias per channel, gates r and i = sigmoid of block-diagonal products of u,
//     log a = -c r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu(y + y_bias)
//
//   rglru_conv   biases and convolution; rows leave block by block, as the grouped product of the gates reads them
//   rglru_scan   the gates' products to the output.  Short portions: one thread per channel walks a sequence's tokens.  Longer ones: a
//                block owns 16 channels and walks 256 tokens at a time, every thread 8 of them; the threads' decays and contributions
//                meet in shared memory, and each goes over its tokens again, still in registers, from the state before them
//   rglru_step   all of it in one launch for steps of up to 32 rows: a block convolves one block's channels, multiplies 16 of them
//                through both gates and walks their recurrences
//
// From the gates' products on everything is fp32, so are the convolution's inputs in the state (the projected rows with their
// bias).  A step reads one state slot and writes another.
#include "cafd_api.h"
#include "common.cuh"
#include "delta.cuh"

namespace cafd {

struct RglruArgs {
  const void* proj;           // [T, ld] E: sections x and y
  const float* y_bias;        // [width]
  const float* x_bias;        // [width]
  const float* conv_w;        // [taps, width], last row = the current token
  const float* conv_b;        // [width]
  const float* lam;           // [width]
  const void* w;              // [blocks, 2 * u_pitch, u_pitch] E: rows of r, then of i
  const float* gate_bias;     // [blocks, 2 * u_pitch]
  void* u;                    // [blocks, t_pad, u_pitch] E
  const float* gates;         // [blocks, t_pad, 2 * u_pitch]
  void* out;                  // [T, ldo] E
  float* state;               // pool, slot_stride floats per slot: [width] at s_off, [taps - 1, width] at c_off
  const int* state_in;        // [S]
  const int* state_out;       // [S]
  const int* q_start;         // [S + 1]
  long long slot_stride, s_off, c_off;
  int T, S, ld, x_off, y_off, width, blocks, taps, u_pitch, t_pad, ldo, max_q;
  float c;
};

__device__ __forceinline__ int rg_seq_of(const int* q_start, int S, int t) {
  int s = 0, hi = S;
  while (hi - s > 1) {
    const int mid = (s + hi) >> 1;
    if (q_start[mid] <= t) s = mid; else hi = mid;
  }
  return s;
}

template <typename E, int V>
__device__ __forceinline__ void rg_load(const E* q, float (&v)[V]) {
  if constexpr (V == 8) {
    const uint4 x = *reinterpret_cast<const uint4*>(q);
    const uint32_t w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) { v[2 * e] = bf16_lo(w[e]); v[2 * e + 1] = bf16_hi(w[e]); }
  } else if constexpr (V == 4) {
    de_load4(q, v);
  } else {
    v[0] = de_f<E>(*q);
  }
}
template <int V>
__device__ __forceinline__ void rg_loadf(const float* q, float (&v)[V]) {
  if constexpr (V >= 4) {
#pragma unroll
    for (int e = 0; e < V; e += 4) {
      const float4 x = *reinterpret_cast<const float4*>(q + e);
      v[e] = x.x; v[e + 1] = x.y; v[e + 2] = x.z; v[e + 3] = x.w;
    }
  } else {
    v[0] = *q;
  }
}
template <typename E, int V>
__device__ __forceinline__ void rg_store(E* q, const float (&v)[V]) {
  if constexpr (V == 8) *reinterpret_cast<uint4*>(q) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  else if constexpr (V == 4) de_store4(q, v);
  else q[0] = de_e<E>(v[0]);
}

// V channels per thread, blockIdx.y = run of tokens.
template <typename E, int V>
__global__ void __launch_bounds__(128) rglru_conv_kernel(const RglruArgs p, int run) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  pdl_wait();
  pdl_trigger();
  if (c >= p.width) return;
  const int t0 = blockIdx.y * run, t1 = min(p.T, t0 + run), halo = p.taps - 1, bs = p.width / p.blocks;
  int seq = rg_seq_of(p.q_start, p.S, t0), s_lo = p.q_start[seq], s_hi = p.q_start[seq + 1];
  const E* src = static_cast<const E*>(p.proj) + p.x_off + c;
  const int b = c / bs;
  E* dst = static_cast<E*>(p.u) + (static_cast<size_t>(b) * p.t_pad) * p.u_pitch + (c - b * bs);
  float xb[V], cb[V];
  rg_loadf<V>(p.x_bias + c, xb);
  rg_loadf<V>(p.conv_b + c, cb);
  auto input = [&](int row, float (&v)[V]) {     // the convolution's input at row, which may lie before this step
    if (row >= s_lo) {
      rg_load<E, V>(src + static_cast<size_t>(row) * p.ld, v);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += xb[e];
    } else {
      rg_loadf<V>(p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.c_off + c + static_cast<size_t>(halo + row - s_lo) * p.width, v);
    }
  };
  constexpr int kTaps = 4;
  if (p.taps <= kTaps) {                         // earlier inputs in registers, a batch of rows on its way
    constexpr int W = kTaps - 1, kBatch = 4;
    float w[kTaps][V], x[W + kBatch][V];         // w[k]: weight of the input k tokens back
#pragma unroll
    for (int k = 0; k < kTaps; ++k) {
#pragma unroll
      for (int e = 0; e < V; ++e) w[k][e] = 0.f;
      if (k <= halo) rg_loadf<V>(p.conv_w + static_cast<size_t>(halo - k) * p.width + c, w[k]);
    }
#pragma unroll
    for (int i = 0; i < W; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = 0.f;
    for (int t = t0; t < t1; t += kBatch) {
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        rg_load<E, V>(src + static_cast<size_t>(min(t + j, t1 - 1)) * p.ld, x[W + j]);
#pragma unroll
        for (int e = 0; e < V; ++e) x[W + j][e] += xb[e];
      }
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        const int row = t + j;
        if (row >= t1) break;
        if (row == t0 || row == s_hi) {          // the inputs before a run's or a sequence's first token
          while (row == s_hi && seq + 1 < p.S) { ++seq; s_lo = s_hi; s_hi = p.q_start[seq + 1]; }
#pragma unroll
          for (int k = 1; k < kTaps; ++k)
            if (k <= halo) input(row - k, x[W + j - k]);
        }
        float u[V];
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = cb[e];
#pragma unroll
        for (int k = W; k >= 0; --k) {
          if (k <= halo) {                       // (past the taps there may be another sequence's inputs)
#pragma unroll
            for (int e = 0; e < V; ++e) u[e] = fmaf(w[k][e], x[W + j - k][e], u[e]);
          }
        }
        rg_store<E, V>(dst + static_cast<size_t>(row) * p.u_pitch, u);
        if (row == s_hi - 1) {                   // the sequence's last halo inputs, oldest first
          float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.c_off + c;
#pragma unroll
          for (int k = 0; k < W; ++k)
            if (k < halo) {
#pragma unroll
              for (int e = 0; e < V; ++e) so[static_cast<size_t>(halo - 1 - k) * p.width + e] = x[W + j - k][e];
            }
        }
      }
#pragma unroll
      for (int i = 0; i < W; ++i)
#pragma unroll
        for (int e = 0; e < V; ++e) x[i][e] = x[kBatch + i][e];
    }
    return;
  }
  for (int t = t0; t < t1; ++t) {
    while (t == s_hi && seq + 1 < p.S) { ++seq; s_lo = s_hi; s_hi = p.q_start[seq + 1]; }
    float u[V];
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = cb[e];
    for (int j = 0; j <= halo; ++j) {
      float x[V], w[V];
      input(t - halo + j, x);
      rg_loadf<V>(p.conv_w + static_cast<size_t>(j) * p.width + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] = fmaf(w[e], x[e], u[e]);
    }
    rg_store<E, V>(dst + static_cast<size_t>(t) * p.u_pitch, u);
    if (t == s_hi - 1) {
      float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.c_off + c;
      for (int j = 0; j < halo; ++j) {
        float x[V];
        input(t - halo + 1 + j, x);
#pragma unroll
        for (int e = 0; e < V; ++e) so[static_cast<size_t>(j) * p.width + e] = x[e];
      }
    }
  }
}

// One token of one channel: a and sqrt(1 - a^2) i u out of the gates' products.  bf16 engines take the special-function unit's
// exponentials and quotients; 1 - a^2 is a series while a is near one, where the difference would cancel.
template <typename E>
__device__ __forceinline__ void rg_gate(float r, float i, float u, float rate, float& a, float& x) {
  if constexpr (sizeof(E) == 4) {
    const float log_a = rate * sigmoid_f(r);
    a = expf(log_a);
    x = sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i) * u;
  } else {
    const float log_a = __fdividef(rate, 1.0f + __expf(fminf(-r, 80.f)));
    a = __expf(log_a);
    const float y = -2.f * log_a;               // 1 - e^-y = y (1 - y / 2 (1 - y / 3 (1 - ...)))
    const float near = y * (1.f - y * (1.f / 2) * (1.f - y * (1.f / 3) * (1.f - y * (1.f / 4) * (1.f - y * (1.f / 5) * (1.f - y * (1.f / 6))))));
    const float rest = y < 0.25f ? near : fmaf(-a, a, 1.f);
    float root;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(root) : "f"(rest));
    x = __fdividef(root * u, 1.0f + __expf(fminf(-i, 80.f)));
  }
}
template <typename E>
__device__ __forceinline__ float gelu_tanh(float z) {
  const float y = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return 0.5f * z * (1.0f + (sizeof(E) == 4 ? tanhf(y) : tanh_exp2(2.f * 1.4426950408889634f * y)));
}

constexpr int kScanThreads = 64, kScanBatch = 4;

// A thread per channel, blockIdx.y = sequence.
template <typename E>
__global__ void __launch_bounds__(kScanThreads) rglru_scan_kernel(const RglruArgs p) {
  const int c = blockIdx.x * kScanThreads + threadIdx.x, seq = blockIdx.y;
  const bool on = c < p.width;
  const int cc = on ? c : 0, bs = p.width / p.blocks, b = cc / bs, d = cc - b * bs;
  const float rb = p.gate_bias[b * 2 * p.u_pitch + d], ib = p.gate_bias[b * 2 * p.u_pitch + p.u_pitch + d], yb = p.y_bias[cc];
  const float rate = -p.c * softplus(p.lam[cc]);
  pdl_wait();
  pdl_trigger();
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t0 >= t1 || !on) return;
  float S = p.state[static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.s_off + c];
  const float* gr = p.gates + static_cast<size_t>(b) * p.t_pad * 2 * p.u_pitch + d;
  const E* us = static_cast<const E*>(p.u) + static_cast<size_t>(b) * p.t_pad * p.u_pitch + d;
  const E* ys = static_cast<const E*>(p.proj) + p.y_off + c;
  float r[kScanBatch], i[kScanBatch], u[kScanBatch], y[kScanBatch];
  auto fetch = [&](int t) {
#pragma unroll
    for (int j = 0; j < kScanBatch; ++j) {
      const size_t tt = min(t + j, t1 - 1);
      r[j] = gr[tt * 2 * p.u_pitch];
      i[j] = gr[tt * 2 * p.u_pitch + p.u_pitch];
      u[j] = de_f<E>(us[tt * p.u_pitch]);
      y[j] = de_f<E>(ys[tt * p.ld]);
    }
  };
  fetch(t0);
  for (int t = t0; t < t1; t += kScanBatch) {
    float a[kScanBatch], x[kScanBatch], g[kScanBatch];
#pragma unroll
    for (int j = 0; j < kScanBatch; ++j) {
      rg_gate<E>(r[j] + rb, i[j] + ib, u[j], rate, a[j], x[j]);
      g[j] = gelu_tanh<E>(y[j] + yb);
    }
    if (t + kScanBatch < t1) fetch(t + kScanBatch);
#pragma unroll
    for (int j = 0; j < kScanBatch; ++j) {
      if (t + j >= t1) break;
      S = fmaf(a[j], S, x[j]);
      static_cast<E*>(p.out)[static_cast<size_t>(t + j) * p.ldo + c] = de_e<E>(S * g[j]);
    }
  }
  p.state[static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.s_off + c] = S;
}

constexpr int kWalkChans = 16, kWalkSubs = 32, kWalkTok = 8, kWalk = kWalkSubs * kWalkTok, kWalkThreads = kWalkChans * kWalkSubs;

// Long portions: thread (channel, run of 8 of the 256 tokens the block is at).
template <typename E>
__global__ void __launch_bounds__(kWalkThreads) rglru_walk_kernel(const RglruArgs p) {
  __shared__ float2 part[2][kWalkSubs][kWalkChans];
  __shared__ float carry[2][kWalkChans];
  const int ch = threadIdx.x & (kWalkChans - 1), sub = threadIdx.x / kWalkChans, seq = blockIdx.y;
  const int c = blockIdx.x * kWalkChans + ch;
  const bool on = c < p.width;
  const int cc = on ? c : 0, bs = p.width / p.blocks, b = cc / bs, d = cc - b * bs;
  const float rb = p.gate_bias[b * 2 * p.u_pitch + d], ib = p.gate_bias[b * 2 * p.u_pitch + p.u_pitch + d], yb = p.y_bias[cc];
  const float rate = -p.c * softplus(p.lam[cc]);
  pdl_wait();
  pdl_trigger();
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  if (t0 >= t1) return;
  if (sub == 0) carry[0][ch] = p.state[static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.s_off + cc];
  const float* gr = p.gates + static_cast<size_t>(b) * p.t_pad * 2 * p.u_pitch + d;
  const E* us = static_cast<const E*>(p.u) + static_cast<size_t>(b) * p.t_pad * p.u_pitch + d;
  const E* ys = static_cast<const E*>(p.proj) + p.y_off + cc;
  float r[kWalkTok], i[kWalkTok];
  E u[kWalkTok], y[kWalkTok];
  auto fetch = [&](int t) {
#pragma unroll
    for (int j = 0; j < kWalkTok; ++j) {
      const size_t tt = min(t + sub * kWalkTok + j, t1 - 1);
      r[j] = gr[tt * 2 * p.u_pitch];
      i[j] = gr[tt * 2 * p.u_pitch + p.u_pitch];
      u[j] = us[tt * p.u_pitch];
      y[j] = ys[tt * p.ld];
    }
  };
  fetch(t0);
  int buf = 0;
  for (int t = t0; t < t1; t += kWalk, buf ^= 1) {
    const int mine = t + sub * kWalkTok;
    float a[kWalkTok], x[kWalkTok], g[kWalkTok], A = 1.f, B = 0.f;
#pragma unroll
    for (int j = 0; j < kWalkTok; ++j) {
      rg_gate<E>(r[j] + rb, i[j] + ib, de_f<E>(u[j]), rate, a[j], x[j]);
      if (mine + j >= t1) { a[j] = 1.f; x[j] = 0.f; }          // past the end the state stays as it is
      A *= a[j];
      B = fmaf(a[j], B, x[j]);
      g[j] = gelu_tanh<E>(de_f<E>(y[j]) + yb);
    }
    if (t + kWalk < t1) fetch(t + kWalk);
    part[buf][sub][ch] = make_float2(A, B);
    __syncthreads();
    float S = carry[buf][ch];
#pragma unroll
    for (int k = 0; k < kWalkSubs - 1; ++k) {
      const float2 q = part[buf][k][ch];
      if (k < sub) S = fmaf(q.x, S, q.y);
    }
#pragma unroll
    for (int j = 0; j < kWalkTok; ++j) {
      S = fmaf(a[j], S, x[j]);
      if (on && mine + j < t1) static_cast<E*>(p.out)[static_cast<size_t>(mine + j) * p.ldo + c] = de_e<E>(S * g[j]);
    }
    if (sub == kWalkSubs - 1) {
      carry[buf ^ 1][ch] = S;
      if (on && t + kWalk >= t1) p.state[static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.s_off + c] = S;
    }
  }
}

constexpr int kStepRows = 32, kStepChans = 16, kStepThreads = 256;

// Block (block of channels, 16 of its channels).  u of every row in shared memory; thread (gate row, every eighth token) for the products.
template <typename E, int V>
__global__ void __launch_bounds__(kStepThreads) rglru_step_kernel(const RglruArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kTok = kStepRows / 8, kSeqs = kStepRows * kStepChans / kStepThreads;
  const int tid = threadIdx.x, b = blockIdx.x, d0 = blockIdx.y * kStepChans, bs = p.width / p.blocks, kp = p.u_pitch, pitch = kp + 4;
  const int nd = min(kStepChans, bs - d0), halo = p.taps - 1;
  float* su = sm;                                // [T][pitch], as the products read it
  float* sg = su + p.T * pitch;                  // [2][16][T + 1]
  int* s_seq = reinterpret_cast<int*>(sg + 2 * kStepChans * (p.T + 1));   // [T] sequence, [T] its first row, [T] the slot it reads
  E* sw = reinterpret_cast<E*>(s_seq + (3 * p.T + 3) / 4 * 4);            // [32][kp + 8]
  constexpr int kV = 16 / static_cast<int>(sizeof(E));
  // the weights do not depend on anything before this launch
  const E* w = static_cast<const E*>(p.w) + static_cast<size_t>(b) * 2 * kp * kp;
  for (int i = tid; i < 2 * kStepChans * (kp / kV); i += kStepThreads) {
    const int r = i / (kp / kV), c = (i - r * (kp / kV)) * kV, g = r / kStepChans, d = r - g * kStepChans;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (d < nd) x = *reinterpret_cast<const uint4*>(w + static_cast<size_t>(g * kp + d0 + d) * kp + c);
    *reinterpret_cast<uint4*>(sw + r * (kp + 8) + c) = x;
  }
  const int d = tid & (kStepChans - 1), sg0 = tid / kStepChans;           // channel and first sequence of the recurrence
  const int c = b * bs + d0 + min(d, nd - 1);
  const float rate = -p.c * softplus(p.lam[c]), yb = p.y_bias[c];
  pdl_wait();
  pdl_trigger();
  for (int t = tid; t < p.T; t += kStepThreads) {
    const int s = rg_seq_of(p.q_start, p.S, t);
    s_seq[t] = s;
    s_seq[p.T + t] = p.q_start[s];
    s_seq[2 * p.T + t] = p.state_in[s];
  }
  float S0[kSeqs];                               // the states this thread starts from are on their way during the products
#pragma unroll
  for (int k = 0; k < kSeqs; ++k) {
    const int s = sg0 + k * (kStepThreads / kStepChans);
    S0[k] = s < p.S ? p.state[static_cast<size_t>(p.state_in[s]) * p.slot_stride + p.s_off + c] : 0.f;
  }
  __syncthreads();
  const E* proj = static_cast<const E*>(p.proj);
  auto input = [&](int row, int slot, int s_lo, int cc, auto& v) {        // the convolution's input at row, which may lie before this step
    constexpr int kN = sizeof(v) / 4;
    if (row >= s_lo) {
      float xb[kN];
      rg_load<E, kN>(proj + static_cast<size_t>(row) * p.ld + p.x_off + cc, v);
      rg_loadf<kN>(p.x_bias + cc, xb);
#pragma unroll
      for (int e = 0; e < kN; ++e) v[e] += xb[e];
    } else {
      rg_loadf<kN>(p.state + static_cast<size_t>(slot) * p.slot_stride + p.c_off + static_cast<size_t>(halo + row - s_lo) * p.width + cc, v);
    }
  };
  const int vecs = kp / V;                       // (the padding behind a block's channels is less than a vector of 8)
  for (int i = tid; i < p.T * vecs; i += kStepThreads) {
    const int t = i / vecs, dd = (i - t * vecs) * V, cc = b * bs + dd;
    float u[V];
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
    if (dd < bs) {
      const int s_lo = s_seq[p.T + t], slot = s_seq[2 * p.T + t];
      rg_loadf<V>(p.conv_b + cc, u);
#pragma unroll 4
      for (int j = 0; j <= halo; ++j) {
        float x[V], cw[V];
        input(t - halo + j, slot, s_lo, cc, x);
        rg_loadf<V>(p.conv_w + static_cast<size_t>(j) * p.width + cc, cw);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = fmaf(cw[e], x[e], u[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) su[t * pitch + dd + e] = de_f<E>(de_e<E>(u[e]));
  }
  __syncthreads();
  {
    const int r = tid >> 3, t0 = tid & 7;
    float acc[kTok];
#pragma unroll
    for (int j = 0; j < kTok; ++j) acc[j] = 0.f;
    const E* wr = sw + r * (kp + 8);
    const int g = r / kStepChans, dd = r - g * kStepChans;
    const float bias = dd < nd ? p.gate_bias[static_cast<size_t>(b) * 2 * kp + g * kp + d0 + dd] : 0.f;
#pragma unroll 4
    for (int k = 0; k < kp; k += 4) {
      float wv[4];
      de_load4(wr + k, wv);
#pragma unroll
      for (int j = 0; j < kTok; ++j) {
        const int t = t0 + 8 * j;
        if (t < p.T) {
          const float4 x = *reinterpret_cast<const float4*>(su + t * pitch + k);
          acc[j] = fmaf(wv[0], x.x, fmaf(wv[1], x.y, fmaf(wv[2], x.z, fmaf(wv[3], x.w, acc[j]))));
        }
      }
    }
#pragma unroll
    for (int j = 0; j < kTok; ++j)
      if (t0 + 8 * j < p.T) sg[r * (p.T + 1) + t0 + 8 * j] = acc[j] + bias;
  }
  __syncthreads();
  if (d >= nd) return;
#pragma unroll
  for (int k = 0; k < kSeqs; ++k) {
    const int s = sg0 + k * (kStepThreads / kStepChans);
    if (s >= p.S) break;
    const int q0 = p.q_start[s], q1 = p.q_start[s + 1];
    if (q0 >= q1) continue;
    float* so = p.state + static_cast<size_t>(p.state_out[s]) * p.slot_stride;
    const int slot = p.state_in[s];
    float S = S0[k];
    for (int t = q0; t < q1; ++t) {
      float a, x;
      rg_gate<E>(sg[d * (p.T + 1) + t], sg[(kStepChans + d) * (p.T + 1) + t], su[t * pitch + d0 + d], rate, a, x);
      S = fmaf(a, S, x);
      static_cast<E*>(p.out)[static_cast<size_t>(t) * p.ldo + c] =
          de_e<E>(S * gelu_tanh<E>(de_f<E>(proj[static_cast<size_t>(t) * p.ld + p.y_off + c]) + yb));
    }
    so[p.s_off + c] = S;
    for (int j = 0; j < halo; ++j) {
      float x[1];
      input(q1 - halo + j, slot, q0, c, x);
      so[p.c_off + static_cast<size_t>(j) * p.width + c] = x[0];
    }
  }
}

template <typename E>
static size_t rglru_step_smem(int T, int u_pitch) {
  return static_cast<size_t>(T * (u_pitch + 4) + 2 * kStepChans * (T + 1) + (3 * T + 3) / 4 * 4) * 4 + static_cast<size_t>(2 * kStepChans) * (u_pitch + 8) * sizeof(E);
}

template <typename E, int V>
static int launch_rglru_step(const RglruArgs& p, cudaStream_t st) {
  const size_t smem = rglru_step_smem<E>(p.T, p.u_pitch);
  if (p.T > kStepRows || p.S > kStepRows || p.u_pitch % 8 || smem > 200 * 1024) return -12;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(rglru_step_kernel<E, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  launch_pdl(rglru_step_kernel<E, V>, dim3(p.blocks, (p.width / p.blocks + kStepChans - 1) / kStepChans), dim3(kStepThreads), smem, st, p);
  return static_cast<int>(cudaGetLastError());
}

// Channels that a thread may move together: vectors inside a block of channels, on their boundaries everywhere.
static bool rglru_vec(const RglruArgs& p, int v) {
  return p.width / p.blocks % v == 0 && p.ld % v == 0 && p.x_off % v == 0 && p.u_pitch % v == 0 && p.slot_stride % 4 == 0 && p.c_off % 4 == 0;
}

template <typename E>
static int launch_rglru_scan(const RglruArgs& p, cudaStream_t st) {
  if (p.max_q <= 32) launch_pdl(rglru_scan_kernel<E>, dim3((p.width + kScanThreads - 1) / kScanThreads, p.S), dim3(kScanThreads), 0, st, p);
  else launch_pdl(rglru_walk_kernel<E>, dim3((p.width + kWalkChans - 1) / kWalkChans, p.S), dim3(kWalkThreads), 0, st, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename E>
static int launch_rglru_conv(const RglruArgs& p, cudaStream_t st) {
  constexpr int kMax = sizeof(E) == 2 ? 8 : 4;
  const int v = p.T > 64 && kMax == 8 && rglru_vec(p, 8) ? 8 : rglru_vec(p, 4) ? 4 : 1;
  const int cols = (p.width + 128 * v - 1) / (128 * v);
  int run = (p.T * cols + 148 * 6 - 1) / (148 * 6);
  run = p.T <= 64 ? 1 : run < 4 ? 4 : run > 32 ? 32 : run;
  const dim3 grid(cols, (p.T + run - 1) / run);
  if (v == 8) launch_pdl(rglru_conv_kernel<E, kMax>, grid, dim3(128), 0, st, p, run);
  else if (v == 4) launch_pdl(rglru_conv_kernel<E, 4>, grid, dim3(128), 0, st, p, run);
  else launch_pdl(rglru_conv_kernel<E, 1>, grid, dim3(128), 0, st, p, run);
  return static_cast<int>(cudaGetLastError());
}

static bool rglru_args_ok(const RglruArgs& p) {
  return p.S >= 1 && p.blocks >= 1 && p.width >= 1 && p.width % p.blocks == 0 && p.taps >= 1 && p.u_pitch >= p.width / p.blocks && p.t_pad >= p.T &&
         p.ldo >= p.width && p.proj && p.u && p.state && p.state_in && p.state_out && p.q_start;
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_rglru_conv(const RglruArgs* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (!rglru_args_ok(*p)) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return is_f32 ? launch_rglru_conv<float>(*p, st) : launch_rglru_conv<__nv_bfloat16>(*p, st);
}

// max_q: the longest portion of the step.
extern "C" int cafd_rglru_scan(const RglruArgs* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (!rglru_args_ok(*p) || !p->gates || !p->out || p->max_q < 1) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return is_f32 ? launch_rglru_scan<float>(*p, st) : launch_rglru_scan<__nv_bfloat16>(*p, st);
}

// Steps of up to 32 rows: convolution, gates and recurrence in one launch (u and gates are not used).
extern "C" int cafd_rglru_step(const RglruArgs* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (!rglru_args_ok(*p) || !p->w || !p->gate_bias || !p->out) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (!rglru_vec(*p, 4)) return is_f32 ? launch_rglru_step<float, 1>(*p, st) : launch_rglru_step<__nv_bfloat16, 1>(*p, st);
  return is_f32 ? launch_rglru_step<float, 4>(*p, st) : launch_rglru_step<__nv_bfloat16, 4>(*p, st);
}

// Whether cafd_rglru_step takes a step of T rows in blocks of u_pitch (padded) channels.
extern "C" int cafd_rglru_step_ok(int T, int u_pitch, int is_f32) {
  return T <= kStepRows && u_pitch % 8 == 0 && (is_f32 ? rglru_step_smem<float>(T, u_pitch) : rglru_step_smem<__nv_bfloat16>(T, u_pitch)) <= 200 * 1024;
}
