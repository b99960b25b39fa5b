// Gated linear recurrence: u = conv(x + x_bias) + conv_bias per channel, gates r and i = sigmoid of block-diagonal products of u,
//     log a = -c r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu(y + y_bias)
//
//   rglru_conv   biases and convolution; rows leave block by block, as the grouped product of the gates reads them
//   rglru_scan   the gates' products to the output.  One thread per channel walks a sequence's tokens; long portions are cut into
//                chunks: every chunk's decay and contribution first, then every chunk again from the state that the chunks before it
//                give
//   rglru_step   all of it in one launch for steps of up to 32 rows: a block convolves one block's channels, multiplies 32 of them
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
  float* carry;               // [S * chunks, 2, width] (long portions)
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
  auto vec = [&](const float* q, float (&v)[V]) {
    if constexpr (V == 4) de_load4(q, v); else v[0] = *q;
  };
  float xb[V], cb[V];
  vec(p.x_bias + c, xb);
  vec(p.conv_b + c, cb);
  for (int t = t0; t < t1; ++t) {
    while (t == s_hi && seq + 1 < p.S) { ++seq; s_lo = s_hi; s_hi = p.q_start[seq + 1]; }
    const float* st = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.c_off + c;
    auto input = [&](int row, float (&v)[V]) {   // the convolution's input at row, which may lie before this step
      if (row >= s_lo) {
        if constexpr (V == 4) de_load4(src + static_cast<size_t>(row) * p.ld, v); else v[0] = de_f<E>(src[static_cast<size_t>(row) * p.ld]);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] += xb[e];
      } else {
        vec(st + static_cast<size_t>(halo + row - s_lo) * p.width, v);
      }
    };
    float u[V];
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = cb[e];
    for (int j = 0; j <= halo; ++j) {
      float x[V], w[V];
      input(t - halo + j, x);
      vec(p.conv_w + static_cast<size_t>(j) * p.width + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] = fmaf(w[e], x[e], u[e]);
    }
    if constexpr (V == 4) de_store4(dst + static_cast<size_t>(t) * p.u_pitch, u); else dst[static_cast<size_t>(t) * p.u_pitch] = de_e<E>(u[0]);
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

__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

constexpr int kScanChunk = 128, kScanThreads = 64, kScanBatch = 4;

enum ScanPart { kScanWhole, kScanSummary, kScanApply };

// blockIdx.y: the sequence, or sequence and chunk.
template <typename E, int kPart>
__global__ void __launch_bounds__(kScanThreads) rglru_scan_kernel(const RglruArgs p, int chunks) {
  const int c = blockIdx.x * kScanThreads + threadIdx.x;
  const int seq = kPart == kScanWhole ? blockIdx.y : blockIdx.y / chunks, chunk = kPart == kScanWhole ? 0 : blockIdx.y - seq * chunks;
  const bool on = c < p.width;
  const int cc = on ? c : 0, bs = p.width / p.blocks, b = cc / bs, d = cc - b * bs;
  const float rb = p.gate_bias[b * 2 * p.u_pitch + d], ib = p.gate_bias[b * 2 * p.u_pitch + p.u_pitch + d], yb = p.y_bias[cc];
  const float rate = -p.c * softplus(p.lam[cc]);
  pdl_wait();
  pdl_trigger();
  const int q0 = p.q_start[seq], q1 = p.q_start[seq + 1];
  const int t0 = kPart == kScanWhole ? q0 : q0 + chunk * kScanChunk, t1 = kPart == kScanWhole ? q1 : min(q1, t0 + kScanChunk);
  if (t0 >= t1 || !on) return;
  float S = 0.f, A = 1.f;
  if (kPart != kScanSummary) {
    S = p.state[static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.s_off + c];
    if (kPart == kScanApply) {
      const float* cr = p.carry + static_cast<size_t>(seq) * chunks * 2 * p.width + c;
#pragma unroll 4
      for (int j = 0; j < chunk; ++j) S = fmaf(cr[static_cast<size_t>(2 * j) * p.width], S, cr[static_cast<size_t>(2 * j + 1) * p.width]);
    }
  }
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
      if (kPart != kScanSummary) y[j] = de_f<E>(ys[tt * p.ld]);
    }
  };
  fetch(t0);
  for (int t = t0; t < t1; t += kScanBatch) {
    float a[kScanBatch], x[kScanBatch], g[kScanBatch];
#pragma unroll
    for (int j = 0; j < kScanBatch; ++j) {
      const float log_a = rate * sigmoid_f(r[j] + rb);
      a[j] = expf(log_a);
      x[j] = sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i[j] + ib) * u[j];
      if (kPart != kScanSummary) g[j] = gelu_tanh(y[j] + yb);
    }
    if (t + kScanBatch < t1) fetch(t + kScanBatch);
#pragma unroll
    for (int j = 0; j < kScanBatch; ++j) {
      if (t + j >= t1) break;
      S = fmaf(a[j], S, x[j]);
      A *= a[j];
      if (kPart != kScanSummary) static_cast<E*>(p.out)[static_cast<size_t>(t + j) * p.ldo + c] = de_e<E>(S * g[j]);
    }
  }
  if (kPart == kScanSummary) {
    float* cr = p.carry + (static_cast<size_t>(seq) * chunks + chunk) * 2 * p.width + c;
    cr[0] = A;
    cr[p.width] = S;
  } else if (t1 == q1) {
    p.state[static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.s_off + c] = S;
  }
}

constexpr int kStepRows = 32, kStepChans = 32, kStepThreads = 256;

// Block (block of channels, 32 of its channels).  u of every row in shared memory; thread (gate row, every fourth token) for the products.
template <typename E>
__global__ void __launch_bounds__(kStepThreads) rglru_step_kernel(const RglruArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kTok = kStepRows / 4;
  const int tid = threadIdx.x, b = blockIdx.x, d0 = blockIdx.y * kStepChans, bs = p.width / p.blocks, kp = p.u_pitch, pitch = kp + 4;
  const int nd = min(kStepChans, bs - d0), halo = p.taps - 1;
  float* su = sm;                                // [T][pitch], as the products read it
  float* sg = su + p.T * pitch;                  // [2][32][T + 1]
  int* s_seq = reinterpret_cast<int*>(sg + 2 * kStepChans * (p.T + 1));   // [T] sequence, [T] its first row
  E* sw = reinterpret_cast<E*>(s_seq + (2 * p.T + 3) / 4 * 4);            // [64][kp + 8]
  constexpr int kV = 16 / static_cast<int>(sizeof(E));
  // the weights do not depend on anything before this launch
  const E* w = static_cast<const E*>(p.w) + static_cast<size_t>(b) * 2 * kp * kp;
  for (int i = tid; i < 2 * kStepChans * (kp / kV); i += kStepThreads) {
    const int r = i / (kp / kV), c = (i - r * (kp / kV)) * kV, g = r / kStepChans, d = r - g * kStepChans;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (d < nd) x = *reinterpret_cast<const uint4*>(w + static_cast<size_t>(g * kp + d0 + d) * kp + c);
    *reinterpret_cast<uint4*>(sw + r * (kp + 8) + c) = x;
  }
  pdl_wait();
  pdl_trigger();
  for (int t = tid; t < p.T; t += kStepThreads) {
    const int s = rg_seq_of(p.q_start, p.S, t);
    s_seq[t] = s;
    s_seq[p.T + t] = p.q_start[s];
  }
  __syncthreads();
  const E* proj = static_cast<const E*>(p.proj);
  auto input = [&](int row, int s, int s_lo, int c) {   // the convolution's input at row, which may lie before this step
    return row >= s_lo ? de_f<E>(proj[static_cast<size_t>(row) * p.ld + p.x_off + c]) + p.x_bias[c]
                       : p.state[static_cast<size_t>(p.state_in[s]) * p.slot_stride + p.c_off + static_cast<size_t>(halo + row - s_lo) * p.width + c];
  };
  for (int i = tid; i < p.T * kp; i += kStepThreads) {
    const int t = i / kp, d = i - t * kp;
    float u = 0.f;
    if (d < bs) {
      const int c = b * bs + d, s = s_seq[t], s_lo = s_seq[p.T + t];
      u = p.conv_b[c];
#pragma unroll 4
      for (int j = 0; j <= halo; ++j) u = fmaf(p.conv_w[static_cast<size_t>(j) * p.width + c], input(t - halo + j, s, s_lo, c), u);
    }
    su[t * pitch + d] = de_f<E>(de_e<E>(u));
  }
  __syncthreads();
  {
    const int r = tid >> 2, t0 = tid & 3;
    float acc[kTok];
#pragma unroll
    for (int j = 0; j < kTok; ++j) acc[j] = 0.f;
    const E* wr = sw + r * (kp + 8);
    for (int k = 0; k < kp; k += 4) {
      float wv[4];
      de_load4(wr + k, wv);
#pragma unroll
      for (int j = 0; j < kTok; ++j) {
        const int t = t0 + 4 * j;
        if (t < p.T) {
          const float4 x = *reinterpret_cast<const float4*>(su + t * pitch + k);
          acc[j] = fmaf(wv[0], x.x, fmaf(wv[1], x.y, fmaf(wv[2], x.z, fmaf(wv[3], x.w, acc[j]))));
        }
      }
    }
    const int g = r / kStepChans, d = r - g * kStepChans;
    const float bias = d < nd ? p.gate_bias[static_cast<size_t>(b) * 2 * kp + g * kp + d0 + d] : 0.f;
#pragma unroll
    for (int j = 0; j < kTok; ++j)
      if (t0 + 4 * j < p.T) sg[r * (p.T + 1) + t0 + 4 * j] = sigmoid_f(acc[j] + bias);
  }
  __syncthreads();
  const int d = tid & (kStepChans - 1);
  if (d >= nd) return;
  const int c = b * bs + d0 + d;
  const float rate = -p.c * softplus(p.lam[c]), yb = p.y_bias[c];
  for (int s = tid / kStepChans; s < p.S; s += kStepThreads / kStepChans) {
    const int q0 = p.q_start[s], q1 = p.q_start[s + 1];
    if (q0 >= q1) continue;
    float* so = p.state + static_cast<size_t>(p.state_out[s]) * p.slot_stride;
    float S = p.state[static_cast<size_t>(p.state_in[s]) * p.slot_stride + p.s_off + c];
    for (int t = q0; t < q1; ++t) {
      const float log_a = rate * sg[d * (p.T + 1) + t];
      const float x = sqrtf(-expm1f(2.f * log_a)) * sg[(kStepChans + d) * (p.T + 1) + t] * su[t * pitch + d0 + d];
      S = fmaf(expf(log_a), S, x);
      static_cast<E*>(p.out)[static_cast<size_t>(t) * p.ldo + c] = de_e<E>(S * gelu_tanh(de_f<E>(proj[static_cast<size_t>(t) * p.ld + p.y_off + c]) + yb));
    }
    so[p.s_off + c] = S;
    for (int j = 0; j < halo; ++j) so[p.c_off + static_cast<size_t>(j) * p.width + c] = input(q1 - halo + j, s, q0, c);
  }
}

template <typename E>
static size_t rglru_step_smem(int T, int u_pitch) {
  return static_cast<size_t>(T * (u_pitch + 4) + 2 * kStepChans * (T + 1) + (2 * T + 3) / 4 * 4) * 4 + static_cast<size_t>(2 * kStepChans) * (u_pitch + 8) * sizeof(E);
}

template <typename E>
static int launch_rglru_step(const RglruArgs& p, cudaStream_t st) {
  const size_t smem = rglru_step_smem<E>(p.T, p.u_pitch);
  if (p.T > kStepRows || p.u_pitch % 8 || smem > 200 * 1024) return -12;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(rglru_step_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr = true;
  }
  launch_pdl(rglru_step_kernel<E>, dim3(p.blocks, (p.width / p.blocks + kStepChans - 1) / kStepChans), dim3(kStepThreads), smem, st, p);
  return static_cast<int>(cudaGetLastError());
}

template <typename E>
static int launch_rglru_scan(const RglruArgs& p, cudaStream_t st) {
  const int cols = (p.width + kScanThreads - 1) / kScanThreads, chunks = (p.max_q + kScanChunk - 1) / kScanChunk;
  if (chunks <= 1) {
    launch_pdl(rglru_scan_kernel<E, kScanWhole>, dim3(cols, p.S), dim3(kScanThreads), 0, st, p, 1);
  } else {
    if (!p.carry) return -12;
    launch_pdl(rglru_scan_kernel<E, kScanSummary>, dim3(cols, p.S * chunks), dim3(kScanThreads), 0, st, p, chunks);
    launch_pdl(rglru_scan_kernel<E, kScanApply>, dim3(cols, p.S * chunks), dim3(kScanThreads), 0, st, p, chunks);
  }
  return static_cast<int>(cudaGetLastError());
}

template <typename E>
static int launch_rglru_conv(const RglruArgs& p, cudaStream_t st) {
  const int bs = p.width / p.blocks, run = p.T <= 256 ? 1 : 4;
  const bool vec = bs % 4 == 0 && p.ld % 4 == 0 && p.x_off % 4 == 0 && p.u_pitch % 4 == 0 && p.slot_stride % 4 == 0 && p.c_off % 4 == 0;
  const int per = 128 * (vec ? 4 : 1);
  const dim3 grid((p.width + per - 1) / per, (p.T + run - 1) / run);
  if (vec) launch_pdl(rglru_conv_kernel<E, 4>, grid, dim3(128), 0, st, p, run);
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

// max_q: the longest portion of the step; above 128 tokens `carry` holds 2 * width floats for every sequence and 128-token chunk of max_q.
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
  return is_f32 ? launch_rglru_step<float>(*p, st) : launch_rglru_step<__nv_bfloat16>(*p, st);
}

// Whether cafd_rglru_step takes a step of T rows in blocks of u_pitch (padded) channels.
extern "C" int cafd_rglru_step_ok(int T, int u_pitch, int is_f32) {
  return T <= kStepRows && u_pitch % 8 == 0 && (is_f32 ? rglru_step_smem<float>(T, u_pitch) : rglru_step_smem<__nv_bfloat16>(T, u_pitch)) <= 200 * 1024;
}
