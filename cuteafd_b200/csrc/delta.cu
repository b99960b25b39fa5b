// Gated delta rule layers (one decay per head): short causal convolutions with silu on q, k and v, unit norms, the
// recurrence
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// and the output norm under a silu gate.
//
// delta_step runs any mix of portions token by token with the state in registers: decode rows, speculative-verify rows,
// short portions, any sizes, bf16 or fp32 activations.  The state, the convolutions' inputs, the norms, the step size and
// the decay are fp32 throughout.  The state is read from one slot and written to another, so a step can be repeated
// (graph capture, rejected drafts) and a sequence may start from a slot that a cached prefix owns.
#include "cafd_api.h"
#include "common.cuh"
#include "delta.cuh"

namespace cafd {

constexpr int kDeltaRows = 32;      // state rows per thread
constexpr int kDeltaCols = 128;     // state columns per block at most

template <typename E, int MAXT, int NT>
__global__ void __launch_bounds__(NT) delta_step_kernel(const DeltaArgs p) {
  extern __shared__ float sm[];
  const int h = blockIdx.x, seq = blockIdx.y, v0 = blockIdx.z * kDeltaCols;
  const int tid = threadIdx.x, lane = tid & 31;
  const int vt = min(kDeltaCols, p.vdim - v0);
  const int n_slice = (p.dim + kDeltaRows - 1) / kDeltaRows;
  const int slice = tid / vt, col = tid - slice * vt;
  const bool worker = slice < n_slice;
  const int r0 = slice * kDeltaRows;
  const int n_ch = 2 * p.dim + vt;
  float* ch = sm;                                // [2][n_ch]
  float* red = ch + 2 * n_ch;                    // [2][n_slice][vt]
  float* so = red + 2 * n_slice * vt;            // [vt]
  float* sgb = so + vt;                          // [2][2]: decay, beta

  // The state of this step was written a whole step ago: its loads need not wait for the projection.
  float S[kDeltaRows];
  const float* st_in = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride;
  float* st_out = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride;
  const size_t s_base = p.s_off + (static_cast<size_t>(h) * p.dim) * p.vdim + v0 + col;
#pragma unroll
  for (int r = 0; r < kDeltaRows; ++r)
    S[r] = (worker && r0 + r < p.dim) ? st_in[s_base + static_cast<size_t>(r0 + r) * p.vdim] : 0.f;

  // this thread's convolution channel
  const int rep = p.heads / p.kv_heads, kh = h / rep;
  const int kd = p.kv_heads * p.dim, channels = 2 * kd + p.heads * p.vdim;
  int chan = -1, src = 0;
  bool keeper = false;                           // writes the channel's inputs to the new state
  if (tid < p.dim) { chan = kh * p.dim + tid; src = p.q_off + chan; keeper = h == kh * rep && blockIdx.z == 0; }
  else if (tid < 2 * p.dim) { const int c = kh * p.dim + tid - p.dim; chan = kd + c; src = p.k_off + c; keeper = h == kh * rep && blockIdx.z == 0; }
  else if (tid < n_ch) { const int c = h * p.vdim + v0 + tid - 2 * p.dim; chan = 2 * kd + c; src = p.v_off + c; keeper = true; }
  const int halo = p.taps - 1;
  float win[MAXT - 1], cw[MAXT];
#pragma unroll
  for (int j = 0; j < MAXT; ++j) {
    const int tap = j - (MAXT - p.taps);
    cw[j] = (chan >= 0 && tap >= 0) ? p.conv_w[static_cast<size_t>(chan) * p.taps + tap] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < MAXT - 1; ++j) {
    const int i = j - (MAXT - 1 - halo);
    win[j] = (chan >= 0 && i >= 0) ? st_in[p.c_off + static_cast<size_t>(i) * channels + chan] : 0.f;
  }
  const float a_scale = tid == 0 ? -expf(p.A_log[h]) : 0.f, dt = tid == 0 ? p.dt_bias[h] : 0.f;
  const float nw = (slice == 0 && p.out) ? p.norm_w[v0 + col] : 0.f;

  pdl_wait();
  pdl_trigger();
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  const E* proj = static_cast<const E*>(p.proj);
  float x = (chan >= 0 && t0 < t1) ? de_f<E>(proj[static_cast<size_t>(t0) * p.ld + src]) : 0.f;
  for (int t = t0; t < t1; ++t) {
    const int buf = (t - t0) & 1;
    const E* row = proj + static_cast<size_t>(t) * p.ld;
    float* c = ch + buf * n_ch;
    if (chan >= 0) {
      float y = cw[MAXT - 1] * x;
#pragma unroll
      for (int j = 0; j < MAXT - 1; ++j) y = fmaf(cw[j], win[j], y);
#pragma unroll
      for (int j = 0; j + 1 < MAXT - 1; ++j) win[j] = win[j + 1];
      win[MAXT - 2] = x;
      c[tid] = y * sigmoid_f(y);
    }
    if (tid == 0) {
      sgb[2 * buf] = expf(a_scale * softplus(de_f<E>(row[p.a_off + h]) + dt));
      sgb[2 * buf + 1] = sigmoid_f(de_f<E>(row[p.b_off + h]));
    }
    __syncthreads();
    if (chan >= 0 && t + 1 < t1) x = de_f<E>(row[p.ld + src]);
    const float gate = (slice == 0 && p.out) ? de_f<E>(row[p.g_off + h * p.vdim + v0 + col]) : 0.f;
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int i = lane; i < p.dim; i += 32) {
      const float a = c[i], b = c[p.dim + i];
      qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); qk = fmaf(a, b, qk);
    }
    qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
    const float ik = 1.0f / sqrtf(kk + 1e-6f), iq = 1.0f / (sqrtf(qq + 1e-6f) * sqrtf(static_cast<float>(p.dim)));
    float sk = 0.f, sq = 0.f;
    if (worker) {
#pragma unroll
      for (int r = 0; r < kDeltaRows; ++r) {
        if (r0 + r < p.dim) {
          sq = fmaf(S[r], c[r0 + r], sq);
          sk = fmaf(S[r], c[p.dim + r0 + r], sk);
        }
      }
      red[slice * vt + col] = sk;
      red[(n_slice + slice) * vt + col] = sq;
    }
    __syncthreads();
    if (worker) {
      sk = 0.f; sq = 0.f;
      for (int i = 0; i < n_slice; ++i) { sk += red[i * vt + col]; sq += red[(n_slice + i) * vt + col]; }
      const float g = sgb[2 * buf], beta = sgb[2 * buf + 1];
      const float u = beta * (c[2 * p.dim + col] - g * (ik * sk));
      const float uk = u * ik;
#pragma unroll
      for (int r = 0; r < kDeltaRows; ++r)
        if (r0 + r < p.dim) S[r] = fmaf(c[p.dim + r0 + r], uk, g * S[r]);
      if (slice == 0) {
        const float o = g * (iq * sq) + (qk * ik * iq) * u;
        if (p.out) so[col] = o;
        else p.raw[static_cast<size_t>(t) * p.heads * p.vdim + h * p.vdim + v0 + col] = o;
      }
    }
    if (p.out) {
      __syncthreads();
      if ((tid & ~31) < vt) {
        float ss = 0.f;
        for (int i = lane; i < vt; i += 32) ss = fmaf(so[i], so[i], ss);
        ss = warp_sum(ss);
        if (tid < vt) {
          const float inv = 1.0f / sqrtf(ss / static_cast<float>(vt) + p.eps);
          static_cast<E*>(p.out)[(static_cast<size_t>(t) * p.heads + h) * p.out_vd + tid] =
              de_e<E>(so[tid] * inv * nw * gate * sigmoid_f(gate));
        }
      }
    }
  }
  if (t1 > t0) {
    if (worker) {
#pragma unroll
      for (int r = 0; r < kDeltaRows; ++r)
        if (r0 + r < p.dim) st_out[s_base + static_cast<size_t>(r0 + r) * p.vdim] = S[r];
    }
    if (chan >= 0 && keeper) {
#pragma unroll
      for (int j = 0; j < MAXT - 1; ++j) {
        const int i = j - (MAXT - 1 - halo);
        if (i >= 0) st_out[p.c_off + static_cast<size_t>(i) * channels + chan] = win[j];
      }
    }
  }
}

// The same recurrence for heads of 128 columns and D = 64 or 128 rows, as decode steps want it: 256 threads, a warp holds
// D / 8 state rows with four columns per lane (16-byte loads and stores), the output norm stays inside one warp.
template <typename E, int D>
__global__ void __launch_bounds__(256, 2) delta_step128_kernel(const DeltaArgs p) {
  constexpr int kR = D / 8, kCh = 2 * D + 128, kTaps = 4;
  __shared__ __align__(16) float ch[2][kCh];
  __shared__ __align__(16) float red[2][8][128];
  __shared__ float sgb[2][2];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // the state of this step was written a whole step ago: its loads need not wait for the projection
  const float* st_in = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride;
  float* st_out = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride;
  const size_t s_at = p.s_off + (static_cast<size_t>(h) * D + warp * kR) * 128 + 4 * lane;
  float4 S[kR];
#pragma unroll
  for (int r = 0; r < kR; ++r) S[r] = __ldcg(reinterpret_cast<const float4*>(st_in + s_at + r * 128));
  const int rep = p.heads / p.kv_heads, kh = h / rep;
  const int kd = p.kv_heads * D, channels = 2 * kd + p.heads * 128, halo = p.taps - 1;
  constexpr int kN = (kCh + 255) / 256;          // channels per thread
  int chan[kN], src[kN];
  float win[kN][kTaps - 1], cw[kN][kTaps], x[kN];
#pragma unroll
  for (int n = 0; n < kN; ++n) {
    const int c = tid + n * 256;
    chan[n] = -1; src[n] = 0;
    if (c < D) { chan[n] = kh * D + c; src[n] = p.q_off + chan[n]; }
    else if (c < 2 * D) { chan[n] = kd + kh * D + c - D; src[n] = p.k_off + kh * D + c - D; }
    else if (c < kCh) { chan[n] = 2 * kd + h * 128 + c - 2 * D; src[n] = p.v_off + h * 128 + c - 2 * D; }
#pragma unroll
    for (int j = 0; j < kTaps; ++j) {
      const int tap = j - (kTaps - p.taps);
      cw[n][j] = (chan[n] >= 0 && tap >= 0) ? p.conv_w[static_cast<size_t>(chan[n]) * p.taps + tap] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kTaps - 1; ++j) {
      const int i = j - (kTaps - 1 - halo);
      win[n][j] = (chan[n] >= 0 && i >= 0) ? st_in[p.c_off + static_cast<size_t>(i) * channels + chan[n]] : 0.f;
    }
  }
  const float a_scale = tid == 0 ? -expf(p.A_log[h]) : 0.f, dt = tid == 0 ? p.dt_bias[h] : 0.f;
  float nw[4] = {};
  if (warp == 0) de_load4(p.norm_w + 4 * lane, nw);

  pdl_wait();
  pdl_trigger();
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
  const E* proj = static_cast<const E*>(p.proj);
#pragma unroll
  for (int n = 0; n < kN; ++n) x[n] = (chan[n] >= 0 && t0 < t1) ? de_f<E>(proj[static_cast<size_t>(t0) * p.ld + src[n]]) : 0.f;
  for (int t = t0; t < t1; ++t) {
    const int buf = (t - t0) & 1;
    const E* row = proj + static_cast<size_t>(t) * p.ld;
    float* c = ch[buf];
    float gate[4] = {};
    if (warp == 0) {
      if (p.g_off % 4 == 0 && p.ld % 4 == 0) de_load4(row + p.g_off + h * 128 + 4 * lane, gate);
      else
        for (int e = 0; e < 4; ++e) gate[e] = de_f<E>(row[p.g_off + h * 128 + 4 * lane + e]);
    }
    if (tid == 0) {
      sgb[buf][0] = expf(a_scale * softplus(de_f<E>(row[p.a_off + h]) + dt));
      sgb[buf][1] = sigmoid_f(de_f<E>(row[p.b_off + h]));
    }
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      if (chan[n] >= 0) {
        float y = cw[n][kTaps - 1] * x[n];
#pragma unroll
        for (int j = 0; j < kTaps - 1; ++j) y = fmaf(cw[n][j], win[n][j], y);
        win[n][0] = win[n][1]; win[n][1] = win[n][2]; win[n][2] = x[n];
        c[tid + n * 256] = y * sigmoid_f(y);
      }
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < kN; ++n)
      if (chan[n] >= 0 && t + 1 < t1) x[n] = de_f<E>(row[p.ld + src[n]]);
    float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
    for (int i = 0; i < D / 32; ++i) {
      const float a = c[lane + 32 * i], b = c[D + lane + 32 * i];
      qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); qk = fmaf(a, b, qk);
    }
    float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
#pragma unroll
    for (int r = 0; r < kR; ++r) {
      const float qv = c[warp * kR + r], kv = c[D + warp * kR + r];
      sq.x = fmaf(S[r].x, qv, sq.x); sq.y = fmaf(S[r].y, qv, sq.y); sq.z = fmaf(S[r].z, qv, sq.z); sq.w = fmaf(S[r].w, qv, sq.w);
      sk.x = fmaf(S[r].x, kv, sk.x); sk.y = fmaf(S[r].y, kv, sk.y); sk.z = fmaf(S[r].z, kv, sk.z); sk.w = fmaf(S[r].w, kv, sk.w);
    }
    *reinterpret_cast<float4*>(&red[0][warp][4 * lane]) = sk;
    *reinterpret_cast<float4*>(&red[1][warp][4 * lane]) = sq;
    qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
    const float ik = 1.0f / sqrtf(kk + 1e-6f), iq = 1.0f / (sqrtf(qq + 1e-6f) * sqrtf(static_cast<float>(D)));
    __syncthreads();
    sk = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      const float4 v = *reinterpret_cast<const float4*>(&red[0][w][4 * lane]);
      sk.x += v.x; sk.y += v.y; sk.z += v.z; sk.w += v.w;
    }
    const float g = sgb[buf][0], beta = sgb[buf][1], gk = g * ik;
    const float4 v = *reinterpret_cast<const float4*>(c + 2 * D + 4 * lane);
    float u[4] = {beta * (v.x - gk * sk.x), beta * (v.y - gk * sk.y), beta * (v.z - gk * sk.z), beta * (v.w - gk * sk.w)};
    if (warp == 0) {
      sq = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        const float4 z = *reinterpret_cast<const float4*>(&red[1][w][4 * lane]);
        sq.x += z.x; sq.y += z.y; sq.z += z.z; sq.w += z.w;
      }
      const float gq = g * iq, qki = qk * ik * iq;
      float o[4] = {gq * sq.x + qki * u[0], gq * sq.y + qki * u[1], gq * sq.z + qki * u[2], gq * sq.w + qki * u[3]};
      const float ss = warp_sum(o[0] * o[0] + o[1] * o[1] + o[2] * o[2] + o[3] * o[3]);
      const float inv = 1.0f / sqrtf(ss * (1.0f / 128.0f) + p.eps);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] *= inv * nw[e] * gate[e] * sigmoid_f(gate[e]);
      de_store4(static_cast<E*>(p.out) + (static_cast<size_t>(t) * p.heads + h) * p.out_vd + 4 * lane, o);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) u[e] *= ik;
#pragma unroll
    for (int r = 0; r < kR; ++r) {
      const float kv = c[D + warp * kR + r];
      S[r].x = fmaf(kv, u[0], g * S[r].x); S[r].y = fmaf(kv, u[1], g * S[r].y);
      S[r].z = fmaf(kv, u[2], g * S[r].z); S[r].w = fmaf(kv, u[3], g * S[r].w);
    }
  }
  if (t1 > t0) {
#pragma unroll
    for (int r = 0; r < kR; ++r) __stcg(reinterpret_cast<float4*>(st_out + s_at + r * 128), S[r]);
#pragma unroll
    for (int n = 0; n < kN; ++n) {
      const int c = tid + n * 256;
      if (chan[n] >= 0 && (c >= 2 * D || h == kh * rep)) {
#pragma unroll
        for (int j = 0; j < kTaps - 1; ++j) {
          const int i = j - (kTaps - 1 - halo);
          if (i >= 0) st_out[p.c_off + static_cast<size_t>(i) * channels + chan[n]] = win[n][j];
        }
      }
    }
  }
}

template <typename E, int MAXT>
static int launch_delta(const DeltaArgs& p, cudaStream_t st) {
  if (MAXT <= 4 && p.vdim == 128 && (p.dim == 64 || p.dim == 128) && p.out_vd % 4 == 0 && p.s_off % 4 == 0 && p.slot_stride % 4 == 0) {
    if (p.dim == 64) launch_pdl(delta_step128_kernel<E, 64>, dim3(p.heads, p.S), dim3(256), 0, st, p);
    else launch_pdl(delta_step128_kernel<E, 128>, dim3(p.heads, p.S), dim3(256), 0, st, p);
    return static_cast<int>(cudaGetLastError());
  }
  const int vt = p.vdim < kDeltaCols ? p.vdim : kDeltaCols;
  const int n_slice = (p.dim + kDeltaRows - 1) / kDeltaRows;
  int threads = vt * n_slice;
  if (threads < 2 * p.dim + vt) threads = 2 * p.dim + vt;
  threads = (threads + 31) / 32 * 32;
  if (threads > 1024) return -12;
  const size_t smem = static_cast<size_t>(2 * (2 * p.dim + vt) + 2 * n_slice * vt + vt + 4) * 4;
  const int tiles = (p.vdim + kDeltaCols - 1) / kDeltaCols;
  DeltaArgs q = p;
  if (tiles > 1) { if (!p.raw) return -13; q.out = nullptr; }
  const dim3 grid(p.heads, p.S, tiles);
  if (threads <= 512) launch_pdl(delta_step_kernel<E, MAXT, 512>, grid, dim3(threads), smem, st, q);
  else launch_pdl(delta_step_kernel<E, MAXT, 1024>, grid, dim3(threads), smem, st, q);
  if (tiles > 1) {
    const long long rows = static_cast<long long>(p.T) * p.heads;
    const int blocks = static_cast<int>(rows < 8 * 148 * 8 ? (rows + 7) / 8 : 148 * 8);
    launch_pdl(delta_out_kernel<E>, dim3(blocks), dim3(256), 0, st, p);
  }
  return static_cast<int>(cudaGetLastError());
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_delta_step(const DeltaArgs* p, int is_f32, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (p->S < 1 || p->kv_heads < 1 || p->heads % p->kv_heads || p->dim < 1 || p->dim > 256 || p->taps < 1 || p->taps > 16) return -10;
  if (!p->state || !p->state_in || !p->state_out || !p->out || p->out_vd < p->vdim) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (p->taps <= 4) return is_f32 ? launch_delta<float, 4>(*p, st) : launch_delta<__nv_bfloat16, 4>(*p, st);
  return is_f32 ? launch_delta<float, 16>(*p, st) : launch_delta<__nv_bfloat16, 16>(*p, st);
}
