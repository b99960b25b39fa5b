// Residual stream of the per-layer hybrid decoders: everything between two sublayers in one launch.
//
//   x   = embed[token] * e_scale            (first launch; a second table's row may be added)  or the fp32 residual of the previous
//                                           launch, or their sum (a loop's next pass)
//   x  += step                              one vector for all tokens (optional)
//   x  += groupnorm(y) * w_b                y = a mixer's output rows, or the routed experts' rows summed here:
//                                           sum over slots of weight * (expert row, or the input row for an identity slot);
//                                           without w_b: x += y; `base` rows are added to the routed sum as they are
//   x   = sum_j past_w[j] * past[j] + past_w[n] * x       average over depth (optional): earlier results of the same rows; x itself is
//                                           kept for later ones first
//   h   = groupnorm(x) * (w + w_off)        RMS norm in equal runs of channels, each with its own root mean square
//                                           (without w: h = x); a second weight vector gives a second output of the same norm
//   out = h + sum_j c[j] * h(t - taps + 1 + j)     causal convolution over time per channel (optional)
//
// A block walks a run of consecutive tokens with every channel in registers, so the convolution's earlier inputs are the
// registers of the previous iterations; the few inputs before the run are recomputed from the residual, or come from the
// sequence's state when they lie before this step.  The residual is read from one buffer and written to another (the
// neighbouring block recomputes rows of the old one), the convolution state likewise from slot to slot.  A token's
// arithmetic does not depend on where its run or its step begins.
#pragma once

#include "cafd_api.h"
#include "common.cuh"

namespace cafd {

struct NormArgs {
  const int* tokens;          // with embed: token ids
  const void* embed;          // [vocab, H] E, or null
  const float* x_in;          // [T, H] or null (with embed: the embedding row is added to it)
  const void* y;              // [T, ldy] E, or the slot rows [T * top_k, ldy] E with slot_w; null = nothing to add
  const float* slot_w;        // [T, top_k]
  const int* slot_idx;        // [T, top_k]; an index >= n_experts is an identity slot
  const void* ident;          // [T, ldi] E: what identity slots hand through
  const void* w_b;            // [H] E, null = y is added as it is
  const void* w;              // [H] E, null = the rows leave as they are, without a norm
  const void* base;           // [T, ldb] E, null = none; only with slot_w
  const void* step;           // [H] E, null = none
  const void* w2;             // [H] E, null = none: weights of the second output; only without a convolution
  void* h2_out;               // [rows, ldh] E
  const void* conv;           // [taps, H] E, null = no convolution
  float* x_out;               // [T, H] or null
  void* h_out;                // [rows, ldh] E
  const int* row_idx;         // rows to compute (null = all, in order); only without a convolution
  float* state;               // recurrent state pool, slot_stride floats per slot; this launch's inputs at state_off
  const int* state_in;        // [S] slot read
  const int* state_out;       // [S] slot written
  const int* q_start;         // [S + 1]
  const int* rows2;           // [T] rows of the second table, with embed only; null = none
  const void* embed2;         // [vocab2, H] E
  const float* past;          // [n_past][T, H], past_stride floats from one to the next; only without a convolution
  const float* past_w;        // [n_past + 1], null = no average
  float* past_out;            // [T, H] or null: x before the average
  long long slot_stride, state_off, past_stride;
  int T, H, S, ldy, ldh, ldb, ldi, groups, taps, top_k, n_experts, vocab, run, vocab2, n_past;   // ldy, ldh, ldb, ldi: elements from row to row of y, of h_out, of base, of ident
  float eps, w_off, e_scale;
};

template <typename E> __device__ __forceinline__ float ld_e(const E* p);
template <> __device__ __forceinline__ float ld_e<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld_e<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }

template <typename E, int V>
__device__ __forceinline__ void load_vec(const E* p, float (&v)[V]) {
  if constexpr (V == 8 && sizeof(E) == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p), r = *reinterpret_cast<const float4*>(p + 4);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    v[4] = r.x; v[5] = r.y; v[6] = r.z; v[7] = r.w;
  } else if constexpr (V == 8) {
    const uint4 q = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) { v[2 * e] = bf16_lo(w[e]); v[2 * e + 1] = bf16_hi(w[e]); }
  } else if constexpr (V == 4 && sizeof(E) == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  } else if constexpr (V == 4) {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(q.x); v[1] = bf16_hi(q.x); v[2] = bf16_lo(q.y); v[3] = bf16_hi(q.y);
  } else {
    v[0] = ld_e<E>(p);
  }
}
template <typename E, int V>
__device__ __forceinline__ void store_vec(E* p, const float (&v)[V]) {
  if constexpr (V == 8 && sizeof(E) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  } else if constexpr (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else if constexpr (V == 4 && sizeof(E) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
  } else if constexpr (sizeof(E) == 4) {
    *reinterpret_cast<float*>(p) = v[0];
  } else {
    *reinterpret_cast<__nv_bfloat16*>(p) = __float2bfloat16(v[0]);
  }
}

// V elements as they sit in memory: loads of rows to come stay packed in registers until their turn
template <typename E, int V> struct Packed;
template <> struct __align__(16) Packed<float, 8> { float4 q, r; };
template <> struct Packed<__nv_bfloat16, 8> { uint4 q; };
template <> struct Packed<float, 4> { float4 q; };
template <> struct Packed<__nv_bfloat16, 4> { uint2 q; };
template <> struct Packed<float, 1> { float q; };
template <> struct Packed<__nv_bfloat16, 1> { __nv_bfloat16 q; };
template <typename E, int V>
__device__ __forceinline__ Packed<E, V> load_packed(const E* p) { return *reinterpret_cast<const Packed<E, V>*>(p); }
__device__ __forceinline__ void unpack(const Packed<float, 4>& a, float (&v)[4]) { v[0] = a.q.x; v[1] = a.q.y; v[2] = a.q.z; v[3] = a.q.w; }
__device__ __forceinline__ void unpack(const Packed<__nv_bfloat16, 4>& a, float (&v)[4]) {
  v[0] = bf16_lo(a.q.x); v[1] = bf16_hi(a.q.x); v[2] = bf16_lo(a.q.y); v[3] = bf16_hi(a.q.y);
}
__device__ __forceinline__ void unpack(const Packed<float, 8>& a, float (&v)[8]) {
  v[0] = a.q.x; v[1] = a.q.y; v[2] = a.q.z; v[3] = a.q.w;
  v[4] = a.r.x; v[5] = a.r.y; v[6] = a.r.z; v[7] = a.r.w;
}
__device__ __forceinline__ void unpack(const Packed<__nv_bfloat16, 8>& a, float (&v)[8]) {
  const uint32_t w[4] = {a.q.x, a.q.y, a.q.z, a.q.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) { v[2 * e] = bf16_lo(w[e]); v[2 * e + 1] = bf16_hi(w[e]); }
}
__device__ __forceinline__ void unpack(const Packed<float, 1>& a, float (&v)[1]) { v[0] = a.q; }
__device__ __forceinline__ void unpack(const Packed<__nv_bfloat16, 1>& a, float (&v)[1]) { v[0] = __bfloat162float(a.q); }

constexpr int kNormThreads = 512;

// 1 / sqrt(mean of squares + eps) of the group each of this thread's vectors lies in.  `part` holds one number per 32
// vectors when groups are whole multiples of that (fast), else one per vector; `gsum` one per group (slow form only).
template <int V, int KV, bool kExact>
__device__ __forceinline__ void group_inv(const float (&v)[KV][V], float (&inv)[KV], float* part, float* gsum, int nvec, int gvec,
                                          const int (&grp)[KV], float inv_n, bool fast, float eps) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x;
  auto root = [&](float s) { return kExact ? 1.0f / sqrtf(s * inv_n + eps) : rsqrtf(s * inv_n + eps); };
  if (fast) {
#pragma unroll
    for (int k = 0; k < KV; ++k) {
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) s += v[k][e] * v[k][e];
      s = warp_sum(s);
      const int i = tid + k * nt;
      if (lane == 0 && i < nvec) part[i >> 5] = s;
    }
    __syncthreads();
    const int per = gvec >> 5;
#pragma unroll
    for (int k = 0; k < KV; ++k) {
      const int i = tid + k * nt;
      float s = 0.f;
      if (i < nvec) {
        const int g0 = grp[k] * per;
        for (int j = 0; j < per; ++j) s += part[g0 + j];
      }
      inv[k] = root(s);
    }
  } else {
#pragma unroll
    for (int k = 0; k < KV; ++k) {
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) s += v[k][e] * v[k][e];
      const int i = tid + k * nt;
      if (i < nvec) part[i] = s;
    }
    __syncthreads();
    const int ng = nvec / gvec;
    for (int g = warp; g < ng; g += nt >> 5) {
      float s = 0.f;
      for (int j = lane; j < gvec; j += 32) s += part[g * gvec + j];
      s = warp_sum(s);
      if (lane == 0) gsum[g] = s;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < KV; ++k) {
      const int i = tid + k * nt;
      inv[k] = i < nvec ? root(gsum[grp[k]]) : 0.f;
    }
  }
}

template <typename E, int V, int KV, int MAXT, bool kSlots, bool kPast, int kMaxThreads, int kMinBlocks>
__global__ void __launch_bounds__(kMaxThreads, kMinBlocks) norm_conv_kernel(const NormArgs a) {
  extern __shared__ float sm[];
  // routed rows of a token whose loads are in flight together (prompts: several blocks per SM share the registers)
  constexpr int kSlotBatch = kMinBlocks == 1 ? 8 : 4;
  const int tid = threadIdx.x, nt = blockDim.x;
  const int nvec = a.H / V, gvec = nvec / a.groups;
  if (kMinBlocks == 1 && a.run == 1) {
    // decode: the weights (and, when a block is a sequence, its state) are on their way into L2 while the previous
    // kernel drains; nothing is read here
    auto pull = [](const void* q) { asm volatile("prefetch.global.L2 [%0];" ::"l"(q)); };
    const bool own_seq = a.conv && a.S == a.T && a.state;
    const float* st = own_seq ? a.state + static_cast<size_t>(a.state_in[blockIdx.x]) * a.slot_stride + a.state_off : nullptr;
    for (int i = tid * 32; i < a.H; i += nt * 32) {         // one 128-byte line per step
      if (a.w) pull(static_cast<const E*>(a.w) + i);
      if (a.w2) pull(static_cast<const E*>(a.w2) + i);
      if (a.w_b) pull(static_cast<const E*>(a.w_b) + i);
      if (a.conv)
        for (int j = 0; j < a.taps; ++j) pull(static_cast<const E*>(a.conv) + static_cast<size_t>(j) * a.H + i);
      if (st)
        for (int j = 0; j + 1 < a.taps; ++j) pull(st + static_cast<size_t>(j) * a.H + i);
    }
  }
  pdl_wait();
  pdl_trigger();
  const bool fast = (gvec & 31) == 0;
  const int stride = fast ? (nvec >> 5) : nvec + a.groups;   // two alternating reduction buffers
  const int r0 = blockIdx.x * a.run;
  const int r1 = min(a.T, r0 + a.run);
  if (r0 >= a.T) return;
  const int halo = a.conv ? a.taps - 1 : 0;
  const E* conv_w = static_cast<const E*>(a.conv);
  const float inv_n = 1.0f / static_cast<float>(gvec * V);
  int grp[KV];
#pragma unroll
  for (int k = 0; k < KV; ++k) grp[k] = (tid + k * nt) / gvec;

  float win[MAXT > 1 ? MAXT - 1 : 1][KV][V];   // the last taps - 1 convolution inputs, oldest first, at the array's end
#pragma unroll
  for (int j = 0; j < MAXT - 1; ++j)
#pragma unroll
    for (int k = 0; k < KV; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) win[j][k][e] = 0.f;

  int seq = 0, s_lo = 0, s_hi = a.T;
  int t = r0;
  if (a.conv) {
    int hi = a.S;                               // sequence of row r0: last s with q_start[s] <= r0
    while (hi - seq > 1) {
      const int mid = (seq + hi) >> 1;
      if (a.q_start[mid] <= r0) seq = mid; else hi = mid;
    }
    s_lo = a.q_start[seq];
    s_hi = a.q_start[seq + 1];
    t = max(s_lo, r0 - halo);
  }
  auto load_state = [&]() {
    const float* st = a.state + static_cast<size_t>(a.state_in[seq]) * a.slot_stride + a.state_off;
#pragma unroll
    for (int j = 0; j < MAXT - 1; ++j) {
      const int src = j - (MAXT - 1 - halo);
      if (src >= 0) {
#pragma unroll
        for (int k = 0; k < KV; ++k) {
          const int i = tid + k * nt;
          if (i < nvec) load_vec<float, V>(st + static_cast<size_t>(src) * a.H + i * V, win[j][k]);
        }
      }
    }
  };
  if (a.conv && t == s_lo && halo > 0) load_state();
  int flip = 0;
  // The residual and the sublayer's output of the next token are loaded while this one is normalised.
  const E* const plain = static_cast<const E*>(kSlots ? a.base : a.y);
  const int ld_plain = kSlots ? a.ldb : a.ldy;
  Packed<float, V> nx[KV];
  Packed<E, V> ny[KV];
  auto fetch = [&](int tt) {
    const int row = a.row_idx ? a.row_idx[tt] : tt;
    if (a.x_in) {
      const float* src = a.x_in + static_cast<size_t>(row) * a.H;
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) nx[k] = load_packed<float, V>(src + i * V);
      }
    }
    if (plain) {
      const E* src = plain + static_cast<size_t>(row) * ld_plain;
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) ny[k] = load_packed<E, V>(src + i * V);
      }
    }
  };
  fetch(t);
  for (; t < r1; ++t) {
    if (a.conv && t == s_hi) {                  // next sequence (empty ones are skipped)
      do { ++seq; s_lo = s_hi; s_hi = a.q_start[seq + 1]; } while (s_hi == s_lo && seq + 1 < a.S);
      if (halo > 0) load_state();
    }
    const int row = a.row_idx ? a.row_idx[t] : t;
    const bool own = t >= r0;
    float x[KV][V], y[KV][V];
#pragma unroll
    for (int k = 0; k < KV; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) { x[k][e] = 0.f; y[k][e] = 0.f; }
    if (a.x_in) {
#pragma unroll
      for (int k = 0; k < KV; ++k)
        if (tid + k * nt < nvec) unpack(nx[k], x[k]);
    }
    if (a.embed) {
      int tok = a.tokens[row];
      tok = tok < 0 ? 0 : tok >= a.vocab ? a.vocab - 1 : tok;
      const E* src = static_cast<const E*>(a.embed) + static_cast<size_t>(tok) * a.H;
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) {
          float v[V];
          load_vec<E, V>(src + i * V, v);
#pragma unroll
          for (int e = 0; e < V; ++e) x[k][e] = fmaf(v[e], a.e_scale, x[k][e]);
        }
      }
      if (a.rows2) {
        const int r2 = min(max(a.rows2[row], 0), a.vocab2 - 1);
        src = static_cast<const E*>(a.embed2) + static_cast<size_t>(r2) * a.H;
#pragma unroll
        for (int k = 0; k < KV; ++k) {
          const int i = tid + k * nt;
          if (i < nvec) {
            float v[V];
            load_vec<E, V>(src + i * V, v);
#pragma unroll
            for (int e = 0; e < V; ++e) x[k][e] += v[e];
          }
        }
      }
    }
    if (a.step) {
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) {
          float v[V];
          load_vec<E, V>(static_cast<const E*>(a.step) + i * V, v);
#pragma unroll
          for (int e = 0; e < V; ++e) x[k][e] += v[e];
        }
      }
    }
    if (plain) {
#pragma unroll
      for (int k = 0; k < KV; ++k)
        if (tid + k * nt < nvec) unpack(ny[k], y[k]);
    }
    if constexpr (kSlots) {
      const float* sw = a.slot_w + static_cast<size_t>(row) * a.top_k;
      const int* si = a.slot_idx + static_cast<size_t>(row) * a.top_k;
      for (int s0 = 0; s0 < a.top_k; s0 += kSlotBatch) {
        int src[kSlotBatch];                    // row offsets; identity slots: the input row, marked by a negative number
        float g[kSlotBatch];
#pragma unroll
        for (int j = 0; j < kSlotBatch; ++j) {
          const int s = min(s0 + j, a.top_k - 1);
          g[j] = s0 + j < a.top_k ? sw[s] : 0.f;
          src[j] = si[s] >= a.n_experts ? -1 : row * a.top_k + s;
        }
#pragma unroll
        for (int k = 0; k < KV; ++k) {
          const int i = tid + k * nt;
          if (i < nvec) {
            Packed<E, V> raw[kSlotBatch];
#pragma unroll
            for (int j = 0; j < kSlotBatch; ++j)
              if (s0 + j < a.top_k)
                raw[j] = load_packed<E, V>((src[j] < 0 ? static_cast<const E*>(a.ident) + static_cast<size_t>(row) * a.ldi
                                                       : static_cast<const E*>(a.y) + static_cast<size_t>(src[j]) * a.ldy) + i * V);
#pragma unroll
            for (int j = 0; j < kSlotBatch; ++j) {
              if (s0 + j < a.top_k) {
                float v[V];
                unpack(raw[j], v);
#pragma unroll
                for (int e = 0; e < V; ++e) y[k][e] += g[j] * v[e];
              }
            }
          }
        }
      }
    }
    if (t + 1 < r1) {
      fetch(t + 1);
      if constexpr (kSlots && kMinBlocks > 1) {               // the next token's routed rows on their way into L2
        const int lines = (a.H * static_cast<int>(sizeof(E)) + 127) / 128;
        for (int l = tid; l < a.top_k * lines; l += nt) {
          const int s = l / lines, nrow = (t + 1) * a.top_k + s;
          if (a.slot_idx[nrow] < a.n_experts)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const uint8_t*>(static_cast<const E*>(a.y) + static_cast<size_t>(nrow) * a.ldy) + (l - s * lines) * 128));
        }
      }
    }
    if (a.y && !a.w_b) {
#pragma unroll
      for (int k = 0; k < KV; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) x[k][e] += y[k][e];
    } else if (a.y) {
      float inv[KV];
      group_inv<V, KV, sizeof(E) == 4>(y, inv, sm + flip * stride, sm + flip * stride + nvec, nvec, gvec, grp, inv_n, fast, a.eps);
      flip ^= 1;
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) {
          float wb[V];
          load_vec<E, V>(static_cast<const E*>(a.w_b) + i * V, wb);
#pragma unroll
          for (int e = 0; e < V; ++e) x[k][e] += y[k][e] * inv[k] * wb[e];
        }
      }
    }
    if constexpr (kPast) {
      constexpr int kBatch = 4;                 // earlier results whose loads are in flight together
      const float wx = a.past_w[a.n_past];
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) {
          const size_t at = static_cast<size_t>(row) * a.H + i * V;
          if (a.past_out) store_vec<float, V>(a.past_out + at, x[k]);
#pragma unroll
          for (int e = 0; e < V; ++e) x[k][e] *= wx;
          for (int j0 = 0; j0 < a.n_past; j0 += kBatch) {
            Packed<float, V> raw[kBatch];
            float g[kBatch];
#pragma unroll
            for (int j = 0; j < kBatch; ++j) {
              const int jj = min(j0 + j, a.n_past - 1);
              g[j] = a.past_w[jj];
              if (j0 + j < a.n_past) raw[j] = load_packed<float, V>(a.past + jj * a.past_stride + at);
            }
#pragma unroll
            for (int j = 0; j < kBatch; ++j) {
              if (j0 + j < a.n_past) {
                float v[V];
                unpack(raw[j], v);
#pragma unroll
                for (int e = 0; e < V; ++e) x[k][e] = fmaf(g[j], v[e], x[k][e]);
              }
            }
          }
        }
      }
    }
    if (own && a.x_out) {
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) store_vec<float, V>(a.x_out + static_cast<size_t>(row) * a.H + i * V, x[k]);
      }
    }
    if (a.w) {
    float inv[KV];
    group_inv<V, KV, sizeof(E) == 4>(x, inv, sm + flip * stride, sm + flip * stride + nvec, nvec, gvec, grp, inv_n, fast, a.eps);
    flip ^= 1;
#pragma unroll
    for (int k = 0; k < KV; ++k) {                                           // x now holds h
      const int i = tid + k * nt;
      if (i < nvec) {
        float wn[V];
        if (a.w2 && own) {
          float o[V];
          load_vec<E, V>(static_cast<const E*>(a.w2) + i * V, wn);
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = x[k][e] * inv[k] * (wn[e] + a.w_off);
          store_vec<E, V>(static_cast<E*>(a.h2_out) + static_cast<size_t>(t) * a.ldh + i * V, o);
        }
        load_vec<E, V>(static_cast<const E*>(a.w) + i * V, wn);
#pragma unroll
        for (int e = 0; e < V; ++e) x[k][e] = x[k][e] * inv[k] * (wn[e] + a.w_off);
      }
    }
    }
    if (own) {
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int i = tid + k * nt;
        if (i < nvec) {
          float o[V];
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = x[k][e];
          if (a.conv) {
            float c[V];
            load_vec<E, V>(conv_w + static_cast<size_t>(a.taps - 1) * a.H + i * V, c);
            float acc[V];
#pragma unroll
            for (int e = 0; e < V; ++e) acc[e] = c[e] * x[k][e];
#pragma unroll
            for (int j = 0; j < MAXT - 1; ++j) {
              const int tap = j - (MAXT - 1 - halo);
              if (tap >= 0) {
                load_vec<E, V>(conv_w + static_cast<size_t>(tap) * a.H + i * V, c);
#pragma unroll
                for (int e = 0; e < V; ++e) acc[e] += c[e] * win[j][k][e];
              }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) o[e] += acc[e];
          }
          store_vec<E, V>(static_cast<E*>(a.h_out) + static_cast<size_t>(t) * a.ldh + i * V, o);
        }
      }
    }
#pragma unroll
    for (int j = 0; j + 1 < MAXT - 1; ++j)
#pragma unroll
      for (int k = 0; k < KV; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) win[j][k][e] = win[j + 1][k][e];
    if (MAXT > 1) {
#pragma unroll
      for (int k = 0; k < KV; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) win[MAXT > 1 ? MAXT - 2 : 0][k][e] = x[k][e];
    }
    if (own && halo > 0 && t == s_hi - 1) {
      float* st = a.state + static_cast<size_t>(a.state_out[seq]) * a.slot_stride + a.state_off;
#pragma unroll
      for (int j = 0; j < MAXT - 1; ++j) {
        const int dst = j - (MAXT - 1 - halo);
        if (dst >= 0) {
#pragma unroll
          for (int k = 0; k < KV; ++k) {
            const int i = tid + k * nt;
            if (i < nvec) store_vec<float, V>(st + static_cast<size_t>(dst) * a.H + i * V, win[j][k]);
          }
        }
      }
    }
  }
}

template <typename E, int V, int KV, int MAXT, int kMaxThreads, int kMinBlocks, bool kPast = false>
static int launch_norm(NormArgs a, cudaStream_t st) {
  const int nvec = a.H / V, gvec = nvec / a.groups;
  const int threads = ((nvec + KV - 1) / KV + 31) / 32 * 32;
  const int stride = (gvec % 32 == 0) ? nvec / 32 : nvec + a.groups;
  const size_t smem = static_cast<size_t>(2 * stride) * 4;
  if (threads > kMaxThreads || smem > 48 * 1024) return -12;
  if (a.run <= 0) {
    // decode: one token per block; prompts: one wave of blocks, each with a run of tokens
    const int run = (a.T + kMinBlocks * 148 - 1) / (kMinBlocks * 148);
    a.run = run <= 2 ? 1 : run > 64 ? 64 : run;
  }
  const dim3 grid((a.T + a.run - 1) / a.run);
  if (a.slot_w) launch_pdl(norm_conv_kernel<E, V, KV, MAXT, true, kPast, kMaxThreads, kMinBlocks>, grid, dim3(threads), smem, st, a);
  else launch_pdl(norm_conv_kernel<E, V, KV, MAXT, false, kPast, kMaxThreads, kMinBlocks>, grid, dim3(threads), smem, st, a);
  return static_cast<int>(cudaGetLastError());
}

template <typename E>
static int dispatch_norm(const NormArgs& a, cudaStream_t st) {
  const int per_group = a.H / a.groups;
  const bool few = !a.conv || a.taps <= 4;
  if (a.past_w) {                               // (never with a convolution)
    if (per_group % 8 == 0) {
      if (a.T > 256 && a.H <= 2048) return launch_norm<E, 8, 1, 1, 256, 3, true>(a, st);
      if (a.T > 256 && a.H <= 4096) return launch_norm<E, 8, 2, 1, 256, 2, true>(a, st);
      if (a.H <= 4096) return launch_norm<E, 8, 1, 1, 512, 1, true>(a, st);
      return a.H <= 8192 ? launch_norm<E, 8, 2, 1, 512, 1, true>(a, st) : -13;
    }
    if (per_group % 4 == 0) return a.H <= 8192 ? launch_norm<E, 4, 4, 1, 512, 1, true>(a, st) : -13;
    return a.H <= 4096 ? launch_norm<E, 1, 8, 1, 512, 1, true>(a, st) : -13;
  }
  if (!a.conv && per_group % 8 == 0) {          // no convolution: no window of earlier rows in registers
    if (a.T > 256 && a.H <= 2048) return launch_norm<E, 8, 1, 1, 256, 4>(a, st);
    if (a.T > 256 && a.H <= 4096) return launch_norm<E, 8, 2, 1, 256, 3>(a, st);
    if (a.H <= 4096) return launch_norm<E, 8, 1, 1, 512, 1>(a, st);
    if (a.H <= 8192) return launch_norm<E, 8, 2, 1, 512, 1>(a, st);
    return -13;
  }
  if (few && per_group % 8 == 0) {
    // eight channels per thread: a thread's channels share their group, so one reduction serves them all
    // prompts: several blocks per SM, each at its own token, hide the loads and barriers; decode: one block per token
    if (a.T > 256 && a.H <= 2048) return launch_norm<E, 8, 1, 4, 256, 3>(a, st);
    if (a.T > 256 && a.H <= 4096) return launch_norm<E, 8, 2, 4, 256, 2>(a, st);
    if (a.H <= 4096) return launch_norm<E, 8, 1, 4, 512, 1>(a, st);
    if (a.H <= 8192) return launch_norm<E, 8, 2, 4, 512, 1>(a, st);
    return -13;
  }
  if (per_group % 4 == 0) {
    if (a.H <= 2048) return few ? launch_norm<E, 4, 1, 4, 512, 1>(a, st) : launch_norm<E, 4, 1, 16, 512, 1>(a, st);
    if (a.H <= 8192) return few ? launch_norm<E, 4, 4, 4, 512, 1>(a, st) : launch_norm<E, 4, 4, 16, 512, 1>(a, st);
    return -13;
  }
  if (a.H > 4096) return -13;
  return few ? launch_norm<E, 1, 8, 4, 512, 1>(a, st) : launch_norm<E, 1, 8, 16, 512, 1>(a, st);
}

}  // namespace cafd
