// Gated delta rule over prompt portions in chunks of 64 tokens.
//
// Within a chunk (G the running sum of log decays, S the state before it) the recurrence
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// has the closed form
//     (I + L) u = beta (v - e^G S^T k)          L_ij = beta_i (k_i . k_j) e^(G_i - G_j),  j < i
//     o_i = e^(G_i) S^T q_i + sum_(j <= i) (q_i . k_j) e^(G_i - G_j) u_j
//     S  <- e^(G_63) S + sum_j e^(G_63 - G_j) k_j u_j^T
// so with T = (I + L)^-1, W = T (beta e^G k), U = T (beta v), P_ij = (q_i . k_j) e^(G_i - G_j):
//     u = U - W S,   o = (e^G q) S + P u,   S <- e^(G_63) S + (e^(G_63 - G) k)^T u.
//
//   delta_prepare  one block per (chunk, head), all chunks at once: convolutions, silu, unit norms, decays, T, W, U, P
//   delta_scan     one block per (sequence, head, 32 state columns), chunk after chunk: the three lines above with the
//                  state in fp32 accumulators; the next chunk's operands are on their way while this one multiplies
//
// Everything that enters the recurrence stays at 32-bit accuracy: the operands of the tensor-core products are split into
// two bf16 halves (16 significant bits together) and multiplied as hi hi + hi lo + lo hi with fp32 accumulation; the
// triangular inverse, decays and norms are fp32.  delta_prepare leaves its results in the order of the mma fragments, so
// delta_scan loads operands straight into registers, 16 bytes per lane.
#include <type_traits>

#include "cafd_api.h"
#include "common.cuh"
#include "delta.cuh"

namespace cafd {

constexpr int kChunk = 64;
constexpr int kSlice = 32;            // state columns per block of delta_scan
constexpr int kChunkThreads = 256;
constexpr int kTPitch = 68;
constexpr float kLogTiny = -104.f;    // e^-104 is below the smallest fp32 number: decays under it are zero

struct ChunkBufs {
  uint4* w;       // [unit][4][D / 16][2][32]
  uint4* q;       // [unit][4][D / 16][2][32]
  uint4* k;       // [unit][D / 16][4][2][32]
  uint4* p;       // [unit][4][4][2][32]
  float4* u;      // [unit][4][vdim / 8][32]
  float* g;       // [unit]: decay over the whole chunk
  int chunk0;     // first chunk of this slab
  int chunks;     // chunks of a slab
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Four neighbouring n tiles of a split product: hi hi, hi lo and lo hi over all four in turn, so that no product waits for
// the one before it.
__device__ __forceinline__ void mma_split4(float (*c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[2][4],
                                           const uint32_t (&bl)[2][4]) {
#pragma unroll
  for (int nt = 0; nt < 4; ++nt) mma16816(c[nt], ah, bh[nt >> 1][(nt & 1) * 2], bh[nt >> 1][(nt & 1) * 2 + 1]);
#pragma unroll
  for (int nt = 0; nt < 4; ++nt) mma16816(c[nt], ah, bl[nt >> 1][(nt & 1) * 2], bl[nt >> 1][(nt & 1) * 2 + 1]);
#pragma unroll
  for (int nt = 0; nt < 4; ++nt) mma16816(c[nt], al, bh[nt >> 1][(nt & 1) * 2], bh[nt >> 1][(nt & 1) * 2 + 1]);
}
// two values -> packed high halves and packed low halves
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
// silu on the special-function unit; the clamp keeps the denominator finite (below -80 the result rounds to zero anyway)
__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.0f + __expf(fminf(-x, 80.f))); }
__device__ __forceinline__ uint4 as4(const uint32_t (&r)[4]) { return make_uint4(r[0], r[1], r[2], r[3]); }

// Chunk `c` of the step -> its sequence and place.  False past the last chunk.
__device__ __forceinline__ bool find_chunk(const int* q_start, int S, int c, int& seq, int& t0, int& len, int& off) {
  for (seq = 0; seq < S; ++seq) {
    t0 = q_start[seq];
    len = q_start[seq + 1] - t0;
    const int n = (len + kChunk - 1) / kChunk;
    if (c < n) { off = c * kChunk; return true; }
    c -= n;
  }
  return false;
}

template <int D>
__global__ void __launch_bounds__(kChunkThreads, 2) delta_prepare_kernel(const DeltaArgs p, const ChunkBufs b) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  constexpr int kP = D + 8;                               // row pitch in elements
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* kl = kh + kChunk * kP;
  __nv_bfloat16* yh = kl + kChunk * kP;                   // q, then 64 columns of v at a time
  __nv_bfloat16* yl = yh + kChunk * kP;
  float* Lm = reinterpret_cast<float*>(yl + kChunk * kP); // [64][kTPitch]
  float* Tm = Lm + kChunk * kTPitch;
  __shared__ float sG[kChunk], sB[kChunk], sIq[kChunk], sIk[kChunk], sW[kChunk], sE[kChunk];

  pdl_wait();
  pdl_trigger();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y;
  int seq, t0, len, off;
  if (!find_chunk(p.q_start, p.S, b.chunk0 + blockIdx.x, seq, t0, len, off)) return;
  const int n_tok = min(kChunk, len - off);
  const size_t unit = static_cast<size_t>(blockIdx.x) * p.heads + h;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj);
  const float* st_in = p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + p.c_off;
  const int rep = p.heads / p.kv_heads, kvh = h / rep;
  const int kd = p.kv_heads * p.dim, channels = 2 * kd + p.heads * p.vdim;

  // convolution + silu of kCols channels from channel `chan0` (column src0 of the projection) into hi / lo tiles: a thread
  // takes two channels of kPer consecutive tokens, all their loads in flight at once
  auto conv = [&](auto cols_c, __nv_bfloat16* dh, __nv_bfloat16* dl, int src0, int chan0) {
    constexpr int kCols = decltype(cols_c)::value, kPairs = kCols / 2, kGroups = kChunkThreads / kPairs, kPer = kChunk / kGroups;
    const int pr = tid % kPairs, grp = tid / kPairs;
    const int c = chan0 + 2 * pr, i0 = off + grp * kPer;
    const __nv_bfloat16* src = proj + static_cast<size_t>(t0) * p.ld + src0 + 2 * pr;
    uint32_t raw[kPer + 3];
#pragma unroll
    for (int j = 0; j < kPer + 3; ++j) {
      const int i = min(max(i0 - 3 + j, 0), len - 1);
      raw[j] = *reinterpret_cast<const uint32_t*>(src + static_cast<size_t>(i) * p.ld);
    }
    float w0[4], w1[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int tap = j - (4 - p.taps);
      w0[j] = tap >= 0 ? p.conv_w[static_cast<size_t>(c) * p.taps + tap] : 0.f;
      w1[j] = tap >= 0 ? p.conv_w[static_cast<size_t>(c + 1) * p.taps + tap] : 0.f;
    }
    float x0[4], x1[4];
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      const int i = i0 - 3 + j;
      x0[j + 1] = bf16_lo(raw[j]); x1[j + 1] = bf16_hi(raw[j]);
      if (i < 0) {                                          // before the portion: the state's inputs
        const bool have = i + p.taps - 1 >= 0;
        const float* s = st_in + static_cast<size_t>(have ? i + p.taps - 1 : 0) * channels + c;
        x0[j + 1] = have ? s[0] : 0.f; x1[j + 1] = have ? s[1] : 0.f;
      }
    }
#pragma unroll
    for (int r = 0; r < kPer; ++r) {
#pragma unroll
      for (int j = 0; j < 3; ++j) { x0[j] = x0[j + 1]; x1[j] = x1[j + 1]; }
      x0[3] = bf16_lo(raw[r + 3]); x1[3] = bf16_hi(raw[r + 3]);
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) { y0 = fmaf(w0[j], x0[j], y0); y1 = fmaf(w1[j], x1[j], y1); }
      const bool live = i0 + r < len;
      y0 = live ? silu_fast(y0) : 0.f;
      y1 = live ? silu_fast(y1) : 0.f;
      uint32_t hi, lo;
      split2(y0, y1, hi, lo);
      const int at = (grp * kPer + r) * kP + 2 * pr;
      *reinterpret_cast<uint32_t*>(dh + at) = hi;
      *reinterpret_cast<uint32_t*>(dl + at) = lo;
    }
  };

  if (warp == 0) {                                          // decays, step sizes and their running sums
    const float a_scale = -expf(p.A_log[h]), dt = p.dt_bias[h];
    float lg[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = 2 * lane + j;
      lg[j] = 0.f;
      float be = 0.f;
      if (i < n_tok) {
        const __nv_bfloat16* row = proj + static_cast<size_t>(t0 + off + i) * p.ld;
        lg[j] = fmaxf(a_scale * softplus(__bfloat162float(row[p.a_off + h]) + dt), kLogTiny);
        be = sigmoid_f(__bfloat162float(row[p.b_off + h]));
      }
      sB[i] = be;
    }
    float run = lg[0] + lg[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    sG[2 * lane] = run - lg[1];
    sG[2 * lane + 1] = run;
  }
  conv(std::integral_constant<int, D>{}, kh, kl, p.k_off + kvh * D, kd + kvh * D);
  conv(std::integral_constant<int, D>{}, yh, yl, p.q_off + kvh * D, kvh * D);
  __syncthreads();
  // inverse norms of q (with 1 / sqrt(dim)) and k
  for (int r = warp; r < 2 * kChunk; r += 8) {
    const bool is_q = r >= kChunk;
    const __nv_bfloat16* hh = (is_q ? yh : kh) + (r & 63) * kP;
    const __nv_bfloat16* ll = (is_q ? yl : kl) + (r & 63) * kP;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < D / 32; ++i) {
      const float v = __bfloat162float(hh[lane + 32 * i]) + __bfloat162float(ll[lane + 32 * i]);
      s = fmaf(v, v, s);
    }
    s = warp_sum(s);
    if (lane == 0) {
      if (is_q) sIq[r & 63] = 1.0f / (sqrtf(s + 1e-6f) * sqrtf(static_cast<float>(D)));
      else {
        const float ik = 1.0f / sqrtf(s + 1e-6f), G = sG[r];
        sIk[r] = ik;
        sW[r] = sB[r] * ik * expf(G);                       // beta e^G / |k|
        sE[r] = ik * expf(sG[kChunk - 1] - G);              // e^(G_63 - G) / |k|
      }
    }
  }
  __syncthreads();

  const int m0 = (warp & 3) * 16, nh = warp >> 2;           // this warp's 16 rows and half of the columns
  const int gr = lane >> 2, tc = (lane & 3) * 2;
  const int r_lo = m0 + gr, r_hi = r_lo + 8;
  const float G_lo = sG[r_lo], G_hi = sG[r_hi];
  {
    // K K^T -> L (strictly lower) and Q K^T -> P (lower), 64 x 64 each
    float ck[4][4] = {}, cq[4][4] = {};
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t ah[4], al[4], qh[4], ql[4];
      const int ao = (m0 + (lane & 15)) * kP + ks * 16 + (lane >> 4) * 8;
      ldsm4(ah, kh + ao); ldsm4(al, kl + ao); ldsm4(qh, yh + ao); ldsm4(ql, yl + ao);
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
        uint32_t bh[4], bl[4];
        const int bo = (nh * 32 + nn * 16 + (lane >> 4) * 8 + (lane & 7)) * kP + ks * 16 + ((lane >> 3) & 1) * 8;
        ldsm4(bh, kh + bo); ldsm4(bl, kl + bo);
        // (neighbouring products go to different accumulators: one that waits for the previous would stall the warp)
#pragma unroll
        for (int term = 0; term < 3; ++term) {
          const uint32_t (&bb)[4] = term == 1 ? bl : bh;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma16816(ck[2 * nn + e], term == 2 ? al : ah, bb[2 * e], bb[2 * e + 1]);
            mma16816(cq[2 * nn + e], term == 2 ? ql : qh, bb[2 * e], bb[2 * e + 1]);
          }
        }
      }
    }
    const float bk_lo = sB[r_lo] * sIk[r_lo], bk_hi = sB[r_hi] * sIk[r_hi], iq_lo = sIq[r_lo], iq_hi = sIq[r_hi];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = nh * 32 + nt * 8 + tc + e;
        const float Gc = sG[col], ikc = sIk[col];
        const float d_lo = col <= r_lo ? expf(G_lo - Gc) * ikc : 0.f, d_hi = col <= r_hi ? expf(G_hi - Gc) * ikc : 0.f;
        Lm[r_lo * kTPitch + col] = col < r_lo ? ck[nt][e] * bk_lo * d_lo : 0.f;
        Lm[r_hi * kTPitch + col] = col < r_hi ? ck[nt][2 + e] * bk_hi * d_hi : 0.f;
        cq[nt][e] *= iq_lo * d_lo;
        cq[nt][2 + e] *= iq_hi * d_hi;
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {                           // accumulator tiles 2j, 2j + 1 = one A fragment
      uint32_t hi[4], lo[4];
      split2(cq[2 * j][0], cq[2 * j][1], hi[0], lo[0]);
      split2(cq[2 * j][2], cq[2 * j][3], hi[1], lo[1]);
      split2(cq[2 * j + 1][0], cq[2 * j + 1][1], hi[2], lo[2]);
      split2(cq[2 * j + 1][2], cq[2 * j + 1][3], hi[3], lo[3]);
      uint4* dst = b.p + ((unit * 4 + (m0 >> 4)) * 4 + nh * 2 + j) * 64 + lane;
      dst[0] = as4(hi);
      dst[32] = as4(lo);
    }
  }
  // e^G q as A fragments (rows = tokens): the two warps of a row tile take alternate k steps
  {
    const float s_lo = sIq[r_lo] * expf(G_lo), s_hi = sIq[r_hi] * expf(G_hi);
#pragma unroll
    for (int ks = nh; ks < D / 16; ks += 2) {
      uint32_t ah[4], al[4], hi[4], lo[4];
      const int ao = (m0 + (lane & 15)) * kP + ks * 16 + (lane >> 4) * 8;
      ldsm4(ah, yh + ao); ldsm4(al, yl + ao);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float s = (e & 1) ? s_hi : s_lo;
        split2((bf16_lo(ah[e]) + bf16_lo(al[e])) * s, (bf16_hi(ah[e]) + bf16_hi(al[e])) * s, hi[e], lo[e]);
      }
      uint4* dst = b.q + ((unit * 4 + (m0 >> 4)) * (D / 16) + ks) * 64 + lane;
      dst[0] = as4(hi);
      dst[32] = as4(lo);
    }
  }
  const float G_end = sG[kChunk - 1];
  // (e^(G_63 - G) k)^T as A fragments (rows = dims, k = tokens)
  for (int i = warp; i < (D / 16) * 4; i += 8) {
    const int mt = i >> 2, ks = i & 3;
    uint32_t ah[4], al[4], hi[4], lo[4];
    const int q = lane >> 3;
    const int ao = (ks * 16 + (q >> 1) * 8 + (lane & 7)) * kP + mt * 16 + (q & 1) * 8;
    ldsm4t(ah, kh + ao); ldsm4t(al, kl + ao);
    float s[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = ks * 16 + (e >> 1) * 8 + tc + (e & 1);
      s[e] = sE[t];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
      split2((bf16_lo(ah[e]) + bf16_lo(al[e])) * s[(e >> 1) * 2], (bf16_hi(ah[e]) + bf16_hi(al[e])) * s[(e >> 1) * 2 + 1], hi[e], lo[e]);
    uint4* dst = b.k + ((unit * (D / 16) + mt) * 4 + ks) * 64 + lane;
    dst[0] = as4(hi);
    dst[32] = as4(lo);
  }
  if (tid == 0) b.g[unit] = expf(G_end);
  __syncthreads();                                          // L complete; q is done with

  // T = (I + L)^-1: the four 16 x 16 diagonal blocks, then block rows below them; the blocks above the diagonal of Tm
  // hold the intermediate products
  if (tid < 64) {
    const int o = tid & ~15, j = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = i == j ? 1.f : 0.f;
#pragma unroll
      for (int k = 0; k < i; ++k) s = fmaf(-Lm[(o + i) * kTPitch + o + k], x[k], s);
      x[i] = s;
      Tm[(o + i) * kTPitch + o + j] = s;
    }
  }
  __syncthreads();
  for (int d = 1; d < 4; ++d) {
    const int er = tid >> 4, ec = tid & 15;
    for (int j = 0; j + d < 4; ++j) {
      const int i = j + d;
      float s = 0.f;
      for (int k = 16 * j; k < 16 * i; ++k) s = fmaf(Lm[(16 * i + er) * kTPitch + k], Tm[k * kTPitch + 16 * j + ec], s);
      Tm[(16 * j + er) * kTPitch + 16 * i + ec] = s;        // above the diagonal: block (j, i)
    }
    __syncthreads();
    for (int j = 0; j + d < 4; ++j) {
      const int i = j + d;
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < 16; ++k) s = fmaf(Tm[(16 * i + er) * kTPitch + 16 * i + k], Tm[(16 * j + k) * kTPitch + 16 * i + ec], s);
      Tm[(16 * i + er) * kTPitch + 16 * j + ec] = -s;
    }
    __syncthreads();
  }

  // a row tile of T with its columns scaled, as A fragments; only the blocks on and below the diagonal
  auto t_frag = [&](int ks, bool with_k, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = (e & 1) ? r_hi : r_lo, col = ks * 16 + (e >> 1) * 8 + tc;
      const float2 v = *reinterpret_cast<const float2*>(Tm + row * kTPitch + col);
      const float s0 = with_k ? sW[col] : sB[col], s1 = with_k ? sW[col + 1] : sB[col + 1];
      split2(v.x * s0, v.y * s1, hi[e], lo[e]);
    }
  };
  const int mt = m0 >> 4;
  {
    // W = T (beta e^G k): this warp's half of the D columns
    constexpr int NT = D / 16;                              // n tiles of 8 per warp
    float c[NT][4] = {};
    for (int ks = 0; ks <= mt; ++ks) {
      uint32_t ah[4], al[4];
      t_frag(ks, true, ah, al);
#pragma unroll
      for (int n0 = 0; n0 < NT / 2; n0 += 2) {
        uint32_t bh[2][4], bl[2][4];
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          const int bo = (ks * 16 + (lane & 15)) * kP + nh * (D / 2) + (n0 + nn) * 16 + (lane >> 4) * 8;
          ldsm4t(bh[nn], kh + bo); ldsm4t(bl[nn], kl + bo);
        }
        mma_split4(&c[2 * n0], ah, al, bh, bl);
      }
    }
#pragma unroll
    for (int j = 0; j < NT / 2; ++j) {
      uint32_t hi[4], lo[4];
      split2(c[2 * j][0], c[2 * j][1], hi[0], lo[0]);
      split2(c[2 * j][2], c[2 * j][3], hi[1], lo[1]);
      split2(c[2 * j + 1][0], c[2 * j + 1][1], hi[2], lo[2]);
      split2(c[2 * j + 1][2], c[2 * j + 1][3], hi[3], lo[3]);
      uint4* dst = b.w + ((unit * 4 + mt) * (D / 16) + nh * (D / 32) + j) * 64 + lane;
      dst[0] = as4(hi);
      dst[32] = as4(lo);
    }
  }
  for (int v0 = 0; v0 < p.vdim; v0 += 64) {
    const int cols = min(64, p.vdim - v0);
    if (v0) __syncthreads();
    const int v_src = p.v_off + h * p.vdim + v0, v_chan = 2 * kd + h * p.vdim + v0;
    if (cols == 64) conv(std::integral_constant<int, 64>{}, yh, yl, v_src, v_chan);
    else conv(std::integral_constant<int, 32>{}, yh, yl, v_src, v_chan);
    __syncthreads();
    if (nh * 32 < cols) {
      float c[4][4] = {};
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t ah[4], al[4];
        t_frag(ks, false, ah, al);
        uint32_t bh[2][4], bl[2][4];
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          const int bo = (ks * 16 + (lane & 15)) * kP + nh * 32 + nn * 16 + (lane >> 4) * 8;
          ldsm4t(bh[nn], yh + bo); ldsm4t(bl[nn], yl + bo);
        }
        mma_split4(c, ah, al, bh, bl);
      }
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
        b.u[((unit * 4 + mt) * (p.vdim >> 3) + ((v0 + nh * 32) >> 3) + nt) * 32 + lane] = make_float4(c[nt][0], c[nt][1], c[nt][2], c[nt][3]);
    }
  }
  // the sequence's last chunk leaves the convolutions' last inputs in the new state
  if (off + n_tok == len && p.taps > 1) {
    float* st_out = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + p.c_off;
    const int n_ch = 2 * D + p.vdim;
    for (int i = tid; i < n_ch * (p.taps - 1); i += kChunkThreads) {
      const int r = i / n_ch, cc = i - r * n_ch;
      int chan, src;
      if (cc < 2 * D) {
        if (h != kvh * rep) continue;
        const int k_part = cc >= D;
        chan = k_part * kd + kvh * D + (cc - k_part * D);
        src = (k_part ? p.k_off : p.q_off) + kvh * D + (cc - k_part * D);
      } else {
        chan = 2 * kd + h * p.vdim + cc - 2 * D;
        src = p.v_off + h * p.vdim + cc - 2 * D;
      }
      const int tt = len - (p.taps - 1) + r;
      st_out[static_cast<size_t>(r) * channels + chan] =
          tt >= 0 ? __bfloat162float(proj[static_cast<size_t>(t0 + tt) * p.ld + src]) : st_in[static_cast<size_t>(tt + p.taps - 1) * channels + chan];
    }
  }
}

template <int D>
__global__ void __launch_bounds__(kChunkThreads, 1) delta_scan_kernel(const DeltaArgs p, const ChunkBufs b) {
  constexpr int kKS = D / 16, kSP = kSlice + 8;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* sh = reinterpret_cast<__nv_bfloat16*>(smem_raw);   // the state's halves [D][kSP] each, then u's [64][kSP]
  __nv_bfloat16* sl = sh + D * kSP;
  __nv_bfloat16* vh = sl + D * kSP;
  __nv_bfloat16* vl = vh + kChunk * kSP;
  uint4* ring = reinterpret_cast<uint4*>(vl + kChunk * kSP);        // per warp and parity: K fragments, then P fragments or U
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.x, v0 = blockIdx.y * kSlice, seq = blockIdx.z;
  int c0 = 0;                                               // the sequence's first chunk
  for (int s = 0; s < seq; ++s) c0 += (p.q_start[s + 1] - p.q_start[s] + kChunk - 1) / kChunk;
  const int t0 = p.q_start[seq], len = p.q_start[seq + 1] - t0;
  const int c_lo = max(c0, b.chunk0), c_hi = min(c0 + (len + kChunk - 1) / kChunk, b.chunk0 + b.chunks);
  if (c_lo >= c_hi) return;
  const int mt = warp & 3, gr = lane >> 2, tc = (lane & 3) * 2;
  const bool first = warp < 4;                              // warps 0-3: u = U - W S; warps 4-7: o
  const bool holds = warp < D / 16;                         // this warp keeps state rows [16 warp, 16 warp + 16)

  const float* st = p.state + static_cast<size_t>(c_lo == c0 ? p.state_in[seq] : p.state_out[seq]) * p.slot_stride;
  const size_t s_at = p.s_off + (static_cast<size_t>(h) * D + 16 * warp + gr) * p.vdim + v0 + tc;
  float S[4][4];
  auto put_state = [&]() {                                  // the state's two halves for the next chunk's products
    if (holds) {
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        uint32_t hi, lo;
        const int at = (16 * warp + gr) * kSP + nt * 8 + tc;
        split2(S[nt][0], S[nt][1], hi, lo);
        *reinterpret_cast<uint32_t*>(sh + at) = hi;
        *reinterpret_cast<uint32_t*>(sl + at) = lo;
        split2(S[nt][2], S[nt][3], hi, lo);
        *reinterpret_cast<uint32_t*>(sh + at + 8 * kSP) = hi;
        *reinterpret_cast<uint32_t*>(sl + at + 8 * kSP) = lo;
      }
    }
  };
  if (holds) {
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      const float2 a = *reinterpret_cast<const float2*>(st + s_at + nt * 8), c = *reinterpret_cast<const float2*>(st + s_at + 8 * static_cast<size_t>(p.vdim) + nt * 8);
      S[nt][0] = a.x; S[nt][1] = a.y; S[nt][2] = c.x; S[nt][3] = c.y;
    }
  }
  put_state();

  // operands of the first product, always one chunk ahead
  uint4 fa[kKS][2];
  auto load_a = [&](int c) {
    const size_t unit = static_cast<size_t>(c - b.chunk0) * p.heads + h;
    const uint4* src = (first ? b.w : b.q) + (unit * 4 + mt) * kKS * 64 + lane;
#pragma unroll
    for (int ks = 0; ks < kKS; ++ks) { fa[ks][0] = __ldcg(src + ks * 64); fa[ks][1] = __ldcg(src + ks * 64 + 32); }
  };
  // operands of the second half travel through shared memory, also one chunk ahead; a warp reads only what its own lanes
  // copied, so waiting for the copies is all the ordering they need
  constexpr int kRing = 512;                                // uint4 per warp and parity: 256 K, 256 P (or 128 U)
  auto copy_b = [&](int c) {
    const size_t unit = static_cast<size_t>(c - b.chunk0) * p.heads + h;
    uint4* dst = ring + ((c & 1) * 8 + warp) * kRing + lane;
    auto cp = [&](uint4* d, const void* s) {
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(d)), "l"(s) : "memory");
    };
    if (holds) {
      const uint4* src = b.k + (unit * kKS + warp) * 4 * 64 + lane;
#pragma unroll
      for (int i = 0; i < 8; ++i) cp(dst + i * 32, src + i * 32);
    }
    if (first) {
      const float4* src = b.u + ((unit * 4 + mt) * (p.vdim >> 3) + (v0 >> 3)) * 32 + lane;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) cp(dst + 256 + nt * 32, src + nt * 32);
    } else {
      const uint4* src = b.p + (unit * 4 + mt) * 4 * 64 + lane;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if ((i >> 1) <= mt) cp(dst + 256 + i * 32, src + i * 32);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_a(c_lo);
  copy_b(c_lo);
  __syncthreads();
  for (int c = c_lo; c < c_hi; ++c) {
    const size_t unit = static_cast<size_t>(c - b.chunk0) * p.heads + h;
    const float g_end = __ldcg(b.g + unit);
    const uint4* mine = ring + ((c & 1) * 8 + warp) * kRing + lane;
    float acc[4][4] = {};
#pragma unroll
    for (int ks = 0; ks < kKS; ++ks) {
      const uint32_t ah[4] = {fa[ks][0].x, fa[ks][0].y, fa[ks][0].z, fa[ks][0].w}, al[4] = {fa[ks][1].x, fa[ks][1].y, fa[ks][1].z, fa[ks][1].w};
      uint32_t bh[2][4], bl[2][4];
#pragma unroll
      for (int nn = 0; nn < 2; ++nn) {
        const int bo = (ks * 16 + (lane & 15)) * kSP + nn * 16 + (lane >> 4) * 8;
        ldsm4t(bh[nn], sh + bo); ldsm4t(bl[nn], sl + bo);
      }
      mma_split4(acc, ah, al, bh, bl);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
    if (c + 1 < c_hi) {
      load_a(c + 1);
      copy_b(c + 1);
    }
    if (first) {
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        uint32_t hi, lo;
        const int at = (16 * mt + gr) * kSP + nt * 8 + tc;
        const float4 u = *reinterpret_cast<const float4*>(mine + 256 + nt * 32);
        split2(u.x - acc[nt][0], u.y - acc[nt][1], hi, lo);
        *reinterpret_cast<uint32_t*>(vh + at) = hi;
        *reinterpret_cast<uint32_t*>(vl + at) = lo;
        split2(u.z - acc[nt][2], u.w - acc[nt][3], hi, lo);
        *reinterpret_cast<uint32_t*>(vh + at + 8 * kSP) = hi;
        *reinterpret_cast<uint32_t*>(vl + at + 8 * kSP) = lo;
      }
    }
    __syncthreads();                                        // u is there, and nobody reads the old state any more
    if (holds) {
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= g_end;
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      const bool want_o = !first && ks <= mt;
      if (holds || want_o) {
        uint32_t bh[2][4], bl[2][4];
#pragma unroll
        for (int nn = 0; nn < 2; ++nn) {
          const int bo = (ks * 16 + (lane & 15)) * kSP + nn * 16 + (lane >> 4) * 8;
          ldsm4t(bh[nn], vh + bo); ldsm4t(bl[nn], vl + bo);
        }
        auto mul = [&](float (&d)[4][4], const uint4& fh, const uint4& fl) {
          const uint32_t ah[4] = {fh.x, fh.y, fh.z, fh.w}, al[4] = {fl.x, fl.y, fl.z, fl.w};
          mma_split4(d, ah, al, bh, bl);
        };
        if (holds) mul(S, mine[ks * 64], mine[ks * 64 + 32]);
        if (want_o) mul(acc, mine[256 + ks * 64], mine[256 + ks * 64 + 32]);
      }
    }
    put_state();
    if (!first) {
      const int row = (c - c0) * kChunk + 16 * mt + gr;
      float* o = p.raw + (static_cast<size_t>(t0 + row) * p.heads + h) * p.vdim + v0 + tc;
      const size_t step8 = static_cast<size_t>(8) * p.heads * p.vdim;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        if (row < len) *reinterpret_cast<float2*>(o + nt * 8) = make_float2(acc[nt][0], acc[nt][1]);
        if (row + 8 < len) *reinterpret_cast<float2*>(o + step8 + nt * 8) = make_float2(acc[nt][2], acc[nt][3]);
      }
    }
    __syncthreads();                                        // the new state is there, and nobody reads u any more
  }
  if (holds) {
    float* so = p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      *reinterpret_cast<float2*>(so + s_at + nt * 8) = make_float2(S[nt][0], S[nt][1]);
      *reinterpret_cast<float2*>(so + s_at + 8 * static_cast<size_t>(p.vdim) + nt * 8) = make_float2(S[nt][2], S[nt][3]);
    }
  }
}

constexpr size_t unit_bytes(int D, int vdim) {
  return static_cast<size_t>(4) * (D / 16) * 1024 * 2 + (D / 16) * 4 * 1024 + 16 * 1024 + static_cast<size_t>(4) * (vdim / 8) * 512 + 16;
}

template <int D>
static int launch_chunks(const DeltaArgs& p, void* scratch, long long scratch_bytes, cudaStream_t st) {
  constexpr size_t smem = static_cast<size_t>(4) * kChunk * (D + 8) * 2 + 2 * kChunk * kTPitch * 4;
  constexpr size_t scan_smem = static_cast<size_t>(2 * D + 2 * kChunk) * (kSlice + 8) * 2 + 2 * 8 * 512 * 16;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(delta_scan_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(scan_smem)));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(delta_prepare_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    attr = true;
  }
  const size_t per_chunk = unit_bytes(D, p.vdim) * p.heads;
  int slab = static_cast<int>(scratch_bytes / per_chunk);
  if (slab < 1) return -14;
  const int total = (p.T + (kChunk - 1) * p.S) / kChunk;    // every portion ends in at most one chunk that is not full
  const int wave = 2 * 148 / p.heads;                       // chunks whose blocks fill the GPU once (two per SM)
  if (wave > 0 && slab > wave) {                            // whole waves of delta_prepare per slab
    int waves = slab * p.heads / (2 * 148);
    slab = waves * 2 * 148 / p.heads;
  }
  if (slab > total) slab = total;
  const size_t units = static_cast<size_t>(slab) * p.heads;
  ChunkBufs b;
  uint4* base = static_cast<uint4*>(scratch);
  b.w = base;
  b.q = b.w + units * 4 * (D / 16) * 64;
  b.k = b.q + units * 4 * (D / 16) * 64;
  b.p = b.k + units * 4 * (D / 16) * 64;
  b.u = reinterpret_cast<float4*>(b.p + units * 16 * 64);
  b.g = reinterpret_cast<float*>(b.u + units * 4 * (p.vdim / 8) * 32);
  b.chunks = slab;
  for (b.chunk0 = 0; b.chunk0 < total; b.chunk0 += slab) {
    const int n = total - b.chunk0 < slab ? total - b.chunk0 : slab;
    launch_pdl(delta_prepare_kernel<D>, dim3(n, p.heads), dim3(kChunkThreads), smem, st, p, b);
    launch_pdl(delta_scan_kernel<D>, dim3(p.heads, p.vdim / kSlice, p.S), dim3(kChunkThreads), scan_smem, st, p, b);
  }
  const long long rows = static_cast<long long>(p.T) * p.heads;
  const int blocks = static_cast<int>(rows < 8 * 148 * 8 ? (rows + 7) / 8 : 148 * 8);
  launch_pdl(delta_out_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, st, p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace cafd

using namespace cafd;

// Bytes of scratch one 64-token chunk of every head takes; the call works in slabs of as many chunks as fit.
extern "C" long long cafd_delta_chunk_bytes(int heads, int dim, int vdim) { return static_cast<long long>(unit_bytes(dim, vdim)) * heads; }

// The chunked form of cafd_delta_step: bf16 activations, dim 64 or 128, vdim a multiple of 32, at most four taps.  raw
// [T, heads * vdim] fp32 holds o before the output norm.
extern "C" int cafd_delta_chunked(const DeltaArgs* p, void* scratch, long long scratch_bytes, cafd_stream_t s) {
  if (p->T <= 0) return 0;
  if (p->S < 1 || p->kv_heads < 1 || p->heads % p->kv_heads || (p->dim != 64 && p->dim != 128) || p->vdim % kSlice || p->taps < 1 || p->taps > 4)
    return -10;
  if (!p->raw || !p->out || !scratch || (p->slot_stride & 1) || (p->s_off & 1) || (p->ld & 1) || ((p->q_off | p->k_off | p->v_off) & 1)) return -11;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return p->dim == 64 ? launch_chunks<64>(*p, scratch, scratch_bytes, st) : launch_chunks<128>(*p, scratch, scratch_bytes, st);
}
