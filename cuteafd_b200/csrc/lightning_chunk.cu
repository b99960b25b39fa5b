// Linear attention over prompt portions in chunks of 128 tokens.  With S the state before a chunk of n tokens,
//     o_i = decay^(i + 1) S^T q_i + sum_(j <= i) decay^(i - j) (q_i . k_j) v_j
//     S  <- decay^n S + sum_j decay^(n - 1 - j) k_j v_j^T
//
//   chunk_states   block per (chunk, head, run of columns): the sum that the chunk adds to the state
//   chunk_prefix   thread per four state cells of a (sequence, head): walks the sequence's chunks, leaves the state before each in place
//                  of its sum and writes the sequence's new state
//   chunk_outputs  block per (chunk, head, run of columns): the first line above
//
// q, k and v are rounded to bf16 after their silu; everything they are multiplied with stays at 32-bit accuracy: states, decays and
// scores enter the tensor-core products split into two bf16 halves, accumulation is fp32.  mma.sync and not tcgen05: the split operands
// come from registers and shared memory that the block has just computed.
#include "cafd_api.h"
#include "common.cuh"
#include "delta.cuh"
#include "lightning.cuh"

namespace cafd {

constexpr int kLc = 128;            // tokens per chunk
constexpr int kLcThreads = 256;

__device__ __forceinline__ void lc_ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lc_ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void lc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lc_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
__device__ __forceinline__ float lc_silu(float x) { return __fdividef(x, 1.0f + __expf(fminf(-x, 80.f))); }

// Chunk `c` of the step -> its sequence, first row and length.  False past the last chunk.
__device__ __forceinline__ bool lc_find(const int* q_start, int S, int c, int& row0, int& n) {
  for (int s = 0; s < S; ++s) {
    const int t0 = q_start[s], len = q_start[s + 1] - t0, k = (len + kLc - 1) / kLc;
    if (c < k) { row0 = t0 + c * kLc; n = min(kLc, len - c * kLc); return true; }
    c -= k;
  }
  return false;
}

// silu of kCols columns of the chunk's rows into a bf16 tile; rows past its end are zero.  With `w`: row j times w[n - 1 - j], split.
template <int kCols, bool kSplit>
__device__ __forceinline__ void lc_load(const __nv_bfloat16* src, int ld, int n, __nv_bfloat16* hi, __nv_bfloat16* lo, const float* w) {
  constexpr int kP = kCols + 8, kVec = kCols / 8, kIter = kLc * kVec / kLcThreads;
  uint4 raw[kIter];
#pragma unroll
  for (int it = 0; it < kIter; ++it) {
    const int i = threadIdx.x + it * kLcThreads, r = i / kVec, c = i - r * kVec;
    raw[it] = r < n ? *reinterpret_cast<const uint4*>(src + static_cast<size_t>(r) * ld + c * 8) : make_uint4(0, 0, 0, 0);
  }
#pragma unroll
  for (int it = 0; it < kIter; ++it) {
    const int i = threadIdx.x + it * kLcThreads, r = i / kVec, c = i - r * kVec;
    const uint32_t x[4] = {raw[it].x, raw[it].y, raw[it].z, raw[it].w};
    uint32_t h[4], l[4];
    const float f = kSplit && r < n ? w[n - 1 - r] : 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      h[e] = pack_bf16(lc_silu(bf16_lo(x[e])), lc_silu(bf16_hi(x[e])));
      if (kSplit) lc_split2(bf16_lo(h[e]) * f, bf16_hi(h[e]) * f, h[e], l[e]);
    }
    *reinterpret_cast<uint4*>(hi + r * kP + c * 8) = make_uint4(h[0], h[1], h[2], h[3]);
    if (kSplit) *reinterpret_cast<uint4*>(lo + r * kP + c * 8) = make_uint4(l[0], l[1], l[2], l[3]);
  }
}

template <int D, int VT>
__global__ void __launch_bounds__(kLcThreads, 2) lightning_chunk_states_kernel(const LightningArgs p) {
  extern __shared__ __align__(16) uint8_t lc_smem[];
  constexpr int kKP = D + 8, kVP = VT + 8, kRowTiles = D / 16, kNSplit = 8 / kRowTiles, kNT = VT / kNSplit / 16;   // pairs of n tiles per warp
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(lc_smem);
  __nv_bfloat16* vh = sk + kLc * kKP;
  __nv_bfloat16* vl = vh + kLc * kVP;
  __shared__ float pw[kLc];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, v0 = blockIdx.z * VT;
  if (tid < kLc) pw[tid] = powf(p.decay[h], static_cast<float>(tid));
  pdl_wait();
  pdl_trigger();
  int row0, n;
  if (!lc_find(p.q_start, p.S, blockIdx.x, row0, n)) return;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj) + static_cast<size_t>(row0) * p.ld;
  __syncthreads();
  lc_load<D, false>(proj + p.k_off + h * D, p.ld, n, sk, nullptr, nullptr);
  lc_load<VT, true>(proj + p.v_off + h * p.vdim + v0, p.ld, n, vh, vl, pw);
  __syncthreads();
  const int rt = warp % kRowTiles, ns = warp / kRowTiles;
  if (ns >= kNSplit) return;
  const int c0 = ns * (VT / kNSplit);
  float acc[2 * kNT][4];
#pragma unroll
  for (int i = 0; i < 2 * kNT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const int steps = (n + 15) / 16;
  for (int s = 0; s < steps; ++s) {
    // A = k^T: rows are channels, so the tile [token][channel] is read transposed; matrices (token half, channel half)
    uint32_t a[4];
    lc_ldsm4t(a, sk + (s * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * kKP + rt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int j = 0; j < kNT; ++j) {
      uint32_t bh[4], bl[4];
      const int off = (s * 16 + (lane & 15)) * kVP + c0 + j * 16 + (lane >> 4) * 8;
      lc_ldsm4t(bh, vh + off);
      lc_ldsm4t(bl, vl + off);
      lc_mma(acc[2 * j], a, bh[0], bh[1]);
      lc_mma(acc[2 * j + 1], a, bh[2], bh[3]);
      lc_mma(acc[2 * j], a, bl[0], bl[1]);
      lc_mma(acc[2 * j + 1], a, bl[2], bl[3]);
    }
  }
  float* dst = static_cast<float*>(p.scratch) + (static_cast<size_t>(blockIdx.x) * p.heads + h) * D * p.vdim + v0 + c0;
  const int r = rt * 16 + (lane >> 2), c = 2 * (lane & 3);
#pragma unroll
  for (int j = 0; j < 2 * kNT; ++j) {
    *reinterpret_cast<float2*>(dst + static_cast<size_t>(r) * p.vdim + j * 8 + c) = make_float2(acc[j][0], acc[j][1]);
    *reinterpret_cast<float2*>(dst + static_cast<size_t>(r + 8) * p.vdim + j * 8 + c) = make_float2(acc[j][2], acc[j][3]);
  }
}

// The state before a chunk is left as four high halves and then four low halves in each 16 bytes.
__global__ void __launch_bounds__(256) lightning_chunk_prefix_kernel(const LightningArgs p) {
  const int cells = p.dim * p.vdim / 4, i = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const float decay = p.decay[h], d128 = powf(decay, static_cast<float>(kLc));
  pdl_wait();
  pdl_trigger();
  const int len = p.q_start[seq + 1] - p.q_start[seq];
  if (i >= cells || len <= 0) return;
  int first = 0;
  for (int s = 0; s < seq; ++s) first += (p.q_start[s + 1] - p.q_start[s] + kLc - 1) / kLc;
  const int chunks = (len + kLc - 1) / kLc;
  const size_t at = p.s_off + (static_cast<size_t>(h) * cells + i) * 4;
  float4 S = *reinterpret_cast<const float4*>(p.state + static_cast<size_t>(p.state_in[seq]) * p.slot_stride + at);
  float4* sums = static_cast<float4*>(p.scratch) + (static_cast<size_t>(first) * p.heads + h) * cells + i;
  const size_t step = static_cast<size_t>(p.heads) * cells;
  constexpr int kAhead = 16;
  for (int c0 = 0; c0 < chunks; c0 += kAhead) {
    float4 x[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < chunks) x[j] = sums[(c0 + j) * step];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (c0 + j < chunks) {
        uint32_t h0, h1, l0, l1;
        lc_split2(S.x, S.y, h0, l0);
        lc_split2(S.z, S.w, h1, l1);
        *reinterpret_cast<uint4*>(sums + (c0 + j) * step) = make_uint4(h0, h1, l0, l1);
        const int n = min(kLc, len - (c0 + j) * kLc);
        const float f = n == kLc ? d128 : powf(decay, static_cast<float>(n));
        S.x = fmaf(f, S.x, x[j].x); S.y = fmaf(f, S.y, x[j].y); S.z = fmaf(f, S.z, x[j].z); S.w = fmaf(f, S.w, x[j].w);
      }
    }
  }
  *reinterpret_cast<float4*>(p.state + static_cast<size_t>(p.state_out[seq]) * p.slot_stride + at) = S;
}

template <int D, int VT>
__global__ void __launch_bounds__(kLcThreads, 2) lightning_chunk_outputs_kernel(const LightningArgs p) {
  extern __shared__ __align__(16) uint8_t lc_smem[];
  constexpr int kKP = D + 8, kVP = VT + 8, kNT = VT / 16;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(lc_smem);
  __nv_bfloat16* sh = sq + kLc * kKP;             // the state's halves, then k and v in their place
  __nv_bfloat16* sl = sh + D * kVP;
  __nv_bfloat16* sk = sh;
  __nv_bfloat16* sv = sk + kLc * kKP;
  __shared__ float pw[kLc + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, v0 = blockIdx.z * VT;
  if (tid <= kLc) pw[tid] = powf(p.decay[h], static_cast<float>(tid));
  pdl_wait();
  pdl_trigger();
  int row0, n;
  if (!lc_find(p.q_start, p.S, blockIdx.x, row0, n)) return;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(p.proj) + static_cast<size_t>(row0) * p.ld;
  const uint4* st = static_cast<const uint4*>(p.scratch) + ((static_cast<size_t>(blockIdx.x) * p.heads + h) * D * p.vdim + v0) / 4;
  for (int i = tid; i < D * (VT / 4); i += kLcThreads) {
    const int r = i / (VT / 4), c = i - r * (VT / 4);
    const uint4 x = st[static_cast<size_t>(r) * (p.vdim / 4) + c];
    *reinterpret_cast<uint2*>(sh + r * kVP + c * 4) = make_uint2(x.x, x.y);
    *reinterpret_cast<uint2*>(sl + r * kVP + c * 4) = make_uint2(x.z, x.w);
  }
  lc_load<D, false>(proj + p.q_off + h * D, p.ld, n, sq, nullptr, nullptr);
  __syncthreads();
  const int m0 = warp * 16, r = m0 + (lane >> 2), c2 = 2 * (lane & 3);
  float o[2 * kNT][4];
#pragma unroll
  for (int i = 0; i < 2 * kNT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const __nv_bfloat16* qrow = sq + (m0 + (lane & 15)) * kKP + (lane >> 4) * 8;
  if (m0 < n) {
#pragma unroll 2
    for (int s = 0; s < D / 16; ++s) {
      uint32_t a[4];
      lc_ldsm4(a, qrow + s * 16);
#pragma unroll
      for (int j = 0; j < kNT; ++j) {
        uint32_t bh[4], bl[4];
        const int off = (s * 16 + (lane & 15)) * kVP + j * 16 + (lane >> 4) * 8;
        lc_ldsm4t(bh, sh + off);
        lc_ldsm4t(bl, sl + off);
        lc_mma(o[2 * j], a, bh[0], bh[1]);
        lc_mma(o[2 * j + 1], a, bh[2], bh[3]);
        lc_mma(o[2 * j], a, bl[0], bl[1]);
        lc_mma(o[2 * j + 1], a, bl[2], bl[3]);
      }
    }
    const float f0 = pw[r + 1], f1 = pw[r + 9];
#pragma unroll
    for (int j = 0; j < 2 * kNT; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
  }
  __syncthreads();                                // the state has been read
  lc_load<D, false>(proj + p.k_off + h * D, p.ld, n, sk, nullptr, nullptr);
  lc_load<VT, false>(proj + p.v_off + h * p.vdim + v0, p.ld, n, sv, nullptr, nullptr);
  __syncthreads();
  if (m0 >= n) return;
  for (int s = 0; s <= warp; ++s) {               // 16 keys at a time, up to the warp's own rows
    float x[2][4] = {};
#pragma unroll
    for (int k = 0; k < D / 16; ++k) {
      uint32_t a[4], b[4];
      lc_ldsm4(a, qrow + k * 16);
      lc_ldsm4(b, sk + (s * 16 + (lane & 7) + (lane >> 4) * 8) * kKP + k * 16 + ((lane >> 3) & 1) * 8);
      lc_mma(x[0], a, b[0], b[1]);
      lc_mma(x[1], a, b[2], b[3]);
    }
    uint32_t ah[4], al[4];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
      const int j = s * 16 + t * 8 + c2;          // key of x[t][0]; rows r and r + 8
      const float w00 = j <= r ? pw[r - j] : 0.f, w01 = j + 1 <= r ? pw[r - j - 1] : 0.f;
      const float w10 = j <= r + 8 ? pw[r + 8 - j] : 0.f, w11 = j + 1 <= r + 8 ? pw[r + 7 - j] : 0.f;
      lc_split2(x[t][0] * w00, x[t][1] * w01, ah[2 * t], al[2 * t]);
      lc_split2(x[t][2] * w10, x[t][3] * w11, ah[2 * t + 1], al[2 * t + 1]);
    }
#pragma unroll
    for (int j = 0; j < kNT; ++j) {
      uint32_t b[4];
      lc_ldsm4t(b, sv + (s * 16 + (lane & 15)) * kVP + j * 16 + (lane >> 4) * 8);
      lc_mma(o[2 * j], ah, b[0], b[1]);
      lc_mma(o[2 * j + 1], ah, b[2], b[3]);
      lc_mma(o[2 * j], al, b[0], b[1]);
      lc_mma(o[2 * j + 1], al, b[2], b[3]);
    }
  }
  float* dst = p.raw + (static_cast<size_t>(row0) * p.heads + h) * p.vdim + v0;
  const size_t pitch = static_cast<size_t>(p.heads) * p.vdim;
#pragma unroll
  for (int j = 0; j < 2 * kNT; ++j) {
    if (r < n) *reinterpret_cast<float2*>(dst + r * pitch + j * 8 + c2) = make_float2(o[j][0], o[j][1]);
    if (r + 8 < n) *reinterpret_cast<float2*>(dst + (r + 8) * pitch + j * 8 + c2) = make_float2(o[j][2], o[j][3]);
  }
}

template <int D, int VT>
static int launch_lightning_chunked(const LightningArgs& p, cudaStream_t st) {
  constexpr int kStates = (kLc * (D + 8) + 2 * kLc * (VT + 8)) * 2;
  constexpr int kA = 2 * D * (VT + 8), kB = kLc * (D + 8) + kLc * (VT + 8);
  constexpr int kOutputs = (kLc * (D + 8) + (kA > kB ? kA : kB)) * 2;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(lightning_chunk_states_kernel<D, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kStates));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(lightning_chunk_outputs_kernel<D, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kOutputs));
    attr = true;
  }
  const int chunks = p.T / kLc + p.S;             // at least as many as there are
  if (p.scratch_bytes < static_cast<long long>(chunks) * p.heads * p.dim * p.vdim * 4) return -12;
  const dim3 grid(chunks, p.heads, p.vdim / VT);
  launch_pdl(lightning_chunk_states_kernel<D, VT>, grid, dim3(kLcThreads), kStates, st, p);
  launch_pdl(lightning_chunk_prefix_kernel, dim3((p.dim * p.vdim / 4 + 255) / 256, p.heads, p.S), dim3(256), 0, st, p);
  launch_pdl(lightning_chunk_outputs_kernel<D, VT>, grid, dim3(kLcThreads), kOutputs, st, p);
  const int rc = static_cast<int>(cudaGetLastError());
  return rc ? rc : launch_lightning_out<__nv_bfloat16>(p, st);
}

}  // namespace cafd

using namespace cafd;

// bf16; dim 32, 64, 96 or 128, vdim a multiple of 64, sections on 16-byte boundaries.  scratch: (T / 128 + S) * heads * dim * vdim floats.
extern "C" int cafd_lightning_chunked(const LightningArgs* a, cafd_stream_t s) {
  if (a->T <= 0) return 0;
  const LightningArgs& p = *a;
  if (!lightning_args_ok(p) || !p.scratch || p.vdim % 64 || (p.ld | p.q_off | p.k_off | p.v_off) % 8 || (p.s_off | p.slot_stride) % 4) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  const bool wide = p.vdim % 128 == 0;
  switch (p.dim) {
    case 32: return wide ? launch_lightning_chunked<32, 128>(p, st) : launch_lightning_chunked<32, 64>(p, st);
    case 64: return wide ? launch_lightning_chunked<64, 128>(p, st) : launch_lightning_chunked<64, 64>(p, st);
    case 96: return wide ? launch_lightning_chunked<96, 128>(p, st) : launch_lightning_chunked<96, 64>(p, st);
    case 128: return wide ? launch_lightning_chunked<128, 128>(p, st) : launch_lightning_chunked<128, 64>(p, st);
  }
  return -11;
}
