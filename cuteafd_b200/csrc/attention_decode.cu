// Paged GQA attention for small query counts (decode rows and speculative-verify rows), split
// over the KV length with a fixed-order merge.  The op is HBM-bound (each K/V byte is used by at
// most 16 query rows), so the tiles run on mma.sync m16n8k16 with cp.async double buffering; the
// compute-bound prefill path uses tcgen05 (attention_prefill.cu).
//
//   grid  (sequence x query tile, kv head, split)     block 128 threads (4 warps)
//   tile  16 rows = (16 / group) query tokens x group heads sharing one kv head
//   each warp owns 16 of the 64 tokens of a page; per-warp online softmax; warps merged in
//   shared memory; splits merged by a second kernel in split order (deterministic).
//
// With kMaps = 2 (differential attention: two 64-wide score maps per head over the same 128-wide values; query and key rows
// hold [map 1 | map 2]) a tile's rows are (query token, head, map) and a row's query fragment is zero in the other map's half,
// so the same products serve.  Map 1 - lambda * map 2, its norm over the head's values and a constant factor follow when the
// row is complete: here without splits, in the merge with them.
// A sliding window may come with kept first tokens; their pages are walked before the window's.  A head may have a sink, a number
// whose exponential joins the softmax's denominator, and an output gate (the sigmoid of one number per token and head); both are
// applied where a row is complete, and so is (kTurn) a rotation of the output back by the query's position.  kTurn: scores may be
// capped.
//
// Reference counterparts: split-KV partial + merge drafter attention
// (native/shared/cuda/draft_attention.cu:42-295) and the LSE state merge
// (native/shared/cuda/attention.cu:925).
#include "cafd_api.h"
#include "common.cuh"

namespace cafd {

constexpr int kD = 128;
constexpr int kPage = 64;
constexpr int kTileBytes = kPage * kD * 2;  // 16 KiB for K, same for V

__device__ __forceinline__ void cp_async_16(void* smem_dst, const void* gsrc) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_ptr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(smem_ptr)));
}

__device__ __forceinline__ void load_page(uint8_t* dst, const __nv_bfloat16* cache, int page, int kvh, int Hkv) {
  // 64 rows x 16 chunks of 16 bytes; chunk index XOR-swizzled by the row so that fragment reads
  // from 8 different rows hit different banks.
  for (int i = threadIdx.x; i < kPage * 16; i += blockDim.x) {
    const int tok = i >> 4, ch = i & 15;
    // cache layout [page, kv head, 64 tokens, D]: the tile of one (page, head) is 16 KB of contiguous memory
    const __nv_bfloat16* src = cache + ((static_cast<size_t>(page) * Hkv + kvh) * kPage + tok) * kD + ch * 8;
    cp_async_16(dst + tok * 256 + ((ch ^ (tok & 7)) << 4), src);
  }
}

// partial layout per (tile, kvh, split): [16 rows][kD] fp32 O (unnormalised), then m[16], l[16]
constexpr int kPartialFloats = 16 * kD + 32;

// Context split (the KV of a sequence dealt over several GPUs by page): every rank runs this kernel over the pages it
// holds and stores its partials into EVERY rank's scratch, at split slots [split_offset, split_offset + splits) of
// total_splits, so that each rank's merge walks all ranks' partials in rank order.  n == 0: the single-GPU form.
// kv_base (optional, per sequence): query token qi sees the first min(seq_len, kv_base + qi + 1) local positions; the
// default seq_len - q_len is the causal rule when the new tokens are the last local ones, and a rank that does not
// hold the new tokens passes its local length (everything it holds is in the past of every query).
struct AttnPeers {
  float* scratch[8];
  int n, split_offset, total_splits;
};

// Kept first tokens, output row pitch, with two maps how they are combined, with one sinks and gates.
struct AttnExtras {
  int keep, ldo;
  float lambda = 0.f, out_scale = 1.f, eps = 0.f;
  const float* sink = nullptr;             // [Hq] or null
  const __nv_bfloat16* gate = nullptr;     // row t, head h: gate[t * gate_ld + h]; or null
  int gate_ld = 0;
  const float2* v_table = nullptr;         // [rows, 64] cos, sin; or null; one map only
  float cap_log2 = 0.f;                    // cap * log2(e): scores are cap * tanh(score / cap), and the kernel's scale is 2 log2(e) * scale / cap; 0 = none
};

// kTurn: with cap_log2, v_table and out_scale.  A complete row of one head: M is the maximum its sums L and O refer to, in log2 units.
template <bool kTurn>
__device__ __forceinline__ float finish_row(float O, float L, float M, const AttnExtras& x, int row, int head) {
  if (x.sink) L += exp2f(x.sink[head] * 1.4426950408889634f - M);
  float v = L > 0.f ? O / L : 0.f;
  if (x.gate) v /= 1.0f + expf(-__bfloat162float(x.gate[static_cast<size_t>(row) * x.gate_ld + head]));
  return kTurn ? v * x.out_scale : v;
}

// One head's 128 values, one per thread, turned back by the row's angles (pairs 64 apart); every thread of the block calls.
__device__ __forceinline__ float turn_back(float v, const AttnExtras& x, int row, float* buf) {
  const int d = threadIdx.x;
  buf[d] = v;
  __syncthreads();
  const float o = buf[d ^ 64];
  const float2 a = x.v_table[static_cast<size_t>(row) * 64 + (d & 63)];
  __syncthreads();
  return d < 64 ? v * a.x + o * a.y : v * a.x - o * a.y;
}

// The combined value of one head's 128 values, one per thread: a - lambda * b over its root mean square, times out_scale.
__device__ __forceinline__ float combine_maps(float a, float b, const AttnExtras& x, float* red) {
  const float o = a - x.lambda * b;
  const float ss = warp_sum(o * o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float tot = (red[0] + red[1]) + (red[2] + red[3]);
  __syncthreads();
  return o * (x.out_scale / sqrtf(tot * (1.0f / kD) + x.eps));
}

template <int kMaps, bool kTurn = false>
__global__ void __launch_bounds__(128) attn_decode_kernel(
    const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k_cache,
    const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ page_table, const int* __restrict__ seq_lens,
    const int* __restrict__ q_start, __nv_bfloat16* __restrict__ out, float* __restrict__ partial, int max_pages,
    int Hq, int Hkv, int tiles_per_seq, int splits, float scale_log2, const int* __restrict__ kv_base, int window, int split_pages,
    const AttnPeers peers, const AttnExtras ex) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t smem[];
  const int group = kMaps * (Hq / Hkv);          // rows per query token
  const int q_per_tile = 16 / group;
  const int seq = blockIdx.x / tiles_per_seq;
  const int qt = blockIdx.x % tiles_per_seq;
  const int kvh = blockIdx.y;
  const int split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t4 = lane & 3;

  const int q0 = q_start[seq], q_len = q_start[seq + 1] - q0;
  const int seq_len = seq_lens[seq];
  const int first_q = qt * q_per_tile;
  const size_t part_off = peers.n
      ? (static_cast<size_t>(blockIdx.x) * Hkv + kvh) * peers.total_splits * kPartialFloats +
            static_cast<size_t>(peers.split_offset + split) * kPartialFloats
      : (static_cast<size_t>(blockIdx.x) * Hkv + kvh) * splits * kPartialFloats + static_cast<size_t>(split) * kPartialFloats;
  float* part = partial + part_off;
  if (first_q >= q_len) return;   // tile beyond this sequence's queries: nothing to write
  const int base_vis = kv_base ? kv_base[seq] : seq_len - q_len;

  // ---- Q fragments straight from global memory ------------------------------------------------
  // row r of the tile = query token first_q + r / group, head kvh * group + r % group
  uint32_t qa[8][4];
  int limit[2];   // number of kv positions visible to rows g and g + 8
  int lo[2];      // first visible position (sliding window; 0 without one)
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = g + 8 * half;
    const int qi = first_q + r / group;
    const bool valid = qi < q_len;
    limit[half] = valid ? min(seq_len, base_vis + qi + 1) : 0;
    lo[half] = !valid ? 0x7fffffff : (window > 0 ? max(0, limit[half] - window) : 0);
    const __nv_bfloat16* qrow = q + (static_cast<size_t>(q0 + (valid ? qi : 0)) * Hq + kvh * (group / kMaps) + (r % group) / kMaps) * kD;
#pragma unroll
    for (int ks = 0; ks < 8; ++ks) {
      const bool on = valid && (kMaps == 1 || (ks >> 2) == (r & 1));
      qa[ks][half] = on ? *reinterpret_cast<const uint32_t*>(qrow + 16 * ks + 2 * t4) : 0u;
      qa[ks][half + 2] = on ? *reinterpret_cast<const uint32_t*>(qrow + 16 * ks + 8 + 2 * t4) : 0u;
    }
  }
  int max_limit = limit[0] > limit[1] ? limit[0] : limit[1];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) max_limit = max(max_limit, __shfl_xor_sync(0xffffffffu, max_limit, o));
  int min_lo = lo[0] < lo[1] ? lo[0] : lo[1];
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) min_lo = min(min_lo, __shfl_xor_sync(0xffffffffu, min_lo, o));

  // pages [0, kept) and [first_page, total_pages) hold every position some row of the tile sees; the splits share them
  const int total_pages = (max_limit + kPage - 1) / kPage;
  const int first_page = min(min_lo / kPage, total_pages);
  const int kept = min((ex.keep + kPage - 1) / kPage, first_page);
  const int gap = first_page - kept;             // page of ordinal i: i + (i < kept ? 0 : gap)
  const int n_pages = total_pages - gap;
  // split_pages > 0: split s owns pages [s * split_pages, (s + 1) * split_pages) of every sequence, whatever the step holds
  auto ordinal = [&](int page) { return page <= kept ? page : max(kept, page - gap); };   // visible pages before `page`
  const int per_split = (n_pages + splits - 1) / splits;
  const int p0 = split_pages > 0 ? min(n_pages, ordinal(split * split_pages)) : split * per_split;
  const int p1 = min(n_pages, split_pages > 0 ? ordinal((split + 1) * split_pages) : p0 + per_split);

  float m_run[2] = {-INFINITY, -INFINITY};
  float l_run[2] = {0.f, 0.f};
  float o_acc[16][4];
#pragma unroll
  for (int i = 0; i < 16; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o_acc[i][j] = 0.f;

  const int* pt = page_table + static_cast<size_t>(seq) * max_pages;
  auto page_at = [&](int i) { return i + (i < kept ? 0 : gap); };
  if (p0 < p1) {
    const int first = pt[page_at(p0)];
    load_page(smem, k_cache, first, kvh, Hkv);
    load_page(smem + kTileBytes, v_cache, first, kvh, Hkv);
  }
  cp_async_commit();
  for (int p = p0; p < p1; ++p) {
    const int stage = (p - p0) & 1;
    if (p + 1 < p1) {
      uint8_t* nxt = smem + (stage ^ 1) * 2 * kTileBytes;
      const int page = pt[page_at(p + 1)];
      load_page(nxt, k_cache, page, kvh, Hkv);
      load_page(nxt + kTileBytes, v_cache, page, kvh, Hkv);
    }
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint8_t* ks_ = smem + stage * 2 * kTileBytes;
    const uint8_t* vs_ = ks_ + kTileBytes;

    // ---- S = Q K^T for this warp's 16 tokens --------------------------------------------------
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
      const int tok = warp * 16 + nt * 8 + g;
      const uint8_t* krow = ks_ + tok * 256;
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(krow + (((2 * ks) ^ (tok & 7)) << 4) + 4 * t4);
        const uint32_t b1 = *reinterpret_cast<const uint32_t*>(krow + (((2 * ks + 1) ^ (tok & 7)) << 4) + 4 * t4);
        mma_bf16_16816(s[nt], qa[ks], b0, b1);
      }
    }
    // ---- mask + online softmax (rows g and g + 8) ---------------------------------------------
    const int tok_base = page_at(p) * kPage + warp * 16;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int half = j >> 1;
        const int tok = tok_base + nt * 8 + 2 * t4 + (j & 1);
        const float z = s[nt][j] * scale_log2;
        const float v = (tok < limit[half] && (tok >= lo[half] || tok < ex.keep)) ? (kTurn && ex.cap_log2 > 0.f ? ex.cap_log2 * tanh_exp2(z) : z) : -INFINITY;
        s[nt][j] = v;
        mx[half] = fmaxf(mx[half], v);
      }
    uint32_t pa[4];
    float corr[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      mx[half] = fmaxf(mx[half], __shfl_xor_sync(0xffffffffu, mx[half], 1));
      mx[half] = fmaxf(mx[half], __shfl_xor_sync(0xffffffffu, mx[half], 2));
      const float m_new = fmaxf(m_run[half], mx[half]);
      corr[half] = (m_new == -INFINITY) ? 1.f : exp2f(m_run[half] - m_new);
      const float base = (m_new == -INFINITY) ? 0.f : m_new;
      float rs = 0.f;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const float e0 = exp2f(s[nt][2 * half] - base);
        const float e1 = exp2f(s[nt][2 * half + 1] - base);
        // round to bf16 first so the row sum matches what the P.V product sees
        const uint32_t packed = pack_bf16(e0, e1);
        rs += bf16_lo(packed) + bf16_hi(packed);
        pa[half + 2 * nt] = packed;
      }
      rs += __shfl_xor_sync(0xffffffffu, rs, 1);
      rs += __shfl_xor_sync(0xffffffffu, rs, 2);
      l_run[half] = l_run[half] * corr[half] + rs;
      m_run[half] = m_new;
    }
#pragma unroll
    for (int nd = 0; nd < 16; ++nd) {
      o_acc[nd][0] *= corr[0]; o_acc[nd][1] *= corr[0];
      o_acc[nd][2] *= corr[1]; o_acc[nd][3] *= corr[1];
    }
    // ---- O += P V ----------------------------------------------------------------------------------
#pragma unroll
    for (int nd = 0; nd < 16; nd += 2) {
      const int m = lane >> 3, r = lane & 7;
      const int tok = warp * 16 + (m & 1) * 8 + r;
      const int ch = nd + (m >> 1);
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, vs_ + tok * 256 + ((ch ^ (tok & 7)) << 4));
      mma_bf16_16816(o_acc[nd], pa, vb[0], vb[1]);
      mma_bf16_16816(o_acc[nd + 1], pa, vb[2], vb[3]);
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  __syncthreads();

  // ---- merge the four warps (fixed order) ---------------------------------------------------------
  float* sm_o = reinterpret_cast<float*>(smem);            // [4][16][kD]
  float* sm_m = sm_o + 4 * 16 * kD;                        // [4][16]
  float* sm_l = sm_m + 64;
#pragma unroll
  for (int nd = 0; nd < 16; ++nd) {
    float* o0 = sm_o + (warp * 16 + g) * kD + nd * 8 + 2 * t4;
    float* o1 = sm_o + (warp * 16 + g + 8) * kD + nd * 8 + 2 * t4;
    o0[0] = o_acc[nd][0]; o0[1] = o_acc[nd][1];
    o1[0] = o_acc[nd][2]; o1[1] = o_acc[nd][3];
  }
  if (t4 == 0) {
    sm_m[warp * 16 + g] = m_run[0]; sm_m[warp * 16 + g + 8] = m_run[1];
    sm_l[warp * 16 + g] = l_run[0]; sm_l[warp * 16 + g + 8] = l_run[1];
  }
  __syncthreads();
  float o_map1 = 0.f;                            // kMaps == 2, no splits: the head's first map, one value per thread
  for (int i = threadIdx.x; i < 16 * kD; i += blockDim.x) {   // every iteration: row i / 128, value threadIdx.x
    const int r = i / kD, d = i % kD;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) M = fmaxf(M, sm_m[w * 16 + r]);
    float L = 0.f, O = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = (sm_m[w * 16 + r] == -INFINITY) ? 0.f : exp2f(sm_m[w * 16 + r] - M);
      L += sm_l[w * 16 + r] * f;
      O += sm_o[(w * 16 + r) * kD + d] * f;
    }
    if (peers.n) {
      for (int pr = 0; pr < peers.n; ++pr) {              // plain peer stores; the flag that publishes them follows in stream order
        float* dst = peers.scratch[pr] + part_off;
        dst[r * kD + d] = O;
        if (d == 0) { dst[16 * kD + r] = M; dst[16 * kD + 16 + r] = L; }
      }
    } else if (splits == 1) {
      const int qi = first_q + r / group;
      if (qi < q_len) {
        const int head = kvh * (group / kMaps) + (r % group) / kMaps;
        float v;
        if (kMaps == 2) {
          v = L > 0.f ? O / L : 0.f;
          if ((r & 1) == 0) { o_map1 = v; continue; }
          v = combine_maps(o_map1, v, ex, sm_l + 64);
        } else {
          v = finish_row<kTurn>(O, L, M, ex, q0 + qi, head);
          if (kTurn && ex.v_table) v = turn_back(v, ex, q0 + qi, sm_l + 128);
        }
        out[static_cast<size_t>(q0 + qi) * ex.ldo + head * kD + d] = __float2bfloat16(v);
      }
    } else {
      part[r * kD + d] = O;
      if (d == 0) { part[16 * kD + r] = M; part[16 * kD + 16 + r] = L; }
    }
  }
}

// One block per (tile, kv head, row; with two maps row pair): thread d walks the splits in order for its output element.
template <int kMaps, bool kTurn = false>
__global__ void __launch_bounds__(128) attn_merge_kernel(const float* __restrict__ partial,
                                                         const int* __restrict__ q_start,
                                                         __nv_bfloat16* __restrict__ out, int Hq, int Hkv,
                                                         int tiles_per_seq, int splits, const AttnExtras ex) {
  __shared__ float red[kTurn ? kD : 4];
  pdl_wait();
  pdl_trigger();
  const int group = Hq / Hkv;
  const int q_per_tile = 16 / (group * kMaps);
  const int seq = blockIdx.x / tiles_per_seq, qt = blockIdx.x % tiles_per_seq, kvh = blockIdx.y, r = blockIdx.z;
  const int q0 = q_start[seq], q_len = q_start[seq + 1] - q0;
  const int qi = qt * q_per_tile + r / group;
  if (qi >= q_len) return;
  const int d = threadIdx.x;
  const float* base = partial + (static_cast<size_t>(blockIdx.x) * Hkv + kvh) * splits * kPartialFloats;
  float v[kMaps];
#pragma unroll
  for (int m = 0; m < kMaps; ++m) {
    const int row = r * kMaps + m;
    float M = -INFINITY;
    for (int s = 0; s < splits; ++s) M = fmaxf(M, __ldg(base + s * kPartialFloats + 16 * kD + row));
    float L = 0.f, O = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float mx = __ldg(base + s * kPartialFloats + 16 * kD + row);
      const float f = (mx == -INFINITY) ? 0.f : exp2f(mx - M);
      L += __ldg(base + s * kPartialFloats + 16 * kD + 16 + row) * f;
      O += __ldg(base + s * kPartialFloats + row * kD + d) * f;
    }
    v[m] = kMaps == 1 ? finish_row<kTurn>(O, L, M, ex, q0 + qi, kvh * group + r % group) : L > 0.f ? O / L : 0.f;
  }
  const float o = kMaps == 2 ? combine_maps(v[0], v[kMaps - 1], ex, red) : kTurn && ex.v_table ? turn_back(v[0], ex, q0 + qi, red) : v[0];
  out[static_cast<size_t>(q0 + qi) * ex.ldo + (kvh * group + r % group) * kD + d] = __float2bfloat16(o);
}

}  // namespace cafd

using namespace cafd;

// tokens per kv split for every decode attention kernel of the library (GQA and MLA); 0 = even division.  A multiple
// of 64.
extern "C" int cafd_set_fixed_kv_split(int tokens) {
  if (tokens < 0 || tokens % kPage) return -10;
  fixed_kv_split_tokens() = tokens;
  return 0;
}
extern "C" int cafd_fixed_kv_split() { return fixed_kv_split_tokens(); }

extern "C" long long cafd_attn_decode_scratch_floats(int num_seqs, int tiles_per_seq, int Hkv, int splits) {
  return static_cast<long long>(num_seqs) * tiles_per_seq * Hkv * splits * kPartialFloats;
}

// q [total_q, Hq, 128] (two maps: [total_q, Hq, 2, 64]); caches [pages, Hkv, 64, 128]; page_table [num_seqs, max_pages];
// seq_lens [num_seqs] (kv length including the new tokens); q_start [num_seqs + 1]; out rows of ldo elements, head h's values at
// column 128 h.  max_q_len bounds the query tokens of any sequence; scratch holds the split partials.  keep: kept first tokens
// beside a window; lambda and eps: two maps only; out_scale multiplies the output; sink [Hq], gate rows (gate_ld elements apart) and
// v_table [rows, 64] (cos, sin of the output's rotation back): one map only; cap 0 = scores are not capped.
extern "C" int cafd_attn_decode(const void* q, const void* k_cache, const void* v_cache, const int* page_table,
                                const int* seq_lens, const int* q_start, void* out, float* scratch, int num_seqs,
                                int max_q_len, int max_pages, int Hq, int Hkv, int D, int splits, float scale,
                                int window, int keep, int ldo, int maps, float lambda, float out_scale, float eps, const float* sink,
                                const void* gate, int gate_ld, float cap, const void* v_table, cafd_stream_t s) {
  if (num_seqs <= 0) return 0;
  if (D != kD || Hq % Hkv || window < 0 || keep < 0 || maps < 1 || maps > 2 || ldo < Hq * kD) return -10;
  if ((maps == 2 && (sink || gate || v_table || cap > 0.f)) || (gate && gate_ld < Hq)) return -10;
  const int group = maps * (Hq / Hkv);
  if (group > 16 || 16 % group) return -11;
  if (splits < 1) splits = 1;
  if (splits > 1 && !scratch) return -12;
  // fixed-size splits must cover the widest sequence the page table can describe
  if (fixed_kv_split_tokens() > 0 && static_cast<long long>(splits) * fixed_kv_split_tokens() < static_cast<long long>(max_pages) * kPage) return -14;
  const int q_per_tile = 16 / group;
  const int tiles_per_seq = (max_q_len + q_per_tile - 1) / q_per_tile;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  const int smem = 4 * kTileBytes;   // two stages of K+V; reused for the warp merge (needs 33 KiB)
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_decode_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_decode_kernel<1, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_decode_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr = true;
  }
  dim3 grid(num_seqs * tiles_per_seq, Hkv, splits);
  const AttnExtras ex{window > 0 ? keep : 0, ldo, lambda, out_scale, eps, sink, static_cast<const __nv_bfloat16*>(gate), gate_ld,
                      static_cast<const float2*>(v_table), cap * 1.4426950408889634f};
  const bool turn = maps == 1 && (cap > 0.f || v_table || out_scale != 1.f);
  auto kern = maps == 2 ? attn_decode_kernel<2> : turn ? attn_decode_kernel<1, true> : attn_decode_kernel<1>;
  launch_pdl(kern, grid, dim3(128), smem, st,
      static_cast<const __nv_bfloat16*>(q), static_cast<const __nv_bfloat16*>(k_cache),
      static_cast<const __nv_bfloat16*>(v_cache), page_table, seq_lens, q_start, static_cast<__nv_bfloat16*>(out),
      scratch, max_pages, Hq, Hkv, tiles_per_seq, splits, (cap > 0.f ? 2.f * scale / cap : scale) * 1.4426950408889634f, static_cast<const int*>(nullptr),
      window, fixed_kv_split_tokens() / kPage, AttnPeers{}, ex);
  if (splits > 1) {
    dim3 g2(num_seqs * tiles_per_seq, Hkv, 16 / maps);
    auto merge = maps == 2 ? attn_merge_kernel<2> : turn ? attn_merge_kernel<1, true> : attn_merge_kernel<1>;
    launch_pdl(merge, g2, dim3(128), 0, st, scratch, q_start, static_cast<__nv_bfloat16*>(out), Hq, Hkv, tiles_per_seq, splits, ex);
  }
  return static_cast<int>(cudaGetLastError());
}

// Context-split form, first half: partial attention over this rank's pages, stored into the scratch of every rank of
// the group (peer_scratch[r], r < n_peers; this rank's own buffer included) at split slots
// [my_rank * splits, (my_rank + 1) * splits) of n_peers * splits.  The caller publishes the stores with a flag per peer
// and merges with cafd_attn_merge once every rank's flag has arrived.
extern "C" int cafd_attn_decode_partial(const void* q, const void* k_cache, const void* v_cache, const int* page_table,
                                        const int* seq_lens, const int* kv_base, const int* q_start, void* const* peer_scratch,
                                        int n_peers, int my_rank, int num_seqs, int max_q_len, int max_pages, int Hq, int Hkv,
                                        int D, int splits, float scale, cafd_stream_t s) {
  if (num_seqs <= 0) return 0;
  if (D != kD || Hq % Hkv || n_peers < 1 || n_peers > 8 || my_rank < 0 || my_rank >= n_peers || !peer_scratch) return -10;
  const int group = Hq / Hkv;
  if (group > 16 || 16 % group) return -11;
  if (splits < 1) splits = 1;
  const int q_per_tile = 16 / group;
  const int tiles_per_seq = (max_q_len + q_per_tile - 1) / q_per_tile;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  const int smem = 4 * kTileBytes;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_decode_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr = true;
  }
  AttnPeers peers{};
  for (int r = 0; r < n_peers; ++r) {
    if (!peer_scratch[r]) return -12;
    peers.scratch[r] = static_cast<float*>(peer_scratch[r]);
  }
  peers.n = n_peers; peers.split_offset = my_rank * splits; peers.total_splits = n_peers * splits;
  dim3 grid(num_seqs * tiles_per_seq, Hkv, splits);
  launch_pdl(attn_decode_kernel<1>, grid, dim3(128), smem, st, static_cast<const __nv_bfloat16*>(q),
             static_cast<const __nv_bfloat16*>(k_cache), static_cast<const __nv_bfloat16*>(v_cache), page_table, seq_lens, q_start,
             static_cast<__nv_bfloat16*>(nullptr), peers.scratch[my_rank], max_pages, Hq, Hkv, tiles_per_seq, splits,
             scale * 1.4426950408889634f, kv_base, 0, 0, peers, AttnExtras{0, Hq * kD});
  return static_cast<int>(cudaGetLastError());
}

// Second half: merge total_splits partials per (tile, kv head) from this rank's scratch in slot order.
extern "C" int cafd_attn_merge(const float* scratch, const int* q_start, void* out, int num_seqs, int max_q_len, int Hq, int Hkv,
                               int total_splits, cafd_stream_t s) {
  if (num_seqs <= 0) return 0;
  if (Hq % Hkv || total_splits < 1 || !scratch) return -10;
  const int group = Hq / Hkv;
  if (group > 16 || 16 % group) return -11;
  const int q_per_tile = 16 / group;
  const int tiles_per_seq = (max_q_len + q_per_tile - 1) / q_per_tile;
  dim3 g2(num_seqs * tiles_per_seq, Hkv, 16);
  launch_pdl(attn_merge_kernel<1>, g2, dim3(128), 0, static_cast<cudaStream_t>(s), scratch, q_start, static_cast<__nv_bfloat16*>(out),
             Hq, Hkv, tiles_per_seq, total_splits, AttnExtras{0, Hq * kD});
  return static_cast<int>(cudaGetLastError());
}
