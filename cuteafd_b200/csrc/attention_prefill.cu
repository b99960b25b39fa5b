// Causal GQA prefill attention over the paged KV cache on tcgen05 tensor cores (head_dim 128).
//
// One CTA computes a 128-row query tile of one head.  S = Q K^T and O += P V both run as
// tcgen05.mma with accumulators in TMEM; K/V pages arrive by TMA straight from the page pool
// (a 4-D tensor map indexed by page id), so chunked prefill and prefix-cache hits need no
// gather.  Warp roles:
//   warp 0     TMA producer: Q tile once, then K and V tiles (two stages each)
//   warp 1     MMA issuer: QK^T for tile j+1 is issued before P V of tile j, so the tensor pipe
//              works on the next scores while the softmax warps are busy
//   warps 2-9  online softmax: thread = (query row, half of the tile's kv columns); warps w and w + 4 share a
//              TMEM lane quarter, so each scheduler has two warps to overlap.  A half row of S is read into
//              registers with one tcgen05.ld wait (the S buffer is released right away), the halves exchange
//              their maxima through shared memory, P is written as bf16 into 128B-swizzled shared memory (the
//              A operand of P V; two buffers in the GQA variant), O is rescaled in TMEM only when the reference
//              maximum moved (it moves when a row maximum exceeds it by more than 8 in log2 units)
// TMEM: S double-buffered (2 x 128 columns) + O (128 columns).
//
// The kRope variant serves MLA prefill in its expanded (non-absorbed) form: per-head K_nope / V tiles come from a
// contiguous expansion buffer (kv_b applied to the chunk's latents), and a 64-wide rotary part that all heads share
// is added to the scores with four more MMAs per tile, its keys read straight from the paged latent cache
// (columns 512..575 of every record).  Query dims are then 128 + 64, value dims 128.
//
// With kMaps = 2 a head has two 64-wide score maps over the same 128-wide values (differential attention): query and key
// rows hold [map 1 | map 2], exactly the two 64-wide halves of the Q and K tiles.  The pipeline then runs over units
// (tile, map), maps alternating: S and P buffer = map, one O accumulator per map (TMEM: 2 x 128 + 2 x 128 columns), K and V
// stages released by the tile's second unit.  The epilogue combines the maps: O1 / l1 - lambda O2 / l2, divided by its root
// mean square over the head's values, times a constant.
//
// A sliding window may come with kept first tokens, which every later row sees too: the tiles that hold them are walked
// before the window's.  A head may have a sink (a number whose exponential joins the softmax's denominator) and an output gate
// (the sigmoid of one number per token and head): both enter the epilogue's quotient; with kTurn the output may be rotated back by
// the query's position there.
//
// kTurn: scores may be cap * tanh(score / cap), the output may be turned back.  While every score of a warp's tile is small against the cap, tanh is an odd polynomial
// (two scores per instruction); else it takes an exponential and a division.
//
// Replaces the reference's mma.sync prefill kernels (native/families/glm5/cuda/glm_mla_prefill.cu:78-135)
// and its exported attention programs for the GQA families.
#include "cafd_api.h"
#include "common.cuh"
#include "host_tma.h"

namespace cafd {

constexpr int kHD = 128;          // head dim
constexpr int kBQ = 128;          // query rows per CTA
constexpr int kBKV = 128;         // kv tokens per tile (two 64-token pages)
constexpr int kPageTok = 64;
constexpr int kHalfBytes = 128 * 128;   // 128 rows x 64 bf16 (one swizzle atom wide) = 16 KiB
constexpr int kTileB = 2 * kHalfBytes;  // 32 KiB: a [128 x 128] bf16 tile as two 64-wide halves
constexpr int kPrefillThreads = 320;   // TMA warp, MMA warp, 8 softmax warps
constexpr int kPrefillSmem = 7 * kTileB + 1024;   // Q, K x2, V x2, P x2
constexpr int kPrefillSmemRope = 5 * kTileB + 3 * kHalfBytes + 1024;   // Q, Qr, (K, Kr) x2, V x1, P

struct PrefillDev {
  const int* page_table;   // [seqs, max_pages]
  const int* seq_lens;     // kv length per sequence (including this chunk)
  const int* q_start;      // [seqs + 1] row offsets into q/out
  __nv_bfloat16* out;      // [total_q, Hq, 128]
  uint32_t* status;
  int max_pages;
  int Hq, Hkv;
  float scale_log2;
  int window;              // sliding window: a query at position t sees keys (t - window, t]; 0 = all earlier keys
  int keep;                // with a window: and the keys [0, keep)
  int ldo;                 // elements from row to row of out
  // kMaps == 2 only
  float lambda, out_scale, eps;
  // kMaps == 1 only
  const float* sink;              // [Hq] or null
  const __nv_bfloat16* gate;      // row t, head h: gate[t * gate_ld + h]; or null
  int gate_ld;
  const float2* v_table;          // [rows, 64] cos, sin; or null
  float cap_in, cap_log2;         // scale / cap, cap * log2(e); scale_log2 is then 1.  These two and v_table: kTurn only
  // kRope only
  const int* kv_tmp_start; // [seqs] first row of the sequence in the expansion buffers (multiple of 64)
  int q_head_stride;       // elements between heads in the nope query matrix (192 for [T, heads * 192])
  int qr_head_stride;      // elements between heads in the rope query matrix (576 for the absorbed-query buffer)
  int qr_col0;             // first rope column inside a head of that matrix (512)
};

// tanh(x) / x as a polynomial in x^2, fitted over |x| <= kTanhRange by least squares at Chebyshev nodes: within 2e-8
constexpr float kTanhRange = 0.75f;
__device__ __forceinline__ uint64_t pack_f32x2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
// 64 scores in place: out * tanh(in * score)
__device__ __forceinline__ void cap_scores(uint32_t (&r)[64], float in, float out) {
  float m4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 64; i += 4) {
#pragma unroll
    for (int k = 0; k < 4; ++k) m4[k] = fmaxf(m4[k], fabsf(__uint_as_float(r[i + k])));
  }
  const float top = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * fabsf(in);
  if (__any_sync(0xffffffffu, !(top <= kTanhRange))) {
    const float arg = 2.f * 1.4426950408889634f * in;
#pragma unroll
    for (int i = 0; i < 64; ++i) r[i] = __float_as_uint(out * tanh_exp2(__uint_as_float(r[i]) * arg));
    return;
  }
  constexpr float kC[6] = {0.999999972f, -0.333329667f, 0.133255153f, -0.0533498202f, 0.0195937858f, -0.00472395227f};
  uint64_t c[6];
#pragma unroll
  for (int k = 0; k < 6; ++k) c[k] = pack_f32x2(kC[k] * out, kC[k] * out);
  const uint64_t s = pack_f32x2(in, in);
#pragma unroll
  for (int i = 0; i < 64; i += 2) {
    const uint64_t x = mul_f32x2(pack_f32x2(__uint_as_float(r[i]), __uint_as_float(r[i + 1])), s), y = mul_f32x2(x, x);
    uint64_t q = c[5];
#pragma unroll
    for (int k = 4; k >= 0; --k) q = fma_f32x2(q, y, c[k]);
    q = mul_f32x2(q, x);
    asm("mov.b64 {%0, %1}, %2;" : "=r"(r[i]), "=r"(r[i + 1]) : "l"(q));
  }
}

template <bool kRope, int kMaps, bool kTurn = false>
__global__ void __launch_bounds__(kPrefillThreads, 1)
attn_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                    const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_qr,
                    const __grid_constant__ CUtensorMap tm_kr, const PrefillDev p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int kVS = kRope ? 1 : 2;    // V stages (the rope tiles take the room of the second one)
  // P buffers.  With two, the exponentials of tile j are stored while P V of tile j - 1 still runs; only a
  // rescale of O (rare with the lazy reference maximum) has to wait for that MMA.
  constexpr int kPB = kRope ? 1 : 2;
  uint8_t* sQ = smem;
  uint8_t* sK = smem + kTileB;          // 2 stages
  uint8_t* sV = smem + 3 * kTileB;      // kVS stages
  uint8_t* sP = sV + kVS * kTileB;
  uint8_t* sQr = sP + kPB * kTileB;     // kRope: 128 x 64 rope queries, then two stages of 128 x 64 rope keys
  uint8_t* sKr = sQr + kHalfBytes;

  __shared__ uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2], s_empty[2], p_ready[2], pv_done[2], mx_bar[2];
  // Exchange between the two column halves of a row: maxima as bf16 [tile parity][half][row] (rounded up, so the
  // common reference is never below a score), and at the very end the row sums as fp32 [half][row] in the same bytes.
  __shared__ uint32_t s_xch[256];
  __shared__ uint32_t tmem_slot;

  pdl_wait();      // the page table, lengths and Q come from kernels earlier in the stream
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z;
  const int head = blockIdx.y;
  const int kvh = head / (p.Hq / p.Hkv);
  const int q0 = p.q_start[seq];
  const int q_len = p.q_start[seq + 1] - q0;
  const int kv_len = p.seq_lens[seq];
  const int n_qt = (q_len + kBQ - 1) / kBQ;
  const int qt = n_qt - 1 - static_cast<int>(blockIdx.x);   // heaviest tiles first
  if (qt < 0) return;
  const int row0 = qt * kBQ;                       // first query row of this tile (within the chunk)
  const int pos0 = kv_len - q_len + row0;          // its absolute position
  const int last_pos = min(pos0 + kBQ - 1, kv_len - 1);
  // kv tiles: with a sliding window those wholly before the first row's window are skipped, except the first ones if they hold
  // kept tokens
  const int win_tile = p.window > 0 ? max(0, pos0 - p.window + 1) / kBKV : 0;
  const int kept_tiles = p.window > 0 ? min((p.keep + kBKV - 1) / kBKV, win_tile) : 0;
  const int tile0 = win_tile - kept_tiles;         // tile of ordinal j: j + (j < kept_tiles ? 0 : tile0)
  const int n_tiles = last_pos / kBKV + 1 - tile0;
  const int n_units = n_tiles * kMaps;             // (tile, map) pairs
  const int seq_pages = (kv_len + kPageTok - 1) / kPageTok;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 256);
    }
    for (int i = 0; i < 2; ++i) { mbar_init(&p_ready[i], 256); mbar_init(&pv_done[i], 1); mbar_init(&mx_bar[i], 256); }
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  const uint32_t tS = tmem;            // + 128 * buffer
  const uint32_t tO = tmem + 256;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tm_q); tma_prefetch_desc(&tm_k); tma_prefetch_desc(&tm_v);
      if (kRope) { tma_prefetch_desc(&tm_qr); tma_prefetch_desc(&tm_kr); }
      const int qcol = kRope ? head * p.q_head_stride : head * kHD;
      mbar_expect_tx(&q_full, kTileB + (kRope ? kHalfBytes : 0));
      tma_load_2d(sQ, &tm_q, &q_full, qcol, q0 + row0);
      tma_load_2d(sQ + kHalfBytes, &tm_q, &q_full, qcol + 64, q0 + row0);
      if (kRope) tma_load_2d(sQr, &tm_qr, &q_full, head * p.qr_head_stride + p.qr_col0, q0 + row0);
      const int* pt = p.page_table + static_cast<size_t>(seq) * p.max_pages;
      const int tmp_page0 = kRope ? p.kv_tmp_start[seq] / kPageTok : 0;
      auto pages_of = [&](int jj, int& pa, int& pb, int& ka, int& kb) {
        const int j = jj + (jj < kept_tiles ? 0 : tile0);
        pa = 2 * j < seq_pages ? pt[2 * j] : 0;                      // page 0 is the all-zero page
        pb = 2 * j + 1 < seq_pages ? pt[2 * j + 1] : 0;
        // expanded K / V (kRope) sit in order in their buffer: "page" = row block of 64; past the end TMA fills zeros
        ka = kRope ? tmp_page0 + 2 * j : pa;
        kb = kRope ? tmp_page0 + 2 * j + 1 : pb;
      };
      auto load_k = [&](int j) -> bool {
        const int st = j & 1;
        const uint32_t ph = (j >> 1) & 1;
        int pa, pb, ka, kb;
        pages_of(j, pa, pb, ka, kb);
        if (!mbar_wait(&k_empty[st], ph ^ 1, p.status, kTimeoutEmptyBarrier)) return false;
        uint8_t* kd = sK + st * kTileB;
        mbar_expect_tx(&k_full[st], kTileB + (kRope ? kHalfBytes : 0));
        tma_load_4d(kd, &tm_k, &k_full[st], 0, kvh, 0, ka);
        tma_load_4d(kd + 64 * 128, &tm_k, &k_full[st], 0, kvh, 0, kb);
        tma_load_4d(kd + kHalfBytes, &tm_k, &k_full[st], 64, kvh, 0, ka);
        tma_load_4d(kd + kHalfBytes + 64 * 128, &tm_k, &k_full[st], 64, kvh, 0, kb);
        if (kRope) {
          uint8_t* rd = sKr + st * kHalfBytes;
          tma_load_3d(rd, &tm_kr, &k_full[st], 512, 0, pa);
          tma_load_3d(rd + 64 * 128, &tm_kr, &k_full[st], 512, 0, pb);
        }
        return true;
      };
      auto load_v = [&](int j) -> bool {
        const int vs = kVS == 2 ? (j & 1) : 0;
        const uint32_t vph = kVS == 2 ? ((j >> 1) & 1) : (j & 1);
        int pa, pb, ka, kb;
        pages_of(j, pa, pb, ka, kb);
        if (!mbar_wait(&v_empty[vs], vph ^ 1, p.status, kTimeoutEmptyBarrier)) return false;
        uint8_t* vd = sV + vs * kTileB;
        mbar_expect_tx(&v_full[vs], kTileB);
        tma_load_4d(vd, &tm_v, &v_full[vs], 0, kvh, 0, ka);
        tma_load_4d(vd + 64 * 128, &tm_v, &v_full[vs], 0, kvh, 0, kb);
        tma_load_4d(vd + kHalfBytes, &tm_v, &v_full[vs], 64, kvh, 0, ka);
        tma_load_4d(vd + kHalfBytes + 64 * 128, &tm_v, &v_full[vs], 64, kvh, 0, kb);
        return true;
      };
      // K runs ahead of V by as many tiles as the scores run ahead of P V (see the MMA warp): a K stage is free as
      // soon as its scores are done, long before the V stage of the same tile is.
      constexpr int kLead = kVS == 2 ? 2 : 0;
      bool ok = true;
      for (int j = 0; ok && j < kLead && j < n_tiles; ++j) ok = load_k(j);
      for (int j = 0; ok && j < n_tiles; ++j) {
        if (kLead == 0) ok = load_k(j);
        if (ok) ok = load_v(j);
        if (ok && kLead > 0 && j + kLead < n_tiles) ok = load_k(j + kLead);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc(128, 128, 1, 1, 0, 0);
      constexpr uint32_t idesc_pv = make_idesc(128, 128, 1, 1, 0, 1);   // B = V is MN-major
      const uint32_t aQ = smem_u32(sQ), aP = smem_u32(sP);
      bool ok = mbar_wait(&q_full, 0, p.status, kTimeoutFullBarrier);
      auto issue_qk = [&](int u) -> bool {
        const int j = u / kMaps, st = j & 1, sb = u & 1;
        if ((kMaps == 1 || sb == 0) && !mbar_wait(&k_full[st], (j >> 1) & 1, p.status, kTimeoutFullBarrier)) return false;
        if (!mbar_wait(&s_empty[sb], ((u >> 1) & 1) ^ 1, p.status, kTimeoutTmemEmpty)) return false;
        tc_fence_after();
        const uint32_t aK = smem_u32(sK + st * kTileB);
        if (kMaps == 2) {
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4)
            umma_f16(tS + sb * 128, smem_desc_k_sw128(aQ + sb * kHalfBytes + k4 * 32),
                     smem_desc_k_sw128(aK + sb * kHalfBytes + k4 * 32), idesc_qk, k4 ? 1u : 0u);
          if (sb == 1) umma_commit(&k_empty[st]);
          umma_commit(&s_full[sb]);
          return true;
        }
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4)
            umma_f16(tS + st * 128, smem_desc_k_sw128(aQ + h * kHalfBytes + k4 * 32),
                     smem_desc_k_sw128(aK + h * kHalfBytes + k4 * 32), idesc_qk, (h | k4) ? 1u : 0u);
        if (kRope) {
          const uint32_t aQr = smem_u32(sQr), aKr = smem_u32(sKr + st * kHalfBytes);
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4)
            umma_f16(tS + st * 128, smem_desc_k_sw128(aQr + k4 * 32), smem_desc_k_sw128(aKr + k4 * 32), idesc_qk, 1u);
        }
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[st]);
        return true;
      };
      // Scores run two tiles ahead of P V: the softmax warps release a score buffer as soon as they have read it
      // into registers, so S(j + 2) is computed while they work on tile j and S(j + 1) is already waiting.
      // (The kRope variant has one V stage: its producer cannot load K(j + 2) before P V(j) has freed V, so there
      // the scores stay one tile ahead.)
      constexpr int kAhead = kVS == 2 ? 2 : 1;
      if (ok) ok = issue_qk(0);
      if (ok && kAhead == 2 && n_units > 1) ok = issue_qk(1);
      for (int u = 0; ok && u < n_units; ++u) {
        if (u + kAhead < n_units) { if (!issue_qk(u + kAhead)) { ok = false; break; } }
        const int j = u / kMaps, pb = u % kPB;
        if (!mbar_wait(&p_ready[pb], (u / kPB) & 1, p.status, kTimeoutSoftmax)) { ok = false; break; }
        const int vs = kVS == 2 ? (j & 1) : 0;
        const uint32_t vph = kVS == 2 ? ((j >> 1) & 1) : (j & 1);
        if ((kMaps == 1 || pb == 0) && !mbar_wait(&v_full[vs], vph, p.status, kTimeoutFullBarrier)) { ok = false; break; }
        tc_fence_after();
        const uint32_t tOm = kMaps == 2 ? tO + pb * 128 : tO;
        const uint32_t aV = smem_u32(sV + vs * kTileB);
#pragma unroll
        for (int k8 = 0; k8 < 8; ++k8) {
          // A = P: atom (k8 / 4) of 64 kv columns, 32 bytes per K step inside it
          // B = V: 16 kv rows per step (2 KiB), two 64-wide d halves 16 KiB apart
          umma_f16(tOm, smem_desc_k_sw128(aP + pb * kTileB + (k8 >> 2) * kHalfBytes + (k8 & 3) * 32),
                   smem_desc_mn_sw128(aV + k8 * 2048, kHalfBytes), idesc_pv, (j | k8) ? 1u : 0u);
        }
        if (kMaps == 1 || pb == 1) umma_commit(&v_empty[vs]);
        umma_commit(&pv_done[pb]);
      }
    }
  } else {
    // Eight softmax warps: warps w and w + 4 share a TMEM lane quarter (32 query rows) and split the tile's 128
    // kv columns in halves, so every scheduler has two warps to cover each other's instruction latencies.
    const int quad = warp & 3;
    const int half = (warp - 2) >> 2;                // 0: columns 0..63, 1: columns 64..127
    const int row = quad * 32 + lane;               // row within the tile = TMEM lane
    const int rowpos = pos0 + row;
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    float m_run = -INFINITY, l_run = 0.f;           // l_run: this half's share of the row sum
    float m_alt = -INFINITY, l_alt = 0.f;           // kMaps == 2: the other map's (the pairs change places after every unit)
    bool ok = true;
    for (int u = 0; ok && u < n_units; ++u) {
      const int j = u / kMaps, st = u & 1;
      const uint32_t ph = (u >> 1) & 1;
      const uint32_t tOm = kMaps == 2 ? tO + st * 128 : tO;
      if (!mbar_wait(&s_full[st], ph, p.status, kTimeoutTmemFull)) { ok = false; break; }
      tc_fence_after();
      const uint32_t tSj = tS + st * 128 + lane_off + half * 64;
      const int col0 = (j + (j < kept_tiles ? 0 : tile0)) * kBKV;   // first kv position of this tile
      // uniform over the CTA: the tile reaches past the first row's diagonal, or starts before the last row's window and is not
      // wholly kept
      const bool need_mask = (col0 + kBKV - 1) > pos0 || (p.window > 0 && col0 < pos0 + kBQ - p.window && col0 + kBKV > p.keep);
      const int col_limit = rowpos - col0 - half * 64;          // local columns <= col_limit are visible
      const int col_lo = p.window > 0 ? col_limit - p.window + 1 : -(1 << 30);   // and local columns >= col_lo
      const int col_keep = p.keep - col0 - half * 64;           // or < col_keep
      // This half of the score row goes to registers with one wait; the TMEM buffer is handed back at once, so
      // the MMA warp can start the scores of tile j + 2 while this tile's exponentials run.
      uint32_t r[64];
      tmem_ld_32x32(tSj, *reinterpret_cast<uint32_t(*)[32]>(r));
      tmem_ld_32x32(tSj + 32, *reinterpret_cast<uint32_t(*)[32]>(r + 32));
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&s_empty[st]);
      if constexpr (kTurn) {
        if (p.cap_log2 > 0.f) cap_scores(r, p.cap_in, p.cap_log2);
      }
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < 64; ++i)
          if (i > col_limit || (i < col_lo && i >= col_keep)) r[i] = 0xff800000u;    // -inf
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};   // four chains: the maximum is latency-bound
#pragma unroll
      for (int i = 0; i < 64; i += 4) {
#pragma unroll
        for (int k = 0; k < 4; ++k) mx4[k] = fmaxf(mx4[k], __uint_as_float(r[i + k]));
      }
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // the row maximum over both halves: both use max(ceil_bf16(own), ceil_bf16(other)), the same value
      __nv_bfloat16* xmx = reinterpret_cast<__nv_bfloat16*>(s_xch) + st * 256;
      const __nv_bfloat16 own = __float2bfloat16_ru(mx);
      xmx[half * 128 + row] = own;
      mbar_arrive(&mx_bar[st]);
      if (!mbar_wait(&mx_bar[st], ph, p.status, kTimeoutSoftmax)) { ok = false; break; }
      mx = fmaxf(__bfloat162float(own), __bfloat162float(xmx[(half ^ 1) * 128 + row])) * p.scale_log2;   // scale > 0
      // The reference maximum only moves when the row maximum exceeds it by more than 8 (factor 256): P stays
      // within bf16 / fp32 range and O is rescaled rarely; O and the running sum share the reference, so the
      // quotient is exact all the same.
      const float m_new = (mx > m_run + 8.0f) ? mx : m_run;
      const float base = (m_new == -INFINITY) ? 0.f : m_new;
      const float corr = (m_run == -INFINITY) ? 0.f : fast_exp2(m_run - base);
      // O may be rescaled once P V of the previous tile has completed; P buffer pb is free once the P V that read
      // it (tile j - kPB) has
      const int pb = u % kPB;
      const bool rescale = j > 0 && __any_sync(0xffffffffu, corr != 1.0f);
      if (u >= kPB && !mbar_wait(&pv_done[pb], (u / kPB - 1) & 1, p.status, kTimeoutTmemFull)) { ok = false; break; }
      if (rescale) {
        // (with two maps the P V that last touched this map's O is the one just waited for)
        if (kMaps == 1 && !mbar_wait(&pv_done[(u - 1) % kPB], ((u - 1) / kPB) & 1, p.status, kTimeoutTmemFull)) { ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < 2; ++c) {             // this half's 64 columns of O
          uint32_t o[32];
          tmem_ld_32x32(tOm + lane_off + half * 64 + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
          tmem_st_32x32(tOm + lane_off + half * 64 + c * 32, o);
        }
      }
      // P = exp2(S * scale - m) as bf16 into swizzled shared memory; running sum in fp32
      float rs0 = 0.f, rs1 = 0.f;
      const float nbase = -base;
      // local columns [0, 64) of this half = swizzle atom `half`, 16-byte chunks 0..7
      uint8_t* prow = sP + pb * kTileB + half * kHalfBytes + row * 128;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float e0 = fast_exp2(fmaf(__uint_as_float(r[c * 32 + i]), p.scale_log2, nbase));
          const float e1 = fast_exp2(fmaf(__uint_as_float(r[c * 32 + i + 1]), p.scale_log2, nbase));
          rs0 += e0;
          rs1 += e1;
          pk[i >> 1] = pack_bf16(e0, e1);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int chunk = c * 4 + q;
          *reinterpret_cast<uint4*>(prow + ((chunk ^ (row & 7)) << 4)) =
              make_uint4(pk[4 * q], pk[4 * q + 1], pk[4 * q + 2], pk[4 * q + 3]);
        }
      }
      l_run = l_run * corr + (rs0 + rs1);
      m_run = m_new;
      tmem_st_wait();
      fence_async_smem();
      tc_fence_before();
      mbar_arrive(&p_ready[pb]);
      if (kMaps == 2) {
        float x = m_run; m_run = m_alt; m_alt = x;
        x = l_run; l_run = l_alt; l_alt = x;
      }
    }
    // ---- epilogue: O / l ---------------------------------------------------------------------------
    if (kMaps == 2) {
      // Both maps end with the last tile (n_units is even).  Once their last P V have run the P buffers are free: the row sums
      // and then the squares of the two column halves meet there.
      const uint32_t last = (n_tiles - 1) & 1, fph = n_tiles & 1;      // fph: the barriers' next phase
      float* xl = reinterpret_cast<float*>(sP);
      ok = ok && mbar_wait(&pv_done[0], last, p.status, kTimeoutTmemFull) && mbar_wait(&pv_done[1], last, p.status, kTimeoutTmemFull);
      if (ok) {
        tc_fence_after();
        xl[half * 128 + row] = l_run;
        xl[256 + half * 128 + row] = l_alt;
        mbar_arrive(&mx_bar[0]);
        ok = mbar_wait(&mx_bar[0], fph, p.status, kTimeoutSoftmax);
      }
      float o[64], ss = 0.f;
      if (ok) {
        const float l1 = l_run + xl[(half ^ 1) * 128 + row], l2 = l_alt + xl[256 + (half ^ 1) * 128 + row];
        const float w1 = l1 > 0.f ? 1.0f / l1 : 0.f, w2 = l2 > 0.f ? p.lambda / l2 : 0.f;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t a[32], b[32];
          tmem_ld_32x32(tO + lane_off + half * 64 + c * 32, a);
          tmem_ld_32x32(tO + 128 + lane_off + half * 64 + c * 32, b);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float v = __uint_as_float(a[i]) * w1 - __uint_as_float(b[i]) * w2;
            o[c * 32 + i] = v;
            ss += v * v;
          }
        }
        xl[512 + half * 128 + row] = ss;
        mbar_arrive(&mx_bar[1]);
        ok = mbar_wait(&mx_bar[1], fph, p.status, kTimeoutSoftmax);
      }
      if (ok && row0 + row < q_len) {
        const float k = p.out_scale / sqrtf((ss + xl[512 + (half ^ 1) * 128 + row]) * (1.0f / kHD) + p.eps);
        __nv_bfloat16* orow = p.out + static_cast<size_t>(q0 + row0 + row) * p.ldo + head * kHD + half * 64;
#pragma unroll
        for (int i = 0; i < 64; i += 8)
          *reinterpret_cast<uint4*>(orow + i) = make_uint4(pack_bf16(o[i] * k, o[i + 1] * k), pack_bf16(o[i + 2] * k, o[i + 3] * k),
                                                           pack_bf16(o[i + 4] * k, o[i + 5] * k), pack_bf16(o[i + 6] * k, o[i + 7] * k));
      }
    } else if (ok && mbar_wait(&pv_done[(n_tiles - 1) % kPB], ((n_tiles - 1) / kPB) & 1, p.status, kTimeoutTmemFull)) {
      // The last P V has run, so every softmax thread is past its last read of the exchange buffer: the two halves
      // now add their row sums through it.
      float* xl = reinterpret_cast<float*>(s_xch);
      const int fb = n_tiles & 1;                    // the barrier that tile n_tiles would have used
      xl[half * 128 + row] = l_run;
      mbar_arrive(&mx_bar[fb]);
      if (mbar_wait(&mx_bar[fb], (n_tiles >> 1) & 1, p.status, kTimeoutSoftmax)) l_run += xl[(half ^ 1) * 128 + row];
      else l_run = 0.f;
      tc_fence_after();
      const bool row_ok = (row0 + row) < q_len;
      if (p.sink) l_run += exp2f(p.sink[head] * 1.4426950408889634f - (m_run == -INFINITY ? 0.f : m_run));   // both halves hold the same maximum
      float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
      if (p.gate && row_ok) inv /= 1.0f + expf(-__bfloat162float(p.gate[static_cast<size_t>(q0 + row0 + row) * p.gate_ld + head]));
      if constexpr (kTurn) inv *= p.out_scale;
      if (kTurn && p.v_table) {
        // values m and m + 64 turn together: this thread takes 32 of either half of the head
        uint32_t a[32], b[32];
        tmem_ld_32x32(tO + lane_off + half * 32, a);
        tmem_ld_32x32(tO + lane_off + 64 + half * 32, b);
        tmem_ld_wait();
        if (row_ok) {
          const float4* cs = reinterpret_cast<const float4*>(p.v_table + static_cast<size_t>(q0 + row0 + row) * 64 + half * 32);
          __nv_bfloat16* dst = p.out + static_cast<size_t>(q0 + row0 + row) * p.ldo + head * kHD + half * 32;
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            float u[8], v[8];
#pragma unroll
            for (int e = 0; e < 8; e += 2) {
              const float4 t = cs[(i + e) >> 1];
              const float a0 = __uint_as_float(a[i + e]) * inv, b0 = __uint_as_float(b[i + e]) * inv;
              const float a1 = __uint_as_float(a[i + e + 1]) * inv, b1 = __uint_as_float(b[i + e + 1]) * inv;
              u[e] = a0 * t.x + b0 * t.y; v[e] = b0 * t.x - a0 * t.y;
              u[e + 1] = a1 * t.z + b1 * t.w; v[e + 1] = b1 * t.z - a1 * t.w;
            }
            *reinterpret_cast<uint4*>(dst + i) = make_uint4(pack_bf16(u[0], u[1]), pack_bf16(u[2], u[3]), pack_bf16(u[4], u[5]), pack_bf16(u[6], u[7]));
            *reinterpret_cast<uint4*>(dst + 64 + i) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
          }
        }
      } else {
      __nv_bfloat16* orow = p.out + static_cast<size_t>(q0 + row0 + row) * p.ldo + head * kHD + half * 64;
#pragma unroll 1
      for (int c = 0; c < 2; ++c) {
        uint32_t r[32];
        tmem_ld_32x32(tO + lane_off + half * 64 + c * 32, r);
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 q;
            q.x = pack_bf16(__uint_as_float(r[i]) * inv, __uint_as_float(r[i + 1]) * inv);
            q.y = pack_bf16(__uint_as_float(r[i + 2]) * inv, __uint_as_float(r[i + 3]) * inv);
            q.z = pack_bf16(__uint_as_float(r[i + 4]) * inv, __uint_as_float(r[i + 5]) * inv);
            q.w = pack_bf16(__uint_as_float(r[i + 6]) * inv, __uint_as_float(r[i + 7]) * inv);
            *reinterpret_cast<uint4*>(orow + c * 32 + i) = q;
          }
        }
      }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace cafd

using namespace cafd;

// q [total_q, Hq, 128] bf16 (two maps: [total_q, Hq, 2, 64]); out rows of ldo elements, head h's 128 values at column 128 h;
// caches [num_pages, Hkv, 64, 128] bf16 (page 0 all zero); page_table [num_seqs, max_pages]; seq_lens [num_seqs];
// q_start [num_seqs + 1]; max_q_len = longest chunk (grid sizing).  maps 1: lambda and eps are unused.
// sink [Hq], gate rows (gate_ld elements apart), v_table [total_q, 64] (cos, sin of the output's rotation back) and cap (0 = none): one
// map only.
extern "C" int cafd_attn_prefill(const void* q, const void* k_cache, const void* v_cache, const int* page_table,
                                 const int* seq_lens, const int* q_start, void* out, uint32_t* status, int total_q,
                                 int num_seqs, int max_q_len, int num_pages, int max_pages, int Hq, int Hkv, int D,
                                 float scale, int window, int keep, int ldo, int maps, float lambda, float out_scale, float eps,
                                 const float* sink, const void* gate, int gate_ld, float cap, const void* v_table, cafd_stream_t s) {
  if (num_seqs <= 0 || total_q <= 0) return 0;
  if (D != kHD || Hq % Hkv || window < 0 || keep < 0 || maps < 1 || maps > 2 || ldo < Hq * kHD || ldo % 8) return -10;
  if ((maps == 2 && (sink || gate || v_table || cap > 0.f)) || (gate && gate_ld < Hq)) return -10;
  CUtensorMap tq, tk, tv;
  int rc = cached_tmap_2d(&tq, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, total_q, static_cast<uint64_t>(Hq) * kHD,
                          static_cast<uint64_t>(Hq) * kHD * 2, kBQ, 64);
  if (rc) return rc;
  const uint64_t dims[4] = {static_cast<uint64_t>(kHD), static_cast<uint64_t>(Hkv), kPageTok,
                            static_cast<uint64_t>(num_pages)};
  // The pools are [page, kv head, 64 tokens, D]; the map keeps the coordinate order (d, kv head, token, page) the
  // kernel uses and only names the strides of that memory layout (head stride 64 * D, token stride D).
  const uint64_t strides[3] = {static_cast<uint64_t>(kPageTok) * kHD * 2, static_cast<uint64_t>(kHD) * 2,
                               static_cast<uint64_t>(kPageTok) * Hkv * kHD * 2};
  const uint32_t box[4] = {64, 1, kPageTok, 1};
  rc = make_tmap_nd(&tk, k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dims, strides, box, true);
  if (rc) return rc;
  rc = make_tmap_nd(&tv, v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dims, strides, box, true);
  if (rc) return rc;
  PrefillDev p{};
  p.page_table = page_table;
  p.seq_lens = seq_lens;
  p.q_start = q_start;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.status = status;
  p.max_pages = max_pages;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.scale_log2 = cap > 0.f ? 1.f : scale * 1.4426950408889634f;
  p.v_table = static_cast<const float2*>(v_table);
  p.cap_in = cap > 0.f ? scale / cap : 0.f;
  p.cap_log2 = cap * 1.4426950408889634f;
  p.window = window;
  p.keep = window > 0 ? keep : 0;
  p.ldo = ldo;
  p.lambda = lambda; p.out_scale = out_scale; p.eps = eps;
  p.sink = sink; p.gate = static_cast<const __nv_bfloat16*>(gate); p.gate_ld = gate_ld;
  p.q_head_stride = kHD;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_prefill_kernel<false, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrefillSmem));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_prefill_kernel<false, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrefillSmem));
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_prefill_kernel<false, 1, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrefillSmem));
    attr = true;
  }
  dim3 grid((max_q_len + kBQ - 1) / kBQ, Hq, num_seqs);
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (maps == 2) launch_pdl(attn_prefill_kernel<false, 2>, grid, dim3(kPrefillThreads), kPrefillSmem, st, tq, tk, tv, tq, tq, p);
  else if (cap > 0.f || v_table || out_scale != 1.f) launch_pdl(attn_prefill_kernel<false, 1, true>, grid, dim3(kPrefillThreads), kPrefillSmem, st, tq, tk, tv, tq, tq, p);
  else launch_pdl(attn_prefill_kernel<false, 1>, grid, dim3(kPrefillThreads), kPrefillSmem, st, tq, tk, tv, tq, tq, p);
  return static_cast<int>(cudaGetLastError());
}

// MLA prefill in expanded form.  q_nope [total_q, heads * q_head_stride] bf16, q_pitch elements from row to row (the first
// 128 columns of every head);
// q_rope [total_q, heads * qr_head_stride] bf16 with the rotated 64 rope dims of head h at column
// h * qr_head_stride + qr_col0; k_exp / v_exp [tmp_rows, heads * 128] bf16 = per-head K_nope / V of every cached
// token of the sequences, sequence s starting at row kv_tmp_start[s] (a multiple of 64); latent cache
// [num_pages, 64, 576] supplies the shared rope keys (columns 512..575) through the page table.
// out rows of ldo elements, head h's 128 values at column 128 h.
extern "C" int cafd_attn_prefill_mla(const void* q_nope, int q_pitch, int q_head_stride, const void* q_rope, int qr_head_stride, int qr_col0,
                                     const void* k_exp, const void* v_exp, long long tmp_rows, const int* kv_tmp_start,
                                     const void* latent_cache, const int* page_table, const int* seq_lens, const int* q_start,
                                     void* out, uint32_t* status, int total_q, int num_seqs, int max_q_len, int num_pages,
                                     int max_pages, int heads, float scale, int window, int ldo, cafd_stream_t s) {
  if (num_seqs <= 0 || total_q <= 0) return 0;
  if (ldo < heads * kHD || ldo % 8 || window < 0 || q_pitch < heads * q_head_stride || (q_pitch % 8)) return -10;
  if (tmp_rows % kPageTok || (q_head_stride % 8) || (qr_head_stride % 8) || (qr_col0 % 8)) return -10;
  CUtensorMap tq, tqr, tk, tv, tkr;
  int rc = cached_tmap_2d(&tq, q_nope, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, total_q, static_cast<uint64_t>(heads) * q_head_stride,
                          static_cast<uint64_t>(q_pitch) * 2, kBQ, 64);
  if (rc) return rc;
  rc = cached_tmap_2d(&tqr, q_rope, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, total_q, static_cast<uint64_t>(heads) * qr_head_stride,
                      static_cast<uint64_t>(heads) * qr_head_stride * 2, kBQ, 64);
  if (rc) return rc;
  const uint64_t dims[4] = {static_cast<uint64_t>(kHD), static_cast<uint64_t>(heads), kPageTok, static_cast<uint64_t>(tmp_rows / kPageTok)};
  const uint64_t strides[3] = {static_cast<uint64_t>(kHD) * 2, static_cast<uint64_t>(heads) * kHD * 2,
                               static_cast<uint64_t>(kPageTok) * heads * kHD * 2};
  const uint32_t box[4] = {64, 1, kPageTok, 1};
  rc = make_tmap_nd(&tk, k_exp, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dims, strides, box, true);
  if (rc) return rc;
  rc = make_tmap_nd(&tv, v_exp, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dims, strides, box, true);
  if (rc) return rc;
  const uint64_t ldims[3] = {576, kPageTok, static_cast<uint64_t>(num_pages)};
  const uint64_t lstrides[2] = {576 * 2, static_cast<uint64_t>(kPageTok) * 576 * 2};
  const uint32_t lbox[3] = {64, kPageTok, 1};
  rc = make_tmap_nd(&tkr, latent_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, ldims, lstrides, lbox, true);
  if (rc) return rc;
  PrefillDev p{};
  p.page_table = page_table; p.seq_lens = seq_lens; p.q_start = q_start;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.status = status;
  p.max_pages = max_pages; p.Hq = heads; p.Hkv = heads;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = window;
  p.ldo = ldo;
  p.kv_tmp_start = kv_tmp_start; p.q_head_stride = q_head_stride; p.qr_head_stride = qr_head_stride; p.qr_col0 = qr_col0;
  static bool attr = false;
  if (!attr) {
    CAFD_CHECK_CUDA(cudaFuncSetAttribute(attn_prefill_kernel<true, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, kPrefillSmemRope));
    attr = true;
  }
  dim3 grid((max_q_len + kBQ - 1) / kBQ, heads, num_seqs);
  launch_pdl(attn_prefill_kernel<true, 1>, grid, dim3(kPrefillThreads), kPrefillSmemRope, static_cast<cudaStream_t>(s), tq, tk, tv, tqr, tkr, p);
  return static_cast<int>(cudaGetLastError());
}

CAFD_WAIT_LIMIT_SETTER(cafd_attn_set_wait_limit_ns)
