// 32-bit matrix products (fp32 operands, fp32 accumulation on the FMA pipe, no reduced-precision mode): the same call
// shape as the bf16 tensor-core GEMM (dense or expert-grouped, SwiGLU pair, row map), for engines that run a model with
// every product and activation in 32-bit.  One block computes a 64 x 64 output tile; K is walked in steps of 16.
#include "cafd_api.h"
#include "common.cuh"

namespace cafd {

constexpr int kF32Tile = 64, kF32K = 16, kF32Threads = 256;

struct GemmF32 {
  const float* w0;
  const float* w1;
  const float* x;
  float* out;
  const int* row_dst;
  const int* tile_expert;
  const int* tile_row0;
  const int* num_x_tiles;
  int k, n, x_rows, ldx, ldo, rows_per_expert, tile_rows, sub_tiles;
  Glu glu;
};

template <bool kDual>
__global__ void __launch_bounds__(kF32Threads) gemm_f32_kernel(const GemmF32 p) {
  __shared__ float sx[kF32K][kF32Tile + 4];
  __shared__ float sw[kDual ? 2 : 1][kF32K][kF32Tile + 4];
  pdl_wait();
  pdl_trigger();
  const int tile = blockIdx.x / p.sub_tiles, sub = blockIdx.x - tile * p.sub_tiles;
  if (p.num_x_tiles && tile >= *p.num_x_tiles) return;
  const int row0 = (p.tile_row0 ? p.tile_row0[tile] : tile * p.tile_rows) + sub * kF32Tile;
  const int row_end = min(p.x_rows, (p.tile_row0 ? p.tile_row0[tile] : tile * p.tile_rows) + p.tile_rows);
  const int expert = p.tile_expert ? p.tile_expert[tile] : 0;
  const int col0 = blockIdx.y * kF32Tile;
  const float* w0 = p.w0 + static_cast<size_t>(expert) * p.rows_per_expert * p.k;
  const float* w1 = kDual ? p.w1 + static_cast<size_t>(expert) * p.rows_per_expert * p.k : nullptr;
  const int tid = threadIdx.x, tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  float acc[kDual ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kF32K) {
    for (int i = tid; i < kF32Tile * kF32K; i += kF32Threads) {
      const int r = i / kF32K, c = i - r * kF32K, kk = k0 + c;
      const bool kin = kk < p.k;
      sx[c][r] = (kin && row0 + r < row_end) ? p.x[static_cast<size_t>(row0 + r) * p.ldx + kk] : 0.f;
      const bool win = kin && col0 + r < p.n;
      sw[0][c][r] = win ? w0[static_cast<size_t>(col0 + r) * p.k + kk] : 0.f;
      if (kDual) sw[kDual ? 1 : 0][c][r] = win ? w1[static_cast<size_t>(col0 + r) * p.k + kk] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kF32K; ++c) {
      float xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = sx[c][tr + i];
#pragma unroll
      for (int d = 0; d < (kDual ? 2 : 1); ++d)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wv = sw[d][c][tc + j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[d][i][j] = fmaf(xv[i], wv, acc[d][i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = row0 + tr + i;
    if (row >= row_end) continue;
    int dst = row;
    if (p.row_dst) { dst = p.row_dst[row]; if (dst < 0) continue; }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = col0 + tc + j;
      if (col >= p.n) continue;
      float v = acc[0][i][j];
      if (kDual) {
        float u = acc[kDual ? 1 : 0][i][j], alpha = 1.f;
        if (p.glu.kind) {
          v = fminf(v, p.glu.limit);
          u = fminf(fmaxf(u, -p.glu.limit), p.glu.limit) + p.glu.bias;
          alpha = p.glu.alpha;
        }
        v = v / (1.0f + expf(-alpha * v)) * u;
      }
      p.out[static_cast<size_t>(dst) * p.ldo + col] = v;
    }
  }
}

}  // namespace cafd

using namespace cafd;

// out[row_dst[r] or r] = x[r] @ w[expert of r's tile].T (with w1: the gated unit of both products, cafd_gemm_args.glu).  Dense: tile_expert,
// tile_row0, num_x_tiles and row_dst null, max_x_tiles = 0.  Grouped: tiles of tile_rows rows as the MoE plan writes them.
extern "C" int cafd_gemm_f32(const float* w0, const float* w1, const float* x, float* out, const int* row_dst, const int* tile_expert,
                             const int* tile_row0, const int* num_x_tiles, int k, int n, int x_rows, int ldx, int ldo,
                             int rows_per_expert, int max_x_tiles, int tile_rows, int glu, float glu_limit, float glu_alpha, float glu_bias,
                             cafd_stream_t s) {
  if (x_rows <= 0 || n <= 0) return 0;
  if (!w0 || !x || !out || k <= 0) return -10;
  GemmF32 p{w0, w1, x, out, row_dst, tile_expert, tile_row0, num_x_tiles, k, n, x_rows, ldx, ldo, rows_per_expert, tile_rows, 1,
            Glu{glu, glu_limit, glu_alpha, glu_bias}};
  int tiles = max_x_tiles;
  if (!tile_row0) {
    p.tile_rows = kF32Tile;
    tiles = (x_rows + kF32Tile - 1) / kF32Tile;
  }
  p.sub_tiles = (p.tile_rows + kF32Tile - 1) / kF32Tile;
  const dim3 grid(tiles * p.sub_tiles, (n + kF32Tile - 1) / kF32Tile);
  cudaStream_t st = static_cast<cudaStream_t>(s);
  if (w1) launch_pdl(gemm_f32_kernel<true>, grid, dim3(kF32Threads), 0, st, p);
  else launch_pdl(gemm_f32_kernel<false>, grid, dim3(kF32Threads), 0, st, p);
  return static_cast<int>(cudaGetLastError());
}
