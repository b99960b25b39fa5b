// The launch between two sublayers (hybrid_norm.cuh) for bf16 activations, and its entry point.
#include "hybrid_norm.cuh"

namespace cafd {

// Exchange two id vectors (a device-resident decode loop alternates the state slots it reads and writes).
__global__ void swap_ids_kernel(int* a, int* b, int n) {
  pdl_wait();
  pdl_trigger();
  for (int i = threadIdx.x; i < n; i += blockDim.x) { const int t = a[i]; a[i] = b[i]; b[i] = t; }
}

// Rows of a second embedding table, picked by a token and the one before it: (previous * mul_prev + token * mul_cur) mod buckets, for
// a sequence's first token row `buckets`.  A sequence's slot holds its last token's id plus one as an integer (0: it has none yet).
struct BigramArgs {
  const int* tokens;
  const int* q_start;         // [S + 1]
  const int* state_in;
  const int* state_out;
  float* state;
  int* rows;                  // [T]
  long long slot_stride, state_off, mul_prev, mul_cur, buckets;
  int T, S;
};

__global__ void __launch_bounds__(128) bigram_rows_kernel(const BigramArgs a) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t >= a.T) return;
  int seq = 0, hi = a.S;                          // last s with q_start[s] <= t
  while (hi - seq > 1) {
    const int mid = (seq + hi) >> 1;
    if (a.q_start[mid] <= t) seq = mid; else hi = mid;
  }
  const int cur = a.tokens[t];
  auto word = [&](int slot) { return reinterpret_cast<int*>(a.state + static_cast<size_t>(slot) * a.slot_stride + a.state_off); };
  const int prev = t > a.q_start[seq] ? a.tokens[t - 1] : *word(a.state_in[seq]) - 1;
  long long r = a.buckets;
  if (prev >= 0) {
    r = (prev * a.mul_prev + cur * a.mul_cur) % a.buckets;
    if (r < 0) r += a.buckets;
  }
  a.rows[t] = static_cast<int>(r);
  if (t == a.q_start[seq + 1] - 1) *word(a.state_out[seq]) = cur + 1;
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_norm_conv_f32(const NormArgs* args, cafd_stream_t s);

extern "C" int cafd_bigram_rows(const BigramArgs* a, cafd_stream_t s) {
  if (a->T <= 0) return 0;
  if (a->S < 1 || a->buckets < 1 || !a->tokens || !a->q_start || !a->state || !a->state_in || !a->state_out || !a->rows) return -10;
  launch_pdl(bigram_rows_kernel, dim3((a->T + 127) / 128), dim3(128), 0, static_cast<cudaStream_t>(s), *a);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int cafd_swap_ids(int* a, int* b, int n, cafd_stream_t s) {
  launch_pdl(swap_ids_kernel, dim3(1), dim3(64), 0, static_cast<cudaStream_t>(s), a, b, n);
  return static_cast<int>(cudaGetLastError());
}

// One launch between two sublayers (see the file's head).  `is_f32`: activations and the embedding table are fp32, else bf16.
extern "C" int cafd_norm_conv(const NormArgs* args, int is_f32, cafd_stream_t s) {
  NormArgs a = *args;
  if (a.T <= 0) return 0;
  if (a.H <= 0 || a.groups <= 0 || a.H % a.groups || (a.conv && (a.taps < 1 || a.taps > 16)) || !a.h_out || a.ldh < a.H || a.ldh % 8) return -10;
  if (a.slot_w && (!a.ident || a.ldi < a.H || a.ldi % 8)) return -10;
  if ((!a.w && (a.conv || a.w2)) || (a.w2 && (!a.h2_out || a.conv)) || (a.base && (!a.slot_w || a.ldb < a.H || a.ldb % 8))) return -10;
  if (a.y && (a.ldy < a.H || a.ldy % 8)) return -10;
  if (a.conv && (a.row_idx || !a.q_start || a.S < 1 || (a.taps > 1 && (!a.state || !a.state_in || !a.state_out)))) return -10;
  if (!a.embed && !a.x_in) return -10;
  if (a.rows2 && (!a.embed || !a.embed2 || a.vocab2 < 1)) return -10;
  if (a.past_w && (a.conv || a.n_past < 1 || !a.past)) return -10;
  if (a.x_out && a.x_out == a.x_in) return -11;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return is_f32 ? cafd_norm_conv_f32(&a, s) : dispatch_norm<__nv_bfloat16>(a, st);
}
