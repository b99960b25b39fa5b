// The launch between two sublayers (hybrid_norm.cuh) for bf16 activations, and its entry point.
#include "hybrid_norm.cuh"

namespace cafd {

// Exchange two id vectors (a device-resident decode loop alternates the state slots it reads and writes).
__global__ void swap_ids_kernel(int* a, int* b, int n) {
  pdl_wait();
  pdl_trigger();
  for (int i = threadIdx.x; i < n; i += blockDim.x) { const int t = a[i]; a[i] = b[i]; b[i] = t; }
}

}  // namespace cafd

using namespace cafd;

extern "C" int cafd_norm_conv_f32(const NormArgs* args, cafd_stream_t s);

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
  if (a.x_out && a.x_out == a.x_in) return -11;
  cudaStream_t st = static_cast<cudaStream_t>(s);
  return is_f32 ? cafd_norm_conv_f32(&a, s) : dispatch_norm<__nv_bfloat16>(a, st);
}
