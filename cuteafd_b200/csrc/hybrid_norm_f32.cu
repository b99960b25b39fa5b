// The launch between two sublayers (hybrid_norm.cuh) for fp32 activations.
#include "hybrid_norm.cuh"

using namespace cafd;

// Arguments are checked by cafd_norm_conv.
extern "C" int cafd_norm_conv_f32(const NormArgs* args, cafd_stream_t s) { return dispatch_norm<float>(*args, static_cast<cudaStream_t>(s)); }
