// The recurrence for fp32 activations.
#include "recurrent.cuh"

namespace nckv {

cudaError_t recurrent_f32(const RecurrentParams &p, bool with_out, cudaStream_t s) { return rec_launch<float>(p, with_out, s); }

}  // namespace nckv
