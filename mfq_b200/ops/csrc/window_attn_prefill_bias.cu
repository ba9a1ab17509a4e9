// The form of the prefill attention kernel with a score bias by distance and a sink (a file of its own: it compiles beside the other).
#include "window_attn_prefill.cuh"

namespace mfq {

int window_prefill_extra(const WindowPrefillParams& p, const WindowPrefillCall& c, cudaStream_t stream) {
  return run_window_prefill<true>(p, c, stream);
}

}  // namespace mfq
