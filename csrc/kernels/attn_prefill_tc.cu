// Prefill attention over the paged cache, heads of 64 or 128 (see attn_prefill_tc.cuh).
#include "attn_prefill_tc.cuh"

namespace oxb {

void launch_paged_prefill_tc(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                             const PrefillAttnParams& p, int n_tiles, int head_dim, int* status,
                             cudaStream_t stream) {
  if (n_tiles <= 0) return;
  if (head_dim == 128) {
    if (p.exact_p != 0) launch_tc<128, 128, 128, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
    else launch_tc<128, 128, 128, false>(tmQ, tmK, tmV, p, n_tiles, status, stream);
  } else {
    if (p.exact_p != 0) launch_tc<64, 64, 128, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
    else launch_tc<64, 64, 128, false>(tmQ, tmK, tmV, p, n_tiles, status, stream);
  }
}

}  // namespace oxb
