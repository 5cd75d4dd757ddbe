// Prefill attention for keys and values of unequal or larger sizes, from pages or from plain rows (see
// attn_prefill_tc.cuh). Softmax weights enter the value product as two bf16 terms.
#include "attn_prefill_tc.cuh"

namespace oxb {

// KV positions per tile: what two stages of keys and values, the queries and the weights leave room for
int prefill_wide_tile(int dk, int dv) {
  if (dk == 64 && dv == 64) return 128;
  if (dk == 128 && dv == 128) return 128;
  if (dk == 192 && dv == 128) return 64;
  if (dk == 256 && dv == 256) return 64;
  return 0;
}

void launch_prefill_wide(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                         const PrefillAttnParams& p, int n_tiles, int dk, int dv, int* status, cudaStream_t stream) {
  if (n_tiles <= 0) return;
  if (dk == 64) launch_tc<64, 64, 128, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
  else if (dk == 128) launch_tc<128, 128, 128, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
  else if (dk == 192) launch_tc<192, 128, 64, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
  else launch_tc<256, 256, 64, true>(tmQ, tmK, tmV, p, n_tiles, status, stream);
}

}  // namespace oxb
