// Parameter blocks of the paged attention kernels.
// KV cache layout (per layer): [num_blocks, Hkv, 16 tokens, head_dim] bf16 for K and for V.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace oxb {

struct DecodeAttnParams {
  const __nv_bfloat16* q;  // [B, Hq, D], row stride q_stride (elements)
  long long q_stride;
  const __nv_bfloat16* k_cache;
  const __nv_bfloat16* v_cache;
  const int* block_tables;     // [B, max_blocks]
  const int* seq_lens;         // [B] context length including the current token
  const int* pages_per_split;  // device scalar, >= 1
  float* part_o;               // [B, Hq, max_splits, D]
  float* part_ml;              // [B, Hq, max_splits, 2]  (running max in log2 units, sum)
  __nv_bfloat16* out;          // [B, Hq*D], row stride out_stride
  long long out_stride;
  int max_blocks, Hq, Hkv, max_splits, window;
  int keep_first;    // with a window: the first positions stay visible too (0: none); they keep their true positions
  int out_d;         // values stored per head in `out` (<= D; 0: D). The caches and q are padded to D
  int exact_p;       // 1: softmax weights enter the value product as two bf16 terms (about 16 bits) instead of one
  int chunk;         // > 0: only positions of the query's own chunk are visible (chunks count from position 0)
  float scale_log2;  // softmax scale * log2(e)
  // score (times log2(e)) of a sink: one more term of the softmax denominator, without a value
  float sink_log2 = -INFINITY;
  const float* sinks;   // [Hq] the sinks' scores, one per head, or nullptr
  float out_gain = 1.f; // factor on the result
  // Differential attention (diff != 0): query heads 2 h and 2 h + 1 are the two maps of head h. The merge writes
  // o = a1 - diff_lambda a2, o / sqrt(mean(o^2) + diff_eps) * diff_gain, one row of out_d values per pair.
  int diff;
  float diff_lambda, diff_gain, diff_eps;
  // Bounds check of block-table entries: an id outside [0, num_blocks) is recorded in *status
  // (kStatusBadIndex) and page 0 is read instead. num_blocks <= 0 or status == nullptr: no check.
  int num_blocks;
  int* status;
  // Heavy-hitter statistics (optional, both or neither): the split kernel records for every attended
  // page and query head the pair (reference max in log2 units, sum of 2^(x - max) over the page's 16
  // tokens) in page_ml [B, max_blocks, Hq, 2]; after the merge a third kernel turns them into
  // block_mass [B, max_blocks] = sum over heads of the softmax probability that fell into the page
  // (0 for pages outside the attended range).
  float* page_ml;
  float* block_mass;
  // Optional int8 view of `out` for an integer GEMV that consumes it (blocks of 32 values with an
  // fp32 scale = amax / 127 and scale * sum): q8 [B, Hq*D] int8, q8_d / q8_s [B, Hq*D / 32], written
  // by the merge kernel.
  signed char* q8;
  float* q8_d;
  float* q8_s;
};

// Launches the split kernel and then the merge; the merge is skipped when the first launch failed.
// Coverage rule: pages_per_split * max_splits pages must cover the longest attended window, a
// split beyond max_splits does not exist and its tokens would be left out.
cudaError_t launch_paged_decode(const DecodeAttnParams& p, int batch, int head_dim, cudaStream_t stream);

struct PrefillAttnParams {
  const __nv_bfloat16* q;  // [T, Hq, D] ragged over sequences, row stride q_stride
  long long q_stride;
  const __nv_bfloat16* k_cache;
  const __nv_bfloat16* v_cache;
  const int* block_tables;  // [n_seqs, max_blocks]
  const int* tile_seq;      // [n_tiles] sequence of each 64-row query tile
  const int* tile_q0;       // [n_tiles] first query index of the tile inside its sequence
  const int* q_start;       // [n_seqs] first row of the sequence in q
  const int* q_lens;        // [n_seqs] query tokens of this chunk
  const int* ctx_lens;      // [n_seqs] context length after this chunk (KV tokens in the cache)
  __nv_bfloat16* out;       // [T, Hq*D], row stride out_stride
  long long out_stride;
  int max_blocks, Hq, Hkv, window;
  int keep_first, out_d, exact_p, chunk;  // as in DecodeAttnParams
  float scale_log2;
  float sink_log2 = -INFINITY;
  const float* sinks;   // as in DecodeAttnParams
  float out_gain = 1.f;
  int num_blocks;  // bound for block-table entries (<= 0: unchecked), violations go to *status
  int* status;
  float* out_f32;  // fp32 rows instead of `out` (the same pitch), or nullptr
  // Keys and values in plain rows instead of pages (kv_row0 != nullptr): position t of sequence s is row kv_row0[s] + t,
  // head g's keys start at column g * k_hd, its values at column v_col0 + g * v_hd
  const int* kv_row0;
  int k_hd, v_col0, v_hd;
};

// Head sizes (keys, values) of the plain-row form and of unequal or larger sizes than 128.
void launch_prefill_wide(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                         const PrefillAttnParams& p, int n_tiles, int dk, int dv, int* status, cudaStream_t stream);
int prefill_wide_tile(int dk, int dv);   // KV positions per tile, 0: sizes that are not built

void launch_paged_prefill_tc(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                             const PrefillAttnParams& p, int n_tiles, int head_dim, int* status,
                             cudaStream_t stream);

}  // namespace oxb
