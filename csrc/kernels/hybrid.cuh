// Parameter blocks of the kernels that serve layer-list decoders (attention, retention, ...): residual
// streams with their norms, projections -> heads with norms and rotations, row attention of any head
// size, retention, and the 32-bit matrix product. `dtype` 0: activations, weights and caches are bf16;
// 1: fp32 throughout. Scores, norms, states, residual streams and angles are fp32 in both.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace oxb {

constexpr int kMaxStreams = 16;

// What stands between two sublayers. With N values per row and S residual streams x_s:
//   tokens given : x_s = embed[token] (+ bigram row of the hash of the previous and this token), all s
//   y given      : x_t = sum_s mix[s, t] x_s + out[t] * y      (the sublayer that just ran)
//   then           u = sum_s in[s] x_s   (in == nullptr: the plain sum)
//                  h = u / sqrt(mean(u^2) + eps) * (w_offset + norm_w)
// x is written back when store_x is set; h rows go to row_map[row] (< 0: skipped) or to the same row.
struct StreamNormParams {
  float* x;                 // [rows, S, N]
  int rows, N, S;
  const int* tokens;        // [rows] or nullptr
  const int* prev;          // [rows] token before it in the sequence, -1: none
  const void* embed;        // [vocab, N]
  const void* bigram;       // [buckets + 1, N] or nullptr
  int vocab, buckets;
  long long mul_prev, mul_cur;
  float* y;                 // [rows, ldy] or nullptr
  long long ldy;
  int zero_y;               // clear y after reading it (split-K GEMMs add into it)
  const float* mix;         // [S, S] indexed [from, to]
  const float* out;         // [S]
  const float* in;          // [S] or nullptr
  int store_x;
  const float* norm_w;      // [N]
  float eps, w_offset;
  void* h;                  // [*, ldh]
  long long ldh;
  const int* row_map;
  float* clear;             // [rows, clear_ld] or nullptr: accumulator of a split-K GEMM that follows, zeroed here
  long long clear_ld;
  int clear_n;
  int* status;
};
cudaError_t launch_stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream);

// Rotary positions: pair i turns by position * (freq_hi[i] + freq_lo[i]) (the frequency as an unevaluated
// sum of two floats, so the angle is good to the last bits of a 32-bit float at any position).
struct RotaryParams {
  const float* freq_hi;     // [dims / 2]
  const float* freq_lo;
  int dims;                 // 0: no rotation
  int interleaved;          // pairs (2i, 2i+1), else (i, i + dims/2)
};

// Projection rows q | k | v -> per-head vectors: optional RMS norm over the whole q (k) projection with
// plain weights, rotation of q and k, k times k_scale. q goes to a dense buffer (head stride q_hd); k goes
// to a dense buffer (k_out) or, with v, into the paged cache [blocks, G, 16, DP] / [blocks, G, 16, EP].
struct HeadsParams {
  const void* proj;         // [M, ld], of the storage type, or fp32 when proj_f32 is set (split-K accumulator)
  int proj_f32;
  long long ld;
  int M, H, G, D, E;
  const float* q_norm;      // [H * D] or nullptr
  const float* k_norm;      // [G * D]
  float eps;
  RotaryParams rot;
  const int* positions;     // [M]
  float k_scale;
  void* q_out;              // element (row, head, d) at row * q_ld + head * q_hd + d
  long long q_ld, q_hd;
  float* k_out;             // dense fp32 (then q_out is fp32 too) or nullptr
  long long k_ld, k_hd;
  void* k_cache;
  void* v_cache;
  const long long* slots;   // [M] cache slot of each row, < 0: not stored
  long long num_slots;
  int DP, EP;
  int* status;
};
cudaError_t launch_heads(const HeadsParams& p, int dtype, cudaStream_t stream);

// Softmax attention of single query rows over the paged cache, any head sizes: the fp32 path, and head
// sizes that the tensor-core kernels do not take. Decode rows have tile_seq == nullptr.
struct RowAttnParams {
  const void* q;            // [rows, q_ld], head stride q_hd
  long long q_ld;
  int q_hd;
  const void* k_cache;      // [blocks, G, 16, DP]
  const void* v_cache;      // [blocks, G, 16, EP]
  const int* block_tables;  // [sequences, max_blocks]
  const int* seq_lens;      // decode: [rows]
  const int* tile_seq;      // prompt chunks: 128-row tiles
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_rows;               // decode: rows; chunks: tiles
  int max_blocks, num_blocks;
  int H, G, D, E, DP, EP;
  int window, keep_first;
  float scale;
  void* out;                // [rows, ldo], head stride E
  long long ldo;
  int* status;
};
cudaError_t launch_row_attention(const RowAttnParams& p, int dtype, cudaStream_t stream);

constexpr int kRetChunk = 64;   // rows per chunk of the chunked form (two per 128-row tile of the scheduler)

struct RetentionParams {
  const void* proj;         // [M, ld]: q (H*D) | k (H*D) | v (H*E) | gate (H*E); type as in HeadsParams
  int proj_f32;
  long long ld;
  int H, D, E;
  const float* decay_pow;   // [H, kRetChunk + 1]: decay^0 .. decay^kRetChunk
  RotaryParams rot;
  float k_scale, eps;
  float* state;             // [slots, H, D, E]
  int num_slots;
  // decode rows
  const int* row_slots;     // [rows], < 0: padding row
  const int* positions;     // [rows]; a row at position 0 starts from the zero state
  int rows;
  // prompt chunks
  const int* seq_slots;     // [sequences]
  const int* tile_seq;
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_tiles, n_seqs;
  const float* q_rot;       // fp32, rotated: [H][M][D], heads rot_hd apart (a chunk of a head is one contiguous run)
  const float* k_rot;       // the same layout, rotated and scaled
  long long rot_hd;
  float* ws;                // [2 * n_tiles, H, D, E]: what each chunk adds to the state, then the state before it
  float* o_buf;             // [M, H*E] fp32 (token-by-token form only)
  void* out;                // [M, ldo]: norm(o) * silu(gate)
  long long ldo;
  int* status;
};
// One token per row: rotation, state update, output, head norm and gate in one launch.
cudaError_t launch_retention_decode(const RetentionParams& p, int dtype, cudaStream_t stream);
// Prompt chunks, bf16: chunk sums, scan over the chunks, outputs (3xTF32 products, fp32 accumulation).
cudaError_t launch_retention_chunks(const RetentionParams& p, cudaStream_t stream);
// Prompt chunks token by token in plain fp32 (the fp32 path, and head sizes above the chunked form's).
cudaError_t launch_retention_scan(const RetentionParams& p, int dtype, cudaStream_t stream);
bool retention_chunks_ok(int D, int E);

// out[M, N] = a[M, K] w[N, K]^T in fp32 FMAs.
cudaError_t launch_gemm_f32(const float* a, long long lda, const float* w, long long ldw, float* out, long long ldo,
                            int M, int N, int K, cudaStream_t stream);
// out[m, i] = act(gu[m, i]) * gu[m, I + i]
cudaError_t launch_glu_f32(const float* gu, long long ldg, float* out, long long ldo, int M, int I, int act,
                           cudaStream_t stream);

}  // namespace oxb
