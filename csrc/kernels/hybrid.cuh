// Parameter blocks of the kernels that serve layer-list decoders (attention, retention, ...): residual
// streams with their norms, projections -> heads with norms and rotations, row attention of any head
// size, retention, and the 32-bit matrix product. `dtype` 0: activations, weights and caches are bf16;
// 1: fp32 throughout. Scores, norms, states, residual streams and angles are fp32 in both.
#pragma once
#include <cuda.h>
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

// What stands between two layers whose mixer and feed-forward run side by side on one residual stream x, or between
// two sublayers with a norm on either side. With N values per row:
//   tokens given : x = embed[token] * embed_scale
//   base given   : x = base + sum_b ... (the branches replace the stream)
//   else         : x += sum_b gain[b] * (w[b] ? y_b / sqrt(mean(y_b^2) + eps) * w[b] : y_b)   (dense branches)
//                     + e,   e = sum_c weight[c] * expert_rows[slot[c]]                       (chosen experts)
//                  where y_b of a branch without rows is e, which is then not added a second time
//   then         : h_o = x / sqrt(mean(x^2) + eps) * (w_offset + norm_w[o])                   for every output o
//   split given  : instead of the norms, the operand of a product over [x; embedding]: bf16 rows of three parts, x rounded |
//                  what the rounding left | embed[x0_tokens], or fp32 rows of two, x | embed[x0_tokens]
// x is written back when store_x is set. Where clear_y is set for a branch, its rows are zeroed on the way (the
// split-K GEMM of the layer that follows adds into them).
constexpr int kMaxBranches = 2;
constexpr int kMaxTop = 32;   // most experts that a token may use
struct BranchNormParams {
  float* x;                 // [rows, N]
  int rows, N;
  const int* tokens;        // [rows] or nullptr
  const void* embed;        // [vocab, N]
  int vocab;
  float embed_scale;
  int n_branches;
  float* y[kMaxBranches];   // [rows, ldy], or nullptr: the weighted expert rows
  const float* w[kMaxBranches];
  float gain[kMaxBranches];
  int clear_y[kMaxBranches];
  long long ldy;
  const void* e_rows;       // expert outputs [n_e_rows, lde] or nullptr
  long long lde, n_e_rows;
  const int* e_slot;        // [rows, top], < 0: nothing
  const float* e_weight;    // [rows, top]
  int top;
  int store_x;
  const float* base;        // [N] or nullptr
  void* split;              // [rows, ld_split], parts split_off apart, or nullptr
  long long ld_split;
  int split_off;
  const int* x0_tokens;     // [rows]
  int n_out;
  const float* norm_w[2];
  void* h[2];
  float eps, w_offset;
  long long ldh;
  const int* row_map;       // destination row of h, < 0: skipped
  float* clear;             // [rows, clear_ld] or nullptr, zeroed as in StreamNormParams
  long long clear_ld;
  int clear_n;
  int* status;
};
cudaError_t launch_branch_norm(const BranchNormParams& p, int dtype, cudaStream_t stream);

// Heads of attention over one projection that is key and value (HeadsParams::k_rms): the key is the stored value times
// one number per token and times k_norm, so the cache keeps the values and that number, and k_norm is part of q_norm.

// Rotary positions: pair i turns by position * (freq_hi[i] + freq_lo[i]) (the frequency as an unevaluated
// sum of two floats, so the angle is good to the last bits of a 32-bit float at any position).
struct RotaryParams {
  const float* freq_hi;     // [dims / 2]
  const float* freq_lo;
  int dims;                 // 0: no rotation
  int interleaved;          // pairs (2i, 2i+1), else (i, i + dims/2)
  float gain;               // factor on sin and cos
};

// Projection rows q | k | v -> per-head vectors: optional bias, optional RMS norm over the whole q (k) projection
// with plain weights, rotation of q and k, k times k_scale, q times a temperature that grows with the position
// (1 + t_coef ln(floor((p + 1) / t_every) + 1)). q goes to a dense buffer (head stride q_hd); k goes to a dense buffer
// (k_out) or, with v, into the paged cache [blocks, G / maps, 16, DP] / [blocks, G / maps, 16, EP].
// maps > 1: that many key heads share a value head and lie side by side in one cache row; query head h belongs to
// the map h % maps and goes to the columns of that map, so its product with the whole row is the one with its own key.
struct HeadsParams {
  const void* proj;         // [M, ld], of the storage type, or fp32 when proj_f32 is set (split-K accumulator)
  int proj_f32;
  long long ld;
  int M, H, G, D, E;        // G 0: queries only
  int maps;
  long long q_pd;           // columns between query heads of the projection (D where they are packed); k starts at H * q_pd
  const float* bias;        // [columns of q | k | v] or nullptr
  float t_coef, t_every;    // t_coef 0: no temperature
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
  float* k_rms;             // [cache slots] or nullptr: k goes to the cache as it is, and 1 / sqrt(mean(k^2) + eps) here
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
  int chunk;                // > 0: only positions of the query's own chunk (counted from position 0) are visible
  float scale;
  float sink;               // score of one more term of the softmax denominator, without a value (-inf: none)
  const float* sinks;       // [H] the same per head, or nullptr
  float out_gain;           // factor on the result
  void* out;                // [rows, ldo], heads o_hd apart; fp32 when out_f32 is set
  int out_f32, o_hd;
  long long ldo;
  int* status;
};
cudaError_t launch_row_attention(const RowAttnParams& p, int dtype, cudaStream_t stream);

// Talking heads over keys that are values. The score of head g for key j of a query at position i is
//   c_g = cap tanh(q_g . k_j k_rms_j scale / cap)            (cap 0: as it is)
// head h goes on with sum_g talk[h, g] c_g - bias[h, i - j] (bias: the heads' distance biases, mixed the same way), takes the
// softmax over the visible keys and sums k_j; the result times sigmoid(gate).
struct TalkParams {
  const void* q;            // [rows, q_ld], heads DP apart: normed, times the keys' norm weights
  long long q_ld;
  const void* cache;        // [blocks, G, 16, DP]
  const float* k_rms;       // [blocks, 16]
  const int* block_tables;  // [sequences, max_blocks]
  const int* seq_lens;      // decode: [rows]
  const int* tile_seq;      // prompt chunks: 128-row tiles
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_rows;               // decode: rows; chunks: tiles
  int max_blocks, num_blocks;
  int H, G, D, DP;
  int window;               // 0: all earlier positions
  float scale, cap;
  const float* talk;        // [H, H]
  const float* bias;        // [H, n_bias], distance 0 first
  int n_bias;
  const void* gate;         // [rows, gate_ld] pre-activations, heads D apart; fp32 when gate_f32 is set
  int gate_f32;
  long long gate_ld;
  float* part_o;            // decode: [rows, H, max_splits, DP]
  float* part_ml;           // [rows, H, max_splits, 2]
  int max_splits;
  float* scores;            // prompt chunks: [tiles, H, 128, span] mixed scores times log2(e), keys from the tile's first one on
  int span;                 // a multiple of 32
  void* out;                // [rows, ldo], heads of D
  long long ldo;
  int* status;
};
// Any sizes, fp32 FMAs, one CTA per row: the fp32 path and sizes that the other kernels do not take.
cudaError_t launch_talk_rows(const TalkParams& p, int dtype, cudaStream_t stream);
size_t talk_rows_smem(int H, int D);
// bf16, D padded to 64 or 128. Decoding: split-KV and merge. tmC: cache rows in boxes of talk_decode_box x 64.
cudaError_t launch_talk_decode(const CUtensorMap& tmC, const TalkParams& p, cudaStream_t stream);
int talk_decode_box(int H, int G, int DP);
bool talk_decode_ok(int H, int G, int DP);
// Prompt chunks: mixed scores of a step's tiles, then softmax and sums. tmV: cache rows in boxes of 16 x 64.
cudaError_t launch_talk_prefill(const CUtensorMap& tmV, const TalkParams& p, cudaStream_t stream);
bool talk_prefill_ok(int H, int DP);
int talk_span(int window, int max_ctx);   // keys per row of `scores`

// Gated recurrence whose gates read only the current token (minGRU), element by element over N channels:
//   z = sigmoid(z_in + b_z), u = x_in + b_x, c = u + 1/2 where u >= 0 else sigmoid(u),  S <- (1 - z) S + z c
//   out = S silu(g) * out_gain
struct GruParams {
  const void* proj;         // [M, ld]: z (N) | x (N) | g (N); type as in HeadsParams
  int proj_f32;
  long long ld;
  int N;                    // a multiple of 4
  const float* bias;        // [2 N]: b_z | b_x
  float out_gain;
  float* state;             // [slots, N]
  int num_slots;
  // decode rows
  const int* row_slots;     // [rows], < 0: padding row
  const int* positions;     // [rows]; a row at position 0 starts from the zero state
  int rows;
  // prompt chunks
  const int* seq_slots;
  const int* tile_seq;      // 128-row tiles, those of a sequence one after the other
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_tiles;
  float* ws;                // [n_tiles, 1 + kGruParts, 2, N]: what a tile and its parts make of a state, S -> S + (b - d S)
  void* out;                // [M, ldo]
  long long ldo;
  int* status;
};
constexpr int kGruParts = 4;   // 32-row parts of a tile that are walked at once
cudaError_t launch_gru_decode(const GruParams& p, int dtype, cudaStream_t stream);
cudaError_t launch_gru_prefill(const GruParams& p, int dtype, cudaStream_t stream);

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

// State-space layer with a scalar decay per head and step (Mamba-2). Head h uses group g = h / (H / G):
//   u    = silu(conv(xbc) + bias)              per channel, causal, `taps` taps (the last one: the current token)
//   dt   = softplus(dt_in + dt_bias[h])
//   S_t  = exp(-exp(A_log[h]) dt_t) S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D[h] x_t     (S: [NP, EP])
// A projection row holds z (H * EP) | x (H * EP) | B (G * NP) | C (G * NP) | dt (H); head sizes E and state sizes N
// are padded with zero channels to EP and NP, multiples of 16. conv_state keeps the inputs of the last `taps` tokens
// of a sequence by position modulo taps, so a decode step never overwrites an input that the step still reads.
struct SsdParams {
  const void* proj;         // [M, ld], first column z
  int proj_f32;
  long long ld;
  int H, G, EP, NP, taps;
  const float* conv_w;      // [channels, taps], channels = H * EP + 2 * G * NP
  const float* conv_b;      // [channels]
  const float* dt_bias;     // [H]
  const float* A_log;       // [H]
  const float* D;           // [H]
  float* state;             // [slots, H, NP, EP]
  float* conv_state;        // [slots, taps, channels]
  int num_slots;
  // decode rows
  const int* row_slots;     // [rows], < 0: padding row
  const int* positions;     // [rows]; a row at position 0 starts from the zero state
  int rows;
  // prompt chunks
  const int* seq_slots;     // [sequences]
  const int* tile_seq;      // 128-row tiles
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_tiles, n_seqs;
  void* u;                  // [M, ldu] convolved channels (x | B | C)
  long long ldu;
  void* y;                  // [M, ldy]: H * EP
  long long ldy;
  int segment;              // > 0: sequences are walked in segments of this many rows (a multiple of 128) at once
  float* ws;                // [n_tiles, H, NP, EP] states of the segments, by their first tile
  float* ws_decay;          // [n_tiles, H]
  int* status;
};
// One token per row: convolution, state update and read-out in one launch.
cudaError_t launch_ssd_decode(const SsdParams& p, int dtype, cudaStream_t stream);
// Prompt chunks: convolution of all rows (and the convolution's state).
cudaError_t launch_ssd_conv(const SsdParams& p, int dtype, cudaStream_t stream);
// Prompt chunks, bf16: runs of 64 tokens on tensor cores, fp32 operands split into three bf16 terms.
cudaError_t launch_ssd_chunks(const SsdParams& p, cudaStream_t stream);
// Prompt chunks token by token in fp32 FMAs.
cudaError_t launch_ssd_scan(const SsdParams& p, int dtype, cudaStream_t stream);
bool ssd_chunks_ok(int NP);
int ssd_segment(int H, int EP, int n_tiles, int n_seqs);   // rows per segment that suit the device, 0: whole sequences

// out[row] = rms_groups(y * silu(z)) * w: `groups` equal parts of H * E values, each by its own root mean square.
// y and z hold heads of E values EP apart.
struct GatedNormParams {
  const void* y;            // [M, ldy], storage type
  long long ldy;
  const void* z;            // [M, ldz], storage type or fp32 when z_f32 is set
  int z_f32;
  long long ldz;
  int M, H, E, EP, groups;
  const float* w;           // [H * E]
  float eps;
  void* out;                // [M, ldo]
  long long ldo;
};
cudaError_t launch_gated_norm(const GatedNormParams& p, int dtype, cudaStream_t stream);

// Differential attention: o = a1 - lambda a2 of the two maps of every head, o / sqrt(mean(o^2) + eps) * gain.
struct DiffNormParams {
  const float* a;           // [M, lda]: heads of [map 1: E | map 2: E]
  long long lda;
  int M, H, E;
  float lambda, gain, eps;
  void* out;                // [M, ldo], heads of E
  long long ldo;
};
cudaError_t launch_diff_norm(const DiffNormParams& p, int dtype, cudaStream_t stream);

// Latent attention. What a token keeps is one row of R latent values (normed) and T rotated key values that all
// heads share: cache [blocks, 16, CP]. Projection rows hold the query latent (Q values, kv_col columns wide) and, from
// column kv_col on, the R + T raw values.
struct LatentRowsParams {
  const void* proj;         // [M, ld], storage type or fp32 when proj_f32 is set
  int proj_f32;
  long long ld;
  int M, Q, R, kv_col;      // R 0: the layer reads another one's cache
  const float* q_norm;      // [Q]
  const float* kv_norm;     // [R]
  float eps;
  RotaryParams rot;         // of the last rot.dims values
  const int* positions;
  void* q_out;              // [M, ldq] normed query latent
  long long ldq;
  void* cache;
  int CP;
  const long long* slots;   // [M], < 0: not stored
  long long num_slots;
  int* status;
};
cudaError_t launch_latent_rows(const LatentRowsParams& p, int dtype, cudaStream_t stream);
// Cache rows of a step's prompts -> consecutive rows: position t of sequence s at row row0[s] + t.
struct LatentGatherParams {
  const void* cache;        // [blocks, 16, CP], bf16
  int CP, num_blocks, max_blocks;
  const int* block_tables;  // [sequences, max_blocks]
  const int* ctx_lens;
  const int* row0;
  int seq0, n_seqs, max_pages;
  void* out;                // [rows, CP]
  long long rows;
  int* status;
};
cudaError_t launch_latent_gather(const LatentGatherParams& p, cudaStream_t stream);
// Decoding: all heads of a row against the latents themselves. q rows [H, CP]: the query's product with the key
// expansion (R values), then its rotated part; the output is the weighted sum of latents, per head R values.
struct LatentDecodeParams {
  const int* block_tables;  // [rows, max_blocks]
  const int* seq_lens;
  int rows, H, R, CP, max_blocks, max_splits, num_blocks;
  int n_splits;             // set by the launch: splits in use
  float scale_log2;
  float* part_o;            // [rows, H, max_splits, R]
  float* part_ml;           // [rows, H, max_splits, 2]
  __nv_bfloat16* out;       // [rows, ldo], heads o_hd apart
  long long ldo;
  int o_hd;
  int* status;
};
// tmQ: [rows, H, CP] in boxes of latent_decode_heads(H, R, CP) x 64 (0: sizes that do not fit); tmC: cache rows in boxes of
// 16 x 64.
cudaError_t launch_latent_decode(const CUtensorMap& tmQ, const CUtensorMap& tmC, const LatentDecodeParams& p, cudaStream_t stream);
int latent_decode_heads(int H, int R, int CP);

// Matrix memory with a running maximum (mLSTM). Log gates per head: i = cap tanh(zi / cap), f = logsigmoid(cap tanh(zf / cap));
//   m' = max(f + m, i), S' = exp(f + m - m') S + exp(i - m') k v^T, n' likewise with k alone, m starts at 0
//   o = scale S'^T q / (max(|scale n' q|, exp(-m')) + 1e-6), then o / rms(o) * norm_w * sigmoid(gate)
// state [slots, H, D * E + D]: S row by row, then n; state_m [slots, H].
constexpr int kMemChunk = 64;
struct MemoryParams {
  const void* proj;         // [M, ld]: q (H * D) | k (H * D) | v (H * E) | gate (H * E); type as in HeadsParams
  int proj_f32;
  long long ld;
  int H, D, E;
  const float* z;           // [M, ldz] pre-activations zi (H) | zf (H) without bias (prompt chunks, fp32 path)
  long long ldz;
  const float* z_bias;      // [2 H]
  const void* h;            // decode: normed rows and gate weights instead of z
  long long ldh;
  const void* z_w;          // [2 H, ldw] bf16
  long long ldw;
  int N;
  float cap, scale, eps;
  const float* norm_w;      // [H * E]
  float* state;
  float* state_m;
  int num_slots;
  // decode rows
  const int* row_slots;     // [rows], < 0: padding row
  const int* positions;     // [rows]; a row at position 0 starts from the zero state
  int rows;
  // prompt chunks
  const int* seq_slots;
  const int* tile_seq;
  const int* tile_q0;
  const int* q_start;
  const int* q_lens;
  const int* ctx_lens;
  int n_tiles, n_seqs;
  float* ws;                // [2 n_tiles, H, D * E + D]: what each chunk adds, then the state before it
  float* ws_m;              // [2 n_tiles, H]: maximum before each chunk
  float* o_buf;             // [M, H * E] fp32 (token-by-token form only)
  float* n_buf;             // [n_seqs, H, D + 1] (token-by-token form only)
  void* out;                // [M, ldo]
  long long ldo;
  int* status;
};
cudaError_t launch_memory_decode(const MemoryParams& p, int dtype, cudaStream_t stream);
// Prompt chunks, bf16: chunk sums, scan over the chunks, outputs (fp32 operands in three bf16 terms).
cudaError_t launch_memory_chunks(const MemoryParams& p, cudaStream_t stream);
// Prompt chunks token by token in fp32 FMAs.
cudaError_t launch_memory_scan(const MemoryParams& p, int dtype, cudaStream_t stream);
bool memory_chunks_ok(int D, int E);

// Router of a mixture of experts. softmax 1: scores are a softmax over all experts, the weights the `top` largest ones
// divided by their sum (+ 1e-20). softmax 0: scores are sigmoids, the weights the chosen scores themselves. With
// `groups` > 0 the experts form that many equal groups of neighbours; only experts of the `keep` groups whose two
// largest scores have the largest sum can be chosen.
constexpr int kMaxExperts = 512;
constexpr int kMaxGroups = 32;
struct MoeRouteParams {
  const float* logits;      // [M, ldl], or nullptr: computed here from h and router
  long long ldl;
  const void* h;            // [M, ldh]
  long long ldh;
  const void* router;       // [E, ldr]
  long long ldr;
  int M, N, E, top;
  int softmax, groups, keep;
  float* weight;            // [M, top]
  int* expert;              // [M, top]
  int* slot;                // [M, top]: row of the expert buffers that belongs to the choice
  int mode;                 // 0: slot = its own index; 1: rows of 128-row slabs per expert, h copied there (M <= 128);
                            // 2: slot = rank inside the expert (launch_moe_scatter turns it into a packed row)
  uint32_t* counts;         // [E] rows per expert, zero before the launch (modes 1 and 2)
  void* xs;                 // [E * 128, ldx] (mode 1)
  long long ldx;
  int* status;
};
cudaError_t launch_moe_route(const MoeRouteParams& p, int dtype, cudaStream_t stream);
// slot[i] += first packed row of the expert (whole 128-row tiles per expert); h rows are copied there.
struct MoeScatterParams {
  const void* h;
  long long ldh;
  int M, N, E, top;
  const int* expert;
  int* slot;
  const uint32_t* counts;
  void* xs;                 // [max_rows, ldx]
  long long ldx, max_rows;
  int* status;
};
cudaError_t launch_moe_scatter(const MoeScatterParams& p, cudaStream_t stream);   // bf16
// y[p] = act(W[expert[p]] x[per_pair ? p : p / top]) for every (row, choice) pair p. act 0: none, 2: squared ReLU,
// 3: W holds gate and up rows in units of 32 | 32, y = silu(gate) * up with N / 2 values.
struct MoeRowsParams {
  const void* x;
  long long ldx;
  int per_pair;
  const void* w;            // [E, N, K]
  int pairs, top, E, N, K;
  const int* expert;        // [pairs]
  int act;
  void* y;                  // [pairs, ldy]
  long long ldy;
};
cudaError_t launch_moe_rows(const MoeRowsParams& p, int dtype, cudaStream_t stream);

// out[M, N] = a[M, K] w[N, K]^T in fp32 FMAs.
cudaError_t launch_gemm_f32(const float* a, long long lda, const float* w, long long ldw, float* out, long long ldo,
                            int M, int N, int K, cudaStream_t stream);
// out[m, i] = act(gu[m, i]) * gu[m, I + i]; act 0: silu, 1: tanh form of gelu, 2: relu(gu[m, i])^2 alone
cudaError_t launch_glu_f32(const float* gu, long long ldg, float* out, long long ldo, int M, int I, int act,
                           cudaStream_t stream);

}  // namespace oxb
