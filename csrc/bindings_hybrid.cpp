// Python bindings of the layer-list kernels (torch extension `oxb_hybrid`). Every function launches on
// torch's current CUDA stream and allocates nothing. The argument checks cover what the kernels index with.
#include <ATen/cuda/CUDAContext.h>
#include <cuda_runtime.h>
#include <torch/extension.h>

#include <cmath>
#include <vector>

#include "common/device_info.h"
#include "common/tma_host.h"
#include "kernels/attn.cuh"
#include "kernels/hybrid.cuh"

namespace py = pybind11;
using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

namespace {

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

void check_launch(cudaError_t e, const char* what) {
  const cudaError_t last = cudaGetLastError();
  if (e == cudaSuccess) e = last;
  TORCH_CHECK(e == cudaSuccess, "oxb: launch of ", what, " failed: ", cudaGetErrorString(e));
}

void check_launch(const char* what) { check_launch(cudaSuccess, what); }

int dtype_code(const Tensor& t, const char* what) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == torch::kBFloat16 || t.scalar_type() == torch::kFloat32), what,
              ": CUDA bf16 or fp32 expected");
  return t.scalar_type() == torch::kBFloat16 ? 0 : 1;
}
bool given(const OptTensor& t) { return t.has_value() && t->defined(); }

const float* f32(const Tensor& t, int64_t need, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.numel() >= need && t.is_contiguous(), what,
              ": contiguous CUDA fp32 of at least ", need, " values expected");
  return t.data_ptr<float>();
}
const float* f32(const OptTensor& t, int64_t need, const char* what) { return given(t) ? f32(*t, need, what) : nullptr; }
const int* i32(const Tensor& t, int64_t need, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt32 && t.numel() >= need && t.is_contiguous(), what,
              ": contiguous CUDA int32 of at least ", need, " values expected");
  return t.data_ptr<int>();
}
int* status_ptr(const Tensor& t) { return const_cast<int*>(i32(t, 1, "status")); }
// rows x cols view with unit column stride; returns the row pitch
int64_t pitch(const Tensor& t, int64_t rows, int64_t cols, const char* what) {
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1 && t.size(0) >= rows && t.size(1) >= cols, what, ": [", rows, ", ", cols,
              "] rows expected");
  return t.stride(0);
}
oxb::RotaryParams rotary(const OptTensor& hi, const OptTensor& lo, bool interleaved, double gain, int64_t D) {
  oxb::RotaryParams r{};
  r.gain = static_cast<float>(gain);
  if (given(hi)) {
    r.dims = static_cast<int>(2 * hi->numel());
    TORCH_CHECK(r.dims <= D, "rotary: more dimensions than a head has");
    r.freq_hi = f32(*hi, 1, "rotary");
    TORCH_CHECK(given(lo), "rotary: frequencies are given as two terms");
    r.freq_lo = f32(*lo, hi->numel(), "rotary");
    r.interleaved = interleaved ? 1 : 0;
  }
  return r;
}

void stream_norm(const Tensor& x, int64_t rows, const OptTensor& tokens, const OptTensor& prev, const OptTensor& embed,
                 const OptTensor& bigram, int64_t mul_prev, int64_t mul_cur, const OptTensor& y, bool zero_y, const OptTensor& mix,
                 const OptTensor& out_w, const OptTensor& in_w, bool store_x, const Tensor& norm_w, double eps, double w_offset,
                 const Tensor& h, const OptTensor& row_map, const OptTensor& clear, const Tensor& status) {
  TORCH_CHECK(x.dim() == 3, "stream_norm: x [rows, streams, N]");
  oxb::StreamNormParams p{};
  p.rows = static_cast<int>(rows);
  p.S = static_cast<int>(x.size(1));
  p.N = static_cast<int>(x.size(2));
  TORCH_CHECK(p.S >= 1 && p.S <= oxb::kMaxStreams, "stream_norm: 1..16 streams");
  TORCH_CHECK(p.N <= 32768, "stream_norm: rows of at most 32768 values");
  TORCH_CHECK(x.size(0) >= rows, "stream_norm: rows");
  p.x = const_cast<float*>(f32(x, rows * p.S * p.N, "stream_norm x"));
  const int dt = dtype_code(h, "stream_norm h");
  TORCH_CHECK(given(tokens) != given(y), "stream_norm: either tokens or the sublayer's output");
  if (given(tokens)) {
    TORCH_CHECK(given(embed) && embed->scalar_type() == h.scalar_type() && embed->is_contiguous() && embed->dim() == 2 &&
                    embed->size(1) == p.N,
                "stream_norm: embed [vocab, N] of h's type");
    p.tokens = i32(*tokens, rows, "stream_norm tokens");
    p.embed = embed->data_ptr();
    p.vocab = static_cast<int>(embed->size(0));
    if (given(bigram)) {
      TORCH_CHECK(given(prev) && bigram->scalar_type() == h.scalar_type() && bigram->is_contiguous() && bigram->dim() == 2 &&
                      bigram->size(1) == p.N && bigram->size(0) >= 2 && mul_prev >= 0 && mul_cur >= 0,
                  "stream_norm: bigram [buckets + 1, N], prev, multipliers >= 0");
      p.prev = i32(*prev, rows, "stream_norm prev");
      p.bigram = bigram->data_ptr();
      p.buckets = static_cast<int>(bigram->size(0)) - 1;
      p.mul_prev = mul_prev;
      p.mul_cur = mul_cur;
    }
  } else {
    p.ldy = pitch(*y, rows, p.N, "stream_norm y");
    TORCH_CHECK(y->is_cuda() && y->scalar_type() == torch::kFloat32, "stream_norm: fp32 y");
    p.y = y->data_ptr<float>();
    p.zero_y = zero_y ? 1 : 0;
    TORCH_CHECK(given(mix) && given(out_w), "stream_norm: mix and out belong to y");
    p.mix = f32(*mix, p.S * p.S, "stream_norm mix");
    p.out = f32(*out_w, p.S, "stream_norm out");
  }
  p.in = f32(in_w, p.S, "stream_norm in");
  p.store_x = store_x ? 1 : 0;
  p.norm_w = f32(norm_w, p.N, "stream_norm norm_w");
  p.eps = static_cast<float>(eps);
  p.w_offset = static_cast<float>(w_offset);
  p.ldh = pitch(h, given(row_map) ? 1 : rows, p.N, "stream_norm h");
  p.h = h.data_ptr();
  if (given(row_map)) p.row_map = i32(*row_map, rows, "stream_norm row_map");
  if (given(clear)) {
    p.clear_ld = pitch(*clear, rows, 1, "stream_norm clear");
    TORCH_CHECK(clear->scalar_type() == torch::kFloat32 && clear->is_cuda() && p.clear_ld % 4 == 0 && clear->size(1) % 4 == 0,
                "stream_norm: clear is fp32 in whole 16-byte pieces");
    p.clear = clear->data_ptr<float>();
    p.clear_n = static_cast<int>(clear->size(1));
  }
  p.status = status_ptr(status);
  check_launch(oxb::launch_stream_norm(p, dt, cur_stream()), "stream_norm");
}

void heads(const Tensor& proj, int64_t M, int64_t H, int64_t G, int64_t D, int64_t E, const OptTensor& q_norm,
           const OptTensor& k_norm, double eps, const OptTensor& freq_hi, const OptTensor& freq_lo, bool interleaved,
           double gain, const Tensor& positions, double k_scale, const Tensor& q_out, int64_t q_hd, const OptTensor& k_out,
           const OptTensor& k_cache, const OptTensor& v_cache, const OptTensor& slots, int64_t q_pd, int64_t maps, const OptTensor& bias,
           double t_coef, double t_every, const OptTensor& k_rms, const Tensor& status) {
  oxb::HeadsParams p{};
  // storage type: that of the caches; dense q and k are fp32 whatever the projection is
  const int proj_dt = dtype_code(proj, "heads proj");
  const int dt = given(k_cache) ? dtype_code(*k_cache, "heads k_cache") : (given(k_out) ? proj_dt : dtype_code(q_out, "heads q_out"));
  p.proj_f32 = proj_dt;
  TORCH_CHECK(dt == 0 || proj_dt == 1, "heads: fp32 caches take fp32 projections");
  if (q_pd == 0) q_pd = D;
  TORCH_CHECK(H >= 1 && G >= 0 && D >= 1 && maps >= 1 && G % maps == 0 && q_hd >= (maps - 1) * D + D && q_pd >= D, "heads: sizes");
  p.maps = static_cast<int>(maps);
  p.q_pd = q_pd;
  p.proj = proj.data_ptr();
  p.M = static_cast<int>(M);
  p.H = static_cast<int>(H);
  p.G = static_cast<int>(G);
  p.D = static_cast<int>(D);
  p.E = static_cast<int>(E);
  p.q_norm = f32(q_norm, H * D, "heads q_norm");
  p.k_norm = f32(k_norm, G * D, "heads k_norm");
  TORCH_CHECK((p.q_norm == nullptr) == (p.k_norm == nullptr) || (given(k_rms) && p.k_norm == nullptr), "heads: q and k norm go together");
  p.eps = static_cast<float>(eps);
  TORCH_CHECK(p.q_norm == nullptr || (q_pd == D && !given(bias)), "heads: the norm spans packed heads without bias");
  p.bias = f32(bias, H * q_pd + G * D + G / maps * E, "heads bias");
  TORCH_CHECK(t_coef == 0.0 || t_every > 0.0, "heads: temperature");
  p.t_coef = static_cast<float>(t_coef);
  p.t_every = static_cast<float>(t_every);
  p.rot = rotary(freq_hi, freq_lo, interleaved, gain, D);
  p.positions = i32(positions, M, "heads positions");
  p.k_scale = static_cast<float>(k_scale);
  p.q_out = q_out.data_ptr();
  if (given(k_out)) {
    // dense fp32 q [H, >= M, D] and k [G, >= M, D], rows of a head together
    auto dense = [&](const Tensor& t, int64_t n) {
      TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.dim() == 3 && t.size(0) == n && t.size(1) >= M &&
                      t.size(2) == D && t.stride(2) == 1 && t.stride(1) == D,
                  "heads: dense q and k are fp32 [heads, rows, D]");
      return t.stride(0);
    };
    TORCH_CHECK(maps == 1, "heads: dense keys have one map");
    p.ld = pitch(proj, M, H * q_pd + G * D, "heads proj");
    p.q_hd = dense(q_out, H);
    p.k_hd = dense(*k_out, G);
    p.q_ld = p.k_ld = D;
    p.k_out = k_out->data_ptr<float>();
  } else {
    p.q_ld = pitch(q_out, M, (H - 1) * q_hd + maps * D, "heads q_out");
    p.q_hd = q_hd;
    if (G == 0) {
      TORCH_CHECK(!given(k_cache) && !given(v_cache), "heads: queries only");
      p.ld = pitch(proj, M, (H - 1) * q_pd + D, "heads proj");
      p.status = status_ptr(status);
      check_launch(oxb::launch_heads(p, dt, cur_stream()), "heads");
      return;
    }
    TORCH_CHECK(given(k_cache) && given(v_cache) != given(k_rms) && given(slots), "heads: caches and slots, or k_out");
    TORCH_CHECK(q_out.scalar_type() == k_cache->scalar_type(), "heads: one storage type");
    TORCH_CHECK(k_cache->dim() == 4 && k_cache->is_contiguous() && k_cache->size(1) == G / maps && k_cache->size(2) == 16 &&
                    k_cache->size(3) >= maps * D,
                "heads: caches [blocks, G, 16, >= head size]");
    p.k_cache = k_cache->data_ptr();
    p.DP = static_cast<int>(k_cache->size(3));
    if (given(k_rms)) {   // keys that are values: no value columns, no value cache
      TORCH_CHECK(p.q_norm != nullptr && p.k_norm == nullptr && maps == 1 && k_scale == 1.0, "heads: keys that are values, with a norm");
      p.k_rms = const_cast<float*>(f32(*k_rms, k_cache->size(0) * 16, "heads k_rms"));
      p.ld = pitch(proj, M, H * q_pd + G * D, "heads proj");
    } else {
      TORCH_CHECK(v_cache->scalar_type() == k_cache->scalar_type() && v_cache->dim() == 4 && v_cache->is_contiguous() &&
                      v_cache->size(1) == G / maps && v_cache->size(2) == 16 && k_cache->size(0) == v_cache->size(0) && v_cache->size(3) >= E,
                  "heads: caches [blocks, G, 16, >= head size]");
      p.ld = pitch(proj, M, H * q_pd + G * D + G / maps * E, "heads proj");
      p.v_cache = v_cache->data_ptr();
      p.EP = static_cast<int>(v_cache->size(3));
    }
    TORCH_CHECK(slots->is_cuda() && slots->scalar_type() == torch::kInt64 && slots->numel() >= M, "heads: slots int64");
    p.slots = reinterpret_cast<const long long*>(slots->data_ptr<int64_t>());
    p.num_slots = k_cache->size(0) * 16;
  }
  p.status = status_ptr(status);
  check_launch(oxb::launch_heads(p, dt, cur_stream()), "heads");
}

void row_attention(const Tensor& q, int64_t q_hd, const Tensor& k_cache, const Tensor& v_cache, const Tensor& block_tables,
                   const OptTensor& seq_lens, const OptTensor& tile_seq, const OptTensor& tile_q0, const OptTensor& q_start,
                   const OptTensor& q_lens, const OptTensor& ctx_lens, int64_t n, int64_t H, int64_t D, int64_t E, int64_t window,
                   int64_t keep_first, int64_t chunk, double scale, double sink, const OptTensor& sinks, double out_gain, const Tensor& out, int64_t o_hd,
                   const Tensor& status) {
  oxb::RowAttnParams p{};
  const int dt = dtype_code(q, "row_attention q");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() &&
                  k_cache.size(2) == 16 && v_cache.size(2) == 16 && k_cache.size(1) == v_cache.size(1) &&
                  k_cache.size(0) == v_cache.size(0),
              "row_attention: caches [blocks, G, 16, head size]");
  TORCH_CHECK(k_cache.scalar_type() == q.scalar_type() && v_cache.scalar_type() == q.scalar_type() &&
                  (out.scalar_type() == q.scalar_type() || out.scalar_type() == torch::kFloat32),
              "row_attention: one storage type (or fp32 out)");
  p.out_f32 = out.scalar_type() == torch::kFloat32 ? 1 : 0;
  p.G = static_cast<int>(k_cache.size(1));
  p.H = static_cast<int>(H);
  p.D = static_cast<int>(D);
  p.E = static_cast<int>(E);
  p.DP = static_cast<int>(k_cache.size(3));
  p.EP = static_cast<int>(v_cache.size(3));
  TORCH_CHECK(H % p.G == 0 && D <= p.DP && E <= p.EP && E <= 1024 && D <= 4096 && q_hd >= D, "row_attention: head sizes");
  p.q = q.data_ptr();
  p.q_ld = pitch(q, 1, H * q_hd, "row_attention q");
  p.q_hd = static_cast<int>(q_hd);
  p.k_cache = k_cache.data_ptr();
  p.v_cache = v_cache.data_ptr();
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous(), "row_attention: block_tables");
  p.block_tables = i32(block_tables, 1, "row_attention block_tables");
  p.max_blocks = static_cast<int>(block_tables.size(1));
  p.num_blocks = static_cast<int>(k_cache.size(0));
  p.n_rows = static_cast<int>(n);
  if (given(tile_seq)) {
    p.tile_seq = i32(*tile_seq, n, "row_attention tile_seq");
    p.tile_q0 = i32(*tile_q0, n, "row_attention tile_q0");
    p.q_start = i32(*q_start, 1, "row_attention q_start");
    p.q_lens = i32(*q_lens, 1, "row_attention q_lens");
    p.ctx_lens = i32(*ctx_lens, 1, "row_attention ctx_lens");
  } else {
    TORCH_CHECK(given(seq_lens) && block_tables.size(0) >= n, "row_attention: seq_lens");
    p.seq_lens = i32(*seq_lens, n, "row_attention seq_lens");
  }
  p.window = static_cast<int>(window);
  p.keep_first = static_cast<int>(keep_first);
  TORCH_CHECK(chunk >= 0 && (chunk == 0 || (window == 0 && keep_first == 0)), "row_attention: a window or a chunk");
  p.chunk = static_cast<int>(chunk);
  p.scale = static_cast<float>(scale);
  p.sink = static_cast<float>(sink);
  p.sinks = f32(sinks, H, "row_attention sinks");
  p.out_gain = static_cast<float>(out_gain);
  if (o_hd == 0) o_hd = E;
  TORCH_CHECK(o_hd >= E, "row_attention: o_hd");
  p.o_hd = static_cast<int>(o_hd);
  p.ldo = pitch(out, 1, (H - 1) * o_hd + E, "row_attention out");
  p.out = out.data_ptr();
  p.status = status_ptr(status);
  check_launch(oxb::launch_row_attention(p, dt, cur_stream()), "row_attention");
}

oxb::RetentionParams retention_common(const Tensor& proj, int64_t M, int64_t H, int64_t D, int64_t E, const Tensor& decay_pow,
                                      const Tensor& state, double eps, const Tensor& out, const Tensor& status) {
  oxb::RetentionParams p{};
  p.proj = proj.data_ptr();
  p.ld = pitch(proj, M, 2 * H * (D + E), "retention proj");
  p.H = static_cast<int>(H);
  p.D = static_cast<int>(D);
  p.E = static_cast<int>(E);
  p.decay_pow = f32(decay_pow, H * (oxb::kRetChunk + 1), "retention decay_pow");
  TORCH_CHECK(state.dim() == 4 && state.size(1) == H && state.size(2) == D && state.size(3) == E,
              "retention: state [slots, H, D, E]");
  p.state = const_cast<float*>(f32(state, 1, "retention state"));
  p.num_slots = static_cast<int>(state.size(0));
  p.eps = static_cast<float>(eps);
  p.proj_f32 = dtype_code(proj, "retention proj");
  TORCH_CHECK(dtype_code(out, "retention out") == 0 || p.proj_f32 == 1, "retention: fp32 rows take fp32 projections");
  p.ldo = pitch(out, M, H * E, "retention out");
  p.out = out.data_ptr();
  p.status = status_ptr(status);
  return p;
}

void retention_decode(const Tensor& proj, int64_t rows, int64_t H, int64_t D, int64_t E, const Tensor& decay_pow,
                      const OptTensor& freq_hi, const OptTensor& freq_lo, bool interleaved, double gain, double k_scale, double eps,
                      const Tensor& state, const Tensor& row_slots, const Tensor& positions, const Tensor& out,
                      const Tensor& status) {
  const int dt = dtype_code(out, "retention_decode out");
  oxb::RetentionParams p = retention_common(proj, rows, H, D, E, decay_pow, state, eps, out, status);
  TORCH_CHECK(D <= 4096 && E <= 4096, "retention_decode: head sizes");
  p.rot = rotary(freq_hi, freq_lo, interleaved, gain, D);
  p.k_scale = static_cast<float>(k_scale);
  p.row_slots = i32(row_slots, rows, "retention_decode row_slots");
  p.positions = i32(positions, rows, "retention_decode positions");
  p.rows = static_cast<int>(rows);
  check_launch(oxb::launch_retention_decode(p, dt, cur_stream()), "retention_decode");
}

void retention_prefill(const Tensor& proj, int64_t M, int64_t H, int64_t D, int64_t E, const Tensor& decay_pow, double eps,
                       const Tensor& state, const Tensor& seq_slots, const Tensor& tile_seq, const Tensor& tile_q0,
                       const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens, int64_t n_tiles, int64_t n_seqs,
                       const Tensor& q_rot, const Tensor& k_rot, const OptTensor& ws, const OptTensor& o_buf, const Tensor& out,
                       const Tensor& status) {
  const int dt = dtype_code(out, "retention_prefill out");
  oxb::RetentionParams p = retention_common(proj, M, H, D, E, decay_pow, state, eps, out, status);
  p.seq_slots = i32(seq_slots, n_seqs, "retention_prefill seq_slots");
  p.tile_seq = i32(tile_seq, n_tiles, "retention_prefill tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "retention_prefill tile_q0");
  p.q_start = i32(q_start, n_seqs, "retention_prefill q_start");
  p.q_lens = i32(q_lens, n_seqs, "retention_prefill q_lens");
  p.ctx_lens = i32(ctx_lens, n_seqs, "retention_prefill ctx_lens");
  p.n_tiles = static_cast<int>(n_tiles);
  p.n_seqs = static_cast<int>(n_seqs);
  TORCH_CHECK(q_rot.dim() == 3 && q_rot.size(0) == H && q_rot.size(1) >= M && q_rot.size(2) == D && q_rot.sizes() == k_rot.sizes(),
              "retention_prefill: q_rot and k_rot [H, rows, D]");
  p.q_rot = f32(q_rot, M * H * D, "retention_prefill q_rot");
  p.k_rot = f32(k_rot, M * H * D, "retention_prefill k_rot");
  p.rot_hd = q_rot.stride(0);
  if (given(ws)) {
    TORCH_CHECK(dt == 0 && oxb::retention_chunks_ok(static_cast<int>(D), static_cast<int>(E)), "retention_prefill: chunked form");
    p.ws = const_cast<float*>(f32(*ws, 2 * n_tiles * H * D * E, "retention_prefill ws"));
    check_launch(oxb::launch_retention_chunks(p, cur_stream()), "retention_prefill");
  } else {
    TORCH_CHECK(given(o_buf) && D <= 1600, "retention_prefill: o_buf for the token-by-token form");
    p.o_buf = const_cast<float*>(f32(*o_buf, M * H * E, "retention_prefill o_buf"));
    check_launch(oxb::launch_retention_scan(p, dt, cur_stream()), "retention_prefill");
  }
}

void branch_norm(const Tensor& x, int64_t rows, const OptTensor& tokens, const OptTensor& embed, double embed_scale,
                 const std::vector<OptTensor>& ys, const std::vector<OptTensor>& ws, const std::vector<double>& gains,
                 const std::vector<bool>& clears, const OptTensor& e_rows, const OptTensor& e_slot, const OptTensor& e_weight,
                 int64_t top, bool store_x, const std::vector<Tensor>& norm_ws, const std::vector<Tensor>& hs, double eps,
                 double w_offset, const OptTensor& row_map, const OptTensor& clear, const OptTensor& base, const OptTensor& split,
                 int64_t split_off, const OptTensor& x0_tokens, const Tensor& status) {
  TORCH_CHECK(x.dim() == 2, "branch_norm: x [rows, N]");
  oxb::BranchNormParams p{};
  p.rows = static_cast<int>(rows);
  p.N = static_cast<int>(x.size(1));
  TORCH_CHECK(x.size(0) >= rows && p.N <= 32768, "branch_norm: rows of at most 32768 values");
  p.x = const_cast<float*>(f32(x, rows * p.N, "branch_norm x"));
  TORCH_CHECK(hs.size() <= 2 && hs.size() == norm_ws.size() && hs.empty() == given(split), "branch_norm: one or two outputs, or split rows");
  const Tensor& like = hs.empty() ? *split : hs[0];   // of the storage type
  const int dt = dtype_code(like, "branch_norm h");
  p.n_out = static_cast<int>(hs.size());
  for (size_t o = 0; o < hs.size(); ++o) {
    TORCH_CHECK(hs[o].scalar_type() == hs[0].scalar_type(), "branch_norm: one storage type");
    p.ldh = pitch(hs[o], given(row_map) ? 1 : rows, p.N, "branch_norm h");
    TORCH_CHECK(p.ldh == hs[0].stride(0), "branch_norm: one row pitch of h");
    p.h[o] = hs[o].data_ptr();
    p.norm_w[o] = f32(norm_ws[o], p.N, "branch_norm norm_w");
  }
  TORCH_CHECK(ys.size() <= oxb::kMaxBranches && ws.size() == ys.size() && gains.size() == ys.size() && clears.size() == ys.size(),
              "branch_norm: at most ", oxb::kMaxBranches, " branches");
  p.n_branches = static_cast<int>(ys.size());
  int from_experts = 0;
  for (size_t b = 0; b < ys.size(); ++b) {
    if (given(ys[b])) {
      TORCH_CHECK(ys[b]->is_cuda() && ys[b]->scalar_type() == torch::kFloat32, "branch_norm: fp32 branches");
      const long long ld = pitch(*ys[b], rows, p.N, "branch_norm y");
      TORCH_CHECK(p.ldy == 0 || p.ldy == ld, "branch_norm: one row pitch of the branches");
      p.ldy = ld;
      p.y[b] = ys[b]->data_ptr<float>();
    } else {
      ++from_experts;
      TORCH_CHECK(given(e_rows) && !clears[b] && from_experts == 1, "branch_norm: one branch may be the expert rows");
    }
    p.w[b] = f32(ws[b], p.N, "branch_norm branch weight");
    p.gain[b] = static_cast<float>(gains[b]);
    p.clear_y[b] = clears[b] ? 1 : 0;
  }
  if (given(tokens)) {
    TORCH_CHECK(given(embed) && embed->scalar_type() == like.scalar_type() && embed->is_contiguous() && embed->dim() == 2 &&
                    embed->size(1) == p.N && !given(e_rows) && !given(base),
                "branch_norm: embed [vocab, N] of h's type");
    p.tokens = i32(*tokens, rows, "branch_norm tokens");
    p.embed = embed->data_ptr();
    p.vocab = static_cast<int>(embed->size(0));
    p.embed_scale = static_cast<float>(embed_scale);
  } else {
    TORCH_CHECK(!ys.empty(), "branch_norm: tokens or branches");
  }
  if (given(e_rows)) {
    TORCH_CHECK(given(e_slot) && given(e_weight) && top >= 1 && top <= oxb::kMaxTop && e_rows->scalar_type() == like.scalar_type() && e_rows->is_cuda(),
                "branch_norm: expert rows of h's type, with slots and weights");
    p.lde = pitch(*e_rows, 1, p.N, "branch_norm expert rows");
    p.n_e_rows = e_rows->size(0);
    p.e_rows = e_rows->data_ptr();
    p.e_slot = i32(*e_slot, rows * top, "branch_norm slots");
    p.e_weight = f32(*e_weight, rows * top, "branch_norm weights");
    p.top = static_cast<int>(top);
  }
  p.base = f32(base, p.N, "branch_norm base");
  if (given(split)) {
    TORCH_CHECK(given(x0_tokens) && given(embed) && embed->scalar_type() == like.scalar_type() && embed->is_contiguous() && embed->dim() == 2 &&
                    embed->size(1) == p.N && !given(row_map) && split_off >= p.N,
                "branch_norm: split rows take the embedding and its tokens");
    p.ld_split = pitch(*split, rows, (dt == 0 ? 2 : 1) * split_off + p.N, "branch_norm split");
    p.split = split->data_ptr();
    p.split_off = static_cast<int>(split_off);
    p.x0_tokens = i32(*x0_tokens, rows, "branch_norm x0_tokens");
    p.embed = embed->data_ptr();
    p.vocab = static_cast<int>(embed->size(0));
    p.embed_scale = static_cast<float>(embed_scale);
  }
  p.store_x = store_x ? 1 : 0;
  p.eps = static_cast<float>(eps);
  p.w_offset = static_cast<float>(w_offset);
  if (given(row_map)) p.row_map = i32(*row_map, rows, "branch_norm row_map");
  if (given(clear)) {
    p.clear_ld = pitch(*clear, rows, 1, "branch_norm clear");
    TORCH_CHECK(clear->scalar_type() == torch::kFloat32 && clear->is_cuda() && p.clear_ld % 4 == 0 && clear->size(1) % 4 == 0,
                "branch_norm: clear is fp32 in whole 16-byte pieces");
    p.clear = clear->data_ptr<float>();
    p.clear_n = static_cast<int>(clear->size(1));
  }
  p.status = status_ptr(status);
  check_launch(oxb::launch_branch_norm(p, dt, cur_stream()), "branch_norm");
}

// Sizes, weights and state of a state-space layer. proj: rows z | x | B | C | dt, heads of EP, states of NP.
oxb::SsdParams ssd_common(const Tensor& proj, int64_t M, int64_t H, int64_t G, const std::vector<Tensor>& w, const Tensor& state,
                          const Tensor& conv_state, const Tensor& y, const Tensor& status) {
  oxb::SsdParams p{};
  TORCH_CHECK(state.dim() == 4 && state.size(1) == H && state.size(2) % 16 == 0 && state.size(3) % 16 == 0,
              "ssd: state [slots, H, N, E], N and E multiples of 16");
  p.state = const_cast<float*>(f32(state, 1, "ssd state"));
  p.num_slots = static_cast<int>(state.size(0));
  TORCH_CHECK(G >= 1 && H % G == 0, "ssd: groups divide the heads");
  p.H = static_cast<int>(H);
  p.G = static_cast<int>(G);
  p.NP = static_cast<int>(state.size(2));
  p.EP = static_cast<int>(state.size(3));
  TORCH_CHECK(p.NP <= 1600 && p.EP <= 4096, "ssd: state and head sizes");
  const int64_t inner = H * p.EP, ch = inner + 2 * G * p.NP;
  TORCH_CHECK(w.size() == 5 && w[0].dim() == 2 && w[0].size(0) == ch, "ssd: weights conv [channels, taps], bias, dt_bias, A_log, D");
  p.taps = static_cast<int>(w[0].size(1));
  TORCH_CHECK(p.taps >= 1 && p.taps <= 32, "ssd: 1..32 taps");
  p.conv_w = f32(w[0], ch * p.taps, "ssd conv");
  p.conv_b = f32(w[1], ch, "ssd conv bias");
  p.dt_bias = f32(w[2], H, "ssd dt_bias");
  p.A_log = f32(w[3], H, "ssd A_log");
  p.D = f32(w[4], H, "ssd D");
  p.conv_state = const_cast<float*>(f32(conv_state, static_cast<int64_t>(p.num_slots) * p.taps * ch, "ssd conv_state"));
  p.ld = pitch(proj, M, 2 * inner + 2 * G * p.NP + H, "ssd proj");
  p.proj = proj.data_ptr();
  p.proj_f32 = dtype_code(proj, "ssd proj");
  TORCH_CHECK(p.ld % 4 == 0 && reinterpret_cast<uintptr_t>(p.proj) % 16 == 0, "ssd: projection rows in whole 16-byte pieces");
  TORCH_CHECK(dtype_code(y, "ssd y") == 0 || p.proj_f32 == 1, "ssd: fp32 rows take fp32 projections");
  p.ldy = pitch(y, M, inner, "ssd y");
  TORCH_CHECK(p.ldy % 4 == 0, "ssd: row pitch of y");
  p.y = y.data_ptr();
  p.status = status_ptr(status);
  return p;
}

void ssd_decode(const Tensor& proj, int64_t rows, int64_t H, int64_t G, const std::vector<Tensor>& w, const Tensor& state,
                const Tensor& conv_state, const Tensor& row_slots, const Tensor& positions, const Tensor& y, const Tensor& status) {
  oxb::SsdParams p = ssd_common(proj, rows, H, G, w, state, conv_state, y, status);
  p.row_slots = i32(row_slots, rows, "ssd_decode row_slots");
  p.positions = i32(positions, rows, "ssd_decode positions");
  p.rows = static_cast<int>(rows);
  check_launch(oxb::launch_ssd_decode(p, dtype_code(y, "ssd y"), cur_stream()), "ssd_decode");
}

void ssd_prefill(const Tensor& proj, int64_t M, int64_t H, int64_t G, const std::vector<Tensor>& w, const Tensor& state,
                 const Tensor& conv_state, const Tensor& seq_slots, const Tensor& tile_seq, const Tensor& tile_q0, const Tensor& q_start,
                 const Tensor& q_lens, const Tensor& ctx_lens, int64_t n_tiles, int64_t n_seqs, const Tensor& u, const Tensor& y,
                 bool runs, int64_t segment, const OptTensor& ws, const Tensor& status) {
  oxb::SsdParams p = ssd_common(proj, M, H, G, w, state, conv_state, y, status);
  const int dt = dtype_code(y, "ssd y");
  p.seq_slots = i32(seq_slots, n_seqs, "ssd_prefill seq_slots");
  p.tile_seq = i32(tile_seq, n_tiles, "ssd_prefill tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "ssd_prefill tile_q0");
  p.q_start = i32(q_start, n_seqs, "ssd_prefill q_start");
  p.q_lens = i32(q_lens, n_seqs, "ssd_prefill q_lens");
  p.ctx_lens = i32(ctx_lens, n_seqs, "ssd_prefill ctx_lens");
  p.n_tiles = static_cast<int>(n_tiles);
  p.n_seqs = static_cast<int>(n_seqs);
  TORCH_CHECK(u.scalar_type() == y.scalar_type() && u.is_cuda(), "ssd_prefill: u of y's type");
  p.ldu = pitch(u, M, H * p.EP + 2 * G * p.NP, "ssd_prefill u");
  TORCH_CHECK(p.ldu % 8 == 0 && reinterpret_cast<uintptr_t>(u.data_ptr()) % 16 == 0, "ssd_prefill: u in whole 16-byte pieces");
  p.u = u.data_ptr();
  check_launch(oxb::launch_ssd_conv(p, dt, cur_stream()), "ssd_conv");
  if (runs) {
    TORCH_CHECK(dt == 0 && oxb::ssd_chunks_ok(p.NP), "ssd_prefill: runs on tensor cores");
    TORCH_CHECK(segment >= 0 && segment % 128 == 0 && (segment == 0 || given(ws)), "ssd_prefill: segments of whole tiles, with ws");
    if (segment > 0) {
      const int64_t states = n_tiles * H * p.NP * p.EP;
      p.segment = static_cast<int>(segment);
      p.ws = const_cast<float*>(f32(*ws, states + n_tiles * H, "ssd_prefill ws"));
      p.ws_decay = p.ws + states;
    }
    check_launch(oxb::launch_ssd_chunks(p, cur_stream()), "ssd_prefill");
  } else {
    check_launch(oxb::launch_ssd_scan(p, dt, cur_stream()), "ssd_prefill");
  }
}

void gated_norm(const Tensor& y, const Tensor& z, int64_t M, int64_t H, int64_t E, int64_t EP, int64_t groups, const Tensor& w, double eps,
                const Tensor& out) {
  oxb::GatedNormParams p{};
  const int dt = dtype_code(y, "gated_norm y");
  TORCH_CHECK(H >= 1 && E >= 1 && EP >= E && groups >= 1 && (H * E) % groups == 0 && H * E / groups <= 49152, "gated_norm: sizes");
  TORCH_CHECK(out.scalar_type() == y.scalar_type() && out.is_cuda(), "gated_norm: out of y's type");
  p.z_f32 = dtype_code(z, "gated_norm z");
  TORCH_CHECK(dt == 0 || p.z_f32 == 1, "gated_norm: fp32 rows take an fp32 gate");
  p.ldy = pitch(y, M, H * EP, "gated_norm y");
  p.ldz = pitch(z, M, H * EP, "gated_norm z");
  p.ldo = pitch(out, M, H * E, "gated_norm out");
  auto al = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
  TORCH_CHECK(al(y.data_ptr()) && al(z.data_ptr()) && al(out.data_ptr()), "gated_norm: rows start on 16 bytes");
  p.y = y.data_ptr();
  p.z = z.data_ptr();
  p.M = static_cast<int>(M);
  p.H = static_cast<int>(H);
  p.E = static_cast<int>(E);
  p.EP = static_cast<int>(EP);
  p.groups = static_cast<int>(groups);
  p.w = f32(w, H * E, "gated_norm w");
  p.eps = static_cast<float>(eps);
  p.out = out.data_ptr();
  check_launch(oxb::launch_gated_norm(p, dt, cur_stream()), "gated_norm");
}

// mode: see MoeRouteParams
void moe_route(const Tensor& h, const Tensor& router, const OptTensor& logits, int64_t M, int64_t E, int64_t top, const Tensor& weight,
               const Tensor& expert, const Tensor& slot, int64_t mode, const OptTensor& counts, const OptTensor& xs, bool softmax,
               int64_t groups, int64_t keep, const Tensor& status) {
  oxb::MoeRouteParams p{};
  const int dt = dtype_code(h, "moe_route h");
  TORCH_CHECK(E >= 1 && E <= oxb::kMaxExperts && top >= 1 && top <= oxb::kMaxTop && top <= E, "moe_route: at most ", oxb::kMaxExperts,
              " experts, ", oxb::kMaxTop, " of them chosen");
  TORCH_CHECK(groups == 0 || (groups <= oxb::kMaxGroups && E % groups == 0 && keep >= 1 && keep <= groups && keep * (E / groups) >= top),
              "moe_route: at most ", oxb::kMaxGroups, " equal groups that leave enough experts");
  p.softmax = softmax ? 1 : 0;
  p.groups = static_cast<int>(groups);
  p.keep = static_cast<int>(keep);
  p.N = static_cast<int>(h.size(1));
  TORCH_CHECK(router.dim() == 2 && router.size(0) >= E && router.size(1) == p.N && router.stride(1) == 1 &&
                  router.scalar_type() == h.scalar_type() && router.is_cuda() && p.N % 8 == 0 && p.N <= 32768,
              "moe_route: router [E, N] of h's type");
  auto al = [](const Tensor& t) { return reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0 && t.stride(0) % 8 == 0; };
  p.ldh = pitch(h, M, p.N, "moe_route h");
  p.ldr = router.stride(0);
  TORCH_CHECK(al(h) && al(router), "moe_route: rows in whole 16-byte pieces");
  p.h = h.data_ptr();
  p.router = router.data_ptr();
  p.M = static_cast<int>(M);
  p.E = static_cast<int>(E);
  p.top = static_cast<int>(top);
  p.mode = static_cast<int>(mode);
  if (given(logits)) {
    TORCH_CHECK(logits->is_cuda() && logits->scalar_type() == torch::kFloat32, "moe_route: fp32 logits");
    p.ldl = pitch(*logits, M, E, "moe_route logits");
    p.logits = logits->data_ptr<float>();
  }
  p.weight = const_cast<float*>(f32(weight, M * top, "moe_route weight"));
  p.expert = const_cast<int*>(i32(expert, M * top, "moe_route expert"));
  p.slot = const_cast<int*>(i32(slot, M * top, "moe_route slot"));
  TORCH_CHECK(mode >= 0 && mode <= 2, "moe_route: mode");
  if (mode != 0) {
    TORCH_CHECK(given(counts), "moe_route: counts");
    p.counts = reinterpret_cast<uint32_t*>(const_cast<int*>(i32(*counts, E, "moe_route counts")));
  }
  if (mode == 1) {
    TORCH_CHECK(M <= 128 && given(xs) && xs->scalar_type() == h.scalar_type() && al(*xs), "moe_route: slabs of 128 rows");
    p.ldx = pitch(*xs, E * 128, p.N, "moe_route xs");
    p.xs = xs->data_ptr();
  }
  TORCH_CHECK(mode != 2 || given(logits), "moe_route: ranks take given logits");
  p.status = status_ptr(status);
  check_launch(oxb::launch_moe_route(p, dt, cur_stream()), "moe_route");
}

void moe_scatter(const Tensor& h, int64_t M, int64_t E, int64_t top, const Tensor& expert, const Tensor& slot, const Tensor& counts,
                 const Tensor& xs, const Tensor& status) {
  oxb::MoeScatterParams p{};
  TORCH_CHECK(dtype_code(h, "moe_scatter h") == 0 && xs.scalar_type() == h.scalar_type(), "moe_scatter: bf16");
  TORCH_CHECK(E >= 1 && E <= oxb::kMaxExperts && top >= 1 && top <= oxb::kMaxTop, "moe_scatter: sizes");
  p.N = static_cast<int>(h.size(1));
  p.ldh = pitch(h, M, p.N, "moe_scatter h");
  p.ldx = pitch(xs, 1, p.N, "moe_scatter xs");
  TORCH_CHECK(p.N % 8 == 0 && p.ldh % 8 == 0 && p.ldx % 8 == 0, "moe_scatter: rows in whole 16-byte pieces");
  p.h = h.data_ptr();
  p.M = static_cast<int>(M);
  p.E = static_cast<int>(E);
  p.top = static_cast<int>(top);
  p.expert = i32(expert, M * top, "moe_scatter expert");
  p.slot = const_cast<int*>(i32(slot, M * top, "moe_scatter slot"));
  p.counts = reinterpret_cast<const uint32_t*>(i32(counts, E, "moe_scatter counts"));
  p.xs = xs.data_ptr();
  p.max_rows = xs.size(0);
  p.status = status_ptr(status);
  check_launch(oxb::launch_moe_scatter(p, cur_stream()), "moe_scatter");
}

void moe_rows(const Tensor& x, const Tensor& w, const Tensor& expert, int64_t pairs, int64_t top, bool per_pair, int64_t act,
              const Tensor& y) {
  oxb::MoeRowsParams p{};
  const int dt = dtype_code(x, "moe_rows x");
  TORCH_CHECK(w.dim() == 3 && w.is_contiguous() && w.scalar_type() == x.scalar_type() && y.scalar_type() == x.scalar_type() && top >= 1,
              "moe_rows: w [E, N, K] of x's type");
  p.E = static_cast<int>(w.size(0));
  p.N = static_cast<int>(w.size(1));
  p.K = static_cast<int>(w.size(2));
  p.ldx = pitch(x, per_pair ? pairs : (pairs + top - 1) / top, p.K, "moe_rows x");
  TORCH_CHECK(p.K % 8 == 0 && p.ldx % 8 == 0 && reinterpret_cast<uintptr_t>(x.data_ptr()) % 16 == 0, "moe_rows: whole 16-byte pieces");
  TORCH_CHECK(act != 3 || p.N % 64 == 0, "moe_rows: gate and up rows in units of 32");
  p.ldy = pitch(y, pairs, act == 3 ? p.N / 2 : p.N, "moe_rows y");
  p.x = x.data_ptr();
  p.w = w.data_ptr();
  p.y = y.data_ptr();
  p.pairs = static_cast<int>(pairs);
  p.top = static_cast<int>(top);
  p.per_pair = per_pair ? 1 : 0;
  p.expert = i32(expert, pairs, "moe_rows expert");
  TORCH_CHECK(act == 0 || act == 2 || act == 3, "moe_rows: act 0, 2 or 3");
  p.act = static_cast<int>(act);
  check_launch(oxb::launch_moe_rows(p, dt, cur_stream()), "moe_rows");
}

// Two maps per head -> their difference, normed (DiffNormParams)
void diff_norm(const Tensor& a, int64_t M, int64_t H, int64_t E, double lambda, double gain, double eps, const Tensor& out) {
  oxb::DiffNormParams p{};
  TORCH_CHECK(a.is_cuda() && a.scalar_type() == torch::kFloat32, "diff_norm: fp32 maps");
  p.lda = pitch(a, M, 2 * H * E, "diff_norm a");
  p.a = a.data_ptr<float>();
  p.M = static_cast<int>(M);
  p.H = static_cast<int>(H);
  p.E = static_cast<int>(E);
  p.lambda = static_cast<float>(lambda);
  p.gain = static_cast<float>(gain);
  p.eps = static_cast<float>(eps);
  p.ldo = pitch(out, M, H * E, "diff_norm out");
  p.out = out.data_ptr();
  check_launch(oxb::launch_diff_norm(p, dtype_code(out, "diff_norm out"), cur_stream()), "diff_norm");
}

// kv: columns of the latent, its norm weight and the cache; none for a layer that reads another one's cache
void latent_rows(const Tensor& proj, int64_t M, int64_t Q, const Tensor& q_norm, const Tensor& q_out, int64_t kv_col, int64_t R,
                 const OptTensor& kv_norm, const OptTensor& cache, const OptTensor& slots, const OptTensor& freq_hi,
                 const OptTensor& freq_lo, bool interleaved, double gain, const Tensor& positions, double eps, const Tensor& status) {
  oxb::LatentRowsParams p{};
  const int dt = dtype_code(q_out, "latent_rows q_out");
  p.proj_f32 = dtype_code(proj, "latent_rows proj");
  TORCH_CHECK(dt == 0 || p.proj_f32 == 1, "latent_rows: fp32 rows take fp32 projections");
  TORCH_CHECK(Q >= 1 && R >= 0 && Q + R <= 49152, "latent_rows: sizes");
  p.proj = proj.data_ptr();
  p.M = static_cast<int>(M);
  p.Q = static_cast<int>(Q);
  p.R = static_cast<int>(R);
  p.kv_col = static_cast<int>(kv_col);
  p.q_norm = f32(q_norm, Q, "latent_rows q_norm");
  p.ldq = pitch(q_out, M, Q, "latent_rows q_out");
  p.q_out = q_out.data_ptr();
  p.eps = static_cast<float>(eps);
  p.positions = i32(positions, M, "latent_rows positions");
  p.ld = pitch(proj, M, Q, "latent_rows proj");
  if (R > 0) {
    TORCH_CHECK(given(kv_norm) && given(cache) && given(slots), "latent_rows: norm weight, cache and slots of the latent");
    TORCH_CHECK(cache->scalar_type() == q_out.scalar_type() && cache->is_contiguous() && cache->dim() == 4 && cache->size(1) == 1 &&
                    cache->size(2) == 16,
                "latent_rows: cache [blocks, 1, 16, values]");
    p.CP = static_cast<int>(cache->size(3));
    p.rot = rotary(freq_hi, freq_lo, interleaved, gain, p.CP - R);
    TORCH_CHECK(R + p.rot.dims <= p.CP && kv_col >= Q && p.ld >= kv_col + R + p.rot.dims && proj.size(1) >= kv_col + R + p.rot.dims,
                "latent_rows: columns");
    p.kv_norm = f32(*kv_norm, R, "latent_rows kv_norm");
    p.cache = cache->data_ptr();
    TORCH_CHECK(slots->is_cuda() && slots->scalar_type() == torch::kInt64 && slots->numel() >= M, "latent_rows: slots int64");
    p.slots = reinterpret_cast<const long long*>(slots->data_ptr<int64_t>());
    p.num_slots = cache->size(0) * 16;
  }
  p.status = status_ptr(status);
  check_launch(oxb::launch_latent_rows(p, dt, cur_stream()), "latent_rows");
}

void latent_gather(const Tensor& cache, const Tensor& block_tables, const Tensor& ctx_lens, const Tensor& row0, int64_t seq0, int64_t n_seqs,
                   int64_t max_pages, const Tensor& out, const Tensor& status) {
  oxb::LatentGatherParams p{};
  TORCH_CHECK(dtype_code(cache, "latent_gather cache") == 0 && dtype_code(out, "latent_gather out") == 0 && cache.dim() == 4 &&
                  cache.is_contiguous() && cache.size(1) == 1 && cache.size(2) == 16 && cache.size(3) % 8 == 0,
              "latent_gather: bf16 cache [blocks, 1, 16, values]");
  p.CP = static_cast<int>(cache.size(3));
  TORCH_CHECK(out.dim() == 2 && out.is_contiguous() && out.size(1) == p.CP, "latent_gather: out [rows, values]");
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous() && block_tables.size(0) >= seq0 + n_seqs, "latent_gather: block_tables");
  p.cache = cache.data_ptr();
  p.num_blocks = static_cast<int>(cache.size(0));
  p.block_tables = i32(block_tables, 1, "latent_gather block_tables");
  p.max_blocks = static_cast<int>(block_tables.size(1));
  p.ctx_lens = i32(ctx_lens, seq0 + n_seqs, "latent_gather ctx_lens");
  p.row0 = i32(row0, seq0 + n_seqs, "latent_gather row0");
  p.seq0 = static_cast<int>(seq0);
  p.n_seqs = static_cast<int>(n_seqs);
  p.max_pages = static_cast<int>(max_pages);
  p.out = out.data_ptr();
  p.rows = out.size(0);
  p.status = status_ptr(status);
  check_launch(oxb::launch_latent_gather(p, cur_stream()), "latent_gather");
}

void latent_decode(const Tensor& q, const Tensor& cache, const Tensor& block_tables, const Tensor& seq_lens,
                   int64_t rows, int64_t R, int64_t max_splits, double scale, const Tensor& part_o, const Tensor& part_ml, const Tensor& out,
                   int64_t o_hd, const Tensor& status) {
  oxb::LatentDecodeParams p{};
  TORCH_CHECK(dtype_code(q, "latent_decode q") == 0 && dtype_code(cache, "latent_decode cache") == 0 && dtype_code(out, "latent_decode out") == 0,
              "latent_decode: bf16");
  TORCH_CHECK(cache.dim() == 4 && cache.is_contiguous() && cache.size(1) == 1 && cache.size(2) == 16, "latent_decode: cache [blocks, 1, 16, values]");
  p.CP = static_cast<int>(cache.size(3));
  TORCH_CHECK(q.dim() == 3 && q.size(0) >= rows && q.size(2) == p.CP && q.is_contiguous(), "latent_decode: q [rows, heads, values]");
  p.H = static_cast<int>(q.size(1));
  p.R = static_cast<int>(R);
  p.rows = static_cast<int>(rows);
  const int hn = oxb::latent_decode_heads(p.H, p.R, p.CP);
  TORCH_CHECK(R >= 1 && R <= p.CP && hn > 0 && max_splits >= 1 && max_splits <= 64, "latent_decode: sizes");
  p.num_blocks = static_cast<int>(cache.size(0));
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous() && block_tables.size(0) >= rows, "latent_decode: block_tables");
  p.block_tables = i32(block_tables, 1, "latent_decode block_tables");
  p.max_blocks = static_cast<int>(block_tables.size(1));
  p.seq_lens = i32(seq_lens, rows, "latent_decode seq_lens");
  p.max_splits = static_cast<int>(max_splits);
  p.scale_log2 = static_cast<float>(scale * 1.4426950408889634);
  p.part_o = const_cast<float*>(f32(part_o, rows * p.H * max_splits * R, "latent_decode part_o"));
  p.part_ml = const_cast<float*>(f32(part_ml, rows * p.H * max_splits * 2, "latent_decode part_ml"));
  TORCH_CHECK(o_hd >= R, "latent_decode: o_hd");
  p.o_hd = static_cast<int>(o_hd);
  p.ldo = pitch(out, rows, (p.H - 1) * o_hd + R, "latent_decode out");
  p.out = reinterpret_cast<__nv_bfloat16*>(out.data_ptr());
  p.status = status_ptr(status);
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto sw = CU_TENSOR_MAP_SWIZZLE_128B;
  const uint64_t row = static_cast<uint64_t>(p.CP) * 2;
  CUtensorMap tmQ = oxb::make_tma_map(q.data_ptr(), bf, 2, 3, p.CP, p.H, rows, row, row * p.H, 64, hn, 1, sw);
  CUtensorMap tmC = oxb::make_tma_map(cache.data_ptr(), bf, 2, 2, p.CP, static_cast<uint64_t>(p.num_blocks) * 16, 1, row, 0, 64, 16, 1, sw);
  check_launch(oxb::launch_latent_decode(tmQ, tmC, p, cur_stream()), "latent_decode");
}

// Causal attention of prompt tiles over plain rows of keys and values: kv [rows, columns], head g's keys from column
// g * dk on, its values from v_col0 + g * dv on; position t of sequence s is row row0[s] + t.
void prefill_rows(const Tensor& q, const Tensor& kv, int64_t dk, int64_t dv, int64_t v_col0, int64_t G, const Tensor& row0,
                  const Tensor& tile_seq, const Tensor& tile_q0, const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens,
                  const Tensor& out, int64_t n_tiles, double scale, int64_t out_d, const Tensor& status) {
  const int bkv = oxb::prefill_wide_tile(static_cast<int>(dk), static_cast<int>(dv));
  TORCH_CHECK(bkv > 0, "prefill_rows: head sizes ", dk, ", ", dv);
  TORCH_CHECK(dtype_code(q, "prefill_rows q") == 0 && dtype_code(kv, "prefill_rows kv") == 0, "prefill_rows: bf16");
  TORCH_CHECK(q.dim() == 3 && q.size(2) == dk && q.stride(2) == 1 && q.stride(1) == dk, "prefill_rows: q [rows, heads, dk]");
  TORCH_CHECK(kv.dim() == 2 && kv.stride(1) == 1 && kv.size(1) >= v_col0 + G * dv && v_col0 >= G * dk && v_col0 % 8 == 0 && kv.stride(0) % 8 == 0,
              "prefill_rows: kv columns");
  oxb::PrefillAttnParams p{};
  p.Hq = static_cast<int>(q.size(1));
  p.Hkv = static_cast<int>(G);
  TORCH_CHECK(G >= 1 && p.Hq % p.Hkv == 0 && out_d >= 1 && out_d <= dv, "prefill_rows: heads");
  p.q = reinterpret_cast<const __nv_bfloat16*>(q.data_ptr());
  p.q_stride = q.stride(0);
  TORCH_CHECK(tile_seq.is_cuda() && tile_seq.numel() >= n_tiles && tile_q0.numel() >= n_tiles, "prefill_rows: tiles");
  p.tile_seq = tile_seq.data_ptr<int>();
  p.tile_q0 = tile_q0.data_ptr<int>();
  p.q_start = i32(q_start, 1, "prefill_rows q_start");
  p.q_lens = i32(q_lens, 1, "prefill_rows q_lens");
  p.ctx_lens = i32(ctx_lens, 1, "prefill_rows ctx_lens");
  p.kv_row0 = i32(row0, 1, "prefill_rows row0");
  p.block_tables = p.kv_row0;   // not read in this form
  p.k_hd = static_cast<int>(dk);
  p.v_col0 = static_cast<int>(v_col0);
  p.v_hd = static_cast<int>(dv);
  p.out_stride = pitch(out, 1, p.Hq * out_d, "prefill_rows out");
  if (out.scalar_type() == torch::kFloat32) p.out_f32 = out.data_ptr<float>();
  else p.out = reinterpret_cast<__nv_bfloat16*>(out.data_ptr());
  p.out_d = static_cast<int>(out_d);
  p.exact_p = 1;
  p.scale_log2 = static_cast<float>(scale * 1.4426950408889634);
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto sw = CU_TENSOR_MAP_SWIZZLE_128B;
  CUtensorMap tmQ = oxb::make_tma_map(q.data_ptr(), bf, 2, 2, static_cast<uint64_t>(p.Hq) * dk, q.size(0), 1, static_cast<uint64_t>(q.stride(0)) * 2,
                                      0, 64, 128, 1, sw);
  CUtensorMap tmKV = oxb::make_tma_map(kv.data_ptr(), bf, 2, 2, static_cast<uint64_t>(v_col0 + G * dv), kv.size(0), 1,
                                       static_cast<uint64_t>(kv.stride(0)) * 2, 0, 64, bkv, 1, sw);
  oxb::launch_prefill_wide(tmQ, tmKV, tmKV, p, static_cast<int>(n_tiles), static_cast<int>(dk), static_cast<int>(dv), status_ptr(status), cur_stream());
  check_launch("prefill_rows");
}

// The paged form of the same for heads of up to 256 values: q [rows, H, D], caches [blocks, G, 16, D].
void prefill_pages(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& block_tables, const Tensor& tile_seq,
                   const Tensor& tile_q0, const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens, const Tensor& out,
                   int64_t n_tiles, double scale, int64_t out_d, const Tensor& status) {
  const int dk = static_cast<int>(q.size(2)), dv = static_cast<int>(v_cache.size(3));
  const int bkv = oxb::prefill_wide_tile(dk, dv);
  TORCH_CHECK(bkv > 0, "prefill_pages: head sizes ", dk, ", ", dv);
  TORCH_CHECK(dtype_code(q, "prefill_pages q") == 0 && dtype_code(k_cache, "prefill_pages k") == 0 && dtype_code(v_cache, "prefill_pages v") == 0,
              "prefill_pages: bf16");
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == dk && k_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() &&
                  k_cache.size(2) == 16 && v_cache.size(2) == 16 && k_cache.size(3) == dk && k_cache.size(0) == v_cache.size(0) &&
                  k_cache.size(1) == v_cache.size(1),
              "prefill_pages: q [rows, heads, D], caches [blocks, G, 16, D]");
  oxb::PrefillAttnParams p{};
  p.Hq = static_cast<int>(q.size(1));
  p.Hkv = static_cast<int>(k_cache.size(1));
  TORCH_CHECK(p.Hq % p.Hkv == 0 && out_d >= 1 && out_d <= dv, "prefill_pages: heads");
  p.q = reinterpret_cast<const __nv_bfloat16*>(q.data_ptr());
  p.q_stride = q.stride(0);
  TORCH_CHECK(block_tables.dim() == 2 && block_tables.is_contiguous(), "prefill_pages: block_tables");
  p.block_tables = i32(block_tables, 1, "prefill_pages block_tables");
  p.max_blocks = static_cast<int>(block_tables.size(1));
  p.num_blocks = static_cast<int>(k_cache.size(0));
  p.tile_seq = i32(tile_seq, n_tiles, "prefill_pages tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "prefill_pages tile_q0");
  p.q_start = i32(q_start, 1, "prefill_pages q_start");
  p.q_lens = i32(q_lens, 1, "prefill_pages q_lens");
  p.ctx_lens = i32(ctx_lens, 1, "prefill_pages ctx_lens");
  p.out_stride = pitch(out, 1, p.Hq * out_d, "prefill_pages out");
  if (out.scalar_type() == torch::kFloat32) p.out_f32 = out.data_ptr<float>();
  else p.out = reinterpret_cast<__nv_bfloat16*>(out.data_ptr());
  p.out_d = static_cast<int>(out_d);
  p.exact_p = 1;
  p.scale_log2 = static_cast<float>(scale * 1.4426950408889634);
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto sw = CU_TENSOR_MAP_SWIZZLE_128B;
  const uint64_t kv_rows = static_cast<uint64_t>(p.num_blocks) * p.Hkv * 16;
  CUtensorMap tmQ = oxb::make_tma_map(q.data_ptr(), bf, 2, 2, static_cast<uint64_t>(p.Hq) * dk, q.size(0), 1, static_cast<uint64_t>(q.stride(0)) * 2,
                                      0, 64, 128, 1, sw);
  CUtensorMap tmK = oxb::make_tma_map(k_cache.data_ptr(), bf, 2, 2, dk, kv_rows, 1, static_cast<uint64_t>(dk) * 2, 0, 64, 16, 1, sw);
  CUtensorMap tmV = oxb::make_tma_map(v_cache.data_ptr(), bf, 2, 2, dv, kv_rows, 1, static_cast<uint64_t>(dv) * 2, 0, 64, 16, 1, sw);
  oxb::launch_prefill_wide(tmQ, tmK, tmV, p, static_cast<int>(n_tiles), dk, dv, status_ptr(status), cur_stream());
  check_launch("prefill_pages");
}

// Sizes, gates and state of a matrix memory. proj: rows q | k | v | gate.
oxb::MemoryParams memory_common(const Tensor& proj, int64_t M, int64_t H, int64_t D, int64_t E, const OptTensor& z, const Tensor& z_bias,
                                double cap, double eps, const Tensor& norm_w, const Tensor& state, const Tensor& state_m, const Tensor& out,
                                const Tensor& status) {
  oxb::MemoryParams p{};
  TORCH_CHECK(H >= 1 && D >= 1 && E >= 1 && D <= 4096 && E <= 4096 && cap > 0, "memory: sizes");
  p.proj = proj.data_ptr();
  p.proj_f32 = dtype_code(proj, "memory proj");
  TORCH_CHECK(dtype_code(out, "memory out") == 0 || p.proj_f32 == 1, "memory: fp32 rows take fp32 projections");
  p.ld = pitch(proj, M, 2 * H * (D + E), "memory proj");
  p.H = static_cast<int>(H);
  p.D = static_cast<int>(D);
  p.E = static_cast<int>(E);
  if (given(z)) {
    TORCH_CHECK(z->is_cuda() && z->scalar_type() == torch::kFloat32, "memory: fp32 gate pre-activations");
    p.ldz = pitch(*z, M, 2 * H, "memory z");
    p.z = z->data_ptr<float>();
  }
  p.z_bias = f32(z_bias, 2 * H, "memory z_bias");
  p.cap = static_cast<float>(cap);
  p.scale = static_cast<float>(1.0 / std::sqrt(static_cast<double>(D)));
  p.eps = static_cast<float>(eps);
  p.norm_w = f32(norm_w, H * E, "memory norm_w");
  TORCH_CHECK(state.dim() == 3 && state.size(1) == H && state.size(2) == D * E + D && state_m.dim() == 2 && state_m.size(1) == H &&
                  state_m.size(0) == state.size(0),
              "memory: state [slots, H, D * E + D], maxima [slots, H]");
  p.state = const_cast<float*>(f32(state, 1, "memory state"));
  p.state_m = const_cast<float*>(f32(state_m, 1, "memory state_m"));
  p.num_slots = static_cast<int>(state.size(0));
  p.ldo = pitch(out, M, H * E, "memory out");
  p.out = out.data_ptr();
  p.status = status_ptr(status);
  return p;
}

void memory_decode(const Tensor& proj, int64_t rows, int64_t H, int64_t D, int64_t E, const OptTensor& z, const OptTensor& h, const OptTensor& z_w,
                   const Tensor& z_bias, double cap, double eps, const Tensor& norm_w, const Tensor& state, const Tensor& state_m,
                   const Tensor& row_slots, const Tensor& positions, const Tensor& out, const Tensor& status) {
  oxb::MemoryParams p = memory_common(proj, rows, H, D, E, z, z_bias, cap, eps, norm_w, state, state_m, out, status);
  if (!given(z)) {
    TORCH_CHECK(given(h) && given(z_w) && dtype_code(*h, "memory h") == 0 && dtype_code(*z_w, "memory z_w") == 0 && z_w->dim() == 2 &&
                    z_w->size(0) >= 2 * H && z_w->stride(1) == 1 && h->size(1) == z_w->size(1) && h->size(1) % 4 == 0,
                "memory_decode: bf16 rows and gate weights");
    p.ldh = pitch(*h, rows, h->size(1), "memory h");
    p.h = h->data_ptr();
    p.z_w = z_w->data_ptr();
    p.ldw = z_w->stride(0);
    p.N = static_cast<int>(h->size(1));
    TORCH_CHECK(p.ldh % 4 == 0 && p.ldw % 4 == 0 && reinterpret_cast<uintptr_t>(p.h) % 8 == 0 && reinterpret_cast<uintptr_t>(p.z_w) % 8 == 0,
                "memory_decode: alignment");
  }
  p.row_slots = i32(row_slots, rows, "memory_decode row_slots");
  p.positions = i32(positions, rows, "memory_decode positions");
  p.rows = static_cast<int>(rows);
  check_launch(oxb::launch_memory_decode(p, dtype_code(out, "memory out"), cur_stream()), "memory_decode");
}

void memory_prefill(const Tensor& proj, int64_t M, int64_t H, int64_t D, int64_t E, const Tensor& z, const Tensor& z_bias, double cap, double eps,
                    const Tensor& norm_w, const Tensor& state, const Tensor& state_m, const Tensor& seq_slots, const Tensor& tile_seq,
                    const Tensor& tile_q0, const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens, int64_t n_tiles, int64_t n_seqs,
                    const Tensor& ws, bool chunks, const Tensor& out, const Tensor& status) {
  oxb::MemoryParams p = memory_common(proj, M, H, D, E, z, z_bias, cap, eps, norm_w, state, state_m, out, status);
  const int dt = dtype_code(out, "memory out");
  p.seq_slots = i32(seq_slots, n_seqs, "memory_prefill seq_slots");
  p.tile_seq = i32(tile_seq, n_tiles, "memory_prefill tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "memory_prefill tile_q0");
  p.q_start = i32(q_start, n_seqs, "memory_prefill q_start");
  p.q_lens = i32(q_lens, n_seqs, "memory_prefill q_lens");
  p.ctx_lens = i32(ctx_lens, n_seqs, "memory_prefill ctx_lens");
  p.n_tiles = static_cast<int>(n_tiles);
  p.n_seqs = static_cast<int>(n_seqs);
  if (chunks) {
    TORCH_CHECK(dt == 0 && oxb::memory_chunks_ok(p.D, p.E), "memory_prefill: chunked form");
    const int64_t n = 2 * n_tiles * H;
    p.ws = const_cast<float*>(f32(ws, n * (D * E + D + 3), "memory_prefill ws"));
    p.ws_m = p.ws + n * (D * E + D);
    check_launch(oxb::launch_memory_chunks(p, cur_stream()), "memory_prefill");
  } else {
    TORCH_CHECK(D <= 1600, "memory_prefill: head size");
    p.o_buf = const_cast<float*>(f32(ws, M * H * E + n_seqs * H * (D + 1), "memory_prefill ws"));
    p.n_buf = p.o_buf + M * H * E;
    check_launch(oxb::launch_memory_scan(p, dt, cur_stream()), "memory_prefill");
  }
}

// Talking heads: decode rows (seq_lens) or prompt tiles; rows: the kernel for any sizes
oxb::TalkParams talk_common(const Tensor& q, const Tensor& cache, const Tensor& k_rms, const Tensor& block_tables, int64_t n, int64_t H,
                            int64_t D, int64_t window, double scale, double cap, const Tensor& talk, const Tensor& bias, const Tensor& gate,
                            const Tensor& out, const Tensor& status) {
  oxb::TalkParams p{};
  const int dt = dtype_code(q, "talk q");
  TORCH_CHECK(cache.dim() == 4 && cache.is_contiguous() && cache.size(2) == 16 && cache.scalar_type() == q.scalar_type() &&
                  out.scalar_type() == q.scalar_type(),
              "talk: cache [blocks, G, 16, head size], one storage type");
  p.H = static_cast<int>(H);
  p.G = static_cast<int>(cache.size(1));
  p.D = static_cast<int>(D);
  p.DP = static_cast<int>(cache.size(3));
  TORCH_CHECK(H >= 1 && H % p.G == 0 && D >= 1 && D <= p.DP && window >= 0, "talk: head sizes");
  p.q = q.data_ptr();
  p.q_ld = pitch(q, 1, H * p.DP, "talk q");
  TORCH_CHECK(dt == 1 || p.q_ld % 8 == 0, "talk: q rows in whole 16-byte pieces");
  p.cache = cache.data_ptr();
  p.k_rms = f32(k_rms, cache.size(0) * 16, "talk k_rms");
  p.num_blocks = static_cast<int>(cache.size(0));
  TORCH_CHECK(block_tables.dim() == 2, "talk: block_tables");
  p.block_tables = i32(block_tables, 1, "talk block_tables");
  p.max_blocks = static_cast<int>(block_tables.size(1));
  p.n_rows = static_cast<int>(n);
  p.window = static_cast<int>(window);
  p.scale = static_cast<float>(scale);
  p.cap = static_cast<float>(cap);
  p.talk = f32(talk, H * H, "talk matrix");
  TORCH_CHECK(bias.dim() == 2 && bias.size(0) == H && bias.size(1) >= 1, "talk: bias [H, distances]");
  p.bias = f32(bias, H, "talk bias");
  p.n_bias = static_cast<int>(bias.size(1));
  TORCH_CHECK(bias.size(1) >= 16 * block_tables.size(1) || (window > 0 && bias.size(1) >= window), "talk: a bias for every visible distance");
  p.gate_f32 = dtype_code(gate, "talk gate");
  p.gate = gate.data_ptr();
  p.gate_ld = pitch(gate, 1, H * D, "talk gate");
  p.ldo = pitch(out, 1, H * D, "talk out");
  p.out = out.data_ptr();
  p.status = status_ptr(status);
  return p;
}

// cache rows (one position of one key head) in boxes of `rows` x 64
CUtensorMap talk_cache_map(const Tensor& cache, const oxb::TalkParams& p, int rows) {
  return oxb::make_tma_map(cache.data_ptr(), CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, 2, p.DP, static_cast<uint64_t>(p.num_blocks) * p.G * 16, 1,
                           static_cast<uint64_t>(p.DP) * 2, 0, 64, rows, 1, CU_TENSOR_MAP_SWIZZLE_128B);
}

void talk_decode(const Tensor& q, const Tensor& cache, const Tensor& k_rms, const Tensor& block_tables, const Tensor& seq_lens,
                 int64_t rows, int64_t H, int64_t D, int64_t window, double scale, double cap,
                 const Tensor& talk, const Tensor& bias, const Tensor& gate, const OptTensor& part_o, const OptTensor& part_ml,
                 int64_t max_splits, const Tensor& out, const Tensor& status) {
  oxb::TalkParams p = talk_common(q, cache, k_rms, block_tables, rows, H, D, window, scale, cap, talk, bias, gate, out, status);
  TORCH_CHECK(block_tables.size(0) >= rows && q.size(0) >= rows && out.size(0) >= rows && gate.size(0) >= rows, "talk_decode: rows");
  p.seq_lens = i32(seq_lens, rows, "talk_decode seq_lens");
  if (!given(part_o)) {
    check_launch(oxb::launch_talk_rows(p, dtype_code(q, "talk q"), cur_stream()), "talk_rows");
    return;
  }
  TORCH_CHECK(dtype_code(q, "talk q") == 0 && oxb::talk_decode_ok(p.H, p.G, p.DP) && given(part_ml) && max_splits >= 1,
              "talk_decode: sizes");
  p.part_o = const_cast<float*>(f32(*part_o, rows * H * max_splits * p.DP, "talk_decode part_o"));
  p.part_ml = const_cast<float*>(f32(*part_ml, rows * H * max_splits * 2, "talk_decode part_ml"));
  p.max_splits = static_cast<int>(max_splits);
  CUtensorMap tmC = talk_cache_map(cache, p, oxb::talk_decode_box(p.H, p.G, p.DP));
  check_launch(oxb::launch_talk_decode(tmC, p, cur_stream()), "talk_decode");
}

void talk_prefill(const Tensor& q, const Tensor& cache, const Tensor& k_rms, const Tensor& block_tables, const Tensor& tile_seq,
                  const Tensor& tile_q0, const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens, int64_t n_tiles, int64_t H,
                  int64_t D, int64_t window, double scale, double cap, const Tensor& talk, const Tensor& bias, const Tensor& gate,
                  const OptTensor& scores, int64_t span, const Tensor& out, const Tensor& status) {
  oxb::TalkParams p = talk_common(q, cache, k_rms, block_tables, n_tiles, H, D, window, scale, cap, talk, bias, gate, out, status);
  p.tile_seq = i32(tile_seq, n_tiles, "talk_prefill tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "talk_prefill tile_q0");
  p.q_start = i32(q_start, 1, "talk_prefill q_start");
  p.q_lens = i32(q_lens, 1, "talk_prefill q_lens");
  p.ctx_lens = i32(ctx_lens, 1, "talk_prefill ctx_lens");
  if (!given(scores)) {
    check_launch(oxb::launch_talk_rows(p, dtype_code(q, "talk q"), cur_stream()), "talk_rows");
    return;
  }
  TORCH_CHECK(dtype_code(q, "talk q") == 0 && oxb::talk_prefill_ok(p.H, p.DP) && span > 0 && span % 32 == 0, "talk_prefill: sizes");
  p.scores = const_cast<float*>(f32(*scores, n_tiles * H * 128 * span, "talk_prefill scores"));
  p.span = static_cast<int>(span);
  CUtensorMap tmV = talk_cache_map(cache, p, 16);
  check_launch(oxb::launch_talk_prefill(tmV, p, cur_stream()), "talk_prefill");
}

oxb::GruParams gru_common(const Tensor& proj, int64_t M, const Tensor& bias, double out_gain, const Tensor& state, const Tensor& out,
                          const Tensor& status) {
  oxb::GruParams p{};
  TORCH_CHECK(state.dim() == 2 && state.size(1) % 4 == 0, "gru: state [slots, N], N a multiple of 4");
  p.N = static_cast<int>(state.size(1));
  p.state = const_cast<float*>(f32(state, 1, "gru state"));
  p.num_slots = static_cast<int>(state.size(0));
  p.ld = pitch(proj, M, 3 * p.N, "gru proj");
  p.proj = proj.data_ptr();
  p.proj_f32 = dtype_code(proj, "gru proj");
  TORCH_CHECK(dtype_code(out, "gru out") == 0 || p.proj_f32 == 1, "gru: fp32 rows take fp32 projections");
  p.bias = f32(bias, 2 * p.N, "gru bias");
  p.out_gain = static_cast<float>(out_gain);
  p.ldo = pitch(out, M, p.N, "gru out");
  p.out = out.data_ptr();
  TORCH_CHECK(p.ld % 4 == 0 && p.ldo % 4 == 0 && reinterpret_cast<uintptr_t>(p.proj) % 16 == 0 && reinterpret_cast<uintptr_t>(p.out) % 8 == 0,
              "gru: rows in whole pieces of four values");
  p.status = status_ptr(status);
  return p;
}

void gru_decode(const Tensor& proj, int64_t rows, const Tensor& bias, double out_gain, const Tensor& state, const Tensor& row_slots,
                const Tensor& positions, const Tensor& out, const Tensor& status) {
  oxb::GruParams p = gru_common(proj, rows, bias, out_gain, state, out, status);
  p.row_slots = i32(row_slots, rows, "gru_decode row_slots");
  p.positions = i32(positions, rows, "gru_decode positions");
  p.rows = static_cast<int>(rows);
  check_launch(oxb::launch_gru_decode(p, dtype_code(out, "gru out"), cur_stream()), "gru_decode");
}

void gru_prefill(const Tensor& proj, int64_t M, const Tensor& bias, double out_gain, const Tensor& state, const Tensor& seq_slots,
                 const Tensor& tile_seq, const Tensor& tile_q0, const Tensor& q_start, const Tensor& q_lens, const Tensor& ctx_lens,
                 int64_t n_tiles, const Tensor& ws, const Tensor& out, const Tensor& status) {
  oxb::GruParams p = gru_common(proj, M, bias, out_gain, state, out, status);
  p.seq_slots = i32(seq_slots, 1, "gru_prefill seq_slots");
  p.tile_seq = i32(tile_seq, n_tiles, "gru_prefill tile_seq");
  p.tile_q0 = i32(tile_q0, n_tiles, "gru_prefill tile_q0");
  p.q_start = i32(q_start, 1, "gru_prefill q_start");
  p.q_lens = i32(q_lens, 1, "gru_prefill q_lens");
  p.ctx_lens = i32(ctx_lens, 1, "gru_prefill ctx_lens");
  p.n_tiles = static_cast<int>(n_tiles);
  p.ws = const_cast<float*>(f32(ws, n_tiles * (1 + oxb::kGruParts) * 2 * p.N, "gru_prefill ws"));
  check_launch(oxb::launch_gru_prefill(p, dtype_code(out, "gru out"), cur_stream()), "gru_prefill");
}

void gemm_f32(const Tensor& a, const Tensor& w, const Tensor& out) {
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && out.is_cuda() && a.scalar_type() == torch::kFloat32 &&
                  w.scalar_type() == torch::kFloat32 && out.scalar_type() == torch::kFloat32 && a.dim() == 2 && w.dim() == 2 &&
                  a.stride(1) == 1 && w.stride(1) == 1 && a.size(1) == w.size(1),
              "gemm_f32: fp32 a [M, K], w [N, K]");
  const int64_t M = a.size(0), N = w.size(0), K = a.size(1);
  const int64_t ldo = pitch(out, M, N, "gemm_f32 out");
  check_launch(oxb::launch_gemm_f32(a.data_ptr<float>(), a.stride(0), w.data_ptr<float>(), w.stride(0), out.data_ptr<float>(), ldo,
                                    static_cast<int>(M), static_cast<int>(N), static_cast<int>(K), cur_stream()),
               "gemm_f32");
}

void glu_f32(const Tensor& gu, const Tensor& out, int64_t M, int64_t I, int64_t act) {
  TORCH_CHECK(gu.is_cuda() && gu.scalar_type() == torch::kFloat32 && out.scalar_type() == torch::kFloat32, "glu_f32: fp32");
  const int64_t ldg = pitch(gu, M, act == 2 ? I : 2 * I, "glu_f32 gu"), ldo = pitch(out, M, I, "glu_f32 out");
  check_launch(oxb::launch_glu_f32(gu.data_ptr<float>(), ldg, out.data_ptr<float>(), ldo, static_cast<int>(M),
                                   static_cast<int>(I), static_cast<int>(act), cur_stream()),
               "glu_f32");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.doc() = "sm_100a kernels of layer-list decoders";
  m.attr("RETENTION_CHUNK") = oxb::kRetChunk;
  m.attr("MAX_STREAMS") = oxb::kMaxStreams;
  m.def("set_pdl", [](bool on) { oxb::pdl_enabled() = on; });
  m.def("stream_norm", &stream_norm);
  m.def("heads", &heads);
  m.def("row_attention", &row_attention);
  m.def("retention_decode", &retention_decode);
  m.def("retention_prefill", &retention_prefill);
  m.def("retention_chunks_ok", [](int64_t D, int64_t E) { return oxb::retention_chunks_ok((int)D, (int)E); });
  m.attr("MAX_EXPERTS") = oxb::kMaxExperts;
  m.attr("MAX_TOP") = oxb::kMaxTop;
  m.def("branch_norm", &branch_norm);
  m.def("ssd_decode", &ssd_decode);
  m.def("ssd_prefill", &ssd_prefill);
  m.def("ssd_chunks_ok", [](int64_t NP) { return oxb::ssd_chunks_ok(static_cast<int>(NP)); });
  m.def("ssd_segment", [](int64_t H, int64_t EP, int64_t n_tiles, int64_t n_seqs) {
    return oxb::ssd_segment(static_cast<int>(H), static_cast<int>(EP), static_cast<int>(n_tiles), static_cast<int>(n_seqs));
  });
  m.def("gated_norm", &gated_norm);
  m.def("moe_route", &moe_route);
  m.def("moe_scatter", &moe_scatter);
  m.def("moe_rows", &moe_rows);
  m.def("diff_norm", &diff_norm);
  m.def("latent_rows", &latent_rows);
  m.def("latent_gather", &latent_gather);
  m.def("latent_decode", &latent_decode);
  m.def("latent_decode_heads", [](int64_t H, int64_t R, int64_t CP) {
    return oxb::latent_decode_heads(static_cast<int>(H), static_cast<int>(R), static_cast<int>(CP));
  });
  m.def("prefill_rows", &prefill_rows);
  m.def("prefill_pages", &prefill_pages);
  m.def("prefill_wide_tile", [](int64_t dk, int64_t dv) { return oxb::prefill_wide_tile(static_cast<int>(dk), static_cast<int>(dv)); });
  m.def("memory_decode", &memory_decode);
  m.def("memory_prefill", &memory_prefill);
  m.def("memory_chunks_ok", [](int64_t D, int64_t E) { return oxb::memory_chunks_ok(static_cast<int>(D), static_cast<int>(E)); });
  m.attr("MEMORY_CHUNK") = oxb::kMemChunk;
  m.attr("MAX_GROUPS") = oxb::kMaxGroups;
  m.def("talk_decode", &talk_decode);
  m.def("talk_prefill", &talk_prefill);
  m.def("talk_decode_ok", [](int64_t H, int64_t G, int64_t DP) { return oxb::talk_decode_ok(static_cast<int>(H), static_cast<int>(G), static_cast<int>(DP)); });
  m.def("talk_prefill_ok", [](int64_t H, int64_t DP) { return oxb::talk_prefill_ok(static_cast<int>(H), static_cast<int>(DP)); });
  m.def("talk_span", [](int64_t window, int64_t max_ctx) { return oxb::talk_span(static_cast<int>(window), static_cast<int>(max_ctx)); });
  m.def("gru_decode", &gru_decode);
  m.def("gru_prefill", &gru_prefill);
  m.attr("GRU_PARTS") = oxb::kGruParts;
  m.def("gemm_f32", &gemm_f32);
  m.def("glu_f32", &glu_f32);
}
