// Softmax attention of single query rows over the paged cache, in fp32 FMAs: any head sizes, fp32 or bf16
// storage, sliding window with kept first positions or chunks, optional sink. One CTA per (row, query head) walks the visible keys
// 128 at a time: thread = key for the scores, thread = value dimension for the sums. The 32-bit path and
// head sizes beyond the tensor-core kernels use it; it is not tuned for throughput.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

constexpr int kKeys = 128;
constexpr int kMaxV = 8;  // value dimensions per thread: E <= 1024

template <typename T>
__global__ void __launch_bounds__(kKeys) row_attention_kernel(const RowAttnParams p) {
  extern __shared__ float s_q[];  // D
  __shared__ float s_p[kKeys], s_red[32];
  __shared__ int s_row[kKeys];    // cache row (block * 16 + offset) of every key of the tile
  pdl_wait();
  const int head = blockIdx.y;
  int row, pos, seq;
  if (p.tile_seq == nullptr) {
    row = seq = blockIdx.x;
    pos = p.seq_lens[row] - 1;
  } else {
    const int tile = blockIdx.x >> 7, r = blockIdx.x & 127;
    seq = p.tile_seq[tile];
    const int qi = p.tile_q0[tile] + r;
    if (qi >= p.q_lens[seq]) return;
    row = p.q_start[seq] + qi;
    pos = p.ctx_lens[seq] - p.q_lens[seq] + qi;
  }
  if (pos < 0) return;  // padding row
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  const T* qp = static_cast<const T*>(p.q) + static_cast<long long>(row) * p.q_ld + head * p.q_hd;
  for (int d = threadIdx.x; d < p.D; d += kKeys) s_q[d] = to_f(qp[d]);
  const int kvh = head / (p.H / p.G);
  // visible keys: [0, n_first) and [lo, pos]
  const int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : ((p.window > 0 && pos + 1 > p.window) ? pos + 1 - p.window : 0);
  const int n_first = min(p.keep_first, lo);
  const int n_vis = n_first + (pos + 1 - lo);
  const float sink = p.sinks != nullptr ? p.sinks[head] : p.sink;
  float m_run = sink, l_run = sink == -INFINITY ? 0.f : 1.f, acc[kMaxV];
#pragma unroll
  for (int i = 0; i < kMaxV; ++i) acc[i] = 0.f;
  __syncthreads();
  for (int base = 0; base < n_vis; base += kKeys) {
    const int l = base + threadIdx.x;
    float s = -INFINITY;
    if (l < n_vis) {
      const int j = l < n_first ? l : lo + l - n_first;
      const int pg = j >> 4;
      int b = pg < p.max_blocks ? bt[pg] : -1;
      if (static_cast<unsigned>(b) >= static_cast<unsigned>(p.num_blocks)) {
        set_status_once(p.status, kStatusBadIndex);
        b = 0;
      }
      const int krow = (b * p.G + kvh) * 16 + (j & 15);
      s_row[threadIdx.x] = krow;
      const T* k = static_cast<const T*>(p.k_cache) + static_cast<long long>(krow) * p.DP;
      float d0 = 0.f;
      for (int d = 0; d < p.D; ++d) d0 = fmaf(s_q[d], to_f(k[d]), d0);
      s = d0 * p.scale;
    }
    const float m_new = fmaxf(m_run, block_max_all(s, s_red));
    const float e = l < n_vis ? expf(s - m_new) : 0.f;
    const float alpha = m_run == -INFINITY ? 0.f : expf(m_run - m_new);
    m_run = m_new;
    s_p[threadIdx.x] = e;
    l_run = l_run * alpha + block_sum_all(e, s_red);  // its barriers also publish s_p and s_row
    const int n = min(kKeys, n_vis - base);
#pragma unroll
    for (int i = 0; i < kMaxV; ++i) {
      const int c = threadIdx.x + i * kKeys;
      if (c < p.E) {
        float a = acc[i] * alpha;
        for (int t = 0; t < n; ++t)
          a = fmaf(s_p[t], to_f(static_cast<const T*>(p.v_cache)[static_cast<long long>(s_row[t]) * p.EP + c]), a);
        acc[i] = a;
      }
    }
    __syncthreads();
  }
  const long long at = static_cast<long long>(row) * p.ldo + head * p.o_hd;
#pragma unroll
  for (int i = 0; i < kMaxV; ++i) {
    const int c = threadIdx.x + i * kKeys;
    if (c >= p.E) continue;
    if (p.out_f32) static_cast<float*>(p.out)[at + c] = acc[i] / l_run * p.out_gain;
    else static_cast<T*>(p.out)[at + c] = from_f<T>(acc[i] / l_run * p.out_gain);
  }
}

}  // namespace

cudaError_t launch_row_attention(const RowAttnParams& p, int dtype, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (p.E > kKeys * kMaxV) return cudaErrorInvalidValue;
  const dim3 grid(p.tile_seq == nullptr ? p.n_rows : p.n_rows * 128, p.H);
  const size_t smem = static_cast<size_t>(p.D) * sizeof(float);
  if (dtype == 1) return launch_kernel(row_attention_kernel<float>, grid, dim3(kKeys), smem, stream, true, false, p);
  return launch_kernel(row_attention_kernel<__nv_bfloat16>, grid, dim3(kKeys), smem, stream, true, false, p);
}

}  // namespace oxb
