// Latent attention around the products (sm_100a): a token keeps one row of R latent values and T rotated key values for
// all heads. Decoding against these rows is in latent_decode.cu.
//
// latent_rows: projection rows -> normed query latent, normed latent and rotated key part into the paged cache.
// latent_gather: cache rows of a step's prompts one after the other, the operand of the GEMM that expands them to
//   keys and values per head (prompts run the plain-row form of the prefill attention).
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

template <typename T, typename P>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentRowsParams p) {
  extern __shared__ float s_mem[];   // Q query values, then R latent values
  __shared__ float s_red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld;
  const P* kv = pr + p.kv_col;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x; c < p.Q; c += blockDim.x) {
    const float x = to_f(pr[c]);
    s_mem[c] = x;
    sq = fmaf(x, x, sq);
  }
  for (int c = threadIdx.x; c < p.R; c += blockDim.x) {
    const float x = to_f(kv[c]);
    s_mem[p.Q + c] = x;
    sk = fmaf(x, x, sk);
  }
  const float rq = 1.f / sqrtf(block_sum_all(sq, s_red) / static_cast<float>(p.Q) + p.eps);
  T* q = static_cast<T*>(p.q_out) + static_cast<long long>(row) * p.ldq;
  for (int c = threadIdx.x; c < p.Q; c += blockDim.x) q[c] = from_f<T>(s_mem[c] * rq * p.q_norm[c]);
  if (p.R <= 0) return;
  const float rk = 1.f / sqrtf(block_sum_all(sk, s_red) / static_cast<float>(p.R) + p.eps);
  const long long slot = p.slots[row];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  T* out = static_cast<T*>(p.cache) + slot * p.CP;
  for (int c = threadIdx.x; c < p.R; c += blockDim.x) out[c] = from_f<T>(s_mem[p.Q + c] * rk * p.kv_norm[c]);
  const int pos = p.positions[row];
  for (int i = threadIdx.x; i < (p.rot.dims >> 1); i += blockDim.x) {
    float sn, cs;
    rotary_sincos(p.rot, i, pos, &sn, &cs);
    int a, b;
    rotary_pair(p.rot, i, &a, &b);
    const float u = to_f(kv[p.R + a]), v = to_f(kv[p.R + b]);
    out[p.R + a] = from_f<T>(u * cs - v * sn);
    out[p.R + b] = from_f<T>(v * cs + u * sn);
  }
}

// grid (pages, sequences): one page per CTA, 16-byte pieces.
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = p.seq0 + blockIdx.y, page = blockIdx.x, ctx = p.ctx_lens[seq];
  if (page * 16 >= ctx || page >= p.max_blocks) return;
  int b = p.block_tables[static_cast<long long>(seq) * p.max_blocks + page];
  if (static_cast<unsigned>(b) >= static_cast<unsigned>(p.num_blocks)) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    b = 0;
  }
  const long long row = static_cast<long long>(p.row0[seq]) + page * 16;
  const int n = min(16, ctx - page * 16);
  if (row < 0 || row + n > p.rows) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.cache) + static_cast<long long>(b) * 16 * p.CP);
  uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + row * p.CP);
  for (int i = threadIdx.x; i < n * p.CP / 8; i += 256) dst[i] = src[i];
}

template <typename T, typename P>
cudaError_t launch_rows(const LatentRowsParams& p, cudaStream_t stream) {
  const size_t smem = (static_cast<size_t>(p.Q) + p.R) * sizeof(float);
  ensure_dynamic_smem(latent_rows_kernel<T, P>, smem);
  return launch_kernel(latent_rows_kernel<T, P>, dim3(p.M), dim3(256), smem, stream, true, false, p);
}

}  // namespace

cudaError_t launch_latent_rows(const LatentRowsParams& p, int dtype, cudaStream_t stream) {
  if (p.M <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_rows<float, float>(p, stream);
  return p.proj_f32 ? launch_rows<bf16, float>(p, stream) : launch_rows<bf16, bf16>(p, stream);
}

cudaError_t launch_latent_gather(const LatentGatherParams& p, cudaStream_t stream) {
  if (p.n_seqs <= 0 || p.max_pages <= 0) return cudaSuccess;
  return launch_kernel(latent_gather_kernel, dim3(p.max_pages, p.n_seqs), dim3(256), 0, stream, true, false, p);
}

}  // namespace oxb
