// Residual streams between the sublayers of a layer-list decoder (sm_100a): the hyper-connection update of
// the sublayer that just ran, the read-out for the next one and its RMS norm in one pass over the row,
// with the embedding gather (and its hashed bigram row) folded into the first of them. Streams stay fp32.
// With one stream, mix = in = out = 1 it is residual-add + RMSNorm. `branch_norm` is its counterpart for layers whose
// mixer and feed-forward run side by side: the branches of the layer that just ran, each by its own norm, the weighted
// rows of the chosen experts, and the norms of the next layer's mixer and feed-forward in one pass.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

// One CTA per row (looping). V = 4: rows of whole 16-byte pieces, V = 1: any width. S: largest stream count
// of this instantiation. CH: pieces per thread whose loads are issued together (the kernel is a stream of
// fp32 rows; the bytes in flight set its rate).
template <typename T, int S, int V, int CH>
__global__ void __launch_bounds__(CH == 1 ? 1024 : (CH == 2 ? 512 : 256)) stream_norm_kernel(const StreamNormParams p) {
  extern __shared__ float s_u[];  // N read-out values
  __shared__ float s_red[32];
  __shared__ float s_mix[S * S], s_out[S], s_in[S];
  pdl_launch_dependents();
  const int n_s = p.S, N = p.N;
  for (int i = threadIdx.x; i < n_s * n_s; i += blockDim.x) s_mix[(i / n_s) * S + i % n_s] = p.y != nullptr ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < n_s; i += blockDim.x) {
    s_out[i] = p.y != nullptr ? p.out[i] : 0.f;
    s_in[i] = p.in != nullptr ? p.in[i] : 1.f;
  }
  __syncthreads();
  pdl_wait();  // streams, the sublayer's output and the step's tokens come from earlier kernels
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    float* xr = p.x + static_cast<long long>(row) * n_s * N;
    float* yr = p.y != nullptr ? p.y + static_cast<long long>(row) * p.ldy : nullptr;
    const T* er = nullptr;
    const T* br = nullptr;
    if (p.tokens != nullptr) {
      const int tok = p.tokens[row], prev = p.prev != nullptr ? p.prev[row] : -1;
      const bool ok = tok >= 0 && tok < p.vocab;
      if (!ok && threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
      er = static_cast<const T*>(p.embed) + static_cast<long long>(ok ? tok : 0) * N;
      if (p.bigram != nullptr) {
        const long long b = (prev < 0 || !ok) ? p.buckets : (prev * p.mul_prev + tok * p.mul_cur) % p.buckets;
        br = static_cast<const T*>(p.bigram) + b * N;
      }
    }
    if (p.clear != nullptr) {
      float* z = p.clear + static_cast<long long>(row) * p.clear_ld;
      for (int c = threadIdx.x * 4; c < p.clear_n; c += blockDim.x * 4)
        *reinterpret_cast<float4*>(z + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int dst = p.row_map != nullptr ? p.row_map[row] : row;
    float ssq = 0.f;
    for (int base = 0; base < N; base += blockDim.x * V * CH) {
      float x[CH][S][V], y[CH][V];
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = base + (k * blockDim.x + threadIdx.x) * V;
        if (c >= N) continue;
        if (er != nullptr) {
          float e[V];
          if constexpr (V == 4) {
            load4<T>(er + c, e);
            if (br != nullptr) {
              float b[4];
              load4<T>(br + c, b);
#pragma unroll
              for (int j = 0; j < 4; ++j) e[j] += b[j];
            }
          } else {
            e[0] = to_f(er[c]) + (br != nullptr ? to_f(br[c]) : 0.f);
          }
#pragma unroll
          for (int s = 0; s < S; ++s)
#pragma unroll
            for (int j = 0; j < V; ++j) x[k][s][j] = e[j];
        } else {
#pragma unroll
          for (int s = 0; s < S; ++s)
            if (s < n_s) {
              if constexpr (V == 4) load4<float>(xr + static_cast<long long>(s) * N + c, x[k][s]);
              else x[k][s][0] = xr[static_cast<long long>(s) * N + c];
            }
          if constexpr (V == 4) load4<float>(yr + c, y[k]);
          else y[k][0] = yr[c];
        }
      }
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = base + (k * blockDim.x + threadIdx.x) * V;
        if (c >= N) continue;
        float u[V];
#pragma unroll
        for (int j = 0; j < V; ++j) u[j] = 0.f;
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (t < n_s) {
            float z[V];
            if (yr != nullptr) {
#pragma unroll
              for (int j = 0; j < V; ++j) z[j] = s_out[t] * y[k][j];
#pragma unroll
              for (int s = 0; s < S; ++s)
                if (s < n_s) {
#pragma unroll
                  for (int j = 0; j < V; ++j) z[j] = fmaf(s_mix[s * S + t], x[k][s][j], z[j]);
                }
            } else {
#pragma unroll
              for (int j = 0; j < V; ++j) z[j] = x[k][t][j];
            }
#pragma unroll
            for (int j = 0; j < V; ++j) u[j] = fmaf(s_in[t], z[j], u[j]);
            if (p.store_x) {
              if constexpr (V == 4) store4<float>(xr + static_cast<long long>(t) * N + c, z);
              else xr[static_cast<long long>(t) * N + c] = z[0];
            }
          }
        }
        if (yr != nullptr && p.zero_y) {
          if constexpr (V == 4) *reinterpret_cast<float4*>(yr + c) = make_float4(0.f, 0.f, 0.f, 0.f);
          else yr[c] = 0.f;
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(s_u + c) = make_float4(u[0], u[1], u[2], u[3]);
        else s_u[c] = u[0];
#pragma unroll
        for (int j = 0; j < V; ++j) ssq = fmaf(u[j], u[j], ssq);
      }
    }
    if (dst < 0) continue;  // a row without a logits row; the same for every thread of the CTA
    const float total = block_sum_all(ssq, s_red);
    const float r = 1.f / sqrtf(total / static_cast<float>(N) + p.eps);
    T* hr = static_cast<T*>(p.h) + static_cast<long long>(dst) * p.ldh;
    for (int c = threadIdx.x * V; c < N; c += blockDim.x * V) {
      if constexpr (V == 4) {
        float w[4], o[4];
        load4<float>(p.norm_w + c, w);
        const float4 u = *reinterpret_cast<const float4*>(s_u + c);
        o[0] = u.x * r * (w[0] + p.w_offset);
        o[1] = u.y * r * (w[1] + p.w_offset);
        o[2] = u.z * r * (w[2] + p.w_offset);
        o[3] = u.w * r * (w[3] + p.w_offset);
        store4<T>(hr + c, o);
      } else {
        hr[c] = from_f<T>(s_u[c] * r * (p.norm_w[c] + p.w_offset));
      }
    }
  }
}

template <typename T, int S, int V, int CH>
cudaError_t launch_ch(const StreamNormParams& p, int threads, cudaStream_t stream) {
  auto kern = stream_norm_kernel<T, S, V, CH>;
  const size_t smem = static_cast<size_t>(p.N) * sizeof(float);
  ensure_dynamic_smem(kern, smem);
  const int cap = 8 * sm_count();
  return launch_kernel(kern, dim3(p.rows < cap ? p.rows : cap), dim3(threads), smem, stream, /*pdl=*/true, false, p);
}

template <typename T, int S>
cudaError_t launch_s(const StreamNormParams& p, cudaStream_t stream) {
  constexpr int VW = S <= 8 ? 4 : 1;  // 16 streams x 4 values would spill
  const bool vec = VW == 4 && p.N % 4 == 0 && p.ldy % 4 == 0 && p.ldh % 4 == 0;
  const int v = vec ? 4 : 1;
  int threads = (p.N / v + 31) / 32 * 32;
  if (threads < 32) threads = 32;
  constexpr int CHM = S <= 2 ? 4 : (S <= 4 ? 2 : 1);  // pieces in flight that the registers hold
  if (vec && CHM > 1 && p.rows > 2 * sm_count() && threads > 256) {
    // many rows: several CTAs per SM, each with a whole row (or most of it) in flight
    if (CHM == 4 && threads > 512) return launch_ch<T, S, VW, CHM>(p, 256, stream);
    return launch_ch<T, S, VW, 2>(p, 256, stream);
  }
  if (threads > 1024) threads = 1024;
  return vec ? launch_ch<T, S, VW, 1>(p, threads, stream) : launch_ch<T, S, 1, 1>(p, threads, stream);
}

template <typename T>
cudaError_t launch_t(const StreamNormParams& p, cudaStream_t stream) {
  if (p.S == 1) return launch_s<T, 1>(p, stream);
  if (p.S == 2) return launch_s<T, 2>(p, stream);
  if (p.S <= 4) return launch_s<T, 4>(p, stream);
  if (p.S <= 8) return launch_s<T, 8>(p, stream);
  return launch_s<T, kMaxStreams>(p, stream);
}

// Layers whose mixer and feed-forward run side by side, or one after the other with a norm on either side: four values
// per piece, CH pieces per thread, which stay in registers; NB: branches that it can add.
// The chosen experts' rows of a token wait in shared memory as (row, weight): a row outside the buffer weighs nothing.
struct ChosenRow {
  int row;
  float weight;
};
__device__ __forceinline__ void chosen_rows(const BranchNormParams& p, int row, ChosenRow* s_e) {
  for (int k = threadIdx.x; k < p.top; k += blockDim.x) {
    const int s = p.e_slot[row * p.top + k];
    const bool ok = s >= 0 && s < p.n_e_rows;
    s_e[k] = {ok ? s : 0, ok ? p.e_weight[row * p.top + k] : 0.f};
  }
}
template <typename T>
__device__ __forceinline__ void expert_sum4(const BranchNormParams& p, const ChosenRow* s_e, int c, float (&a)[4]) {
  const T* rows = static_cast<const T*>(p.e_rows) + c;
#pragma unroll 8
  for (int k = 0; k < p.top; ++k) {
    const ChosenRow e = s_e[k];
    float v[4];
    load4_stream(rows + static_cast<long long>(e.row) * p.lde, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) a[j] = fmaf(e.weight, v[j], a[j]);
  }
}
template <typename T>
__device__ __forceinline__ float expert_sum(const BranchNormParams& p, const ChosenRow* s_e, int c) {
  float a = 0.f;
  for (int k = 0; k < p.top; ++k)
    a = fmaf(s_e[k].weight, to_f(static_cast<const T*>(p.e_rows)[static_cast<long long>(s_e[k].row) * p.lde + c]), a);
  return a;
}
__device__ __forceinline__ bool experts_are_branch(const BranchNormParams& p) {
  return (p.n_branches > 0 && p.y[0] == nullptr) || (p.n_branches > 1 && p.y[1] == nullptr);
}
// sums of both branches at once over the block
__device__ __forceinline__ float2 block_sum2(float2 v, float2* scratch) {
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  const int nw = (blockDim.x + 31) >> 5;
  const float2 s = lane < nw ? scratch[lane] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(s.x), warp_sum(s.y));
}

// Operand of the product over [x; embedding] (BranchNormParams::split)
template <typename T>
__device__ __forceinline__ const T* x0_row(const BranchNormParams& p, int row) {
  const int tok = p.x0_tokens[row];
  const bool ok = tok >= 0 && tok < p.vocab;
  if (!ok && threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
  return static_cast<const T*>(p.embed) + static_cast<long long>(ok ? tok : 0) * p.N;
}
template <typename T>
__device__ __forceinline__ void split_row4(const BranchNormParams& p, int row, int c, const float (&x)[4]) {
  T* d = static_cast<T*>(p.split) + static_cast<long long>(row) * p.ld_split + c;
  store4<T>(d, x);
  if constexpr (sizeof(T) == 2) {
    float rest[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) rest[j] = x[j] - to_f(from_f<T>(x[j]));
    d += p.split_off;
    store4<T>(d, rest);
  }
  float e[4];
  load4<T>(x0_row<T>(p, row) + c, e);
#pragma unroll
  for (int j = 0; j < 4; ++j) e[j] *= p.embed_scale;
  store4<T>(d + p.split_off, e);
}

template <typename T, int CH, int NB, int THREADS, int CTAS>
__global__ void __launch_bounds__(THREADS, CTAS) branch_norm_kernel(const BranchNormParams p) {
  __shared__ float s_red[32];
  __shared__ float2 s_red2[32];
  __shared__ ChosenRow s_chosen[2][kMaxTop];   // of this row and of the CTA's next one
  pdl_launch_dependents();
  pdl_wait();
  const int N = p.N;
  const float inv_n = 1.f / static_cast<float>(N);
  const bool e_plain = p.e_rows != nullptr && !experts_are_branch(p);
  if (p.e_rows != nullptr) {
    chosen_rows(p, blockIdx.x, s_chosen[0]);
    __syncthreads();
  }
  int parity = 0;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x, parity ^= 1) {
    float* xr = p.x + static_cast<long long>(row) * N;
    if (p.clear != nullptr) {
      float* z = p.clear + static_cast<long long>(row) * p.clear_ld;
      for (int c = threadIdx.x * 4; c < p.clear_n; c += blockDim.x * 4)
        *reinterpret_cast<float4*>(z + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int dst = p.row_map != nullptr ? p.row_map[row] : row;
    float x[CH][4];
    if (p.tokens != nullptr) {
      const int tok = p.tokens[row];
      const bool ok = tok >= 0 && tok < p.vocab;
      if (!ok && threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
      const T* er = static_cast<const T*>(p.embed) + static_cast<long long>(ok ? tok : 0) * N;
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) x[k][j] = 0.f;
        if (c < N) {
          load4<T>(er + c, x[k]);
#pragma unroll
          for (int j = 0; j < 4; ++j) x[k][j] *= p.embed_scale;
        }
      }
      for (int b = 0; b < NB; ++b)
        if (b < p.n_branches && p.clear_y[b])
          for (int c = threadIdx.x * 4; c < N; c += blockDim.x * 4)
            *reinterpret_cast<float4*>(p.y[b] + static_cast<long long>(row) * p.ldy + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    } else {
      float y[NB][CH][4];
      float ss[NB] = {};
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) x[k][j] = 0.f;
        if (c < N) {
          if (p.base != nullptr) load4<float>(p.base + c, x[k]);
          else load4_stream(xr + c, x[k]);
          if (e_plain) expert_sum4<T>(p, s_chosen[parity], c, x[k]);
        }
#pragma unroll
        for (int b = 0; b < NB; ++b) {
#pragma unroll
          for (int j = 0; j < 4; ++j) y[b][k][j] = 0.f;
          if (b < p.n_branches && c < N) {
            if (p.y[b] != nullptr) load4_stream(p.y[b] + static_cast<long long>(row) * p.ldy + c, y[b][k]);
            else expert_sum4<T>(p, s_chosen[parity], c, y[b][k]);
#pragma unroll
            for (int j = 0; j < 4; ++j) ss[b] = fmaf(y[b][k][j], y[b][k][j], ss[b]);
          }
        }
      }
      // (the barriers of the sums and of the norm below publish the next row's table)
      if (p.e_rows != nullptr && row + gridDim.x < p.rows) chosen_rows(p, row + gridDim.x, s_chosen[parity ^ 1]);
      const float2 tot = block_sum2(make_float2(ss[0], NB > 1 ? ss[NB - 1] : 0.f), s_red2);
      const float r[2] = {1.f / sqrtf(tot.x * inv_n + p.eps), 1.f / sqrtf(tot.y * inv_n + p.eps)};
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * 4;
        if (c >= N) continue;
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int b = 0; b < NB; ++b)
          if (b < p.n_branches) {
            float w[4] = {1.f, 1.f, 1.f, 1.f};
            if (p.w[b] != nullptr) load4<float>(p.w[b] + c, w);
            const float g = p.gain[b] * (p.w[b] != nullptr ? r[b] : 1.f);
#pragma unroll
            for (int j = 0; j < 4; ++j) a[j] = fmaf(g * w[j], y[b][k][j], a[j]);
            if (p.clear_y[b])
              *reinterpret_cast<float4*>(p.y[b] + static_cast<long long>(row) * p.ldy + c) = make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
        for (int j = 0; j < 4; ++j) x[k][j] += a[j];
      }
    }
    float ssq = 0.f;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
      const int c = (k * blockDim.x + threadIdx.x) * 4;
      if (c >= N) continue;
      if (p.store_x) store4<float>(xr + c, x[k]);
#pragma unroll
      for (int j = 0; j < 4; ++j) ssq = fmaf(x[k][j], x[k][j], ssq);
    }
    if (p.split != nullptr) {
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * 4;
        if (c < N) split_row4<T>(p, row, c, x[k]);
      }
      continue;
    }
    if (dst < 0) continue;  // a row without outputs; the same for every thread of the CTA
    const float r = 1.f / sqrtf(block_sum_all(ssq, s_red) * inv_n + p.eps);
#pragma unroll
    for (int o = 0; o < 2; ++o) {
      if (o >= p.n_out) break;
      T* hr = static_cast<T*>(p.h[o]) + static_cast<long long>(dst) * p.ldh;
#pragma unroll
      for (int k = 0; k < CH; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * 4;
        if (c >= N) continue;
        float w[4], v[4];
        load4<float>(p.norm_w[o] + c, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = x[k][j] * r * (w[j] + p.w_offset);
        store4<T>(hr + c, v);
      }
    }
  }
}

// Any row length; the row waits in shared memory.
template <typename T>
__global__ void __launch_bounds__(256) branch_norm_any_kernel(const BranchNormParams p) {
  extern __shared__ float s_u[];  // N values of the row
  __shared__ float s_red[32];
  __shared__ float2 s_red2[32];
  __shared__ ChosenRow s_e[kMaxTop];
  pdl_launch_dependents();
  pdl_wait();
  const int N = p.N;
  const float inv_n = 1.f / static_cast<float>(N);
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    float* xr = p.x + static_cast<long long>(row) * N;
    if (p.e_rows != nullptr) {
      __syncthreads();
      chosen_rows(p, row, s_e);
    }
    if (p.clear != nullptr)
      for (int c = threadIdx.x; c < p.clear_n; c += blockDim.x) p.clear[static_cast<long long>(row) * p.clear_ld + c] = 0.f;
    const int dst = p.row_map != nullptr ? p.row_map[row] : row;
    if (p.e_rows != nullptr) __syncthreads();
    const bool e_plain = p.e_rows != nullptr && !experts_are_branch(p);
    auto branch = [&](int b, int c) {
      return p.y[b] != nullptr ? p.y[b][static_cast<long long>(row) * p.ldy + c] : expert_sum<T>(p, s_e, c);
    };
    const T* er = nullptr;
    float r[kMaxBranches] = {};
    if (p.tokens != nullptr) {
      const int tok = p.tokens[row];
      const bool ok = tok >= 0 && tok < p.vocab;
      if (!ok && threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
      er = static_cast<const T*>(p.embed) + static_cast<long long>(ok ? tok : 0) * N;
    } else {
      float ss[kMaxBranches] = {};
      for (int c = threadIdx.x; c < N; c += blockDim.x)
#pragma unroll
        for (int b = 0; b < kMaxBranches; ++b)
          if (b < p.n_branches) {
            const float y = branch(b, c);
            ss[b] = fmaf(y, y, ss[b]);
          }
      const float2 tot = block_sum2(make_float2(ss[0], ss[1]), s_red2);
      r[0] = 1.f / sqrtf(tot.x * inv_n + p.eps);
      r[1] = 1.f / sqrtf(tot.y * inv_n + p.eps);
    }
    float ssq = 0.f;
    for (int c = threadIdx.x; c < N; c += blockDim.x) {
      float x;
      if (er != nullptr) {
        x = to_f(er[c]) * p.embed_scale;
      } else {
        x = e_plain ? expert_sum<T>(p, s_e, c) : 0.f;
#pragma unroll
        for (int b = 0; b < kMaxBranches; ++b)
          if (b < p.n_branches) {
            const float y = branch(b, c);
            x = fmaf(p.gain[b] * (p.w[b] != nullptr ? r[b] * p.w[b][c] : 1.f), y, x);
          }
        x += p.base != nullptr ? p.base[c] : xr[c];
      }
#pragma unroll
      for (int b = 0; b < kMaxBranches; ++b)
        if (b < p.n_branches && p.clear_y[b]) p.y[b][static_cast<long long>(row) * p.ldy + c] = 0.f;
      if (p.store_x) xr[c] = x;
      if (p.split != nullptr) {
        T* d = static_cast<T*>(p.split) + static_cast<long long>(row) * p.ld_split + c;
        d[0] = from_f<T>(x);
        if constexpr (sizeof(T) == 2) {
          d += p.split_off;
          d[0] = from_f<T>(x - to_f(from_f<T>(x)));
        }
        d[p.split_off] = from_f<T>(to_f(x0_row<T>(p, row)[c]) * p.embed_scale);
      }
      s_u[c] = x;
      ssq = fmaf(x, x, ssq);
    }
    if (dst < 0 || p.split != nullptr) continue;
    const float rr = 1.f / sqrtf(block_sum_all(ssq, s_red) * inv_n + p.eps);
    for (int o = 0; o < p.n_out; ++o) {
      T* hr = static_cast<T*>(p.h[o]) + static_cast<long long>(dst) * p.ldh;
      for (int c = threadIdx.x; c < N; c += blockDim.x) hr[c] = from_f<T>(s_u[c] * rr * (p.norm_w[o][c] + p.w_offset));
    }
  }
}

template <typename T>
cudaError_t launch_branch(const BranchNormParams& p, cudaStream_t stream) {
  const int cap = 8 * sm_count();
  const dim3 grid(p.rows < cap ? p.rows : cap);
  const bool vec = p.N % 4 == 0 && p.ldy % 4 == 0 && p.ldh % 4 == 0 && p.lde % 4 == 0 && p.ld_split % 4 == 0 && p.split_off % 4 == 0;
  const int quads = (p.N + 3) / 4;
  auto threads = [&](int ch) { return dim3(((quads + ch - 1) / ch + 31) / 32 * 32); };
  if (vec && p.n_branches <= 1 && quads <= 1024) {
    // many rows: four CTAs of an SM in different phases of their rows
    if (p.rows > 2 * sm_count())
      return launch_kernel(branch_norm_kernel<T, 2, 1, 512, 4>, grid, threads(2), 0, stream, true, false, p);
    return launch_kernel(branch_norm_kernel<T, 1, 1, 1024, 1>, grid, threads(1), 0, stream, true, false, p);
  }
  // two branches: one piece per thread, as many warps as the row has (measured against two and four pieces)
  if (vec && quads <= 1024) return launch_kernel(branch_norm_kernel<T, 1, 2, 1024, 1>, grid, threads(1), 0, stream, true, false, p);
  if (vec && quads <= 2048) return launch_kernel(branch_norm_kernel<T, 2, 2, 1024, 1>, grid, threads(2), 0, stream, true, false, p);
  const size_t smem = static_cast<size_t>(p.N) * sizeof(float);
  ensure_dynamic_smem(branch_norm_any_kernel<T>, smem);
  return launch_kernel(branch_norm_any_kernel<T>, grid, dim3(256), smem, stream, true, false, p);
}

}  // namespace

cudaError_t launch_branch_norm(const BranchNormParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  return dtype == 0 ? launch_branch<__nv_bfloat16>(p, stream) : launch_branch<float>(p, stream);
}

cudaError_t launch_stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  if (p.S < 1 || p.S > kMaxStreams) return cudaErrorInvalidValue;
  return dtype == 0 ? launch_t<__nv_bfloat16>(p, stream) : launch_t<float>(p, stream);
}

}  // namespace oxb
