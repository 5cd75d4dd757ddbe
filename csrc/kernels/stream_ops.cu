// Residual streams between the sublayers of a layer-list decoder (sm_100a): the hyper-connection update of
// the sublayer that just ran, the read-out for the next one and its RMS norm in one pass over the row,
// with the embedding gather (and its hashed bigram row) folded into the first of them. Streams stay fp32.
// With one stream, mix = in = out = 1 it is residual-add + RMSNorm.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

// One CTA per row (looping). V = 4: rows of whole 16-byte pieces, V = 1: any width. S: largest stream count
// of this instantiation.
template <typename T, int S, int V>
__global__ void __launch_bounds__(1024) stream_norm_kernel(const StreamNormParams p) {
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
    for (int c = threadIdx.x * V; c < N; c += blockDim.x * V) {
      float x[S][V];
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
          for (int j = 0; j < V; ++j) x[s][j] = e[j];
      } else {
#pragma unroll
        for (int s = 0; s < S; ++s) {
          if (s < n_s) {
            if constexpr (V == 4) load4<float>(xr + static_cast<long long>(s) * N + c, x[s]);
            else x[s][0] = xr[static_cast<long long>(s) * N + c];
          }
        }
      }
      float u[V];
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = 0.f;
      if (p.y != nullptr) {
        float y[V];
        float* yp = p.y + static_cast<long long>(row) * p.ldy + c;
        if constexpr (V == 4) {
          load4<float>(yp, y);
          if (p.zero_y) *reinterpret_cast<float4*>(yp) = make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
          y[0] = *yp;
          if (p.zero_y) *yp = 0.f;
        }
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (t < n_s) {
            float z[V];
#pragma unroll
            for (int j = 0; j < V; ++j) z[j] = s_out[t] * y[j];
#pragma unroll
            for (int s = 0; s < S; ++s) {
              if (s < n_s) {
#pragma unroll
                for (int j = 0; j < V; ++j) z[j] = fmaf(s_mix[s * S + t], x[s][j], z[j]);
              }
            }
#pragma unroll
            for (int j = 0; j < V; ++j) u[j] = fmaf(s_in[t], z[j], u[j]);
            if (p.store_x) {
              if constexpr (V == 4) store4<float>(xr + static_cast<long long>(t) * N + c, z);
              else xr[static_cast<long long>(t) * N + c] = z[0];
            }
          }
        }
      } else {
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (t < n_s) {
#pragma unroll
            for (int j = 0; j < V; ++j) u[j] = fmaf(s_in[t], x[t][j], u[j]);
            if (p.store_x) {
              if constexpr (V == 4) store4<float>(xr + static_cast<long long>(t) * N + c, x[t]);
              else xr[static_cast<long long>(t) * N + c] = x[t][0];
            }
          }
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) {
        s_u[c + j] = u[j];
        ssq = fmaf(u[j], u[j], ssq);
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
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = s_u[c + j] * r * (w[j] + p.w_offset);
        store4<T>(hr + c, o);
      } else {
        hr[c] = from_f<T>(s_u[c] * r * (p.norm_w[c] + p.w_offset));
      }
    }
  }
}

template <typename T, int S>
cudaError_t launch_s(const StreamNormParams& p, cudaStream_t stream) {
  constexpr int VW = S <= 8 ? 4 : 1;  // 16 streams x 4 values would spill
  const bool vec = VW == 4 && p.N % 4 == 0 && p.ldy % 4 == 0 && p.ldh % 4 == 0;
  const int v = vec ? 4 : 1;
  int threads = (p.N / v + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 1024 ? 1024 : threads);
  // many rows: smaller CTAs, so that several rows per SM are in flight
  if (p.rows > 2 * sm_count() && threads > 256) threads = 256;
  const int per_sm = 2048 / threads;
  const int cap = sm_count() * per_sm;
  const int grid = p.rows < cap ? p.rows : cap;
  const size_t smem = static_cast<size_t>(p.N) * sizeof(float);
  auto kern = vec ? stream_norm_kernel<T, S, VW> : stream_norm_kernel<T, S, 1>;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(grid), dim3(threads), smem, stream, /*pdl=*/true, false, p);
}

template <typename T>
cudaError_t launch_t(const StreamNormParams& p, cudaStream_t stream) {
  if (p.S == 1) return launch_s<T, 1>(p, stream);
  if (p.S == 2) return launch_s<T, 2>(p, stream);
  if (p.S <= 4) return launch_s<T, 4>(p, stream);
  if (p.S <= 8) return launch_s<T, 8>(p, stream);
  return launch_s<T, kMaxStreams>(p, stream);
}

}  // namespace

cudaError_t launch_stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  if (p.S < 1 || p.S > kMaxStreams) return cudaErrorInvalidValue;
  return dtype == 0 ? launch_t<__nv_bfloat16>(p, stream) : launch_t<float>(p, stream);
}

}  // namespace oxb
