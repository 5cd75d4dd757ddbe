// Residual streams between the sublayers of a layer-list decoder (sm_100a): the hyper-connection update of
// the sublayer that just ran, the read-out for the next one and its RMS norm in one pass over the row,
// with the embedding gather (and its hashed bigram row) folded into the first of them. Streams stay fp32.
// With one stream, mix = in = out = 1 it is residual-add + RMSNorm.
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

}  // namespace

cudaError_t launch_stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  if (p.S < 1 || p.S > kMaxStreams) return cudaErrorInvalidValue;
  return dtype == 0 ? launch_t<__nv_bfloat16>(p, stream) : launch_t<float>(p, stream);
}

}  // namespace oxb
