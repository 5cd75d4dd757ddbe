// Projections -> heads (sm_100a): bias, RMS norm over the whole q / k projection, rotation in either pair layout
// on the first dimensions of every head, write of k and v into the paged cache (or of q and k to dense
// fp32 buffers for a recurrence); the difference of the two maps of differential attention with its norm; plus plain
// fp32 pieces of the 32-bit path (GEMM, gated unit).
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

// grid (rows, head ranges): a range of the H + G (+ G value) heads per CTA. The norm spans heads of other
// CTAs: each CTA re-reads the row's q / k (a few KB from L2) for the sum of squares it needs.
// This thread's share of the sum of squares of n values
template <typename P>
__device__ __forceinline__ float row_ssq(const P* v, int n, long long ld) {
  float ss = 0.f;
  if ((n & 3) == 0 && (ld & 3) == 0 && (reinterpret_cast<uintptr_t>(v) & 15) == 0) {
    for (int c = threadIdx.x * 4; c < n; c += blockDim.x * 4) {
      float x[4];
      load4<P>(v + c, x);
      ss = fmaf(x[0], x[0], fmaf(x[1], x[1], fmaf(x[2], x[2], fmaf(x[3], x[3], ss))));
    }
  } else {
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float x = to_f(v[c]);
      ss = fmaf(x, x, ss);
    }
  }
  return ss;
}

// T: storage type (cache, dense q of the attention), TQ: type of q_out, P: type of the projection rows.
// VEC: every size and pitch is a multiple of 4, values move four at a time.
template <typename T, typename TQ, typename P, bool VEC>
__global__ void __launch_bounds__(256) heads_kernel(const HeadsParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_red[32];
  pdl_launch_dependents();
  const int rot2 = p.rot.dims >> 1;
  float* s_sin = s_mem;
  float* s_cos = s_mem + rot2;
  pdl_wait();  // the projection comes from the kernel before this one
  const int row = blockIdx.x;
  const int H = p.H, G = p.G, D = p.D, E = p.E;
  const int GV = G / p.maps;   // value heads = rows of a cache block
  const int n_heads = H + G + (p.v_cache != nullptr ? GV : 0);
  const int hpc = (n_heads + gridDim.y - 1) / gridDim.y;
  const int h_lo = blockIdx.y * hpc;
  const int h_hi = min(h_lo + hpc, n_heads);
  if (h_lo >= h_hi) return;
  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld;
  const int pos = p.positions[row];
  if (h_lo < H + G)
    for (int i = threadIdx.x; i < rot2; i += blockDim.x) rotary_sincos(p.rot, i, pos, &s_sin[i], &s_cos[i]);
  float rq = 1.f, rk = 1.f;
  if (p.q_norm != nullptr) {
    const bool need_k = h_lo < H + G && h_hi > H;
    const float sq = h_lo < H ? row_ssq(pr, H * D, p.ld) : 0.f;
    const float sk = need_k ? row_ssq(pr + H * D, G * D, p.ld) : 0.f;
    if (h_lo < H) rq = 1.f / sqrtf(block_sum_all(sq, s_red) / static_cast<float>(H * D) + p.eps);
    if (need_k) rk = 1.f / sqrtf(block_sum_all(sk, s_red) / static_cast<float>(G * D) + p.eps);
  }
  const float rw = p.k_norm != nullptr ? rk : 1.f;   // what the stored keys are multiplied by
  const float qt = p.t_coef != 0.f ? 1.f + p.t_coef * logf(floorf(static_cast<float>(pos + 1) / p.t_every) + 1.f) : 1.f;
  const long long k_col = p.q_pd * H;   // k follows q in the projection row
  __syncthreads();
  const long long slot = p.slots != nullptr ? p.slots[row] : -1;
  const bool store_kv = slot >= 0 && slot < p.num_slots;
  if (p.slots != nullptr && slot >= p.num_slots && threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
  const long long blk = slot >> 4;
  const int off = static_cast<int>(slot & 15);
  if (p.k_rms != nullptr && store_kv && h_lo <= H && H < h_hi && threadIdx.x == 0) p.k_rms[slot] = rk;

  if constexpr (VEC) {
    // four values (two pairs of the interleaved layout) or two times four (the other) per item, items of all
    // heads of this CTA dealt out over its threads
    const int r_end = min(h_hi, H + G);
    const int rq4 = p.rot.interleaved ? (2 * rot2) >> 2 : rot2 >> 2;   // rotated items of a head
    const int per = rq4 + ((D - 2 * rot2) >> 2);
    for (int i = threadIdx.x; i < (r_end - h_lo) * per; i += blockDim.x) {
      const int lh = i / per, it = i - lh * per, h = h_lo + lh;
      const bool is_q = h < H;
      if (!is_q && p.k_out == nullptr && !store_kv) continue;
      const long long col = is_q ? h * p.q_pd : k_col + (h - H) * D;
      const P* src = pr + col;
      const float r = is_q ? rq : rw, ks = is_q ? qt : p.k_scale;
      const float* w = is_q ? p.q_norm : p.k_norm;
      if (w != nullptr) w += (is_q ? h : h - H) * D;
      auto get = [&](int d, float (&v)[4]) {
        load4<P>(src + d, v);
        if (p.bias != nullptr) {
          float b4[4];
          load4<float>(p.bias + col + d, b4);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] += b4[j];
        }
        if (w != nullptr) {
          float g4[4];
          load4<float>(w + d, g4);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] *= r * g4[j];
        }
      };
      auto put = [&](int d, float (&v)[4]) {
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] *= ks;
        if (is_q) {
          store4<TQ>(static_cast<TQ*>(p.q_out) + static_cast<long long>(row) * p.q_ld + h * p.q_hd + (h % p.maps) * D + d, v);
          return;
        }
        const int g = h - H;
        if (p.k_out != nullptr) store4<float>(p.k_out + static_cast<long long>(row) * p.k_ld + g * p.k_hd + d, v);
        else store4<T>(static_cast<T*>(p.k_cache) + ((blk * GV + g / p.maps) * 16 + off) * p.DP + (g % p.maps) * D + d, v);
      };
      float x[4];
      if (it >= rq4) {
        const int d = 2 * rot2 + (it - rq4) * 4;
        get(d, x);
        put(d, x);
      } else if (p.rot.interleaved) {
        const int f = it * 2;
        get(it * 4, x);
        float y[4] = {x[0] * s_cos[f] - x[1] * s_sin[f], x[1] * s_cos[f] + x[0] * s_sin[f],
                      x[2] * s_cos[f + 1] - x[3] * s_sin[f + 1], x[3] * s_cos[f + 1] + x[2] * s_sin[f + 1]};
        put(it * 4, y);
      } else {
        const int f = it * 4;
        float z[4], y0[4], y1[4];
        get(f, x);
        get(f + rot2, z);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          y0[j] = x[j] * s_cos[f + j] - z[j] * s_sin[f + j];
          y1[j] = z[j] * s_cos[f + j] + x[j] * s_sin[f + j];
        }
        put(f, y0);
        put(f + rot2, y1);
      }
    }
    if (store_kv && h_hi > H + G) {
      const int v_lo = max(h_lo, H + G), e4 = E >> 2;
      const long long v_col = k_col + G * D;
      for (int i = threadIdx.x; i < (h_hi - v_lo) * e4; i += blockDim.x) {
        const int lh = i / e4, e = (i - lh * e4) * 4, g = v_lo + lh - H - G;
        float x[4];
        load4<P>(pr + v_col + g * E + e, x);
        if (p.bias != nullptr) {
          float b4[4];
          load4<float>(p.bias + v_col + g * E + e, b4);
#pragma unroll
          for (int j = 0; j < 4; ++j) x[j] += b4[j];
        }
        store4<T>(static_cast<T*>(p.v_cache) + ((blk * GV + g) * 16 + off) * p.EP + e, x);
      }
    }
    return;
  }
  // any sizes: one warp per head, a lane takes rotation pairs, then dimensions that pass
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int r_hi = min(h_hi, H + G);
  for (int h = h_lo + warp; h < r_hi; h += nw) {
    const bool is_q = h < H;
    if (!is_q && p.k_out == nullptr && !store_kv) continue;
    const long long col = is_q ? h * p.q_pd : k_col + (h - H) * D;
    const P* src = pr + col;
    const float* bias = p.bias != nullptr ? p.bias + col : nullptr;
    const float r = is_q ? rq : rw;
    const float* w = is_q ? p.q_norm : p.k_norm;
    if (w != nullptr) w += (is_q ? h : h - H) * D;
    const float ks = is_q ? qt : p.k_scale;
    TQ* qd = nullptr;
    float* kd = nullptr;
    T* kc = nullptr;
    if (is_q) qd = static_cast<TQ*>(p.q_out) + static_cast<long long>(row) * p.q_ld + h * p.q_hd + (h % p.maps) * D;
    else if (p.k_out != nullptr) kd = p.k_out + static_cast<long long>(row) * p.k_ld + (h - H) * p.k_hd;
    else kc = static_cast<T*>(p.k_cache) + ((blk * GV + (h - H) / p.maps) * 16 + off) * p.DP + ((h - H) % p.maps) * D;
    auto put = [&](int d, float y) {
      if (qd != nullptr) qd[d] = from_f<TQ>(y * ks);
      else if (kd != nullptr) kd[d] = y * ks;
      else kc[d] = from_f<T>(y * ks);
    };
    for (int it = lane; it < rot2; it += 32) {
      int d0, d1;
      rotary_pair(p.rot, it, &d0, &d1);
      float u = to_f(src[d0]), v = to_f(src[d1]);
      if (bias != nullptr) {
        u += bias[d0];
        v += bias[d1];
      }
      u *= r;
      v *= r;
      if (w != nullptr) {
        u *= w[d0];
        v *= w[d1];
      }
      put(d0, u * s_cos[it] - v * s_sin[it]);
      put(d1, v * s_cos[it] + u * s_sin[it]);
    }
    for (int d = 2 * rot2 + lane; d < D; d += 32) put(d, (to_f(src[d]) + (bias != nullptr ? bias[d] : 0.f)) * r * (w != nullptr ? w[d] : 1.f));
  }
  if (store_kv && h_hi > H + G) {
    for (int h = max(h_lo, H + G) + warp; h < h_hi; h += nw) {
      const int g = h - H - G;
      const long long col = k_col + G * D + g * E;
      T* vc = static_cast<T*>(p.v_cache) + ((blk * GV + g) * 16 + off) * p.EP;
      for (int e = lane; e < E; e += 32) vc[e] = from_f<T>(to_f(pr[col + e]) + (p.bias != nullptr ? p.bias[col + e] : 0.f));
    }
  }
}

// One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) diff_norm_kernel(const DiffNormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(p.M) * p.H) return;
  const long long row = item / p.H;
  const int head = static_cast<int>(item - row * p.H), E = p.E;
  const float* a = p.a + row * p.lda + 2ll * head * E;
  T* out = static_cast<T*>(p.out) + row * p.ldo + static_cast<long long>(head) * E;
  float ss = 0.f;
  if (E % 4 == 0 && p.lda % 4 == 0 && p.ldo % 4 == 0 && E <= 1024) {
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int e = (i * 32 + lane) * 4;
      if (e >= E) break;
      float x[4], y[4];
      load4_stream(a + e, x);
      load4_stream(a + E + e, y);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        o[i][j] = fmaf(-p.lambda, y[j], x[j]);
        ss = fmaf(o[i][j], o[i][j], ss);
      }
    }
    const float r = p.gain / sqrtf(warp_sum(ss) / static_cast<float>(E) + p.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int e = (i * 32 + lane) * 4;
      if (e >= E) break;
#pragma unroll
      for (int j = 0; j < 4; ++j) o[i][j] *= r;
      store4<T>(out + e, o[i]);
    }
    return;
  }
  for (int e = lane; e < E; e += 32) {
    const float o = fmaf(-p.lambda, a[E + e], a[e]);
    ss = fmaf(o, o, ss);
  }
  const float r = p.gain / sqrtf(warp_sum(ss) / static_cast<float>(E) + p.eps);
  for (int e = lane; e < E; e += 32) out[e] = from_f<T>(fmaf(-p.lambda, a[E + e], a[e]) * r);
}

constexpr int kFT = 64, kFK = 16;

// 64 x 64 tiles, 256 threads of 4 x 4 outputs, K in steps of 16.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* a, long long lda, const float* w, long long ldw,
                                                       float* out, long long ldo, int M, int N, int K) {
  __shared__ float sa[kFK][kFT + 4], sw[kFK][kFT + 4];
  pdl_wait();
  const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kFK) {
    for (int i = threadIdx.x; i < kFT * kFK; i += 256) {
      const int r = i / kFK, c = i % kFK;
      const bool kin = k0 + c < K;
      sa[c][r] = (kin && m0 + r < M) ? a[static_cast<long long>(m0 + r) * lda + k0 + c] : 0.f;
      sw[c][r] = (kin && n0 + r < N) ? w[static_cast<long long>(n0 + r) * ldw + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = sa[k][ty * 4 + i];
        y[i] = sw[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N)
        out[static_cast<long long>(m0 + ty * 4 + i) * ldo + n0 + tx * 4 + j] = acc[i][j];
}

// Few rows: one warp per output column, the row values re-read from cache.
constexpr int kFewRows = 8;
__global__ void __launch_bounds__(256) gemv_f32_kernel(const float* a, long long lda, const float* w, long long ldw,
                                                       float* out, long long ldo, int M, int N, int K) {
  pdl_wait();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (n >= N) return;
  float acc[kFewRows] = {};
  for (int k = lane; k < K; k += 32) {
    const float wv = w[static_cast<long long>(n) * ldw + k];
#pragma unroll
    for (int m = 0; m < kFewRows; ++m)
      if (m < M) acc[m] = fmaf(a[static_cast<long long>(m) * lda + k], wv, acc[m]);
  }
#pragma unroll
  for (int m = 0; m < kFewRows; ++m) {
    const float v = warp_sum(acc[m]);
    if (lane == 0 && m < M) out[static_cast<long long>(m) * ldo + n] = v;
  }
}

__global__ void __launch_bounds__(256) glu_f32_kernel(const float* gu, long long ldg, float* out, long long ldo, int M,
                                                      int I, int act) {
  pdl_wait();
  const long long total = static_cast<long long>(M) * I;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const long long m = i / I;
    const int c = static_cast<int>(i - m * I);
    const float g = gu[m * ldg + c];
    if (act == 2) {
      const float r = fmaxf(g, 0.f);
      out[m * ldo + c] = r * r;
      continue;
    }
    const float u = gu[m * ldg + I + c];
    const float a = act == 0 ? silu_f(g)
                             : 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
    out[m * ldo + c] = a * u;
  }
}

}  // namespace

template <bool VEC>
static cudaError_t launch_heads_v(const HeadsParams& p, int dtype, dim3 grid, dim3 block, size_t smem, cudaStream_t stream) {
  using bf16 = __nv_bfloat16;
  auto kern = dtype == 1          ? heads_kernel<float, float, float, VEC>
              : p.k_out != nullptr ? (p.proj_f32 ? heads_kernel<bf16, float, float, VEC> : heads_kernel<bf16, float, bf16, VEC>)
                                   : (p.proj_f32 ? heads_kernel<bf16, bf16, float, VEC> : heads_kernel<bf16, bf16, bf16, VEC>);
  return launch_kernel(kern, grid, block, smem, stream, true, false, p);
}

cudaError_t launch_heads(const HeadsParams& p, int dtype, cudaStream_t stream) {
  if (p.M <= 0) return cudaSuccess;
  const int n_heads = p.H + p.G + (p.v_cache != nullptr ? p.G / p.maps : 0);
  // ranges of at least 4 heads until about two CTAs per SM exist
  int chunks = (2 * sm_count() + p.M - 1) / p.M;
  chunks = chunks > n_heads / 4 ? n_heads / 4 : chunks;
  if (chunks < 1) chunks = 1;
  const size_t smem = static_cast<size_t>(p.rot.dims) * sizeof(float);
  const dim3 grid(p.M, chunks), block(256);
  auto al = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
  const bool vec = p.D % 4 == 0 && p.E % 4 == 0 && p.rot.dims % (p.rot.interleaved ? 4 : 8) == 0 && p.ld % 4 == 0 && p.q_ld % 4 == 0 &&
                   p.q_hd % 4 == 0 && p.q_pd % 4 == 0 && al(p.bias) && p.k_ld % 4 == 0 && p.k_hd % 4 == 0 && p.DP % 4 == 0 && p.EP % 4 == 0 && al(p.proj) &&
                   al(p.q_out) && al(p.k_out) && al(p.q_norm) && al(p.k_norm);
  return vec ? launch_heads_v<true>(p, dtype, grid, block, smem, stream) : launch_heads_v<false>(p, dtype, grid, block, smem, stream);
}

cudaError_t launch_diff_norm(const DiffNormParams& p, int dtype, cudaStream_t stream) {
  const long long items = static_cast<long long>(p.M) * p.H;
  if (items <= 0) return cudaSuccess;
  const dim3 grid(static_cast<unsigned>((items + 7) / 8));
  return dtype == 0 ? launch_kernel(diff_norm_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, true, false, p)
                    : launch_kernel(diff_norm_kernel<float>, grid, dim3(256), 0, stream, true, false, p);
}

cudaError_t launch_gemm_f32(const float* a, long long lda, const float* w, long long ldw, float* out, long long ldo,
                            int M, int N, int K, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return cudaSuccess;
  if (M <= kFewRows)
    return launch_kernel(gemv_f32_kernel, dim3((N + 7) / 8), dim3(256), 0, stream, true, false, a, lda, w, ldw, out,
                         ldo, M, N, K);
  return launch_kernel(gemm_f32_kernel, dim3((N + kFT - 1) / kFT, (M + kFT - 1) / kFT), dim3(256), 0, stream, true,
                       false, a, lda, w, ldw, out, ldo, M, N, K);
}

cudaError_t launch_glu_f32(const float* gu, long long ldg, float* out, long long ldo, int M, int I, int act,
                           cudaStream_t stream) {
  const long long total = static_cast<long long>(M) * I;
  if (total <= 0) return cudaSuccess;
  long long blocks = (total + 255) / 256;
  if (blocks > sm_count() * 16) blocks = sm_count() * 16;
  return launch_kernel(glu_f32_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, stream, true, false, gu, ldg,
                       out, ldo, M, I, act);
}

}  // namespace oxb
