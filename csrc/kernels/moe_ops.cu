// Mixture of experts around the grouped GEMM (sm_100a): router (softmax over all experts with weights divided by their
// sum, or sigmoid scores; best groups of experts first where experts form groups), placement of the chosen rows, and expert products of a handful of rows.
//
// Three ways from the normed rows to expert rows:
//   a step of a few rows (and the 32-bit path): every (row, choice) pair is a row of its own, `moe_rows` streams the
//     chosen expert's matrix once per pair;
//   up to 128 rows: one launch routes and copies each row into its experts' 128-row slabs;
//   more rows: ranks inside the experts first (counted per CTA in shared memory, one global atomic per expert and
//     CTA), then rows packed expert after expert in whole 128-row tiles, so the buffer is as long as the work.
// Router logits are fp32 sums of exact products (weights and rows of the storage type).
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

constexpr int kSlab = 128;   // rows of a slab = rows of a GEMM tile

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// Takes the experts of all but the best groups out of the choice (logit -inf).
template <int R>
__device__ __forceinline__ void keep_groups(float (&l)[R], int E, int groups, int keep, int lane) {
  const int size = E / groups;
  float mine = -INFINITY;   // lane g: score of group g
  for (int g = 0; g < groups; ++g) {
    float a = -INFINITY, b = -INFINITY;   // largest and second largest logit of the group
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int e = lane + 32 * i;
      if (e >= g * size && e < (g + 1) * size) {
        b = fmaxf(b, fminf(a, l[i]));
        a = fmaxf(a, l[i]);
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
      b = fmaxf(fmaxf(b, ob), fminf(a, oa));
      a = fmaxf(a, oa);
    }
    if (lane == g) mine = sigmoid_f(a) + (size > 1 ? sigmoid_f(b) : 0.f);
  }
  unsigned kept = 0;
  for (int c = 0; c < keep; ++c) {
    float best = mine;
    int at = lane;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) {
        best = ob;
        at = oa;
      }
    }
    kept |= 1u << at;
    if (lane == at) mine = -INFINITY;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int e = lane + 32 * i;
    if (e < E && ((kept >> (e / size)) & 1u) == 0) l[i] = -INFINITY;
  }
}

// Chosen experts of one row: logits of expert e in l[e / 32] of lane e % 32. Lane c < top gets choice c and its weight.
template <int R>
__device__ __forceinline__ void choose(float (&l)[R], const MoeRouteParams& p, int lane, int* expert, float* weight) {
  const int E = p.E, top = p.top;
  if (p.groups > 0) keep_groups<R>(l, E, p.groups, p.keep, lane);
  float m = -INFINITY;
#pragma unroll
  for (int i = 0; i < R; ++i) m = fmaxf(m, l[i]);
  m = warp_max(m);
  float z = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i)
    if (lane + 32 * i < E) z += expf(l[i] - m);
  z = warp_sum(z);
  int my_e = 0;
  float my_s = 0.f;
  for (int c = 0; c < top; ++c) {
    float best = -INFINITY;
    int at = 1 << 30;
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (l[i] > best) {
        best = l[i];
        at = lane + 32 * i;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) {
        best = ob;
        at = oa;
      }
    }
    if (at >= E) at = 0;  // not reached with finite logits
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (lane + 32 * i == at) l[i] = -INFINITY;
    if (lane == c) {
      my_e = at;
      my_s = p.softmax ? expf(best - m) / z : sigmoid_f(best);
    }
  }
  if (!p.softmax) {
    *expert = my_e;
    *weight = my_s;
    return;
  }
  const float sum = warp_sum(my_s);
  *expert = my_e;
  *weight = my_s / (sum + 1e-20f);
}

template <typename T>
struct Pack;   // 16 bytes of a row
template <>
struct Pack<__nv_bfloat16> {
  static constexpr int n = 8;
  static __device__ __forceinline__ void get(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
};
template <>
struct Pack<float> {
  static constexpr int n = 4;
  static __device__ __forceinline__ void get(const float* p, float (&v)[4]) { load4<float>(p, v); }
};

// One CTA per row: logits (unless given), choice, slot, and the row's copies (mode 1).
constexpr int kRouteThreads = 1024, kRouteWarps = kRouteThreads / 32;
template <typename T, int R>
__global__ void __launch_bounds__(kRouteThreads) moe_route_row_kernel(const MoeRouteParams p) {
  extern __shared__ float s_h[];   // N values of the row
  __shared__ float s_l[R * 32];
  __shared__ float s_part[kRouteWarps][2];
  __shared__ int s_slot[kMaxTop];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* hr = static_cast<const T*>(p.h) + static_cast<long long>(row) * p.ldh;
  constexpr int W = Pack<T>::n;
  if (p.logits == nullptr) {
    for (int c = threadIdx.x * W; c < p.N; c += kRouteThreads * W) {
      float v[W];
      Pack<T>::get(hr + c, v);
#pragma unroll
      for (int j = 0; j < W; ++j) s_h[c + j] = v[j];
    }
    __syncthreads();
    // two experts per warp; where warps are left over, several share the two experts and split the row
    const int pairs = (p.E + 1) / 2;
    const int ks = pairs >= kRouteWarps ? 1 : kRouteWarps / pairs;
    for (int q0 = 0; q0 < pairs; q0 += kRouteWarps) {
      const int q = ks == 1 ? q0 + warp : warp / ks, part = ks == 1 ? 0 : warp % ks;
      float a0 = 0.f, a1 = 0.f;
      if (q < pairs) {
        const T* w0 = static_cast<const T*>(p.router) + static_cast<long long>(2 * q) * p.ldr;
        const T* w1 = 2 * q + 1 < p.E ? w0 + p.ldr : w0;
#pragma unroll 4
        for (int c = (part * 32 + lane) * W; c < p.N; c += ks * 32 * W) {
          float u[W], v[W];
          Pack<T>::get(w0 + c, u);
          Pack<T>::get(w1 + c, v);
#pragma unroll
          for (int j = 0; j < W; ++j) {
            a0 = fmaf(u[j], s_h[c + j], a0);
            a1 = fmaf(v[j], s_h[c + j], a1);
          }
        }
      }
      a0 = warp_sum(a0);
      a1 = warp_sum(a1);
      if (ks == 1) {
        if (lane == 0 && q < pairs) {
          s_l[2 * q] = a0;
          if (2 * q + 1 < p.E) s_l[2 * q + 1] = a1;
        }
      } else {
        if (lane == 0) {
          s_part[warp][0] = a0;
          s_part[warp][1] = a1;
        }
        __syncthreads();
        for (int e = threadIdx.x; e < p.E; e += kRouteThreads) {
          float t = 0.f;
          for (int k = 0; k < ks; ++k) t += s_part[(e >> 1) * ks + k][e & 1];
          s_l[e] = t;
        }
      }
    }
  } else {
    for (int e = threadIdx.x; e < p.E; e += kRouteThreads) s_l[e] = p.logits[static_cast<long long>(row) * p.ldl + e];
  }
  __syncthreads();
  if (warp == 0) {
    float l[R];
#pragma unroll
    for (int i = 0; i < R; ++i) l[i] = lane + 32 * i < p.E ? s_l[lane + 32 * i] : -INFINITY;
    int e;
    float w;
    choose<R>(l, p, lane, &e, &w);
    if (lane < p.top) {
      const int i = row * p.top + lane;
      int slot = i;
      if (p.mode == 1) {
        const unsigned rank = atomicAdd(p.counts + e, 1u);
        slot = rank < kSlab ? e * kSlab + static_cast<int>(rank) : -1;
        if (slot < 0) set_status_once(p.status, kStatusBadIndex);
      }
      p.expert[i] = e;
      p.weight[i] = w;
      p.slot[i] = slot;
      s_slot[lane] = slot;
    }
  }
  if (p.mode != 1) return;
  __syncthreads();
  for (int c = 0; c < p.top; ++c) {
    const int slot = s_slot[c];
    if (slot < 0) continue;
    T* dst = static_cast<T*>(p.xs) + static_cast<long long>(slot) * p.ldx;
    for (int k = threadIdx.x * W; k < p.N; k += kRouteThreads * W)
      *reinterpret_cast<uint4*>(dst + k) = *reinterpret_cast<const uint4*>(hr + k);
  }
}

// Many rows, logits given: kRows rows per CTA, one warp per row; ranks inside the experts.
constexpr int kRouteRows = 64;
template <int R>
__global__ void __launch_bounds__(256) moe_route_rank_kernel(const MoeRouteParams p) {
  __shared__ unsigned s_cnt[R * 32], s_base[R * 32];
  pdl_launch_dependents();
  for (int e = threadIdx.x; e < p.E; e += 256) s_cnt[e] = 0;
  __syncthreads();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int e[kRouteRows / 8];
  unsigned rank[kRouteRows / 8];
#pragma unroll
  for (int i = 0; i < kRouteRows / 8; ++i) {
    const int row = blockIdx.x * kRouteRows + i * 8 + warp;
    e[i] = -1;
    if (row >= p.M) continue;
    float l[R];
#pragma unroll
    for (int k = 0; k < R; ++k) l[k] = lane + 32 * k < p.E ? p.logits[static_cast<long long>(row) * p.ldl + lane + 32 * k] : -INFINITY;
    float w;
    int ex;
    choose<R>(l, p, lane, &ex, &w);
    if (lane < p.top) {
      e[i] = ex;
      rank[i] = atomicAdd(&s_cnt[ex], 1u);
      p.expert[row * p.top + lane] = ex;
      p.weight[row * p.top + lane] = w;
    }
  }
  __syncthreads();
  for (int x = threadIdx.x; x < p.E; x += 256) s_base[x] = s_cnt[x] > 0 ? atomicAdd(p.counts + x, s_cnt[x]) : 0u;
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kRouteRows / 8; ++i)
    if (e[i] >= 0) p.slot[(blockIdx.x * kRouteRows + i * 8 + warp) * p.top + lane] = static_cast<int>(s_base[e[i]] + rank[i]);
}

__global__ void __launch_bounds__(256) moe_scatter_kernel(const MoeScatterParams p) {
  __shared__ int s_start[kMaxExperts];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    int acc = 0;
    for (int e0 = 0; e0 < p.E; e0 += 32) {
      const int e = e0 + lane;
      const int tiles = e < p.E ? (static_cast<int>(__ldcg(p.counts + e)) + kSlab - 1) / kSlab : 0;
      int incl = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += up;
      }
      if (e < p.E) s_start[e] = (acc + incl - tiles) * kSlab;
      acc += __shfl_sync(0xffffffffu, incl, 31);
    }
  }
  __syncthreads();
  // one warp per row: its values once, then a copy per choice
  for (int row = blockIdx.x * 8 + warp; row < p.M; row += gridDim.x * 8) {
    int slot = -1;
    if (lane < p.top) {
      const int i = row * p.top + lane;
      slot = s_start[p.expert[i]] + p.slot[i];
      if (slot >= p.max_rows) {
        set_status_once(p.status, kStatusBadIndex);
        slot = -1;
      }
      p.slot[i] = slot;
    }
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.h) + static_cast<long long>(row) * p.ldh;
    for (int k0 = 0; k0 < p.N; k0 += 32 * 8 * 4) {
      uint4 v[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int k = k0 + (u * 32 + lane) * 8;
        if (k < p.N) v[u] = *reinterpret_cast<const uint4*>(src + k);
      }
      for (int c = 0; c < p.top; ++c) {
        const int s = __shfl_sync(0xffffffffu, slot, c);
        if (s < 0) continue;
        __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.xs) + static_cast<long long>(s) * p.ldx;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int k = k0 + (u * 32 + lane) * 8;
          if (k < p.N) *reinterpret_cast<uint4*>(dst + k) = v[u];
        }
      }
    }
  }
}

// grid (pairs, N / 16): 8 warps of two rows of W each, which are two outputs or the gate and up row of one.
template <typename T>
__global__ void __launch_bounds__(256) moe_rows_kernel(const MoeRowsParams p) {
  pdl_wait();
  const int pair = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n2 = (blockIdx.y * 8 + warp) * 2;
  if (n2 >= p.N) return;
  const bool glu = p.act == 3;
  const int n0 = glu ? (n2 >> 6) * 64 + ((n2 >> 1) & 31) : n2;
  const int e = p.expert[pair];
  if (static_cast<unsigned>(e) >= static_cast<unsigned>(p.E)) return;
  const T* x = static_cast<const T*>(p.x) + static_cast<long long>(p.per_pair ? pair : pair / p.top) * p.ldx;
  const int n1 = glu ? n0 + 32 : (n0 + 1 < p.N ? n0 + 1 : n0);
  const T* w0 = static_cast<const T*>(p.w) + (static_cast<long long>(e) * p.N + n0) * p.K;
  const T* w1 = static_cast<const T*>(p.w) + (static_cast<long long>(e) * p.N + n1) * p.K;
  constexpr int W = Pack<T>::n;
  float a0 = 0.f, a1 = 0.f;
#pragma unroll 4
  for (int k = lane * W; k < p.K; k += 32 * W) {
    float xv[W], u[W], v[W];
    Pack<T>::get(w0 + k, u);
    Pack<T>::get(w1 + k, v);
    Pack<T>::get(x + k, xv);
#pragma unroll
    for (int j = 0; j < W; ++j) {
      a0 = fmaf(u[j], xv[j], a0);
      a1 = fmaf(v[j], xv[j], a1);
    }
  }
  pdl_launch_dependents();
  a0 = warp_sum(a0);
  a1 = warp_sum(a1);
  if (p.act == 2) {
    a0 = fmaxf(a0, 0.f) * fmaxf(a0, 0.f);
    a1 = fmaxf(a1, 0.f) * fmaxf(a1, 0.f);
  }
  if (lane == 0) {
    T* y = static_cast<T*>(p.y) + static_cast<long long>(pair) * p.ldy + (glu ? n2 >> 1 : n0);
    if (glu) {
      y[0] = from_f<T>(silu_f(a0) * a1);
      return;
    }
    y[0] = from_f<T>(a0);
    if (n1 != n0) y[1] = from_f<T>(a1);
  }
}

template <typename T, int R>
cudaError_t launch_route(const MoeRouteParams& p, cudaStream_t stream) {
  if (p.mode == 2)
    return launch_kernel(moe_route_rank_kernel<R>, dim3((p.M + kRouteRows - 1) / kRouteRows), dim3(256), 0, stream, true, false, p);
  const size_t smem = p.logits == nullptr ? static_cast<size_t>(p.N) * sizeof(float) : 0;
  ensure_dynamic_smem(moe_route_row_kernel<T, R>, smem);
  return launch_kernel(moe_route_row_kernel<T, R>, dim3(p.M), dim3(kRouteThreads), smem, stream, true, false, p);
}

template <typename T>
cudaError_t route_of(const MoeRouteParams& p, cudaStream_t stream) {
  if (p.E <= 64) return launch_route<T, 2>(p, stream);
  if (p.E <= 128) return launch_route<T, 4>(p, stream);
  if (p.E <= 256) return launch_route<T, 8>(p, stream);
  return launch_route<T, kMaxExperts / 32>(p, stream);
}

}  // namespace

cudaError_t launch_moe_route(const MoeRouteParams& p, int dtype, cudaStream_t stream) {
  if (p.M <= 0) return cudaSuccess;
  if (p.E > kMaxExperts || p.top > kMaxTop || p.top > p.E) return cudaErrorInvalidValue;
  if (p.groups > kMaxGroups || (p.groups > 0 && (p.E % p.groups != 0 || p.keep < 1 || p.keep > p.groups))) return cudaErrorInvalidValue;
  return dtype == 0 ? route_of<__nv_bfloat16>(p, stream) : route_of<float>(p, stream);
}

cudaError_t launch_moe_scatter(const MoeScatterParams& p, cudaStream_t stream) {
  if (p.M <= 0) return cudaSuccess;
  if (p.E > kMaxExperts || p.top > kMaxTop) return cudaErrorInvalidValue;
  const int want = (p.M + 7) / 8, cap = 8 * sm_count();
  return launch_kernel(moe_scatter_kernel, dim3(want < cap ? want : cap), dim3(256), 0, stream, true, false, p);
}

cudaError_t launch_moe_rows(const MoeRowsParams& p, int dtype, cudaStream_t stream) {
  if (p.pairs <= 0 || p.N <= 0) return cudaSuccess;
  const dim3 grid(p.pairs, (p.N + 15) / 16);
  return dtype == 0 ? launch_kernel(moe_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, true, false, p)
                    : launch_kernel(moe_rows_kernel<float>, grid, dim3(256), 0, stream, true, false, p);
}

}  // namespace oxb
