// Retention (linear attention with a fixed decay per head) on sm_100a:
//     S_t = decay S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t,   out_t = o_t / rms(o_t) * silu(gate_t)
//
// Decode: one thread-block cluster per (row, head) streams that head's fp32 state once through the SMs:
//   rotation of q and k, state update, read-out, head norm and gate in one launch. The CTAs of a cluster
//   own column slices of the state and exchange their parts of the norm through distributed shared memory.
// Prompt chunks of 64 rows, three launches, parallel over chunks:
//   1. U_c = sum_j decay^(n-1-j) k_j v_j^T           what chunk c adds to the state
//   2. scan over the chunks of a sequence: replaces U_c by the state before chunk c, stores the final state
//   3. O = ((Q K^T) o decay^(i-j)) V + decay^(i+1) (Q S_before), then head norm and gate
//   q, k, scores, weights and states are fp32: the tensor-core products split every fp32 operand into two
//   TF32 numbers (3xTF32: hi*hi + hi*lo + lo*hi, fp32 accumulation), which keeps about 21 bits; bf16 values
//   are exact in TF32 and need no second term.
// Token-by-token form in fp32 FMAs for the 32-bit path and for head sizes above the chunked form's.
#include <cooperative_groups.h>

#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace cg = cooperative_groups;

namespace oxb {

namespace {

// ------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256;
constexpr int kDecUnroll = 8;

// grid (slices, H, rows), cluster (slices, 1, 1). V columns of the state per thread and access. T: storage
// type, P: type of the projection rows. Values enter the state as the storage type holds them.
template <typename T, typename P, int V>
__global__ void __launch_bounds__(kDecThreads) retention_decode_kernel(const RetentionParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_red[32];
  __shared__ float s_part;
  const int D = p.D, E = p.E;
  const int Es = E / static_cast<int>(gridDim.x);
  float* s_q = s_mem;            // D
  float* s_k = s_q + D;          // D
  float* s_o = s_k + D;          // [lanes][Es]
  const int head = blockIdx.y, row = blockIdx.z, e0 = blockIdx.x * Es;
  pdl_wait();  // the projection comes from the kernel before this one
  const int slot = p.row_slots[row];
  if (slot < 0) return;  // padding row (the whole cluster leaves)
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const int pos = p.positions[row];
  const bool fresh = pos == 0;
  const float gamma = p.decay_pow[head * (kRetChunk + 1) + 1];
  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld;
  const P* qp = pr + head * D;
  const P* kp = pr + (p.H + head) * D;
  const P* vp = pr + 2 * p.H * D + head * E + e0;
  const P* gp = pr + 2 * p.H * D + p.H * E + head * E + e0;
  const int rot2 = p.rot.dims >> 1;
  for (int i = threadIdx.x; i < D - rot2; i += kDecThreads) {
    if (i < rot2) {
      float sn, cs;
      rotary_sincos(p.rot, i, pos, &sn, &cs);
      int u, v;
      rotary_pair(p.rot, i, &u, &v);
      const float qu = to_f(qp[u]), qv = to_f(qp[v]), ku = to_f(kp[u]), kv = to_f(kp[v]);
      s_q[u] = qu * cs - qv * sn;
      s_q[v] = qv * cs + qu * sn;
      s_k[u] = (ku * cs - kv * sn) * p.k_scale;
      s_k[v] = (kv * cs + ku * sn) * p.k_scale;
    } else {
      s_q[rot2 + i] = to_f(qp[rot2 + i]);
      s_k[rot2 + i] = to_f(kp[rot2 + i]) * p.k_scale;
    }
  }
  __syncthreads();
  const int groups = Es / V;
  const int gt = groups < kDecThreads ? groups : kDecThreads;
  const int lanes = kDecThreads / gt;
  const int cgi = threadIdx.x % gt, dl = threadIdx.x / gt;
  float* S = p.state + (static_cast<long long>(slot) * p.H + head) * D * E + e0;
  if (dl < lanes) {
    for (int c = cgi; c < groups; c += gt) {
      float v[V], acc[V];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        v[j] = to_f(from_f<T>(to_f(vp[c * V + j])));
        acc[j] = 0.f;
      }
      for (int d0 = dl; d0 < D; d0 += lanes * kDecUnroll) {
        float s[kDecUnroll][V];
#pragma unroll
        for (int i = 0; i < kDecUnroll; ++i) {
          const int d = d0 + i * lanes;
#pragma unroll
          for (int j = 0; j < V; ++j) s[i][j] = 0.f;
          if (d < D && !fresh) {
            const float* sp = S + static_cast<long long>(d) * E + c * V;
            if constexpr (V == 4) load4<float>(sp, s[i]);
            else s[i][0] = *sp;
          }
        }
#pragma unroll
        for (int i = 0; i < kDecUnroll; ++i) {
          const int d = d0 + i * lanes;
          if (d < D) {
            const float kd = s_k[d], qd = s_q[d];
#pragma unroll
            for (int j = 0; j < V; ++j) {
              s[i][j] = fmaf(gamma, s[i][j], kd * v[j]);
              acc[j] = fmaf(qd, s[i][j], acc[j]);
            }
            float* sp = S + static_cast<long long>(d) * E + c * V;
            if constexpr (V == 4) store4<float>(sp, s[i]);
            else *sp = s[i][0];
          }
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) s_o[dl * Es + c * V + j] = acc[j];
    }
  }
  pdl_launch_dependents();  // the state stream of this CTA is done
  __syncthreads();
  float ssq = 0.f;
  for (int e = threadIdx.x; e < Es; e += kDecThreads) {
    float o = 0.f;
    for (int i = 0; i < lanes; ++i) o += s_o[i * Es + e];
    s_o[e] = o;   // column e of lane 0: read above by this thread only
    ssq = fmaf(o, o, ssq);
  }
  float total = block_sum_all(ssq, s_red);
  if (gridDim.x > 1) {
    cg::cluster_group cl = cg::this_cluster();
    if (threadIdx.x == 0) s_part = total;
    cl.sync();
    total = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) total += *cl.map_shared_rank(&s_part, r);
    cl.sync();  // nobody leaves while a neighbour still reads its part
  }
  const float r = 1.f / sqrtf(total / static_cast<float>(E) + p.eps);
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + head * E + e0;
  for (int e = threadIdx.x; e < Es; e += kDecThreads) out[e] = from_f<T>(s_o[e] * r * silu_f(to_f(gp[e])));
}

// ------------------------------------------------------------------------------------------------
// chunked form
// ------------------------------------------------------------------------------------------------
constexpr int C = kRetChunk;
constexpr int kChThreads = 256;
constexpr int KT = 32;           // head dimensions per step of the Q K^T / Q S loop
constexpr int kLdQ = KT + 4;     // row pitches that make the fragment reads conflict-free
constexpr int kLdP = C + 4;

struct Tf {
  uint32_t hi, lo;
};
// x = hi + lo with both parts representable in TF32 (10 stored bits; the rest is cut off, so lo keeps the
// bits that hi lost and the pair carries about 21)
constexpr uint32_t kTf32Mask = 0xffffe000u;
__device__ __forceinline__ Tf split_tf32(float x) {
  Tf t;
  t.hi = __float_as_uint(x) & kTf32Mask;
  t.lo = __float_as_uint(x - __uint_as_float(t.hi)) & kTf32Mask;
  return t;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 "
      "{%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// A fragment (16 x 8) split in two
struct FragA {
  Tf v[4];
};
// c += A B with both operands split
__device__ __forceinline__ void mma_3x(float (&c)[4], const FragA& a, const Tf& b0, const Tf& b1) {
  mma_tf32(c, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, b0.hi, b1.hi);
  mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b0.lo, b1.lo);
  mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b0.hi, b1.hi);
}
// c += A B where B is exact in TF32
__device__ __forceinline__ void mma_2x(float (&c)[4], const FragA& a, uint32_t b0, uint32_t b1) {
  mma_tf32(c, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, b0, b1);
  mma_tf32(c, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b0, b1);
}

__device__ __forceinline__ void cp_async16(float* dst, const float* src, bool in) {
  const int n = in ? 16 : 0;  // 0 bytes read: the destination is zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// [R x CW] fp32 tile from global (row pitch ldg) into shared memory (row pitch lds); rows >= r_ok and
// columns >= c_ok become zero. vec: source rows are 16-byte aligned and c_ok is a multiple of 4.
template <int R, int CW>
__device__ __forceinline__ void tile_f32(float* dst, int lds, const float* src, long long ldg, int r_ok, int c_ok, bool vec) {
  if (vec) {
    for (int i = threadIdx.x; i < R * (CW / 4); i += kChThreads) {
      const int r = i / (CW / 4), c = (i % (CW / 4)) * 4;
      const bool in = r < r_ok && c < c_ok;
      cp_async16(dst + r * lds + c, in ? src + r * ldg + c : src, in);
    }
  } else {
    for (int i = threadIdx.x; i < R * CW; i += kChThreads) {
      const int r = i / CW, c = i % CW;
      dst[r * lds + c] = (r < r_ok && c < c_ok) ? src[r * ldg + c] : 0.f;
    }
  }
}
// [C x ET] value rows of the projection buffer, rounded to bf16, into fp32 shared memory
template <int ET, typename P>
__device__ __forceinline__ void tile_values(float* dst, int lds, const P* src, long long ldg, int r_ok, int e_ok, bool vec) {
  if (vec) {
    for (int i = threadIdx.x; i < C * (ET / 4); i += kChThreads) {
      const int r = i / (ET / 4), c = (i % (ET / 4)) * 4;
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (r < r_ok && c < e_ok) load4<P>(src + r * ldg + c, v);
      if constexpr (sizeof(P) == 4) {
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = __bfloat162float(__float2bfloat16(v[j]));
      }
      store4<float>(dst + r * lds + c, v);
    }
  } else {
    for (int i = threadIdx.x; i < C * ET; i += kChThreads) {
      const int r = i / ET, c = i % ET;
      dst[r * lds + c] = (r < r_ok && c < e_ok) ? __bfloat162float(from_f<__nv_bfloat16>(to_f(src[r * ldg + c]))) : 0.f;
    }
  }
}

struct ChunkPos {
  int row0, n;  // first row of the chunk in the step, rows in it (<= 0: empty)
};
__device__ __forceinline__ ChunkPos chunk_pos(const RetentionParams& p, int chunk) {
  const int tile = chunk >> 1;
  const int seq = p.tile_seq[tile];
  const int q0 = p.tile_q0[tile] + (chunk & 1) * C;
  const int left = p.q_lens[seq] - q0;
  return {p.q_start[seq] + q0, left < C ? left : C};
}

// 1. grid (chunks, H): U_c[d, e], 64 head dimensions at a time, the next keys on their way meanwhile.
template <int ET>
struct SumSmem {
  static constexpr int kLdK = 64 + 8, kLdV = ET + 8;
  static constexpr int kFloats = 2 * C * kLdK + C * kLdV;
};
template <int ET, typename P>
__global__ void __launch_bounds__(kChThreads) retention_chunk_sum_kernel(const RetentionParams p) {
  using L = SumSmem<ET>;
  extern __shared__ __align__(16) float s_mem[];
  __shared__ float s_w[C];                    // decay of every row of the chunk up to its end
  float* sV = s_mem + 2 * C * L::kLdK;        // [C][ET]
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x, head = blockIdx.y;
  const ChunkPos cp = chunk_pos(p, chunk);
  if (cp.n <= 0) return;
  const int D = p.D, E = p.E;
  const long long ldk = D;
  const float* ksrc = p.k_rot + head * p.rot_hd + cp.row0 * ldk;
  const int n_it = (D + 63) / 64;
  auto load_k = [&](int it) {
    tile_f32<C, 64>(s_mem + (it & 1) * C * L::kLdK, L::kLdK, ksrc + it * 64, ldk, cp.n, D - it * 64, D % 4 == 0);
    cp_commit();
  };
  load_k(0);
  const P* vsrc = static_cast<const P*>(p.proj) + cp.row0 * p.ld + 2 * p.H * D + head * E;
  const bool vec_v = (E % 4 == 0) && (p.ld % 4 == 0) && ((2 * p.H * D) % 4 == 0);
  tile_values<ET, P>(sV, L::kLdV, vsrc, p.ld, cp.n, E, vec_v);
  for (int r = threadIdx.x; r < C; r += kChThreads) s_w[r] = r < cp.n ? p.decay_pow[head * (C + 1) + cp.n - 1 - r] : 0.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int m0 = (warp & 3) * 16;
  constexpr int NT = ET / 16;     // 8-column tiles of this warp's half
  const int n0 = (warp >> 2) * (ET / 2);
  float* w = p.ws + (static_cast<long long>(chunk) * p.H + head) * D * E;
  for (int it = 0; it < n_it; ++it) {
    if (it + 1 < n_it) {
      load_k(it + 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const float* sK = s_mem + (it & 1) * C * L::kLdK;
    float acc[NT][4] = {};
#pragma unroll 2
    for (int kk = 0; kk < C; kk += 8) {
      const float w0 = s_w[kk + t], w1 = s_w[kk + t + 4];
      FragA a;
      a.v[0] = split_tf32(sK[(kk + t) * L::kLdK + m0 + g] * w0);
      a.v[1] = split_tf32(sK[(kk + t) * L::kLdK + m0 + g + 8] * w0);
      a.v[2] = split_tf32(sK[(kk + t + 4) * L::kLdK + m0 + g] * w1);
      a.v[3] = split_tf32(sK[(kk + t + 4) * L::kLdK + m0 + g + 8] * w1);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const uint32_t b0 = __float_as_uint(sV[(kk + t) * L::kLdV + n0 + n * 8 + g]);
        const uint32_t b1 = __float_as_uint(sV[(kk + t + 4) * L::kLdV + n0 + n * 8 + g]);
        mma_2x(acc[n], a, b0, b1);
      }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = it * 64 + m0 + g + 8 * h, e = n0 + n * 8 + 2 * t;
        if (d < D) {
          if (e + 1 < E && (E & 1) == 0) {
            *reinterpret_cast<float2*>(w + static_cast<long long>(d) * E + e) = make_float2(acc[n][2 * h], acc[n][2 * h + 1]);
          } else {
            if (e < E) w[static_cast<long long>(d) * E + e] = acc[n][2 * h];
            if (e + 1 < E) w[static_cast<long long>(d) * E + e + 1] = acc[n][2 * h + 1];
          }
        }
      }
    __syncthreads();  // the stage may be refilled
  }
}

// 2. grid (D E / (256 V CH), H, sequences): walks the chunks of a sequence, U chunks of CH pieces per thread in
// flight (a CTA covers CH x 4 KB of a state in one run).
template <int V, int CH, int U>
__global__ void __launch_bounds__(256) retention_scan_chunks_kernel(const RetentionParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const long long DE = static_cast<long long>(p.D) * p.E;
  const long long i0 = (static_cast<long long>(blockIdx.x) * 256 * CH + threadIdx.x) * V;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (i0 == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  int tile0 = 0;
  for (int s = 0; s < seq; ++s) tile0 += (p.q_lens[s] + 127) >> 7;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + C - 1) / C;
  const float* pw = p.decay_pow + head * (C + 1);
  const float g_full = pw[C], g_last = pw[len - (n_chunks - 1) * C];
  float* st = p.state + (static_cast<long long>(slot) * p.H + head) * DE + i0;
  float* w = p.ws + (static_cast<long long>(2 * tile0) * p.H + head) * DE + i0;
  const long long step = static_cast<long long>(p.H) * DE;
  const bool past = p.ctx_lens[seq] != len;
  float S[CH][V];
  bool in[CH];
#pragma unroll
  for (int h = 0; h < CH; ++h) {
    in[h] = i0 + h * 256 * V < DE;
#pragma unroll
    for (int j = 0; j < V; ++j) S[h][j] = 0.f;
    if (past && in[h]) {
      if constexpr (V == 4) load4<float>(st + h * 256 * V, S[h]);
      else S[h][0] = st[h * 256 * V];
    }
  }
  for (int c0 = 0; c0 < n_chunks; c0 += U) {
    float u[U][CH][V];
#pragma unroll
    for (int k = 0; k < U; ++k)
#pragma unroll
      for (int h = 0; h < CH; ++h)
        if (c0 + k < n_chunks && in[h]) {
          if constexpr (V == 4) load4<float>(w + (c0 + k) * step + h * 256 * V, u[k][h]);
          else u[k][h][0] = w[(c0 + k) * step + h * 256 * V];
        }
#pragma unroll
    for (int k = 0; k < U; ++k)
#pragma unroll
      for (int h = 0; h < CH; ++h)
        if (c0 + k < n_chunks && in[h]) {
          if constexpr (V == 4) store4<float>(w + (c0 + k) * step + h * 256 * V, S[h]);
          else w[(c0 + k) * step + h * 256 * V] = S[h][0];
          const float g = c0 + k == n_chunks - 1 ? g_last : g_full;
#pragma unroll
          for (int j = 0; j < V; ++j) S[h][j] = fmaf(g, S[h][j], u[k][h][j]);
        }
  }
#pragma unroll
  for (int h = 0; h < CH; ++h)
    if (in[h]) {
      if constexpr (V == 4) store4<float>(st + h * 256 * V, S[h]);
      else st[h * 256 * V] = S[h][0];
    }
}

// 3. grid (chunks, H): the chunk's outputs over all value dimensions.
template <int ET>
struct OutSmem {
  static constexpr int kLdS = ET + 8;
  static constexpr int kQK = C * kLdQ;                       // one stage of Q (or K)
  static constexpr int kS = KT * kLdS;                       // one stage of the state
  static constexpr int kStage = 2 * kQK + kS;
  static constexpr int kV = C * kLdS;
  static constexpr bool kShareV = kV <= kStage;             // the values reuse the second stage after the loop
  static constexpr int kFloats = 2 * kStage + (kShareV ? 0 : kV);
  static_assert(C * kLdP <= kStage, "the weights reuse the first stage");
};

template <int ET, typename P>
__global__ void __launch_bounds__(kChThreads, ET <= 128 ? 3 : 1) retention_chunk_out_kernel(const RetentionParams p) {
  using L = OutSmem<ET>;
  extern __shared__ __align__(16) float s_mem[];
  __shared__ float s_pw[C + 1];
  __shared__ float s_ssq[2][C];
  float* sV = s_mem + (L::kShareV ? L::kStage : 2 * L::kStage);
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x, head = blockIdx.y;
  const ChunkPos cp = chunk_pos(p, chunk);
  if (cp.n <= 0) return;
  const int D = p.D, E = p.E;
  const long long ldq = D;
  const float* qsrc = p.q_rot + head * p.rot_hd + cp.row0 * ldq;
  const float* ksrc = p.k_rot + head * p.rot_hd + cp.row0 * ldq;
  const float* ssrc = p.ws + (static_cast<long long>(chunk) * p.H + head) * D * E;
  const P* prow = static_cast<const P*>(p.proj) + cp.row0 * p.ld + 2 * p.H * D + head * E;
  const bool vec_d = D % 4 == 0, vec_e = E % 4 == 0;
  const bool vec_v = vec_e && (p.ld % 4 == 0) && ((2 * p.H * D) % 4 == 0);
  for (int i = threadIdx.x; i <= C; i += kChThreads) s_pw[i] = p.decay_pow[head * (C + 1) + i];

  auto load_stage = [&](int it) {
    float* st = s_mem + (it & 1) * L::kStage;
    const int k0 = it * KT;
    tile_f32<C, KT>(st, kLdQ, qsrc + k0, ldq, cp.n, D - k0, vec_d);
    tile_f32<C, KT>(st + L::kQK, kLdQ, ksrc + k0, ldq, cp.n, D - k0, vec_d);
    tile_f32<KT, ET>(st + 2 * L::kQK, L::kLdS, ssrc + static_cast<long long>(k0) * E, E, D - k0, E, vec_e);
    cp_commit();
  };
  const int n_it = (D + KT - 1) / KT;
  load_stage(0);
  if constexpr (!L::kShareV) tile_values<ET, P>(sV, L::kLdS, prow, p.ld, cp.n, E, vec_v);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int m0 = (warp & 3) * 16, half = warp >> 2;
  constexpr int NT = ET / 16;
  const int n0 = half * (ET / 2);
  float sc[4][4] = {};    // scores: rows m0.., columns half * 32 ..
  float os[NT][4] = {};   // outputs: rows m0.., columns n0 ..
  for (int it = 0; it < n_it; ++it) {
    if (it + 1 < n_it) {
      load_stage(it + 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const float* sQ = s_mem + (it & 1) * L::kStage;
    const float* sK = sQ + L::kQK;
    const float* sS = sK + L::kQK;
#pragma unroll
    for (int kk = 0; kk < KT; kk += 8) {
      FragA a;
      a.v[0] = split_tf32(sQ[(m0 + g) * kLdQ + kk + t]);
      a.v[1] = split_tf32(sQ[(m0 + g + 8) * kLdQ + kk + t]);
      a.v[2] = split_tf32(sQ[(m0 + g) * kLdQ + kk + t + 4]);
      a.v[3] = split_tf32(sQ[(m0 + g + 8) * kLdQ + kk + t + 4]);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int j0 = half * 32 + n * 8;
        if (j0 > m0 + 15) continue;  // above the diagonal
        const Tf b0 = split_tf32(sK[(j0 + g) * kLdQ + kk + t]), b1 = split_tf32(sK[(j0 + g) * kLdQ + kk + t + 4]);
        mma_3x(sc[n], a, b0, b1);
      }
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const Tf b0 = split_tf32(sS[(kk + t) * L::kLdS + n0 + n * 8 + g]);
        const Tf b1 = split_tf32(sS[(kk + t + 4) * L::kLdS + n0 + n * 8 + g]);
        mma_3x(os[n], a, b0, b1);
      }
    }
    __syncthreads();  // the stage may be refilled
  }
  if constexpr (L::kShareV) tile_values<ET, P>(sV, L::kLdS, prow, p.ld, cp.n, E, vec_v);
  // weights of the chunk's own rows, and decay of what came before it
  float* sP = s_mem;
  const int i0 = m0 + g, i1 = m0 + g + 8;
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int i = x < 2 ? i0 : i1, j = half * 32 + n * 8 + 2 * t + (x & 1);
      sP[i * kLdP + j] = j <= i ? sc[n][x] * s_pw[i - j] : 0.f;
    }
  const float f0 = s_pw[i0 + 1], f1 = s_pw[i1 + 1];
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    os[n][0] *= f0;
    os[n][1] *= f0;
    os[n][2] *= f1;
    os[n][3] *= f1;
  }
  __syncthreads();
  for (int kk = 0; kk < m0 + 16; kk += 8) {  // keys above the diagonal weigh nothing
    FragA a;
    a.v[0] = split_tf32(sP[(m0 + g) * kLdP + kk + t]);
    a.v[1] = split_tf32(sP[(m0 + g + 8) * kLdP + kk + t]);
    a.v[2] = split_tf32(sP[(m0 + g) * kLdP + kk + t + 4]);
    a.v[3] = split_tf32(sP[(m0 + g + 8) * kLdP + kk + t + 4]);
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const uint32_t b0 = __float_as_uint(sV[(kk + t) * L::kLdS + n0 + n * 8 + g]);
      const uint32_t b1 = __float_as_uint(sV[(kk + t + 4) * L::kLdS + n0 + n * 8 + g]);
      mma_2x(os[n], a, b0, b1);
    }
  }
  // head norm over the value dimensions: the two column halves meet in shared memory
  float q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    q0 = fmaf(os[n][0], os[n][0], fmaf(os[n][1], os[n][1], q0));
    q1 = fmaf(os[n][2], os[n][2], fmaf(os[n][3], os[n][3], q1));
  }
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    q0 += __shfl_xor_sync(0xffffffffu, q0, o);
    q1 += __shfl_xor_sync(0xffffffffu, q1, o);
  }
  if (t == 0) {
    s_ssq[half][i0] = q0;
    s_ssq[half][i1] = q1;
  }
  __syncthreads();
  const float r0 = 1.f / sqrtf((s_ssq[0][i0] + s_ssq[1][i0]) / static_cast<float>(E) + p.eps);
  const float r1 = 1.f / sqrtf((s_ssq[0][i1] + s_ssq[1][i1]) / static_cast<float>(E) + p.eps);
  const P* grow = prow + p.H * E;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + cp.row0 * p.ldo + head * E;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = h == 0 ? i0 : i1, e = n0 + n * 8 + 2 * t;
      const float r = h == 0 ? r0 : r1;
      if (i >= cp.n) continue;
#pragma unroll
      for (int x = 0; x < 2; ++x)
        if (e + x < E)
          out[i * p.ldo + e + x] = __float2bfloat16(os[n][2 * h + x] * r * silu_f(to_f(grow[i * p.ld + e + x])));
    }
}

// ------------------------------------------------------------------------------------------------
// token by token
// ------------------------------------------------------------------------------------------------
constexpr int kScanCols = 32;

// grid (E / 32, H, sequences): 32 state columns in shared memory, 8 warps split the head dimensions.
template <typename T, typename P>
__global__ void __launch_bounds__(256) retention_scan_kernel(const RetentionParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_o[8][kScanCols];
  pdl_wait();
  const int D = p.D, E = p.E;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int e = blockIdx.x * kScanCols + lane;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  float* st = p.state + (static_cast<long long>(slot) * p.H + head) * D * E;
  const int len = p.q_lens[seq];
  const bool fresh = p.ctx_lens[seq] == len;
  for (int d = w; d < D; d += 8) s_mem[d * kScanCols + lane] = (fresh || e >= E) ? 0.f : st[static_cast<long long>(d) * E + e];
  const float gamma = p.decay_pow[head * (kRetChunk + 1) + 1];
  for (int i = 0; i < len; ++i) {
    const long long row = p.q_start[seq] + i;
    const float* q = p.q_rot + head * p.rot_hd + row * D;
    const float* k = p.k_rot + head * p.rot_hd + row * D;
    const float v = e < E ? to_f(from_f<T>(to_f(static_cast<const P*>(p.proj)[row * p.ld + 2 * p.H * D + head * E + e]))) : 0.f;
    float acc = 0.f;
    for (int d = w; d < D; d += 8) {
      const float s = fmaf(gamma, s_mem[d * kScanCols + lane], k[d] * v);
      s_mem[d * kScanCols + lane] = s;
      acc = fmaf(q[d], s, acc);
    }
    s_o[w][lane] = acc;
    __syncthreads();
    if (w == 0 && e < E) {
      float o = 0.f;
#pragma unroll
      for (int x = 0; x < 8; ++x) o += s_o[x][lane];
      p.o_buf[(row * p.H + head) * E + e] = o;
    }
    __syncthreads();
  }
  if (e < E)
    for (int d = w; d < D; d += 8) st[static_cast<long long>(d) * E + e] = s_mem[d * kScanCols + lane];
}

// grid (128-row tiles x 128, H): head norm and gate of the rows that the kernel above wrote.
template <typename T, typename P>
__global__ void __launch_bounds__(128) retention_head_norm_kernel(const RetentionParams p) {
  __shared__ float s_red[32];
  pdl_wait();
  const int tile = blockIdx.x >> 7, r = blockIdx.x & 127, head = blockIdx.y;
  const int seq = p.tile_seq[tile], qi = p.tile_q0[tile] + r;
  if (qi >= p.q_lens[seq]) return;
  const long long row = p.q_start[seq] + qi;
  const float* o = p.o_buf + (row * p.H + head) * p.E;
  float ss = 0.f;
  for (int e = threadIdx.x; e < p.E; e += 128) ss = fmaf(o[e], o[e], ss);
  const float rr = 1.f / sqrtf(block_sum_all(ss, s_red) / static_cast<float>(p.E) + p.eps);
  const P* gp = static_cast<const P*>(p.proj) + row * p.ld + 2 * p.H * p.D + p.H * p.E + head * p.E;
  T* out = static_cast<T*>(p.out) + row * p.ldo + head * p.E;
  for (int e = threadIdx.x; e < p.E; e += 128) out[e] = from_f<T>(o[e] * rr * silu_f(to_f(gp[e])));
}

template <typename T, typename P, int V>
cudaError_t launch_decode(const RetentionParams& p, int slices, cudaStream_t stream) {
  const int Es = p.E / slices;
  const int groups = Es / V, gt = groups < kDecThreads ? groups : kDecThreads, lanes = kDecThreads / gt;
  const size_t smem = (2 * static_cast<size_t>(p.D) + static_cast<size_t>(lanes) * Es) * sizeof(float);
  auto kern = retention_decode_kernel<T, P, V>;
  ensure_dynamic_smem(kern, smem);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(slices, p.H, p.rows);
  cfg.blockDim = dim3(kDecThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = slices;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.numAttrs = 1;
  if (pdl_enabled()) {
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.numAttrs = 2;
  }
  cfg.attrs = attr;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

template <int ET, typename P>
cudaError_t launch_chunks(const RetentionParams& p, cudaStream_t stream) {
  const int chunks = 2 * p.n_tiles;
  const size_t smem1 = SumSmem<ET>::kFloats * sizeof(float);
  const size_t smem3 = OutSmem<ET>::kFloats * sizeof(float);
  ensure_dynamic_smem(retention_chunk_sum_kernel<ET, P>, smem1);
  ensure_dynamic_smem(retention_chunk_out_kernel<ET, P>, smem3);
  cudaError_t e = launch_kernel(retention_chunk_sum_kernel<ET, P>, dim3(chunks, p.H), dim3(kChThreads), smem1,
                                stream, true, false, p);
  if (e != cudaSuccess) return e;
  const long long de = static_cast<long long>(p.D) * p.E;
  const int v = p.E % 4 == 0 ? 4 : 1;
  // whole runs of 16 KB per CTA where that still leaves enough CTAs
  const bool wide = v == 4 && de >= 4096 && (de / 4096) * p.H * p.n_seqs >= 2 * sm_count();
  const long long per = 256ll * v * (wide ? 4 : 1);
  const dim3 grid2(static_cast<unsigned>((de + per - 1) / per), p.H, p.n_seqs);
  auto scan = wide ? retention_scan_chunks_kernel<4, 4, 2> : (v == 4 ? retention_scan_chunks_kernel<4, 1, 8> : retention_scan_chunks_kernel<1, 1, 8>);
  e = launch_kernel(scan, grid2, dim3(256), 0, stream, true, false, p);
  if (e != cudaSuccess) return e;
  return launch_kernel(retention_chunk_out_kernel<ET, P>, dim3(chunks, p.H), dim3(kChThreads), smem3, stream, true, false, p);
}

template <typename T, typename P>
cudaError_t launch_scan(const RetentionParams& p, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(p.D) * kScanCols * sizeof(float);
  ensure_dynamic_smem(retention_scan_kernel<T, P>, smem);
  cudaError_t e = launch_kernel(retention_scan_kernel<T, P>, dim3((p.E + kScanCols - 1) / kScanCols, p.H, p.n_seqs), dim3(256),
                                smem, stream, true, false, p);
  if (e != cudaSuccess) return e;
  return launch_kernel(retention_head_norm_kernel<T, P>, dim3(p.n_tiles * 128, p.H), dim3(128), 0, stream, true, false, p);
}

}  // namespace

bool retention_chunks_ok(int D, int E) { return D <= 1024 && E <= 256; }

cudaError_t launch_retention_decode(const RetentionParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  // column slices per head: enough CTAs for about two per SM, whole 16-byte pieces, at least 16 columns
  int slices = 1;
  while (slices < 8 && p.rows * p.H * slices < 2 * sm_count() && p.E % (slices * 2 * 4) == 0 && p.E / (slices * 2) >= 16)
    slices *= 2;
  const bool vec = p.E % 4 == 0;
  if (!vec) slices = 1;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return vec ? launch_decode<float, float, 4>(p, slices, stream) : launch_decode<float, float, 1>(p, slices, stream);
  if (p.proj_f32) return vec ? launch_decode<bf16, float, 4>(p, slices, stream) : launch_decode<bf16, float, 1>(p, slices, stream);
  return vec ? launch_decode<bf16, bf16, 4>(p, slices, stream) : launch_decode<bf16, bf16, 1>(p, slices, stream);
}

template <typename P>
static cudaError_t chunks_of(const RetentionParams& p, cudaStream_t stream) {
  if (p.E <= 32) return launch_chunks<32, P>(p, stream);
  if (p.E <= 64) return launch_chunks<64, P>(p, stream);
  if (p.E <= 128) return launch_chunks<128, P>(p, stream);
  if (p.E <= 256) return launch_chunks<256, P>(p, stream);
  return cudaErrorInvalidValue;
}

cudaError_t launch_retention_chunks(const RetentionParams& p, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  return p.proj_f32 ? chunks_of<float>(p, stream) : chunks_of<__nv_bfloat16>(p, stream);
}

cudaError_t launch_retention_scan(const RetentionParams& p, int dtype, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_scan<float, float>(p, stream);
  return p.proj_f32 ? launch_scan<bf16, float>(p, stream) : launch_scan<bf16, bf16>(p, stream);
}

}  // namespace oxb
