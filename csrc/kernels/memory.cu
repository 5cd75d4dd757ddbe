// Matrix memory with a running maximum (mLSTM) on sm_100a. Per head, with log gates f_t and i_t:
//     m_t = max(f_t + m_(t-1), i_t),  S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,  n_t likewise with k_t
//     o_t = S_t^T q_t / (max(|n_t q_t|, exp(-m_t)) + 1e-6),   out_t = o_t / rms(o_t) * w * sigmoid(gate_t)
//
// Decode: one thread-block cluster per (row, head) streams that head's fp32 state once through the SMs: gate
//   pre-activations, state and normaliser update, read-out, head norm and gate in one launch. The CTAs of a cluster own
//   column slices of the state and exchange their parts of the norm through distributed shared memory.
// Prompt chunks of 64 rows, three launches, parallel over chunks. With b_t the sum of f up to row t of a chunk, g its
// value at the chunk's end and M the maximum before the chunk:
//   1. U_c = sum_s exp(g - b_s + i_s - a) k_s v_s^T, a the largest exponent; likewise for n
//   2. scan over the chunks of a sequence: M' = max(g + M, a), S' = exp(g + M - M') S + exp(a - M') U_c; replaces U_c by
//      the state before chunk c and stores the final state
//   3. m_t = b_t + max(M, max_{s <= t}(i_s - b_s)); o_t from exp(b_t - b_s + i_s - m_t) (q_t k_s) over the chunk's own rows
//      and exp(b_t + M - m_t) q_t S before them, then the normaliser, head norm and gate
//   q, k and v are bf16 (outputs of the projection), so q k is exact products summed in fp32; weighted scores, weighted
//   keys and states enter their products as three bf16 terms, which carry all 24 bits.
// Token-by-token form in fp32 FMAs for the 32-bit path and for head sizes above the chunked form's.
#include <cooperative_groups.h>

#include "../common/device_info.h"
#include "hybrid_dev.cuh"
#include "hybrid_mma.cuh"

namespace cg = cooperative_groups;

namespace oxb {

namespace {

constexpr int C = kMemChunk;

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ long long state_size(const MemoryParams& p) { return static_cast<long long>(p.D) * p.E + p.D; }

// ------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256;
constexpr int kDecUnroll = 8;

// grid (slices, H, rows), cluster (slices, 1, 1). V columns of the state per thread and access. T: storage type, P: type
// of the projection rows. q, k and v enter the state as the storage type holds them.
template <typename T, typename P, int V>
__global__ void __launch_bounds__(kDecThreads) memory_decode_kernel(const MemoryParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_red[32], s_red2[32];
  __shared__ float s_part;
  const int D = p.D, E = p.E;
  const int Es = E / static_cast<int>(gridDim.x);
  float* s_q = s_mem;            // D
  float* s_k = s_q + D;          // D, times the input gate
  float* s_n = s_k + D;          // D, the new normaliser
  float* s_o = s_n + D;          // [lanes][Es]
  const int head = blockIdx.y, row = blockIdx.z, e0 = blockIdx.x * Es;
  pdl_wait();  // the projection comes from the kernel before this one
  const int slot = p.row_slots[row];
  if (slot < 0) return;  // padding row (the whole cluster leaves)
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const bool fresh = p.positions[row] == 0;
  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld;
  const P* qp = pr + head * D;
  const P* kp = pr + (p.H + head) * D;
  const P* vp = pr + 2 * p.H * D + head * E + e0;
  const P* gp = pr + 2 * p.H * D + p.H * E + head * E + e0;
  // gate pre-activations
  float zi, zf;
  if (p.z != nullptr) {
    zi = p.z[row * p.ldz + head];
    zf = p.z[row * p.ldz + p.H + head];
  } else {
    const __nv_bfloat16* h = static_cast<const __nv_bfloat16*>(p.h) + row * p.ldh;
    const __nv_bfloat16* wi = static_cast<const __nv_bfloat16*>(p.z_w) + head * p.ldw;
    const __nv_bfloat16* wf = wi + p.H * p.ldw;
    float a = 0.f, b = 0.f;
    for (int c = threadIdx.x * 4; c < p.N; c += kDecThreads * 4) {
      float x[4], u[4], v[4];
      load4<__nv_bfloat16>(h + c, x);
      load4<__nv_bfloat16>(wi + c, u);
      load4<__nv_bfloat16>(wf + c, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        a = fmaf(x[j], u[j], a);
        b = fmaf(x[j], v[j], b);
      }
    }
    zi = block_sum_all(a, s_red);
    zf = block_sum_all(b, s_red2);
  }
  const float gi = log_input_gate(zi + p.z_bias[head], p.cap), gf = log_forget_gate(zf + p.z_bias[p.H + head], p.cap);
  float* mp = p.state_m + static_cast<long long>(slot) * p.H + head;
  const float m_old = fresh ? 0.f : *mp;
  const float m = fmaxf(gf + m_old, gi);
  const float keep = expf(gf + m_old - m), add = expf(gi - m);
  float* S0 = p.state + (static_cast<long long>(slot) * p.H + head) * state_size(p);
  float* np = S0 + static_cast<long long>(D) * E;
  float nq = 0.f;
  for (int d = threadIdx.x; d < D; d += kDecThreads) {
    const float q = to_f(from_f<T>(to_f(qp[d]))) * p.scale, k = to_f(from_f<T>(to_f(kp[d])));
    s_q[d] = q;
    s_k[d] = add * k;
    const float n = fmaf(keep, fresh ? 0.f : np[d], add * k);
    s_n[d] = n;
    nq = fmaf(n, q, nq);
  }
  nq = block_sum_all(nq, s_red);
  const float den = fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
  const int groups = Es / V;
  const int gt = groups < kDecThreads ? groups : kDecThreads;
  const int lanes = kDecThreads / gt;
  const int cgi = threadIdx.x % gt, dl = threadIdx.x / gt;
  float* S = S0 + e0;
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
              s[i][j] = fmaf(keep, s[i][j], kd * v[j]);
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
    o /= den;
    s_o[e] = o;   // column e of lane 0: read above by this thread only
    ssq = fmaf(o, o, ssq);
  }
  float total = block_sum_all(ssq, s_red2);
  if (gridDim.x > 1) {
    cg::cluster_group cl = cg::this_cluster();
    if (threadIdx.x == 0) s_part = total;
    cl.sync();   // (also: every CTA has read the old normaliser and maximum)
    total = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) total += *cl.map_shared_rank(&s_part, r);
    cl.sync();  // nobody leaves while a neighbour still reads its part
  }
  if (blockIdx.x == 0) {
    for (int d = threadIdx.x; d < D; d += kDecThreads) np[d] = s_n[d];
    if (threadIdx.x == 0) *mp = m;
  }
  const float r = 1.f / sqrtf(total / static_cast<float>(E) + p.eps);
  const float* nw = p.norm_w + head * E + e0;
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + head * E + e0;
  for (int e = threadIdx.x; e < Es; e += kDecThreads) out[e] = from_f<T>(s_o[e] * r * nw[e] * sigmoid_f(to_f(gp[e])));
}

// ------------------------------------------------------------------------------------------------
// chunked form
// ------------------------------------------------------------------------------------------------
constexpr int kChThreads = 256, kChWarps = kChThreads / 32;
constexpr int ET = 128;                    // value columns per CTA
constexpr int kPitchV = ET * 2 + 16;       // bytes; odd multiples of 16: rows start in different banks
constexpr int kPitchW = C * 2 + 16;

struct ChunkPos {
  int row0, n, seq, q0;  // first row of the chunk in the step, rows in it (<= 0: empty)
};
__device__ __forceinline__ ChunkPos chunk_pos(const MemoryParams& p, int chunk) {
  const int tile = chunk >> 1;
  const int seq = p.tile_seq[tile];
  const int q0 = p.tile_q0[tile] + (chunk & 1) * C;
  const int left = p.q_lens[seq] - q0;
  return {p.q_start[seq] + q0, left < C ? left : C, seq, q0};
}

// [C x w] values of the projection rows, as bf16, into shared memory; rows >= n and columns >= w_ok become zero. w is a
// multiple of 16. bf16 rows of whole 16-byte pieces go asynchronously (wait with cp_wait<0>); otherwise eight or four
// pieces per thread are on their way together.
template <typename P>
__device__ __forceinline__ void tile_bf16(uint8_t* dst, int pitch, const P* src, long long ld, int n, int w, int w_ok) {
  const bool row16 = ((reinterpret_cast<uintptr_t>(src) | (ld * sizeof(P))) & 15) == 0;
  if (sizeof(P) == 2 && row16 && w_ok % 8 == 0) {
    const int per = w >> 3;
    int r = threadIdx.x / per, c = threadIdx.x - r * per;
    const int dr = kChThreads / per, dc = kChThreads - dr * per;
    while (r < C) {
      const bool in = r < n && c * 8 < w_ok;
      cp_async16(smem_u32(dst) + r * pitch + c * 16, in ? src + r * ld + c * 8 : src, in);
      r += dr;
      c += dc;
      if (c >= per) {
        c -= per;
        ++r;
      }
    }
    cp_commit();
  } else if (sizeof(P) == 4 && row16 && w_ok % 4 == 0) {
    const int per = w >> 2, total = C * per;
    for (int i0 = threadIdx.x; i0 < total; i0 += kChThreads * 8) {
      float v[8][4];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = i0 + k * kChThreads, r = i / per, c = (i - r * per) * 4;
#pragma unroll
        for (int x = 0; x < 4; ++x) v[k][x] = 0.f;
        if (i < total && r < n && c < w_ok) load4<P>(src + r * ld + c, v[k]);
      }
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = i0 + k * kChThreads, r = i / per, c = (i - r * per) * 4;
        if (i >= total) break;
        uint2 x;
        x.x = pack_bf16x2(v[k][0], v[k][1]);
        x.y = pack_bf16x2(v[k][2], v[k][3]);
        *reinterpret_cast<uint2*>(dst + r * pitch + c * 2) = x;
      }
    }
  } else {
    for (int i = threadIdx.x; i < C * w; i += kChThreads) {
      const int r = i / w, c = i - r * w;
      reinterpret_cast<__nv_bfloat16*>(dst + r * pitch)[c] =
          (r < n && c < w_ok) ? from_f<__nv_bfloat16>(to_f(src[r * ld + c])) : __float2bfloat16(0.f);
    }
  }
}

// Gates of a chunk by one warp, lane -> rows 2 lane and 2 lane + 1: running sums of f in s_b, log input gates in s_i (rows
// past the end add nothing), running maximum of i - b in `mx`.
__device__ __forceinline__ void chunk_gates(const MemoryParams& p, const ChunkPos& cp, int head, int lane, float* s_b, float* s_i, float (&mx)[2]) {
  float f[2], gi[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int r = 2 * lane + x;
    const bool in = r < cp.n;
    const float* z = p.z + (cp.row0 + (in ? r : 0)) * p.ldz;
    f[x] = in ? log_forget_gate(z[p.H + head] + p.z_bias[p.H + head], p.cap) : 0.f;
    gi[x] = in ? log_input_gate(z[head] + p.z_bias[head], p.cap) : -INFINITY;
  }
  float incl = f[0] + f[1];
  const float pair = incl;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, incl, o);
    if (lane >= o) incl += up;
  }
  const float b0 = incl - pair + f[0], b1 = incl;
  float m1 = fmaxf(gi[0] - b0, gi[1] - b1), run = m1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run = fmaxf(run, up);
  }
  const float before = __shfl_up_sync(0xffffffffu, run, 1);
  mx[0] = fmaxf(lane > 0 ? before : -INFINITY, gi[0] - b0);
  mx[1] = run;
  s_b[2 * lane] = b0;
  s_b[2 * lane + 1] = b1;
  s_i[2 * lane] = gi[0];
  s_i[2 * lane + 1] = gi[1];
}

// 1. grid (chunks, H, column slices)
template <typename P>
__global__ void __launch_bounds__(kChThreads) memory_chunk_sum_kernel(const MemoryParams p) {
  extern __shared__ __align__(16) uint8_t s_raw[];
  __shared__ float s_b[C], s_i[C], s_w[C];
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x, head = blockIdx.y, e0 = blockIdx.z * ET;
  const ChunkPos cp = chunk_pos(p, chunk);
  if (cp.n <= 0) return;
  const int D = p.D, E = p.E, Dp = (D + 15) & ~15, pitch = Dp * 2 + 16;
  uint8_t* sK = s_raw;
  uint8_t* sV = s_raw + C * pitch;
  const P* prow = static_cast<const P*>(p.proj) + cp.row0 * p.ld;
  const int k_col = (p.H + head) * D, v_col = 2 * p.H * D + head * E + e0;
  tile_bf16<P>(sK, pitch, prow + k_col, p.ld, cp.n, Dp, D);
  tile_bf16<P>(sV, kPitchV, prow + v_col, p.ld, cp.n, ET, min(ET, E - e0));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  if (warp == 0) {
    float mx[2];
    chunk_gates(p, cp, head, lane, s_b, s_i, mx);
    __syncwarp();
    const float end = s_b[C - 1], a = end + __shfl_sync(0xffffffffu, mx[1], 31);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = 2 * lane + x;
      s_w[r] = r < cp.n ? expf(end - s_b[r] + s_i[r] - a) : 0.f;
    }
    if (lane == 0 && blockIdx.z == 0) {
      float* w = p.ws_m + (static_cast<long long>(chunk) * p.H + head) * 3;
      w[1] = end;
      w[2] = a;
    }
  }
  cp_wait<0>();
  __syncthreads();
  float* U = p.ws + (static_cast<long long>(chunk) * p.H + head) * state_size(p);
  if (blockIdx.z == 0)
    for (int d = threadIdx.x; d < D; d += kChThreads) {
      float a = 0.f;
      for (int s = 0; s < cp.n; ++s) a = fmaf(s_w[s], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sK + s * pitch + d * 2)), a);
      U[static_cast<long long>(D) * E + d] = a;
    }
  const int lr = lane & 7, lm = lane >> 3;
  const int row_a = (lm & 1) * 8 + lr, col_a = (lm >> 1) * 16;
  const int row_b = (lm >> 1) * 8 + lr, col_b = (lm & 1) * 16;
  const uint32_t aK = smem_u32(sK), aV = smem_u32(sV);
  const int pairs = min(ET, (E - e0 + 15) & ~15) >> 4;   // pairs of 8-column tiles in use
  for (int dt = warp; dt * 16 < D; dt += kChWarps) {
    float acc[ET / 8][4];
#pragma unroll
    for (int i = 0; i < ET / 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[i][x] = 0.f;
#pragma unroll
    for (int kj = 0; kj < C / 16; ++kj) {
      uint32_t kv[4], a[4][3];   // keys, transposed: (d lo, s lo) (d hi, s lo) (d lo, s hi) (d hi, s hi)
      ldsm4t(aK + (kj * 16 + row_b) * pitch + dt * 32 + col_b, kv);
      const int s0 = kj * 16 + 2 * t;
      const float w0 = s_w[s0], w1 = s_w[s0 + 1], w2 = s_w[s0 + 8], w3 = s_w[s0 + 9];
#pragma unroll
      for (int x = 0; x < 4; ++x)
        split3(__uint_as_float(kv[x] << 16) * (x < 2 ? w0 : w2), __uint_as_float(kv[x] & 0xffff0000u) * (x < 2 ? w1 : w3), a[x]);
#pragma unroll
      for (int q = 0; q < ET / 16; ++q) {
        if (q >= pairs) break;
        uint32_t b[4];
        ldsm4t(aV + (kj * 16 + row_a) * kPitchV + q * 32 + col_a, b);
#pragma unroll
        for (int x = 2; x >= 0; --x) {
          mma_bf16(acc[2 * q], a[0][x], a[1][x], a[2][x], a[3][x], b[0], b[1]);
          mma_bf16(acc[2 * q + 1], a[0][x], a[1][x], a[2][x], a[3][x], b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < ET / 8; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = dt * 16 + g + 8 * h, e = e0 + i * 8 + 2 * t;
        if (d >= D) continue;
        float* o = U + static_cast<long long>(d) * E + e;
        if ((E & 1) == 0 && (D & 1) == 0) {
          if (e < E) *reinterpret_cast<float2*>(o) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
        } else {
          if (e < E) o[0] = acc[i][2 * h];
          if (e + 1 < E) o[1] = acc[i][2 * h + 1];
        }
      }
  }
}

// 2. grid (state pieces, H, sequences): walks the chunks of a sequence, K chunks of N pieces per thread in flight.
template <int V, int N, int K>
__global__ void __launch_bounds__(256) memory_scan_chunks_kernel(const MemoryParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const long long size = state_size(p);
  const long long i0 = (static_cast<long long>(blockIdx.x) * 256 * N + threadIdx.x) * V;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (i0 == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  int tile0 = 0;
  for (int s = 0; s < seq; ++s) tile0 += (p.q_lens[s] + 127) >> 7;
  const int len = p.q_lens[seq];
  const int n_chunks = (len + C - 1) / C;
  const bool past = p.ctx_lens[seq] != len;
  float* st = p.state + (static_cast<long long>(slot) * p.H + head) * size + i0;
  const long long at0 = static_cast<long long>(2 * tile0) * p.H + head;
  float* w = p.ws + at0 * size + i0;
  float* wm = p.ws_m + at0 * 3;
  const long long step = p.H * size;
  float m = past ? p.state_m[static_cast<long long>(slot) * p.H + head] : 0.f;
  float S[N][V];
  bool in[N];
#pragma unroll
  for (int h = 0; h < N; ++h) {
    in[h] = i0 + h * 256 * V < size;
#pragma unroll
    for (int j = 0; j < V; ++j) S[h][j] = 0.f;
    if (past && in[h]) {
      if constexpr (V == 4) load4<float>(st + h * 256 * V, S[h]);
      else S[h][0] = st[h * 256 * V];
    }
  }
  for (int c0 = 0; c0 < n_chunks; c0 += K) {
    float u[K][N][V], ga[K][2];
#pragma unroll
    for (int k = 0; k < K; ++k)
      if (c0 + k < n_chunks) {
        const float* z = wm + static_cast<long long>(c0 + k) * p.H * 3;
        ga[k][0] = z[1];
        ga[k][1] = z[2];
#pragma unroll
        for (int h = 0; h < N; ++h)
          if (in[h]) {
            if constexpr (V == 4) load4<float>(w + (c0 + k) * step + h * 256 * V, u[k][h]);
            else u[k][h][0] = w[(c0 + k) * step + h * 256 * V];
          }
      }
#pragma unroll
    for (int k = 0; k < K; ++k)
      if (c0 + k < n_chunks) {
        if (i0 == 0) wm[static_cast<long long>(c0 + k) * p.H * 3] = m;
        const float m2 = fmaxf(ga[k][0] + m, ga[k][1]);
        const float keep = expf(ga[k][0] + m - m2), add = expf(ga[k][1] - m2);
        m = m2;
#pragma unroll
        for (int h = 0; h < N; ++h)
          if (in[h]) {
            if constexpr (V == 4) store4<float>(w + (c0 + k) * step + h * 256 * V, S[h]);
            else w[(c0 + k) * step + h * 256 * V] = S[h][0];
#pragma unroll
            for (int j = 0; j < V; ++j) S[h][j] = fmaf(keep, S[h][j], add * u[k][h][j]);
          }
      }
  }
#pragma unroll
  for (int h = 0; h < N; ++h)
    if (in[h]) {
      if constexpr (V == 4) store4<float>(st + h * 256 * V, S[h]);
      else st[h * 256 * V] = S[h][0];
    }
}

// 3. grid (chunks, H, column slices), cluster (1, 1, slices). Warp w owns columns 16 w .. of the slice, all 64 rows.
struct OutSmem {
  int pitch, k, v, w, n, total;
  __host__ __device__ explicit OutSmem(int D) {
    pitch = ((D + 15) & ~15) * 2 + 16;
    k = C * pitch;
    v = 2 * C * pitch;
    w = v + C * kPitchV;
    n = w + 3 * C * kPitchW;
    total = n + ((D + 31) & ~31) * 4;
  }
};
template <typename P>
__global__ void __launch_bounds__(kChThreads, 2) memory_chunk_out_kernel(const MemoryParams p) {
  extern __shared__ __align__(16) uint8_t s_raw[];
  __shared__ float s_b[C], s_i[C], s_m[C], s_in[C], s_qn[C];   // s_in: weight of what came before the chunk
  __shared__ float s_sum[C / 16][C], s_ssq[kChWarps][C], s_part[C];
  pdl_launch_dependents();
  pdl_wait();
  const int chunk = blockIdx.x, head = blockIdx.y, e0 = blockIdx.z * ET;
  const ChunkPos cp = chunk_pos(p, chunk);
  if (cp.n <= 0) return;   // the whole cluster leaves
  const int D = p.D, E = p.E, Dp = (D + 15) & ~15;
  const OutSmem L(D);
  const P* prow = static_cast<const P*>(p.proj) + cp.row0 * p.ld;
  const int q_col = head * D, k_col = (p.H + head) * D, v_col = 2 * p.H * D + head * E + e0;
  const float* S0 = p.ws + (static_cast<long long>(chunk) * p.H + head) * state_size(p);
  float* s_n = reinterpret_cast<float*>(s_raw + L.n);
  tile_bf16<P>(s_raw, L.pitch, prow + q_col, p.ld, cp.n, Dp, D);
  tile_bf16<P>(s_raw + L.k, L.pitch, prow + k_col, p.ld, cp.n, Dp, D);
  tile_bf16<P>(s_raw + L.v, kPitchV, prow + v_col, p.ld, cp.n, ET, min(ET, E - e0));
  for (int d = threadIdx.x; d < ((D + 31) & ~31); d += kChThreads) s_n[d] = d < D ? S0[static_cast<long long>(D) * E + d] : 0.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const float* wm = p.ws_m + (static_cast<long long>(chunk) * p.H + head) * 3;
  if (warp == 0) {
    const float M = wm[0];
    float mx[2];
    chunk_gates(p, cp, head, lane, s_b, s_i, mx);
    __syncwarp();
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = 2 * lane + x;
      const float m = s_b[r] + fmaxf(M, mx[x]);
      s_m[r] = m;
      s_in[r] = expf(s_b[r] + M - m);
    }
    // the sequence's last chunk leaves the maximum behind
    if (lane == 0 && blockIdx.z == 0 && cp.q0 + cp.n == p.q_lens[cp.seq]) {
      const int slot = p.seq_slots[cp.seq];
      if (slot >= 0 && slot < p.num_slots) p.state_m[static_cast<long long>(slot) * p.H + head] = fmaxf(wm[1] + M, wm[2]);
    }
  }
  for (int i = threadIdx.x; i < C / 16 * C; i += kChThreads) (&s_sum[0][0])[i] = 0.f;
  cp_wait<0>();
  __syncthreads();
  const uint32_t aQ = smem_u32(s_raw), aK = aQ + L.k, aV = aQ + L.v, aW = aQ + L.w;
  const int lr = lane & 7, lm = lane >> 3;
  const int row_a = (lm & 1) * 8 + lr, col_a = (lm >> 1) * 16;
  const int row_b = (lm >> 1) * 8 + lr, col_b = (lm & 1) * 16;
  // ---- weighted scores: 16 x 16 blocks on and below the diagonal ----
  for (int it = warp; it < 10; it += kChWarps) {
    int mi = 0, nj = it;
    while (nj > mi) {
      nj -= mi + 1;
      ++mi;
    }
    float sc[2][4] = {};
#pragma unroll 4
    for (int k = 0; k < Dp / 16; ++k) {
      uint32_t a[4], b[4];
      ldsm4(aQ + (mi * 16 + row_a) * L.pitch + k * 32 + col_a, a);
      ldsm4(aK + (nj * 16 + row_b) * L.pitch + k * 32 + col_b, b);
      mma_bf16(sc[0], a, b[0], b[1]);
      mma_bf16(sc[1], a, b[2], b[3]);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = mi * 16 + g + r * 8;
      const float bi = s_b[i] - s_m[i];
      float sum = 0.f;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int j = nj * 16 + h * 8 + 2 * t;
        const float v0 = j <= i ? sc[h][2 * r] * p.scale * expf(bi - s_b[j] + s_i[j]) : 0.f;
        const float v1 = j + 1 <= i ? sc[h][2 * r + 1] * p.scale * expf(bi - s_b[j + 1] + s_i[j + 1]) : 0.f;
        sum += v0 + v1;
        uint32_t tm[3];
        split3(v0, v1, tm);
#pragma unroll
        for (int x = 0; x < 3; ++x)
          asm volatile("st.shared.u32 [%0], %1;" ::"r"(aW + (x * C + i) * kPitchW + j * 2), "r"(tm[x]) : "memory");
      }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if (t == 0) s_sum[nj][i] = sum;
    }
  }
  // ---- q n: four threads per row ----
  {
    const int r = threadIdx.x >> 2, part = threadIdx.x & 3;
    float a = 0.f;
    for (int d = part * 8; d < Dp; d += 32) {
      float x[8], y[4];
      load4<__nv_bfloat16>(reinterpret_cast<const __nv_bfloat16*>(s_raw + r * L.pitch) + d, *reinterpret_cast<float(*)[4]>(x));
      load4<__nv_bfloat16>(reinterpret_cast<const __nv_bfloat16*>(s_raw + r * L.pitch) + d + 4, *reinterpret_cast<float(*)[4]>(x + 4));
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        load4<float>(s_n + d + 4 * h, y);
#pragma unroll
        for (int k = 0; k < 4; ++k) a = fmaf(x[4 * h + k], y[k], a);
      }
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    if (part == 0) s_qn[r] = a * p.scale;
  }
  // ---- q S: the state's values go from global memory straight into fragments ----
  const int ec = e0 + warp * 16;      // this warp's columns
  const bool active = ec < E;
  float Y[4][2][4] = {};
  if (active) {
    const bool c0 = ec + g < E, c1 = ec + 8 + g < E;
    const float* Sp = S0 + ec + g;
    auto fetch = [&](int k, float (&v)[2][4]) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = k * 16 + 2 * t + (x & 1) + (x >> 1) * 8;
        const float* sp = Sp + static_cast<long long>(d) * E;
        v[0][x] = d < D && c0 ? __ldcg(sp) : 0.f;
        v[1][x] = d < D && c1 ? __ldcg(sp + 8) : 0.f;
      }
    };
    constexpr int kAhead = 4;   // steps whose values are on their way
    float v[kAhead][2][4];
    const int steps = Dp / 16;
#pragma unroll
    for (int j = 0; j < kAhead; ++j) fetch(j, v[j]);
    for (int k0 = 0; k0 < steps; k0 += kAhead) {
#pragma unroll
      for (int j = 0; j < kAhead; ++j) {
        const int k = k0 + j;
        if (k >= steps) break;
        uint32_t b[2][2][3];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          split3(v[j][h][0], v[j][h][1], b[h][0]);
          split3(v[j][h][2], v[j][h][3], b[h][1]);
        }
        fetch(k + kAhead, v[j]);
        uint32_t a[4][4];
#pragma unroll
        for (int mi = 0; mi < 4; ++mi) ldsm4(aQ + (mi * 16 + row_a) * L.pitch + k * 32 + col_a, a[mi]);
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
          for (int mi = 0; mi < 4; ++mi)
#pragma unroll
            for (int h = 0; h < 2; ++h) mma_bf16(Y[mi][h], a[mi], b[h][0][x], b[h][1][x]);
      }
    }
#pragma unroll
    for (int mi = 0; mi < 4; ++mi) {
      const float f0 = s_in[mi * 16 + g] * p.scale, f1 = s_in[mi * 16 + g + 8] * p.scale;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        Y[mi][h][0] *= f0;
        Y[mi][h][1] *= f0;
        Y[mi][h][2] *= f1;
        Y[mi][h][3] *= f1;
      }
    }
  }
  __syncthreads();   // weights and their sums are there
  if (active) {
#pragma unroll
    for (int kj = 0; kj < 4; ++kj) {
      uint32_t vb[4];
      ldsm4t(aV + (kj * 16 + row_a) * kPitchV + warp * 32 + col_a, vb);
#pragma unroll
      for (int x = 2; x >= 0; --x)
#pragma unroll
        for (int mi = kj; mi < 4; ++mi) {
          uint32_t a[4];
          ldsm4(aW + (x * C + mi * 16 + row_a) * kPitchW + kj * 32 + col_a, a);
          mma_bf16(Y[mi][0], a, vb[0], vb[1]);
          mma_bf16(Y[mi][1], a, vb[2], vb[3]);
        }
    }
  }
  // ---- normaliser; the rows wait in shared memory (where values and weights were) for their norm over all columns ----
  __syncthreads();
  constexpr int kPitchO = ET + 4;
  float* s_o = reinterpret_cast<float*>(s_raw + L.v);
  static_assert(C * kPitchO * 4 <= C * kPitchV + 3 * C * kPitchW, "rows fit where values and weights were");
#pragma unroll
  for (int mi = 0; mi < 4; ++mi)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = mi * 16 + g + r * 8;
      const float nq = s_qn[i] * s_in[i] + s_sum[0][i] + s_sum[1][i] + s_sum[2][i] + s_sum[3][i];
      const float inv = 1.f / (fmaxf(fabsf(nq), expf(-s_m[i])) + 1e-6f);
      float ss = 0.f;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float2 o = make_float2(Y[mi][h][2 * r] * inv, Y[mi][h][2 * r + 1] * inv);
        ss = fmaf(o.x, o.x, fmaf(o.y, o.y, ss));
        *reinterpret_cast<float2*>(s_o + i * kPitchO + warp * 16 + h * 8 + 2 * t) = o;
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (t == 0) s_ssq[warp][i] = ss;
    }
  __syncthreads();
  if (threadIdx.x < C) {
    float a = 0.f;
#pragma unroll
    for (int x = 0; x < kChWarps; ++x) a += s_ssq[x][threadIdx.x];
    s_part[threadIdx.x] = a;
  }
  if (gridDim.z > 1) {
    cg::cluster_group cl = cg::this_cluster();
    cl.sync();
    if (threadIdx.x < C) {
      float a = 0.f;
      for (unsigned x = 0; x < gridDim.z; ++x) a += cl.map_shared_rank(s_part, x)[threadIdx.x];
      s_qn[threadIdx.x] = 1.f / sqrtf(a / static_cast<float>(E) + p.eps);
    }
    cl.sync();  // nobody leaves while a neighbour still reads its part
  } else {
    __syncthreads();
    if (threadIdx.x < C) s_qn[threadIdx.x] = 1.f / sqrtf(s_part[threadIdx.x] / static_cast<float>(E) + p.eps);
    __syncthreads();
  }
  const P* grow = prow + 2 * p.H * D + p.H * E + head * E + e0;
  const float* nw = p.norm_w + head * E + e0;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + cp.row0 * p.ldo + head * E + e0;
  const int cols = min(ET, E - e0);
  if (cols % 4 == 0 && E % 4 == 0 && D % 2 == 0 && p.ld % 4 == 0 && p.ldo % 4 == 0 && (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0) {
    // four columns per thread, a warp per row: gate, weight and output in whole runs
    const int e = lane * 4;
    if (e < cols) {
      float w4[4];
      load4<float>(nw + e, w4);
#pragma unroll
      for (int i0 = 0; i0 < C; i0 += kChWarps * 4) {
        float gt[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int i = i0 + k * kChWarps + warp;
          if (i < cp.n) load4<P>(grow + i * p.ld + e, gt[k]);
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int i = i0 + k * kChWarps + warp;
          if (i >= cp.n) continue;
          float o[4];
          load4<float>(s_o + i * kPitchO + e, o);
#pragma unroll
          for (int x = 0; x < 4; ++x) o[x] *= s_qn[i] * w4[x] * sigmoid_f(gt[k][x]);
          store4<__nv_bfloat16>(out + i * p.ldo + e, o);
        }
      }
    }
  } else {
    for (int i = warp; i < cp.n; i += kChWarps)
      for (int e = lane; e < cols; e += 32)
        out[i * p.ldo + e] = __float2bfloat16(s_o[i * kPitchO + e] * s_qn[i] * nw[e] * sigmoid_f(to_f(grow[i * p.ld + e])));
  }
}

// ------------------------------------------------------------------------------------------------
// token by token
// ------------------------------------------------------------------------------------------------
constexpr int kScanCols = 32;

// grid (E / 32, H, sequences): 32 state columns in shared memory, 8 warps split the key dimensions. Every CTA carries the
// normaliser and the maximum; the first one hands them to the kernel below, which stores them when no CTA reads them any more.
template <typename T, typename P>
__global__ void __launch_bounds__(256) memory_scan_kernel(const MemoryParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_o[8][kScanCols], s_nq[8];
  pdl_wait();
  const int D = p.D, E = p.E;
  float* s_n = s_mem + D * kScanCols;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int e = blockIdx.x * kScanCols + lane;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  float* st = p.state + (static_cast<long long>(slot) * p.H + head) * state_size(p);
  const int len = p.q_lens[seq];
  const bool fresh = p.ctx_lens[seq] == len;
  for (int d = w; d < D; d += 8) s_mem[d * kScanCols + lane] = (fresh || e >= E) ? 0.f : st[static_cast<long long>(d) * E + e];
  for (int d = threadIdx.x; d < D; d += 256) s_n[d] = fresh ? 0.f : st[static_cast<long long>(D) * E + d];
  float m = fresh ? 0.f : p.state_m[static_cast<long long>(slot) * p.H + head];
  __syncthreads();
  for (int i = 0; i < len; ++i) {
    const long long row = p.q_start[seq] + i;
    const P* pr = static_cast<const P*>(p.proj) + row * p.ld;
    const P* q = pr + head * D;
    const P* k = pr + (p.H + head) * D;
    const float gi = log_input_gate(p.z[row * p.ldz + head] + p.z_bias[head], p.cap);
    const float gf = log_forget_gate(p.z[row * p.ldz + p.H + head] + p.z_bias[p.H + head], p.cap);
    const float m2 = fmaxf(gf + m, gi), keep = expf(gf + m - m2), add = expf(gi - m2);
    m = m2;
    const float v = e < E ? to_f(from_f<T>(to_f(pr[2 * p.H * D + head * E + e]))) : 0.f;
    float acc = 0.f, nq = 0.f;
    for (int d = w; d < D; d += 8) {
      const float kd = add * to_f(from_f<T>(to_f(k[d]))), qd = to_f(from_f<T>(to_f(q[d]))) * p.scale;
      const float s = fmaf(keep, s_mem[d * kScanCols + lane], kd * v);
      s_mem[d * kScanCols + lane] = s;
      acc = fmaf(qd, s, acc);
      if (lane == 0) {
        const float n = fmaf(keep, s_n[d], kd);
        s_n[d] = n;
        nq = fmaf(qd, n, nq);
      }
    }
    s_o[w][lane] = acc;
    if (lane == 0) s_nq[w] = nq;
    __syncthreads();
    if (w == 0 && e < E) {
      float o = 0.f, n = 0.f;
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        o += s_o[x][lane];
        n += s_nq[x];
      }
      p.o_buf[(row * p.H + head) * E + e] = o / (fmaxf(fabsf(n), expf(-m)) + 1e-6f);
    }
    __syncthreads();
  }
  if (e < E)
    for (int d = w; d < D; d += 8) st[static_cast<long long>(d) * E + e] = s_mem[d * kScanCols + lane];
  if (blockIdx.x == 0) {
    float* nb = p.n_buf + (static_cast<long long>(seq) * p.H + head) * (D + 1);
    for (int d = threadIdx.x; d < D; d += 256) nb[d] = s_n[d];
    if (threadIdx.x == 0) nb[D] = m;
  }
}

// grid (128-row tiles x 128, H): head norm and gate of the rows that the kernel above wrote; normaliser and maximum.
template <typename T, typename P>
__global__ void __launch_bounds__(128) memory_head_norm_kernel(const MemoryParams p) {
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
  for (int e = threadIdx.x; e < p.E; e += 128) out[e] = from_f<T>(o[e] * rr * p.norm_w[head * p.E + e] * sigmoid_f(to_f(gp[e])));
  if (qi == p.q_lens[seq] - 1) {
    const int slot = p.seq_slots[seq];
    if (slot < 0 || slot >= p.num_slots) return;
    const float* nb = p.n_buf + (static_cast<long long>(seq) * p.H + head) * (p.D + 1);
    float* n = p.state + (static_cast<long long>(slot) * p.H + head) * state_size(p) + static_cast<long long>(p.D) * p.E;
    for (int d = threadIdx.x; d < p.D; d += 128) n[d] = nb[d];
    if (threadIdx.x == 0) p.state_m[static_cast<long long>(slot) * p.H + head] = nb[p.D];
  }
}

template <typename T, typename P, int V>
cudaError_t launch_decode(const MemoryParams& p, int slices, cudaStream_t stream) {
  const int Es = p.E / slices;
  const int groups = Es / V, gt = groups < kDecThreads ? groups : kDecThreads, lanes = kDecThreads / gt;
  const size_t smem = (3 * static_cast<size_t>(p.D) + static_cast<size_t>(lanes) * Es) * sizeof(float);
  auto kern = memory_decode_kernel<T, P, V>;
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

template <typename P>
cudaError_t launch_chunks(const MemoryParams& p, cudaStream_t stream) {
  const int chunks = 2 * p.n_tiles, slices = (p.E + ET - 1) / ET;
  const OutSmem L(p.D);
  const size_t smem1 = static_cast<size_t>(C) * (L.pitch + kPitchV);
  ensure_dynamic_smem(memory_chunk_sum_kernel<P>, smem1);
  cudaError_t e = launch_kernel(memory_chunk_sum_kernel<P>, dim3(chunks, p.H, slices), dim3(kChThreads), smem1, stream, true, false, p);
  if (e != cudaSuccess) return e;
  const long long size = static_cast<long long>(p.D) * p.E + p.D;
  const int v = p.E % 4 == 0 && p.D % 4 == 0 ? 4 : 1;
  // whole runs of 16 KB per CTA where that still leaves enough CTAs
  const bool wide = v == 4 && size >= 4096 && (size / 4096) * p.H * p.n_seqs >= 2 * sm_count();
  const long long per = 256ll * v * (wide ? 4 : 1);
  const dim3 grid2(static_cast<unsigned>((size + per - 1) / per), p.H, p.n_seqs);
  auto scan = wide ? memory_scan_chunks_kernel<4, 4, 2> : (v == 4 ? memory_scan_chunks_kernel<4, 1, 8> : memory_scan_chunks_kernel<1, 1, 8>);
  e = launch_kernel(scan, grid2, dim3(256), 0, stream, true, false, p);
  if (e != cudaSuccess) return e;
  auto kern = memory_chunk_out_kernel<P>;
  ensure_dynamic_smem(kern, static_cast<size_t>(L.total));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(chunks, p.H, slices);
  cfg.blockDim = dim3(kChThreads);
  cfg.dynamicSmemBytes = L.total;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = slices;
  cfg.numAttrs = 1;
  if (pdl_enabled()) {
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.numAttrs = 2;
  }
  cfg.attrs = attr;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

template <typename T, typename P>
cudaError_t launch_scan(const MemoryParams& p, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(p.D) * (kScanCols + 1) * sizeof(float);
  ensure_dynamic_smem(memory_scan_kernel<T, P>, smem);
  cudaError_t e = launch_kernel(memory_scan_kernel<T, P>, dim3((p.E + kScanCols - 1) / kScanCols, p.H, p.n_seqs), dim3(256), smem, stream,
                                true, false, p);
  if (e != cudaSuccess) return e;
  return launch_kernel(memory_head_norm_kernel<T, P>, dim3(p.n_tiles * 128, p.H), dim3(128), 0, stream, true, false, p);
}

}  // namespace

bool memory_chunks_ok(int D, int E) { return D <= 512 && E <= 8 * ET; }

cudaError_t launch_memory_decode(const MemoryParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  // column slices per head: enough CTAs for about two per SM, whole 16-byte pieces, at least 16 columns
  const bool vec = p.E % 4 == 0 && p.D % 4 == 0;
  int slices = 1;
  while (vec && slices < 8 && p.rows * p.H * slices < 2 * sm_count() && p.E % (slices * 2 * 4) == 0 && p.E / (slices * 2) >= 16) slices *= 2;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return vec ? launch_decode<float, float, 4>(p, slices, stream) : launch_decode<float, float, 1>(p, slices, stream);
  if (p.proj_f32) return vec ? launch_decode<bf16, float, 4>(p, slices, stream) : launch_decode<bf16, float, 1>(p, slices, stream);
  return vec ? launch_decode<bf16, bf16, 4>(p, slices, stream) : launch_decode<bf16, bf16, 1>(p, slices, stream);
}

cudaError_t launch_memory_chunks(const MemoryParams& p, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  return p.proj_f32 ? launch_chunks<float>(p, stream) : launch_chunks<__nv_bfloat16>(p, stream);
}

cudaError_t launch_memory_scan(const MemoryParams& p, int dtype, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_scan<float, float>(p, stream);
  return p.proj_f32 ? launch_scan<bf16, float>(p, stream) : launch_scan<bf16, bf16>(p, stream);
}

}  // namespace oxb
