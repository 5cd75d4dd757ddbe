// State-space layer with one decay per head and step (Mamba-2) on sm_100a:
//     S_t = a_t S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   a_t = exp(-exp(A_log) dt_t)
// with x, B and C from a short causal convolution, B and C shared by the heads of a group.
//
// Decode: one CTA per (row, head, column slice) does the convolution of the channels it needs, the step size, the
//   state update and the read-out; the head's fp32 state is streamed once. The inputs of the last `taps` tokens lie
//   in a ring by position, where a step writes an entry that no CTA of the step reads, so the convolution of the
//   shared B and C channels needs no order between CTAs.
// Prompt chunks: a convolution kernel over all rows, then one CTA per (sequence, head, column slice) that walks runs
//   of 64 tokens with the state in the accumulator registers of its warps (S^T: 16 columns of x per warp). With
//   l_i = sum_{k <= i} log a_k inside the run:
//       P_ij = (C_i . B_j) exp(l_i - l_j) dt_j  (j <= i)
//       Y    = P x + exp(l_i) C S,         S <- exp(l_end) S + sum_j exp(l_end - l_j) dt_j B_j x_j^T
//   Where sequences and heads are too few for the SMs, sequences are cut into segments: a first launch leaves every
//   segment's own contribution to the state, a scan turns these into the states before the segments, and the walk then
//   runs over all segments at once.
//   x, B and C are bf16, so C B^T is exact products summed in fp32. P, S and the weighted x are fp32: each enters its
//   product as three bf16 terms, which carry all 24 bits. An accumulator of S^T is at the same time the B-operand
//   fragment of C S, so the state never leaves the registers between runs.
// Token by token in fp32 FMAs for the 32-bit path and for state sizes above the run form's.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"
#include "hybrid_mma.cuh"

namespace oxb {

namespace {

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ int ssd_channels(const SsdParams& p) { return p.H * p.EP + 2 * p.G * p.NP; }

// ------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------
constexpr int kDecThreads = 256;
constexpr int kDecUnroll = 8;

// Convolution of one channel at the newest token: history from the ring, `cur` goes there. TAPS 0: any number.
template <int TAPS>
__device__ __forceinline__ float conv_step(const SsdParams& p, const float* ring, int c, int ch, int r0, int pos, float cur) {
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const float* w = p.conv_w + static_cast<long long>(c) * taps;
  float acc = p.conv_b[c];
  if constexpr (TAPS > 0) {
    float h[TAPS], wv[TAPS];   // all loads before the first use
#pragma unroll
    for (int k = 1; k < TAPS; ++k) {
      const int r = r0 >= k ? r0 - k : r0 - k + TAPS;
      h[k] = k <= pos ? ring[static_cast<long long>(r) * ch + c] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < TAPS; ++k) wv[k] = w[TAPS - 1 - k];
    acc = fmaf(wv[0], cur, acc);
#pragma unroll
    for (int k = 1; k < TAPS; ++k) acc = fmaf(wv[k], h[k], acc);
  } else {
    acc = fmaf(w[taps - 1], cur, acc);
    for (int k = 1; k < taps && k <= pos; ++k) {
      const int r = r0 >= k ? r0 - k : r0 - k + taps;
      acc = fmaf(w[taps - 1 - k], ring[static_cast<long long>(r) * ch + c], acc);
    }
  }
  return silu_f(acc);
}

// grid (slices, H, rows). T: storage type, P: type of the projection rows.
template <typename T, typename P, int TAPS>
__global__ void __launch_bounds__(kDecThreads, 3) ssd_decode_kernel(const SsdParams p) {
  extern __shared__ float s_mem[];
  const int EP = p.EP, NP = p.NP;
  const int Es = EP / static_cast<int>(gridDim.x);
  float* s_x = s_mem;              // Es
  float* s_b = s_x + Es;           // NP
  float* s_c = s_b + NP;           // NP
  float* s_y = s_c + NP;           // [lanes][Es]
  const int head = blockIdx.y, row = blockIdx.z, e0 = blockIdx.x * Es;
  const int group = head / (p.H / p.G);
  pdl_wait();  // the projection comes from the kernel before this one
  const int slot = p.row_slots[row];
  if (slot < 0) return;  // padding row
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const int pos = p.positions[row];
  const bool fresh = pos == 0;
  // this thread's first pieces of the state are on their way while the convolution runs
  const int groups = Es >> 2;
  const int gt = groups < kDecThreads ? groups : kDecThreads;
  const int lanes = kDecThreads / gt;
  const int cgi = threadIdx.x % gt, dl = threadIdx.x / gt;
  float* S = p.state + (static_cast<long long>(slot) * p.H + head) * NP * EP + e0;
  const int per_pass = lanes * kDecUnroll;
  float s[kDecUnroll][4];
  auto load = [&](int c, int n0) {
#pragma unroll
    for (int i = 0; i < kDecUnroll; ++i) {
      const int n = n0 + i * lanes;
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
      if (n < NP && !fresh && dl < lanes) load4<float>(S + static_cast<long long>(n) * EP + c * 4, s[i]);
    }
  };
  load(cgi, dl);

  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld;
  const int inner = p.H * EP, ch = ssd_channels(p), taps = p.taps;
  float* ring = p.conv_state + static_cast<long long>(slot) * taps * ch;
  const int r0 = pos % taps;
  const bool shared_owner = head % (p.H / p.G) == 0 && blockIdx.x == 0;   // writes the inputs of B and C
#pragma unroll 2
  for (int i = threadIdx.x; i < Es + 2 * NP; i += kDecThreads) {
    int c;                                           // channel
    if (i < Es) c = head * EP + e0 + i;
    else if (i < Es + NP) c = inner + group * NP + i - Es;
    else c = inner + p.G * NP + group * NP + i - Es - NP;
    const float cur = to_f(pr[inner + c]);
    s_x[i] = conv_step<TAPS>(p, ring, c, ch, r0, pos, cur);   // s_x, s_b and s_c follow one another
    if (i < Es || shared_owner) ring[static_cast<long long>(r0) * ch + c] = cur;
  }
  const float dt = softplus_f(to_f(pr[2 * inner + 2 * p.G * NP + head]) + p.dt_bias[head]);
  const float a = expf(-expf(p.A_log[head]) * dt);
  __syncthreads();
  if (dl < lanes) {
    for (int c = cgi; c < groups; c += gt) {
      float x[4], acc[4] = {};
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] = dt * s_x[c * 4 + j];
      for (int n0 = dl; n0 < NP; n0 += per_pass) {
        if (n0 != dl || c != cgi) load(c, n0);
#pragma unroll
        for (int i = 0; i < kDecUnroll; ++i) {
          const int n = n0 + i * lanes;
          if (n < NP) {
            const float b = s_b[n], cc = s_c[n];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              s[i][j] = fmaf(a, s[i][j], b * x[j]);
              acc[j] = fmaf(cc, s[i][j], acc[j]);
            }
            store4<float>(S + static_cast<long long>(n) * EP + c * 4, s[i]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) s_y[dl * Es + c * 4 + j] = acc[j];
    }
  }
  pdl_launch_dependents();  // the state stream of this CTA is done
  __syncthreads();
  T* y = static_cast<T*>(p.y) + static_cast<long long>(row) * p.ldy + head * EP + e0;
  const float D = p.D[head];
  for (int e = threadIdx.x; e < Es; e += kDecThreads) {
    float o = D * s_x[e];
    for (int i = 0; i < lanes; ++i) o += s_y[i * Es + e];
    y[e] = from_f<T>(o);
  }
}

// ------------------------------------------------------------------------------------------------
// convolution of prompt chunks
// ------------------------------------------------------------------------------------------------
constexpr int kConvRows = 32;   // rows per CTA, four pieces per 128-row tile

// grid (tiles * 4, channels / 1024): four channels per thread. Only the first piece of a sequence's portion reads
// inputs from before it (taps <= kConvRows), and the same thread writes the channel's new state after that.
// TAPS 0: any number of taps, inputs re-read.
template <typename T, typename P, int TAPS>
__global__ void __launch_bounds__(256, 3) ssd_conv_kernel(const SsdParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int tile = blockIdx.x >> 2, piece = blockIdx.x & 3;
  const int seq = p.tile_seq[tile];
  const int q0 = p.tile_q0[tile] + piece * kConvRows;
  const int len = p.q_lens[seq];
  const int ch = ssd_channels(p);
  const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
  if (q0 >= len || c >= ch) return;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const int past = p.ctx_lens[seq] - len;      // position of the portion's first row
  const int inner = p.H * p.EP;
  const P* src = static_cast<const P*>(p.proj) + static_cast<long long>(p.q_start[seq]) * p.ld + inner + c;
  T* dst = static_cast<T*>(p.u) + static_cast<long long>(p.q_start[seq]) * p.ldu + c;
  float* ring = p.conv_state + static_cast<long long>(slot) * taps * ch + c;
  auto input = [&](int q, float (&v)[4]) {     // input of the portion's row q, also before its start
    if (q >= 0) {
      load4<P>(src + q * p.ld, v);
    } else if (past + q >= 0) {
      load4<float>(ring + static_cast<long long>((past + q) % taps) * ch, v);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = 0.f;
    }
  };
  float b[4];
  load4<float>(p.conv_b + c, b);
  const int q1 = min(q0 + kConvRows, len);
  if constexpr (TAPS > 0) {
    constexpr int kConvBatch = sizeof(P) == 2 ? 8 : 4;   // rows whose loads are issued together
    constexpr int H = TAPS - 1;                // rows of history before a batch
    float w[4][TAPS], v[H + kConvBatch][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int k = 0; k < TAPS; ++k) w[j][k] = p.conv_w[static_cast<long long>(c + j) * TAPS + k];
#pragma unroll
    for (int k = 0; k < H; ++k) input(q0 - H + k, v[k]);
    for (int q = q0; q < q1; q += kConvBatch) {
#pragma unroll
      for (int i = 0; i < kConvBatch; ++i) {
        const int qi = q + i < q1 ? q + i : q1 - 1;   // rows past the end are not stored
        load4<P>(src + qi * p.ld, v[H + i]);
      }
#pragma unroll
      for (int i = 0; i < kConvBatch; ++i) {
        float o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float acc = b[j];
#pragma unroll
          for (int k = 0; k < TAPS; ++k) acc = fmaf(w[j][k], v[i + k][j], acc);
          o[j] = silu_as<T>(acc);
        }
        if (q + i < q1) store4<T>(dst + (q + i) * p.ldu, o);
      }
#pragma unroll
      for (int k = 0; k < H; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j) v[k][j] = v[kConvBatch + k][j];
    }
  } else {
    for (int q = q0; q < q1; ++q) {
      float acc[4] = {b[0], b[1], b[2], b[3]};
      for (int k = 0; k < taps; ++k) {
        float v[4];
        input(q - k, v);
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[j] = fmaf(p.conv_w[static_cast<long long>(c + j) * taps + taps - 1 - k], v[j], acc[j]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j] = silu_as<T>(acc[j]);
      store4<T>(dst + q * p.ldu, acc);
    }
  }
  if (q0 == 0)  // nobody else reads or writes this sequence's ring in this launch
    for (int q = max(0, len - taps); q < len; ++q) {
      float v[4];
      load4<P>(src + q * p.ld, v);
      store4<float>(ring + static_cast<long long>((past + q) % taps) * ch, v);
    }
}

// ------------------------------------------------------------------------------------------------
// runs of 64 tokens
// ------------------------------------------------------------------------------------------------
constexpr int C = 64;

// Shared memory of a CTA of W warps, state size up to 8 * NT: two stages of [C | B | x], P in three terms, step sizes.
template <int NT>
struct RunSmem {
  static constexpr int kN = NT * 8;
  static constexpr int kPitch = kN * 2 + 16;                  // bytes of a row of C or B
  static constexpr int kCB = C * kPitch;
  static constexpr int kP = C * C * 2;                        // one term, rows of 128 bytes, 16-byte chunks swizzled
  __host__ __device__ static constexpr int x_pitch(int W) { return W * 32 + 16; }
  __host__ __device__ static constexpr int stage(int W) { return 2 * kCB + C * x_pitch(W); }
  __host__ __device__ static constexpr int total(int W) { return 2 * stage(W) + 3 * kP + 7 * C * 4; }
};

// grid (column slices, H, sequences or tiles), W warps. PART 0: whole sequences; 1: what every segment (but a
// sequence's last) adds to the state; 2: outputs of every segment. A segment is named by its first tile.
template <int NT, typename P, int PART>
__global__ void __launch_bounds__(128) ssd_run_kernel(const SsdParams p) {
  using L = RunSmem<NT>;
  extern __shared__ __align__(16) uint8_t s_raw[];
  const int W = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int xp = L::x_pitch(W), stage_bytes = L::stage(W);
  const uint32_t smem = smem_u32(s_raw);
  const uint32_t sP = smem + 2 * stage_bytes;
  float* s_la = reinterpret_cast<float*>(s_raw + 2 * stage_bytes + 3 * L::kP);   // l_i
  float* s_dt = s_la + C;
  float* s_ea = s_dt + C;                                                       // exp(l_i)
  float* s_w = s_ea + C;                                                        // exp(l_end - l_j) dt_j
  // exp(l_i - l_j) dt_j of a 16 x 16 block left of the diagonal, with r the block's first row:
  // exp(l_i - l_r) times exp(l_r - l_j) dt_j, both factors at most 1 (times dt_j)
  float* s_row = s_w + C;                                                       // exp(l_i - l_(first row of i's block))
  auto col_factor = [&](int mi, int j) -> float& {                              // mi 1..3, j < 16 mi: 96 values
    return s_row[C + (mi == 1 ? 0 : (mi == 2 ? 16 : 48)) + j];
  };
  // columns of C and B beyond the state size stay zero
  const int NP = p.NP, EP = p.EP, H = p.H;
  if (NP < L::kN)
    for (int i = threadIdx.x; i < 2 * 2 * C; i += blockDim.x) {
      uint8_t* r = s_raw + (i / (2 * C)) * stage_bytes + (i % (2 * C)) * L::kPitch;
      for (int b = NP * 2; b < L::kN * 2; b += 16) *reinterpret_cast<uint4*>(r + b) = make_uint4(0, 0, 0, 0);
    }
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.y, e_cta = blockIdx.x * W * 16;
  const int tile = PART == 0 ? 0 : blockIdx.z;
  const int seq = PART == 0 ? blockIdx.z : p.tile_seq[tile];
  const int group = head / (H / p.G);
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const int q_first = PART == 0 ? 0 : p.tile_q0[tile];
  if (PART != 0 && q_first % p.segment != 0) return;
  int len = p.q_lens[seq] - q_first;           // rows of this CTA
  const bool last = PART == 0 || len <= p.segment;
  if (!last) len = p.segment;
  if (len <= 0 || (PART == 1 && last)) return;
  const long long row0 = p.q_start[seq] + q_first;
  const int inner = H * EP;
  const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(p.u) + row0 * p.ldu;
  const __nv_bfloat16* xsrc = u + head * EP + e_cta;
  const __nv_bfloat16* bsrc = u + inner + group * NP;
  const __nv_bfloat16* csrc = bsrc + p.G * NP;
  const P* dtsrc = static_cast<const P*>(p.proj) + row0 * p.ld + 2 * inner + 2 * p.G * NP + head;
  const float A = expf(p.A_log[head]), dt_bias = p.dt_bias[head], Dh = p.D[head];
  const int n_runs = (len + C - 1) / C;

  const int x_cols = min(W * 16, EP - e_cta);
  auto load_stage = [&](int c) {
    const int q0 = c * C;
    const uint32_t st = smem + (c & 1) * stage_bytes;
    // thread -> 16-byte piece of a row, rows apart by the same step every time
    {
      const int k = threadIdx.x % NT, dr = blockDim.x / NT;
      int r = threadIdx.x / NT;
      if (k * 8 < NP) {
        const long long step = dr * p.ldu;
        long long off = (q0 + r) * p.ldu + k * 8;
        uint32_t dst = st + r * L::kPitch + k * 16;
        for (; r < C; r += dr, off += step, dst += dr * L::kPitch) {
          const bool in = q0 + r < len;
          if constexpr (PART != 1) cp_async16(dst, in ? csrc + off : csrc, in);
          cp_async16(dst + L::kCB, in ? bsrc + off : bsrc, in);
        }
      }
    }
    {
      const int k = threadIdx.x % (2 * W), dr = 16;   // 2 W pieces per row, 32 W threads
      int r = threadIdx.x / (2 * W);
      const bool cols = k * 8 < x_cols;
      long long off = (q0 + r) * p.ldu + k * 8;
      uint32_t dst = st + 2 * L::kCB + r * xp + k * 16;
#pragma unroll
      for (int i = 0; i < C / 16; ++i, r += dr, off += dr * p.ldu, dst += dr * xp) {
        const bool in = cols && q0 + r < len;
        cp_async16(dst, in ? xsrc + off : xsrc, in);
      }
    }
    cp_commit();
  };
  float dt_next[2];            // last warp: raw step sizes of rows 2 lane, 2 lane + 1 of the next run
  auto load_dt = [&](int c) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int q = c * C + 2 * lane + i;
      dt_next[i] = q < len ? to_f(dtsrc[q * p.ld]) : 0.f;
    }
  };
  load_stage(0);
  if (warp == W - 1) load_dt(0);

  const int e_w = e_cta + warp * 16;   // this warp's columns
  const bool active = e_w < EP;
  float S[NT][4];                      // S^T: rows e_w + g (+ 8), columns 8 i + 2 t (+ 1)
  float* st_g = p.state + (static_cast<long long>(slot) * H + head) * NP * EP + e_w + g;
  float* ws_g = PART == 0 ? nullptr : p.ws + (static_cast<long long>(tile) * H + head) * NP * EP + e_w + g;
  const float* from = PART == 2 ? ws_g : st_g;
  const bool past = PART == 2 || (PART == 0 && p.ctx_lens[seq] != len);
  float decay_all = 1.f;               // over the rows of this CTA
#pragma unroll
  for (int i = 0; i < NT; ++i) {
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int n = i * 8 + 2 * t + (x & 1);
      S[i][x] = (past && active && n < NP) ? from[static_cast<long long>(n) * EP + (x >> 1) * 8] : 0.f;
    }
  }
  // fragment addresses: 8x8 matrices of an x4 load, rows lane & 7 of matrix lane / 8
  const int lr = lane & 7, lm = lane >> 3;
  const int row_a = (lm & 1) * 8 + lr, col_a = (lm >> 1) * 16;        // [rows 0-7 | 8-15] x [k 0-7 | 8-15]: A operands
  const int row_b = (lm >> 1) * 8 + lr, col_b = (lm & 1) * 16;        // two n tiles x [k 0-7 | 8-15]: B operands, k contiguous

  __nv_bfloat16* yrow = static_cast<__nv_bfloat16*>(p.y) + row0 * p.ldy + head * EP + e_w;
  for (int c = 0; c < n_runs; ++c) {
    const int n = min(C, len - c * C);   // rows past the end are zero and have step 0: they change nothing
    cp_wait<0>();
    __syncthreads();   // this run's stage has landed, the other stage and P have been read
    const float raw0 = dt_next[0], raw1 = dt_next[1];
    if (c + 1 < n_runs) {
      load_stage(c + 1);
      if (warp == W - 1) load_dt(c + 1);
    }
    const uint32_t sC = smem + (c & 1) * stage_bytes, sB = sC + L::kCB, sX = sB + L::kCB;
    if (warp == W - 1) {
      // step sizes and running log decays
      const float d0 = 2 * lane < n ? softplus_f(raw0 + dt_bias) : 0.f;
      const float d1 = 2 * lane + 1 < n ? softplus_f(raw1 + dt_bias) : 0.f;
      const float l0 = -A * d0, pair = l0 - A * d1;
      float incl = pair;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += up;
      }
      const float before = incl - pair;
      const float end = __shfl_sync(0xffffffffu, incl, 31);
      const float la0 = before + l0, la1 = incl;
      s_dt[2 * lane] = d0;
      s_dt[2 * lane + 1] = d1;
      s_la[2 * lane] = la0;
      s_la[2 * lane + 1] = la1;
      s_ea[2 * lane] = expf(la0);
      s_ea[2 * lane + 1] = expf(la1);
      s_w[2 * lane] = expf(end - la0) * d0;
      s_w[2 * lane + 1] = expf(end - la1) * d1;
      if constexpr (PART != 1) {
        const float ref = __shfl_sync(0xffffffffu, la0, lane & 24);   // first row of this row's block
        s_row[2 * lane] = expf(la0 - ref);
        s_row[2 * lane + 1] = expf(la1 - ref);
#pragma unroll
        for (int mi = 1; mi < 4; ++mi) {
          const float lr = __shfl_sync(0xffffffffu, la0, mi * 8);
          if (lane < mi * 8) {
            col_factor(mi, 2 * lane) = expf(lr - la0) * d0;
            col_factor(mi, 2 * lane + 1) = expf(lr - la1) * d1;
          }
        }
      }
    }
    // ---- C B^T of this warp's 16 x 16 blocks on and below the diagonal, kPar of them at a time ----
    constexpr int kItems = 10, kPar = 3;
    if constexpr (PART == 1) __syncthreads();   // step sizes are there
    for (int it0 = PART == 1 ? kItems : warp; it0 < kItems; it0 += kPar * W) {
      float cb[kPar][2][4] = {};
      int mis[kPar], njs[kPar];
#pragma unroll
      for (int y = 0; y < kPar; ++y) {
        const int it = it0 + y * W;
        mis[y] = 0;
        njs[y] = it < kItems ? it : 0;
        while (njs[y] > mis[y]) {
          njs[y] -= mis[y] + 1;
          ++mis[y];
        }
      }
#pragma unroll
      for (int k = 0; k < NT / 2; ++k)
#pragma unroll
        for (int y = 0; y < kPar; ++y)
        {   // (a block past the last one repeats the first and is not used)
          uint32_t a[4], b[4];
          ldsm4(sC + (mis[y] * 16 + row_a) * L::kPitch + k * 32 + col_a, a);
          ldsm4(sB + (njs[y] * 16 + row_b) * L::kPitch + k * 32 + col_b, b);
          mma_bf16(cb[y][0], a[0], a[1], a[2], a[3], b[0], b[1]);
          mma_bf16(cb[y][1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
      if (it0 == warp) __syncthreads();   // step sizes are there (every warp passes here once)
#pragma unroll
      for (int y = 0; y < kPar; ++y) {
        const int mi = mis[y], nj = njs[y];
        if (it0 + y * W >= kItems) continue;
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int i = mi * 16 + g + r * 8, j = nj * 16 + h * 8 + 2 * t;
            float v0, v1;
            if (nj < mi) {
              const float f = s_row[i];
              v0 = cb[y][h][2 * r] * (f * col_factor(mi, j));
              v1 = cb[y][h][2 * r + 1] * (f * col_factor(mi, j + 1));
            } else {
              const float li = s_la[i];
              v0 = j <= i ? cb[y][h][2 * r] * (expf(li - s_la[j]) * s_dt[j]) : 0.f;
              v1 = j + 1 <= i ? cb[y][h][2 * r + 1] * (expf(li - s_la[j + 1]) * s_dt[j + 1]) : 0.f;
            }
            uint32_t tm[3];
            split3(v0, v1, tm);
            const uint32_t off = i * 128 + (((j >> 3) ^ (i & 7)) << 4) + (j & 7) * 2;
#pragma unroll
            for (int x = 0; x < 3; ++x)
              asm volatile("st.shared.u32 [%0], %1;" ::"r"(sP + x * L::kP + off), "r"(tm[x]) : "memory");
          }
      }
    }
    // ---- exp(l_i) C S ----
    float Y[4][2][4] = {};
    if (PART != 1 && active) {
#pragma unroll
      for (int k = 0; k < NT / 2; ++k) {
        uint32_t b[2][2][3];   // [column tile][k half][term]
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int q = 0; q < 2; ++q) split3(S[2 * k + q][2 * h], S[2 * k + q][2 * h + 1], b[h][q]);
        uint32_t a[4][4];
#pragma unroll
        for (int mi = 0; mi < 4; ++mi)
          ldsm4(sC + (mi * 16 + row_a) * L::kPitch + k * 32 + col_a, a[mi]);
        // eight independent products between two of one accumulator
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
          for (int mi = 0; mi < 4; ++mi)
#pragma unroll
            for (int h = 0; h < 2; ++h) mma_bf16(Y[mi][h], a[mi][0], a[mi][1], a[mi][2], a[mi][3], b[h][0][x], b[h][1][x]);
      }
#pragma unroll
      for (int mi = 0; mi < 4; ++mi) {
        const float f0 = s_ea[mi * 16 + g], f1 = s_ea[mi * 16 + g + 8];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          Y[mi][h][0] *= f0;
          Y[mi][h][1] *= f0;
          Y[mi][h][2] *= f1;
          Y[mi][h][3] *= f1;
        }
      }
    }
    if constexpr (PART != 1) __syncthreads();   // P is there
    if constexpr (PART == 1) decay_all *= s_ea[C - 1];
    if (active) {
      const float a_end = s_ea[C - 1];
#pragma unroll
      for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) S[i][x] *= a_end;
#pragma unroll
      for (int kj = 0; kj < 4; ++kj) {
        // x rows of this block as B operand [k = j][n = e] and, transposed, as A operand [m = e][k = j]
        uint32_t xb[4];
        ldsm4t(sX + (kj * 16 + row_a) * xp + warp * 32 + col_a, xb);   // (j lo, e lo) (j hi, e lo) (j lo, e hi) (j hi, e hi)
        // ---- Y += P x ----
#pragma unroll
        for (int x = 2; x >= 0; --x)
#pragma unroll
          for (int mi = kj; mi < 4; ++mi)
            if (PART != 1) {
              const int pr = mi * 16 + row_a;
              uint32_t a[4];
              ldsm4(sP + x * L::kP + pr * 128 + (((kj * 2 + (col_a >> 4)) ^ (pr & 7)) << 4), a);
              mma_bf16(Y[mi][0], a[0], a[1], a[2], a[3], xb[0], xb[1]);
              mma_bf16(Y[mi][1], a[0], a[1], a[2], a[3], xb[2], xb[3]);
            }
        // ---- S^T += (w_j x_j)^T B_j ----
        uint32_t av[4][3];   // A fragments: (e lo, j lo) (e hi, j lo) (e lo, j hi) (e hi, j hi)
        const int j0 = kj * 16 + 2 * t;
        const float w0 = s_w[j0], w1 = s_w[j0 + 1], w2 = s_w[j0 + 8], w3 = s_w[j0 + 9];
        auto weigh = [&](uint32_t v, float p0, float p1, uint32_t (&o)[3]) {
          split3(__uint_as_float(v << 16) * p0, __uint_as_float(v & 0xffff0000u) * p1, o);
        };
        weigh(xb[0], w0, w1, av[0]);
        weigh(xb[2], w0, w1, av[1]);
        weigh(xb[1], w2, w3, av[2]);
        weigh(xb[3], w2, w3, av[3]);
        constexpr int kPairs = NT >= 8 ? 4 : NT / 2;   // pairs of column tiles at a time
#pragma unroll
        for (int i = 0; i < NT; i += 2 * kPairs) {
          uint32_t b[kPairs][4];   // (j lo, n lo) (j hi, n lo) (j lo, n hi) (j hi, n hi)
#pragma unroll
          for (int q = 0; q < kPairs; ++q) ldsm4t(sB + (kj * 16 + row_a) * L::kPitch + (i + 2 * q) * 16 + col_a, b[q]);
#pragma unroll
          for (int x = 2; x >= 0; --x)
#pragma unroll
            for (int q = 0; q < kPairs; ++q) {
              mma_bf16(S[i + 2 * q], av[0][x], av[1][x], av[2][x], av[3][x], b[q][0], b[q][1]);
              mma_bf16(S[i + 2 * q + 1], av[0][x], av[1][x], av[2][x], av[3][x], b[q][2], b[q][3]);
            }
        }
      }
      // ---- Y + D x ----
#pragma unroll
      for (int mi = 0; mi < 4; ++mi)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int i = mi * 16 + g + r * 8;
          if (PART == 1 || i >= n) continue;
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int e = h * 8 + 2 * t;
            uint32_t xv;
            asm volatile("ld.shared.u32 %0, [%1];" : "=r"(xv) : "r"(sX + i * xp + warp * 32 + e * 2));
            const float y0 = fmaf(Dh, __uint_as_float(xv << 16), Y[mi][h][2 * r]);
            const float y1 = fmaf(Dh, __uint_as_float(xv & 0xffff0000u), Y[mi][h][2 * r + 1]);
            *reinterpret_cast<uint32_t*>(yrow + static_cast<long long>(c * C + i) * p.ldy + e) = pack_bf16x2(y0, y1);
          }
        }
    }
  }
  if (active && (PART == 1 || last)) {
    float* to = PART == 1 ? ws_g : st_g;
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int nn = i * 8 + 2 * t + (x & 1);
        if (nn < NP) to[static_cast<long long>(nn) * EP + (x >> 1) * 8] = S[i][x];
      }
  }
  if (PART == 1 && threadIdx.x == 0 && blockIdx.x == 0) p.ws_decay[static_cast<long long>(tile) * H + head] = decay_all;
}

// Contributions of the segments -> states before the segments. grid (NP EP / 1024, H, sequences).
__global__ void __launch_bounds__(256) ssd_segment_scan_kernel(const SsdParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const long long ne = static_cast<long long>(p.NP) * p.EP;
  const long long i0 = (static_cast<long long>(blockIdx.x) * 256 + threadIdx.x) * 4;
  if (i0 >= ne) return;
  const int slot = p.seq_slots[seq], len = p.q_lens[seq];
  if (slot < 0 || slot >= p.num_slots) return;
  int tile0 = 0;
  for (int s = 0; s < seq; ++s) tile0 += (p.q_lens[s] + 127) >> 7;
  const int n_seg = (len + p.segment - 1) / p.segment, per = p.segment >> 7;
  float S[4] = {0.f, 0.f, 0.f, 0.f};
  if (p.ctx_lens[seq] != len) load4<float>(p.state + (static_cast<long long>(slot) * p.H + head) * ne + i0, S);
  constexpr int U = 4;   // segments whose loads are issued together
  for (int s0 = 0; s0 < n_seg; s0 += U) {
    float u[U][4], a[U];
#pragma unroll
    for (int k = 0; k < U; ++k)
      if (s0 + k < n_seg - 1) {
        const long long at = static_cast<long long>(tile0 + (s0 + k) * per) * p.H + head;
        load4<float>(p.ws + at * ne + i0, u[k]);
        a[k] = p.ws_decay[at];
      }
#pragma unroll
    for (int k = 0; k < U; ++k)
      if (s0 + k < n_seg) {
        store4<float>(p.ws + (static_cast<long long>(tile0 + (s0 + k) * per) * p.H + head) * ne + i0, S);
        if (s0 + k < n_seg - 1) {
#pragma unroll
          for (int j = 0; j < 4; ++j) S[j] = fmaf(a[k], S[j], u[k][j]);
        }
      }
  }
}

// ------------------------------------------------------------------------------------------------
// token by token
// ------------------------------------------------------------------------------------------------
constexpr int kScanCols = 32;

// grid (EP / 32, H, sequences): 32 state columns in shared memory, 8 warps split the state dimension.
template <typename T, typename P>
__global__ void __launch_bounds__(256) ssd_scan_kernel(const SsdParams p) {
  extern __shared__ float s_mem[];
  __shared__ float s_o[8][kScanCols];
  pdl_wait();
  const int NP = p.NP, EP = p.EP;
  const int seq = blockIdx.z, head = blockIdx.y, group = head / (p.H / p.G);
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int e = blockIdx.x * kScanCols + lane;
  const int slot = p.seq_slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    return;
  }
  float* st = p.state + (static_cast<long long>(slot) * p.H + head) * NP * EP;
  const int len = p.q_lens[seq];
  const bool fresh = p.ctx_lens[seq] == len;
  for (int d = w; d < NP; d += 8) s_mem[d * kScanCols + lane] = (fresh || e >= EP) ? 0.f : st[static_cast<long long>(d) * EP + e];
  const int inner = p.H * EP;
  const float A = expf(p.A_log[head]), dt_bias = p.dt_bias[head], D = p.D[head];
  for (int i = 0; i < len; ++i) {
    const long long row = p.q_start[seq] + i;
    const T* u = static_cast<const T*>(p.u) + row * p.ldu;
    const T* b = u + inner + group * NP;
    const T* cc = b + p.G * NP;
    const float dt = softplus_f(to_f(static_cast<const P*>(p.proj)[row * p.ld + 2 * inner + 2 * p.G * NP + head]) + dt_bias);
    const float a = expf(-A * dt);
    const float x = e < EP ? to_f(u[head * EP + e]) : 0.f;
    const float dx = dt * x;
    float acc = 0.f;
    for (int d = w; d < NP; d += 8) {
      const float s = fmaf(a, s_mem[d * kScanCols + lane], to_f(b[d]) * dx);
      s_mem[d * kScanCols + lane] = s;
      acc = fmaf(to_f(cc[d]), s, acc);
    }
    s_o[w][lane] = acc;
    __syncthreads();
    if (w == 0 && e < EP) {
      float o = D * x;
#pragma unroll
      for (int k = 0; k < 8; ++k) o += s_o[k][lane];
      static_cast<T*>(p.y)[row * p.ldy + head * EP + e] = from_f<T>(o);
    }
    __syncthreads();
  }
  if (e < EP)
    for (int d = w; d < NP; d += 8) st[static_cast<long long>(d) * EP + e] = s_mem[d * kScanCols + lane];
}

// ------------------------------------------------------------------------------------------------
// gate and norm
// ------------------------------------------------------------------------------------------------
// One (row, part) per CTA, or per warp (WARPS) where a part is small; the gated values of a part wait in shared
// memory for its root mean square.
template <typename T, typename P, bool WARPS>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNormParams p) {
  extern __shared__ __align__(16) float s_mem[];
  __shared__ float s_red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int inner = p.H * p.E, part = inner / p.groups;
  const int TPG = WARPS ? 32 : blockDim.x;
  const int sub = WARPS ? threadIdx.x >> 5 : 0, tid = WARPS ? threadIdx.x & 31 : threadIdx.x;
  const long long item = WARPS ? static_cast<long long>(blockIdx.x) * 8 + sub : blockIdx.x;
  const bool on = item < static_cast<long long>(p.M) * p.groups;
  const long long row = on ? item / p.groups : 0;
  const int c0 = on ? static_cast<int>(item - row * p.groups) * part : 0;
  float* s_g = s_mem + static_cast<long long>(sub) * part;
  const T* y = static_cast<const T*>(p.y) + row * p.ldy;
  const P* z = static_cast<const P*>(p.z) + row * p.ldz;
  T* out = static_cast<T*>(p.out) + row * p.ldo + c0;
  const bool vec = p.E == p.EP && part % 4 == 0 && p.ldy % 4 == 0 && p.ldz % 4 == 0 && p.ldo % 4 == 0;
  float ss = 0.f;
  if (on) {
    if (vec) {
#pragma unroll 4
      for (int c = tid * 4; c < part; c += TPG * 4) {
        float a[4], b[4];
        load4<T>(y + c0 + c, a);
        load4<P>(z + c0 + c, b);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          a[j] *= silu_as<T>(b[j]);
          ss = fmaf(a[j], a[j], ss);
        }
        store4<float>(s_g + c, a);
      }
    } else {
      for (int c = tid; c < part; c += TPG) {
        const int h = (c0 + c) / p.E, k = h * p.EP + (c0 + c) - h * p.E;
        const float a = to_f(y[k]) * silu_as<T>(to_f(z[k]));
        ss = fmaf(a, a, ss);
        s_g[c] = a;
      }
    }
  }
  const float total = WARPS ? warp_sum(ss) : block_sum_all(ss, s_red);
  if (!on) return;
  const float r = 1.f / sqrtf(total / static_cast<float>(part) + p.eps);
  if (vec) {
    for (int c = tid * 4; c < part; c += TPG * 4) {
      float a[4], w[4];
      load4<float>(s_g + c, a);
      load4<float>(p.w + c0 + c, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) a[j] *= r * w[j];
      store4<T>(out + c, a);
    }
  } else {
    for (int c = tid; c < part; c += TPG) out[c] = from_f<T>(s_g[c] * r * p.w[c0 + c]);
  }
}

template <typename T, typename P>
cudaError_t launch_decode(const SsdParams& p, int slices, cudaStream_t stream) {
  const int Es = p.EP / slices, groups = Es >> 2;
  const int gt = groups < kDecThreads ? groups : kDecThreads, lanes = kDecThreads / gt;
  const size_t smem = (Es + 2 * static_cast<size_t>(p.NP) + static_cast<size_t>(lanes) * Es) * sizeof(float);
  auto kern = p.taps == 4 ? ssd_decode_kernel<T, P, 4> : ssd_decode_kernel<T, P, 0>;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(slices, p.H, p.rows), dim3(kDecThreads), smem, stream, true, false, p);
}

template <typename T, typename P>
cudaError_t launch_conv(const SsdParams& p, cudaStream_t stream) {
  const int ch = p.H * p.EP + 2 * p.G * p.NP;
  const dim3 grid(p.n_tiles * 4, (ch + 1023) / 1024);
  if (p.taps == 4) return launch_kernel(ssd_conv_kernel<T, P, 4>, grid, dim3(256), 0, stream, true, false, p);
  return launch_kernel(ssd_conv_kernel<T, P, 0>, grid, dim3(256), 0, stream, true, false, p);
}

int run_warps(int EP) { return EP / 16 < 2 ? 1 : (EP / 16 < 4 ? 2 : 4); }   // of 16 columns each

template <int NT, typename P>
cudaError_t launch_run(const SsdParams& p, cudaStream_t stream) {
  const int W = run_warps(p.EP);
  const size_t smem = RunSmem<NT>::total(W);
  const int slices = (p.EP + W * 16 - 1) / (W * 16);
  if (p.segment <= 0) {
    ensure_dynamic_smem(ssd_run_kernel<NT, P, 0>, smem);
    return launch_kernel(ssd_run_kernel<NT, P, 0>, dim3(slices, p.H, p.n_seqs), dim3(W * 32), smem, stream, true, false, p);
  }
  ensure_dynamic_smem(ssd_run_kernel<NT, P, 1>, smem);
  ensure_dynamic_smem(ssd_run_kernel<NT, P, 2>, smem);
  const dim3 grid(slices, p.H, p.n_tiles);
  cudaError_t e = launch_kernel(ssd_run_kernel<NT, P, 1>, grid, dim3(W * 32), smem, stream, true, false, p);
  if (e != cudaSuccess) return e;
  const dim3 sgrid((p.NP * p.EP + 1023) / 1024, p.H, p.n_seqs);
  e = launch_kernel(ssd_segment_scan_kernel, sgrid, dim3(256), 0, stream, true, false, p);
  if (e != cudaSuccess) return e;
  return launch_kernel(ssd_run_kernel<NT, P, 2>, grid, dim3(W * 32), smem, stream, true, false, p);
}
template <typename P>
cudaError_t run_of(const SsdParams& p, cudaStream_t stream) {
  if (p.NP <= 32) return launch_run<4, P>(p, stream);
  if (p.NP <= 64) return launch_run<8, P>(p, stream);
  if (p.NP <= 128) return launch_run<16, P>(p, stream);
  if (p.NP <= 256) return launch_run<32, P>(p, stream);
  return cudaErrorInvalidValue;
}

template <typename T, typename P>
cudaError_t launch_scan(const SsdParams& p, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(p.NP) * kScanCols * sizeof(float);
  ensure_dynamic_smem(ssd_scan_kernel<T, P>, smem);
  return launch_kernel(ssd_scan_kernel<T, P>, dim3((p.EP + kScanCols - 1) / kScanCols, p.H, p.n_seqs), dim3(256), smem, stream, true,
                       false, p);
}

template <typename T, typename P>
cudaError_t launch_gated(const GatedNormParams& p, cudaStream_t stream) {
  const int part = p.H * p.E / p.groups;
  const long long items = static_cast<long long>(p.M) * p.groups;
  if (part <= 128 || (part <= 1024 && items >= 32ll * sm_count())) {
    const size_t smem = 8 * static_cast<size_t>(part) * sizeof(float);
    return launch_kernel(gated_norm_kernel<T, P, true>, dim3(static_cast<unsigned>((items + 7) / 8)), dim3(256), smem, stream, true,
                         false, p);
  }
  const size_t smem = static_cast<size_t>(part) * sizeof(float);
  ensure_dynamic_smem(gated_norm_kernel<T, P, false>, smem);
  const int threads = part >= 1024 ? 256 : (part / 4 + 31) / 32 * 32;
  return launch_kernel(gated_norm_kernel<T, P, false>, dim3(static_cast<unsigned>(items)), dim3(threads), smem, stream, true, false, p);
}

}  // namespace

bool ssd_chunks_ok(int NP) { return NP <= 256; }

int ssd_segment(int H, int EP, int n_tiles, int n_seqs) {
  const int W = run_warps(EP), slices = (EP + W * 16 - 1) / (W * 16);
  const int slots = 2 * sm_count();   // CTAs that run at a time
  if (static_cast<long long>(slices) * H * n_seqs * 4 >= 3ll * slots || n_tiles < 3 * n_seqs) return 0;
  int seg = 256;
  while (seg < 2048 && static_cast<long long>(n_tiles) * 128 / seg * slices * H > 4ll * slots) seg *= 2;
  return seg;
}

cudaError_t launch_ssd_decode(const SsdParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  int slices = 1;   // of at least 16 columns, until about two CTAs per SM exist
  while (p.rows * p.H * slices < 2 * sm_count() && p.EP % (slices * 2 * 4) == 0 && p.EP / (slices * 2) >= 16) slices *= 2;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_decode<float, float>(p, slices, stream);
  return p.proj_f32 ? launch_decode<bf16, float>(p, slices, stream) : launch_decode<bf16, bf16>(p, slices, stream);
}

cudaError_t launch_ssd_conv(const SsdParams& p, int dtype, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  if (p.taps > kConvRows) return cudaErrorInvalidValue;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_conv<float, float>(p, stream);
  return p.proj_f32 ? launch_conv<bf16, float>(p, stream) : launch_conv<bf16, bf16>(p, stream);
}

cudaError_t launch_ssd_chunks(const SsdParams& p, cudaStream_t stream) {
  if (p.n_seqs <= 0) return cudaSuccess;
  return p.proj_f32 ? run_of<float>(p, stream) : run_of<__nv_bfloat16>(p, stream);
}

cudaError_t launch_ssd_scan(const SsdParams& p, int dtype, cudaStream_t stream) {
  if (p.n_seqs <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_scan<float, float>(p, stream);
  return p.proj_f32 ? launch_scan<bf16, float>(p, stream) : launch_scan<bf16, bf16>(p, stream);
}

cudaError_t launch_gated_norm(const GatedNormParams& p, int dtype, cudaStream_t stream) {
  if (p.M <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  if (dtype == 1) return launch_gated<float, float>(p, stream);
  return p.z_f32 ? launch_gated<bf16, float>(p, stream) : launch_gated<bf16, bf16>(p, stream);
}

}  // namespace oxb
