// Gated recurrence whose gates read only the current token (minGRU, sm_100a): S <- (1 - z) S + z c, element by element. It is
// computed as S + z (c - S): with 1 - z as a factor its rounding would add up over the thousands of tokens that a small z keeps.
// A run of tokens makes S -> S + (b - d S) of a state (d = 1 - the product of all 1 - z, b: what the run makes of 0).
// Prompts: every 32-row part of a tile is walked by itself for its (d, b), then,
// knowing what the rows before it make of the sequence's state, walked again for the outputs; both passes are streams of the
// projection rows. Decoding: one launch, a thread per four channels of a row. Gates, candidates and states are fp32.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

constexpr int kTileRows = 128;
constexpr int kPartRows = kTileRows / kGruParts;
constexpr int kQuads = 64;   // four-channel columns per CTA

// z and c of one channel. FAST: hardware exponential and reciprocal (both good to about 2^-22), for rows that come
// as bf16 products.
template <bool FAST>
__device__ __forceinline__ void gates(float zin, float u, float* z, float* c) {
  if constexpr (FAST) {   // one reciprocal for both
    const float a = 1.f + __expf(-fmaxf(zin, -40.f)), b = 1.f + __expf(fminf(-u, 40.f));
    const float r = __fdividef(1.f, a * b);
    *z = r * b;
    *c = u >= 0.f ? u + 0.5f : r * a;
  } else {
    *z = 1.f / (1.f + expf(-fmaxf(zin, -80.f)));
    *c = u >= 0.f ? u + 0.5f : 1.f / (1.f + expf(fminf(-u, 80.f)));
  }
}
// a state (or a run's b) one token on; a state after a run
__device__ __forceinline__ float step_of(float s, float z, float c) { return fmaf(z, c - s, s); }
__device__ __forceinline__ float after(float s, float d, float b) { return s + fmaf(-d, s, b); }
template <bool FAST>
__device__ __forceinline__ float silu_of(float g) {
  return FAST ? __fdividef(g, 1.f + __expf(fminf(-g, 80.f))) : g / (1.f + expf(fminf(-g, 80.f)));
}

template <typename T, typename P>
__global__ void __launch_bounds__(128) gru_decode_kernel(const GruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  pdl_launch_dependents();
  const int row = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * 4, N = p.N;
  if (c >= N) return;
  float bz[4], bx[4], z[4], u[4], g[4], s[4] = {0.f, 0.f, 0.f, 0.f};
  load4<float>(p.bias + c, bz);
  load4<float>(p.bias + N + c, bx);
  pdl_wait();  // the projection and the step's slots come from earlier kernels
  const int slot = p.row_slots[row];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    set_status_once(p.status, kStatusBadIndex);
    return;
  }
  const P* pr = static_cast<const P*>(p.proj) + static_cast<long long>(row) * p.ld + c;
  float* st = p.state + static_cast<long long>(slot) * N + c;
  load4_stream(pr, z);
  load4_stream(pr + N, u);
  load4_stream(pr + 2 * N, g);
  if (p.positions[row] > 0) load4_stream(st, s);
  float o[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    float zj, cj;
    gates<FAST>(z[j] + bz[j], u[j] + bx[j], &zj, &cj);
    s[j] = step_of(s[j], zj, cj);
    o[j] = s[j] * silu_of<FAST>(g[j]) * p.out_gain;
  }
  store4<float>(st, s);
  store4<T>(static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + c, o);
}

struct TileRows {
  int n;          // rows of the tile
  long long row;  // first one
  int first;      // the sequence's first tile in this step
  int slot;
  bool fresh, last;
};
__device__ __forceinline__ TileRows tile_rows(const GruParams& p, int tile) {
  TileRows t;
  const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile], len = p.q_lens[seq];
  t.n = min(kTileRows, len - q0);
  t.row = p.q_start[seq] + q0;
  t.first = tile - q0 / kTileRows;
  t.slot = p.seq_slots[seq];
  t.fresh = p.ctx_lens[seq] == len;
  t.last = q0 + kTileRows >= len;
  return t;
}
// (d, b) of a tile (part 0) or of one of its parts (1 ..)
__device__ __forceinline__ float* ws_of(const GruParams& p, int tile, int part) {
  return p.ws + (static_cast<long long>(tile) * (1 + kGruParts) + part) * 2 * p.N;
}

// What every part and every tile makes of a state. The first tile of a sequence takes the state itself: b is the state after
// it, d the state before it.
template <typename T, typename P>
__global__ void __launch_bounds__(kQuads * kGruParts) gru_sums_kernel(const GruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float4 s_d[kGruParts][kQuads], s_b[kGruParts][kQuads];
  pdl_launch_dependents();
  pdl_wait();
  const int part = threadIdx.y, N = p.N, c = (blockIdx.x * kQuads + threadIdx.x) * 4, tile = blockIdx.y;
  const TileRows t = tile_rows(p, tile);
  const bool in = c < N;
  if (in) {
    float bz[4], bx[4], d[4] = {}, b[4] = {};
    load4<float>(p.bias + c, bz);
    load4<float>(p.bias + N + c, bx);
    const int r0 = part * kPartRows, r1 = min(r0 + kPartRows, t.n);
    const P* pr = static_cast<const P*>(p.proj) + t.row * p.ld + c;
#pragma unroll 8
    for (int r = r0; r < r1; ++r) {
      float z[4], u[4];
      load4_stream(pr + r * p.ld, z);
      load4_stream(pr + r * p.ld + N, u);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float zj, cj;
        gates<FAST>(z[j] + bz[j], u[j] + bx[j], &zj, &cj);
        d[j] = step_of(d[j], zj, 1.f);
        b[j] = step_of(b[j], zj, cj);
      }
    }
    float* w = ws_of(p, tile, 1 + part);
    store4<float>(w + c, d);
    store4<float>(w + N + c, b);
    s_d[part][threadIdx.x] = make_float4(d[0], d[1], d[2], d[3]);
    s_b[part][threadIdx.x] = make_float4(b[0], b[1], b[2], b[3]);
  }
  __syncthreads();
  if (!in || part != 0) return;
  const bool first = tile == t.first;
  float d[4] = {}, b[4] = {}, start[4] = {};
  if (first && !t.fresh) {
    if (t.slot >= 0 && t.slot < p.num_slots) load4_stream(p.state + static_cast<long long>(t.slot) * N + c, start);
    else set_status_once(p.status, kStatusBadIndex);
#pragma unroll
    for (int j = 0; j < 4; ++j) b[j] = start[j];
  }
#pragma unroll
  for (int k = 0; k < kGruParts; ++k) {
    const float4 x = s_d[k][threadIdx.x], y = s_b[k][threadIdx.x];
    const float xd[4] = {x.x, x.y, x.z, x.w}, yb[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      b[j] = after(b[j], xd[j], yb[j]);
      d[j] = after(d[j], xd[j], xd[j]);
    }
  }
  float* w = ws_of(p, tile, 0);
  store4<float>(w + c, first ? start : d);
  store4<float>(w + N + c, b);
}

// The state before each part, then its rows once more for the outputs. The parts share the walk over the sequence's earlier
// tiles; the last tile's last part leaves the new state.
template <typename T, typename P>
__global__ void __launch_bounds__(kQuads * kGruParts) gru_outputs_kernel(const GruParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float4 s_d[kGruParts][kQuads], s_b[kGruParts][kQuads];
  pdl_launch_dependents();
  pdl_wait();
  const int part = threadIdx.y, N = p.N, c = (blockIdx.x * kQuads + threadIdx.x) * 4, tile = blockIdx.y;
  const TileRows t = tile_rows(p, tile);
  const bool in = c < N;
  const int before = tile - t.first;
  if (in) {
    const int per = (before + kGruParts - 1) / kGruParts;
    const int k0 = t.first + part * per, k1 = min(k0 + per, tile);
    float d[4] = {}, b[4] = {};
#pragma unroll 4
    for (int k = k0; k < k1; ++k) {
      const float* w = ws_of(p, k, 0);
      float x[4], y[4];
      load4_stream(w + c, x);
      load4_stream(w + N + c, y);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float xd = k == t.first ? 1.f : x[j];   // nothing comes before the first tile: b is the state after it
        b[j] = after(b[j], xd, y[j]);
        d[j] = after(d[j], xd, xd);
      }
    }
    s_d[part][threadIdx.x] = make_float4(d[0], d[1], d[2], d[3]);
    s_b[part][threadIdx.x] = make_float4(b[0], b[1], b[2], b[3]);
  }
  __syncthreads();
  if (!in) return;
  float s[4] = {};
  if (before == 0) {
    load4_stream(ws_of(p, tile, 0) + c, s);
  } else {
#pragma unroll
    for (int k = 0; k < kGruParts; ++k) {
      const float4 x = s_d[k][threadIdx.x], y = s_b[k][threadIdx.x];
      const float xd[4] = {x.x, x.y, x.z, x.w}, yb[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j] = after(s[j], xd[j], yb[j]);
    }
  }
  for (int k = 0; k < part; ++k) {
    const float* w = ws_of(p, tile, 1 + k);
    float x[4], y[4];
    load4_stream(w + c, x);
    load4_stream(w + N + c, y);
#pragma unroll
    for (int j = 0; j < 4; ++j) s[j] = after(s[j], x[j], y[j]);
  }
  float bz[4], bx[4];
  load4<float>(p.bias + c, bz);
  load4<float>(p.bias + N + c, bx);
  const int r0 = part * kPartRows, r1 = min(r0 + kPartRows, t.n);
  const P* pr = static_cast<const P*>(p.proj) + t.row * p.ld + c;
  T* out = static_cast<T*>(p.out) + t.row * p.ldo + c;
#pragma unroll 4
  for (int r = r0; r < r1; ++r) {
    float z[4], u[4], g[4], o[4];
    load4_stream(pr + r * p.ld, z);
    load4_stream(pr + r * p.ld + N, u);
    load4_stream(pr + r * p.ld + 2 * N, g);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float zj, cj;
      gates<FAST>(z[j] + bz[j], u[j] + bx[j], &zj, &cj);
      s[j] = step_of(s[j], zj, cj);
      o[j] = s[j] * silu_of<FAST>(g[j]) * p.out_gain;
    }
    store4<T>(out + r * p.ldo, o);
  }
  if (t.last && r0 < t.n && r1 == t.n) {
    if (t.slot >= 0 && t.slot < p.num_slots) store4<float>(p.state + static_cast<long long>(t.slot) * N + c, s);
    else set_status_once(p.status, kStatusBadIndex);
  }
}

}  // namespace

cudaError_t launch_gru_decode(const GruParams& p, int dtype, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  auto kern = dtype == 1 ? gru_decode_kernel<float, float> : (p.proj_f32 ? gru_decode_kernel<bf16, float> : gru_decode_kernel<bf16, bf16>);
  return launch_kernel(kern, dim3((p.N / 4 + 127) / 128, p.rows), dim3(128), 0, stream, true, false, p);
}

cudaError_t launch_gru_prefill(const GruParams& p, int dtype, cudaStream_t stream) {
  if (p.n_tiles <= 0) return cudaSuccess;
  using bf16 = __nv_bfloat16;
  auto sums = dtype == 1 ? gru_sums_kernel<float, float> : (p.proj_f32 ? gru_sums_kernel<bf16, float> : gru_sums_kernel<bf16, bf16>);
  auto outs = dtype == 1 ? gru_outputs_kernel<float, float> : (p.proj_f32 ? gru_outputs_kernel<bf16, float> : gru_outputs_kernel<bf16, bf16>);
  const dim3 grid((p.N / 4 + kQuads - 1) / kQuads, p.n_tiles), block(kQuads, kGruParts);
  const cudaError_t e = launch_kernel(sums, grid, block, 0, stream, true, false, p);
  if (e != cudaSuccess) return e;
  return launch_kernel(outs, grid, block, 0, stream, true, false, p);
}

}  // namespace oxb
