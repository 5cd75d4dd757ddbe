// Latent attention (sm_100a): a token keeps one row of R latent values and T rotated key values for all heads.
//
// latent_rows: projection rows -> normed query latent, normed latent and rotated key part into the paged cache.
// latent_gather: cache rows of a step's prompts one after the other, the operand of the GEMM that expands them to
//   keys and values per head (prompts run the plain-row form of the prefill attention).
// latent_decode: decode rows against the latents themselves. With the key expansion moved to the query (q' = W_uk^T q)
//   and the value expansion behind the sum, all heads of a row share one key, which is also the value: the cache row is
//   read once for scores and sums. One CTA = (row, 16 or 32 heads, KV split); tiles of two pages are staged by cp.async
//   (the next one on its way), eight warps share the products of a tile by keys and halves of the row (scores), by
//   value columns (sums). Heads are the M dimension of mma.sync m16n8k16: sixteen query rows against a stream that is
//   bound by HBM cannot fill a 128-row tcgen05 tile.
#include "../common/device_info.h"
#include "hybrid_dev.cuh"
#include "hybrid_mma.cuh"

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

// ------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------
constexpr int kLatWarps = 8, kLatKeys = 32, kLatStages = 2;
constexpr int kPitchS = kLatKeys + 4;        // fp32 scores
constexpr int kPitchP = kLatKeys * 2 + 16;   // bytes of a row of bf16 weights

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct LatentSmem {
  int pitch, q, tile, s, pw, alpha, total;
  __host__ __device__ LatentSmem(int CP, int heads) {
    pitch = CP * 2 + 16;      // rows start in different banks
    q = 0;
    tile = heads * pitch;
    s = tile + kLatStages * kLatKeys * pitch;
    pw = s + 2 * heads * kPitchS * 4;
    alpha = pw + 2 * heads * kPitchP;
    total = alpha + heads * 4;
  }
};

// HT: tiles of 16 heads; NP: pairs of 8-column value tiles per warp.
template <int HT, int NP>
__global__ void __launch_bounds__(kLatWarps * 32, HT * NP <= 4 ? 2 : 1) latent_decode_kernel(const LatentDecodeParams p) {
  extern __shared__ __align__(16) uint8_t s_raw[];
  constexpr int kHeads = HT * 16;
  const LatentSmem L(p.CP, kHeads);
  const uint32_t smem = smem_u32(s_raw);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int row = blockIdx.x, h0 = blockIdx.y * kHeads, split = blockIdx.z;
  pdl_wait();
  const int seq_len = p.seq_lens[row];
  int n_pages = (seq_len + 15) / 16;
  if (n_pages > p.max_blocks) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    n_pages = p.max_blocks;
  }
  const int pps = (*p.pages_per_split + 1) & ~1;
  const int pg_lo = split * pps, pg_hi = min(pg_lo + pps, n_pages);
  const long long part0 = (static_cast<long long>(row) * p.H + h0) * p.max_splits + split;
  if (pg_lo >= pg_hi) {
    for (int h = threadIdx.x; h < kHeads && h0 + h < p.H; h += blockDim.x) {
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2] = -INFINITY;
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2 + 1] = 0.f;
    }
    return;
  }
  const int cpr = p.CP >> 3;   // 16-byte pieces of a row
  // queries (heads past the last one are zero)
  for (int r = warp; r < kHeads; r += kLatWarps) {
    const bool in = h0 + r < p.H;
    const __nv_bfloat16* src = p.q + (static_cast<long long>(row) * p.H + (in ? h0 + r : 0)) * p.CP;
    for (int c = lane; c < cpr; c += 32) cp_async16(smem + L.q + r * L.pitch + c * 16, src + c * 8, in);
  }
  const int* bt = p.block_tables + static_cast<long long>(row) * p.max_blocks;
  auto issue = [&](int it) {
    const uint32_t dst0 = smem + L.tile + (it & 1) * kLatKeys * L.pitch;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int page = pg_lo + it * 2 + half;
      const bool in = page < pg_hi;
      int b = in ? bt[page] : 0;
      if (static_cast<unsigned>(b) >= static_cast<unsigned>(p.num_blocks)) {
        if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
        b = 0;
      }
      const __nv_bfloat16* src = p.cache + static_cast<long long>(b) * 16 * p.CP;
#pragma unroll
      for (int i = 0; i < 16 / kLatWarps; ++i) {
        const int r = warp + i * kLatWarps;
        const uint32_t dst = dst0 + (half * 16 + r) * L.pitch;
        for (int c = lane; c < cpr; c += 32) cp_async16(dst + c * 16, src + r * p.CP + c * 8, in);
      }
    }
    cp_commit();
  };
  const int n_it = (pg_hi - pg_lo + 1) / 2;
  issue(0);

  float o[HT][NP][2][4];
#pragma unroll
  for (int i = 0; i < HT; ++i)
#pragma unroll
    for (int j = 0; j < NP; ++j)
#pragma unroll
      for (int x = 0; x < 4; ++x) o[i][j][0][x] = o[i][j][1][x] = 0.f;
  constexpr int kRows = kHeads / kLatWarps;   // score rows of this warp: rows warp * kRows ..
  float m_run[kRows], l_run[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  const int lr = lane & 7, lm = lane >> 3;
  const int row_a = (lm & 1) * 8 + lr, col_a = (lm >> 1) * 16;   // A operands: [rows 0-7 | 8-15] x [k 0-7 | 8-15]
  const int steps = p.CP >> 4, half_steps = (steps + 1) >> 1;
  const int kt = warp & 3, kh = warp >> 2;                       // this warp's 8 keys and its part of the row
  const int k_lo = kh * half_steps, k_hi = min(k_lo + half_steps, steps);
  const int n_pairs = (p.R + 15) >> 4;
  float* s_s = reinterpret_cast<float*>(s_raw + L.s);
  float* s_alpha = reinterpret_cast<float*>(s_raw + L.alpha);

  for (int it = 0; it < n_it; ++it) {
    cp_wait<0>();
    __syncthreads();   // the tile has landed; the other stage, the scores and the weights have been read
    if (it + 1 < n_it) issue(it + 1);
    const uint32_t tile = smem + L.tile + (it & 1) * kLatKeys * L.pitch;
    // ---- scores: 16 HT heads x 8 keys over half of the row ----
    {
      float sc[HT][2][4] = {};   // two accumulators hide the latency of one chain
      const uint32_t kb = tile + (kt * 8 + lr) * L.pitch + lm * 16;
      const uint32_t qa = smem + L.q + row_a * L.pitch + col_a;
      int k = k_lo;
      for (; k + 2 <= k_hi; k += 2) {
        uint32_t b[4];
        ldsm4(kb + k * 32, b);
#pragma unroll
        for (int i = 0; i < HT; ++i) {
          uint32_t a[4], a2[4];
          ldsm4(qa + i * 16 * L.pitch + k * 32, a);
          ldsm4(qa + i * 16 * L.pitch + k * 32 + 32, a2);
          mma_bf16(sc[i][0], a, b[0], b[1]);
          mma_bf16(sc[i][1], a2, b[2], b[3]);
        }
      }
      if (k < k_hi) {
        uint32_t b[2];
        ldsm2(tile + (kt * 8 + lr) * L.pitch + (lm & 1) * 16 + k * 32, b);
#pragma unroll
        for (int i = 0; i < HT; ++i) {
          uint32_t a[4];
          ldsm4(qa + i * 16 * L.pitch + k * 32, a);
          mma_bf16(sc[i][0], a, b[0], b[1]);
        }
      }
#pragma unroll
      for (int i = 0; i < HT; ++i) {
        float* d = s_s + (kh * kHeads + i * 16 + g) * kPitchS + kt * 8 + 2 * t;
        *reinterpret_cast<float2*>(d) = make_float2(sc[i][0][0] + sc[i][1][0], sc[i][0][1] + sc[i][1][1]);
        *reinterpret_cast<float2*>(d + 8 * kPitchS) = make_float2(sc[i][0][2] + sc[i][1][2], sc[i][0][3] + sc[i][1][3]);
      }
    }
    __syncthreads();
    // ---- softmax: lane = key ----
    const bool seen = (pg_lo + it * 2) * 16 + lane < min(seq_len, pg_hi * 16);
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int r = warp * kRows + i;
      const float x = seen ? (s_s[r * kPitchS + lane] + s_s[(kHeads + r) * kPitchS + lane]) * p.scale_log2 : -INFINITY;
      const float mn = fmaxf(m_run[i], warp_max(x));   // the first key of a tile is always visible
      const float alpha = ex2(m_run[i] - mn), w = ex2(x - mn);
      m_run[i] = mn;
      l_run[i] = l_run[i] * alpha + w;
      const __nv_bfloat16 hi = __float2bfloat16(w);
      __nv_bfloat16* d = reinterpret_cast<__nv_bfloat16*>(s_raw + L.pw + r * kPitchP) + lane;
      *d = hi;
      *reinterpret_cast<__nv_bfloat16*>(reinterpret_cast<uint8_t*>(d) + kHeads * kPitchP) = __float2bfloat16(w - __bfloat162float(hi));
      if (lane == 0) s_alpha[r] = alpha;
    }
    __syncthreads();
    // ---- sums: this warp's value columns ----
#pragma unroll
    for (int i = 0; i < HT; ++i) {
      const float a0 = s_alpha[i * 16 + g], a1 = s_alpha[i * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o[i][j][n][0] *= a0;
          o[i][j][n][1] *= a0;
          o[i][j][n][2] *= a1;
          o[i][j][n][3] *= a1;
        }
    }
#pragma unroll
    for (int k = 0; k < kLatKeys / 16; ++k) {
      uint32_t a[HT][2][4];   // weights: high and low terms
#pragma unroll
      for (int i = 0; i < HT; ++i)
#pragma unroll
        for (int x = 0; x < 2; ++x)
          ldsm4(smem + L.pw + (x * kHeads + i * 16 + row_a) * kPitchP + k * 32 + col_a, a[i][x]);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int pair = warp * NP + j;
        if (pair < n_pairs) {
          uint32_t b[4];   // (keys lo, cols lo) (keys hi, cols lo) (keys lo, cols hi) (keys hi, cols hi)
          ldsm4t(tile + (k * 16 + row_a) * L.pitch + pair * 32 + col_a, b);
#pragma unroll
          for (int i = 0; i < HT; ++i)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              mma_bf16(o[i][j][0], a[i][x], b[0], b[1]);
              mma_bf16(o[i][j][1], a[i][x], b[2], b[3]);
            }
        }
      }
    }
  }
  pdl_launch_dependents();
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int h = warp * kRows + i;
    const float l = warp_sum(l_run[i]);
    if (lane == 0 && h0 + h < p.H) {
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2] = m_run[i];
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2 + 1] = l;
    }
  }
#pragma unroll
  for (int i = 0; i < HT; ++i)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int h = i * 16 + g + 8 * x;
      if (h0 + h >= p.H) continue;
      float* d = p.part_o + (part0 + static_cast<long long>(h) * p.max_splits) * p.R;
#pragma unroll
      for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int c = (warp * NP + j) * 16 + n * 8 + 2 * t;
          if (c < p.R) d[c] = o[i][j][n][2 * x];
          if (c + 1 < p.R) d[c + 1] = o[i][j][n][2 * x + 1];
        }
    }
}

// grid (rows, heads)
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentDecodeParams p) {
  __shared__ float s_w[64];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, head = blockIdx.y;
  const long long base = (static_cast<long long>(row) * p.H + head) * p.max_splits;
  // weight of every split: max_splits <= 64
  if (threadIdx.x < 32) {
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    const float m0 = s0 < p.max_splits ? p.part_ml[(base + s0) * 2] : -INFINITY, m1 = s1 < p.max_splits ? p.part_ml[(base + s1) * 2] : -INFINITY;
    const float M = warp_max(fmaxf(m0, m1));
    const float w0 = m0 == -INFINITY ? 0.f : ex2(m0 - M), w1 = m1 == -INFINITY ? 0.f : ex2(m1 - M);
    const float l = warp_sum((w0 > 0.f ? w0 * p.part_ml[(base + s0) * 2 + 1] : 0.f) + (w1 > 0.f ? w1 * p.part_ml[(base + s1) * 2 + 1] : 0.f));
    const float inv = l > 0.f ? 1.f / l : 0.f;
    s_w[s0] = w0 * inv;
    s_w[s1] = w1 * inv;
  }
  __syncthreads();
  __nv_bfloat16* out = p.out + static_cast<long long>(row) * p.ldo + static_cast<long long>(head) * p.o_hd;
  for (int c = threadIdx.x; c < p.R; c += 128) {
    float a = 0.f;
    for (int s = 0; s < p.max_splits; ++s) {
      const float w = s_w[s];
      if (w > 0.f) a = fmaf(w, p.part_o[(base + s) * p.R + c], a);
    }
    out[c] = __float2bfloat16(a);
  }
}

template <int HT>
cudaError_t launch_lat(const LatentDecodeParams& p, cudaStream_t stream) {
  const int pairs = (p.R + 15) / 16, np = (pairs + kLatWarps - 1) / kLatWarps;
  auto kern = np <= 1 ? latent_decode_kernel<HT, 1> : (np <= 2 ? latent_decode_kernel<HT, 2> : latent_decode_kernel<HT, 4>);
  const LatentSmem L(p.CP, HT * 16);
  ensure_dynamic_smem(kern, static_cast<size_t>(L.total));
  const dim3 grid(p.rows, (p.H + HT * 16 - 1) / (HT * 16), p.max_splits);
  return launch_kernel(kern, grid, dim3(kLatWarps * 32), static_cast<size_t>(L.total), stream, true, false, p);
}

template <typename T, typename P>
cudaError_t launch_rows(const LatentRowsParams& p, cudaStream_t stream) {
  const size_t smem = (static_cast<size_t>(p.Q) + p.R) * sizeof(float);
  ensure_dynamic_smem(latent_rows_kernel<T, P>, smem);
  return launch_kernel(latent_rows_kernel<T, P>, dim3(p.M), dim3(256), smem, stream, true, false, p);
}

}  // namespace

bool latent_decode_ok(int R, int CP) { return R <= 16 * 4 * kLatWarps && CP <= 1024 && CP % 16 == 0; }

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

cudaError_t launch_latent_decode(const LatentDecodeParams& p, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  if (!latent_decode_ok(p.R, p.CP) || p.max_splits > 64) return cudaErrorInvalidValue;
  const cudaError_t e = p.H <= 16 ? launch_lat<1>(p, stream) : launch_lat<2>(p, stream);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_merge_kernel, dim3(p.rows, p.H), dim3(128), 0, stream, true, false, p);
}

}  // namespace oxb
