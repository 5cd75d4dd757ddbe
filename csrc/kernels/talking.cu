// Talking heads over keys that are values (sm_100a): the softmax of a head runs over a mix of all heads' scores, so the scores of
// all heads have to meet before any weight is known. The cache keeps one tensor, the keys before their norm (which are the
// values), and the norm's factor per token; a page is read once for both products.
//
// Decoding (talk_decode): one CTA = (sequence, KV split) walks its pages with all heads. A block of pages in shared memory is
// first the key operand (warps take page x key head), the capped scores meet in shared memory and are mixed there in fp32
// (lanes are positions), and then the same block is the value operand (warps own pieces of the output, [16 dims x 8 heads]).
//
// Prompts: the sums of all heads of a query tile do not fit an SM, the scores of a tile do. talk_scores: one CTA = 16 queries, 32 keys
// at a time; the scores of all heads (mma.sync: a head's 16 x 32 tile is too small for a 128-row tcgen05 tile) meet in shared memory,
// are mixed as a product with the heads' matrix and written out. talk_values: softmax and sums per head from there.
//
// talk_rows takes any sizes in fp32 FMAs, one row per CTA.
#include "../common/device_info.h"
#include "hybrid_mma.cuh"

namespace oxb {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2t(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// cap tanh(x / cap) = cap - 2 cap / (e^(2 x / cap) + 1); k2 = 2 log2(e) / cap. Good to about cap * 2^-22.
__device__ __forceinline__ float capped(float x, float cap, float k2) {
  return cap > 0.f ? cap - __fdividef(2.f * cap, fminf(ex2t(x * k2), 1e30f) + 1.f) : x;
}
__device__ __forceinline__ float gate_at(const TalkParams& p, long long row, int col) {
  const float z = p.gate_f32 ? static_cast<const float*>(p.gate)[row * p.gate_ld + col]
                             : to_f(static_cast<const __nv_bfloat16*>(p.gate)[row * p.gate_ld + col]);
  return 1.f / (1.f + expf(-z));
}
// block id of page pg of a sequence; ids outside the pool are recorded and replaced by 0
__device__ __forceinline__ int block_of(const TalkParams& p, const int* bt, int pg) {
  const int b = pg < p.max_blocks ? bt[pg] : -1;
  if (static_cast<unsigned>(b) < static_cast<unsigned>(p.num_blocks)) return b;
  set_status_once(p.status, kStatusBadIndex);
  return 0;
}

// ---------------------------------------------------------------- any sizes
constexpr int kRowKeys = 32;

template <typename T>
__global__ void __launch_bounds__(256) talk_rows_kernel(const TalkParams p) {
  extern __shared__ float s_mem[];
  __shared__ int s_tok[kRowKeys];
  __shared__ float s_r[kRowKeys];
  pdl_wait();
  const int H = p.H, D = p.D, HD = H * D, R = H / p.G, tid = threadIdx.x;
  float* s_q = s_mem;
  float* s_o = s_q + HD;
  float* s_c = s_o + HD;
  float* s_p = s_c + H * (kRowKeys + 1);
  float* s_t = s_p + H * (kRowKeys + 1);
  float* s_m = s_t + H * H;
  float* s_l = s_m + H;
  float* s_a = s_l + H;
  int row, pos, seq;
  if (p.tile_seq == nullptr) {
    row = seq = blockIdx.x;
    pos = p.seq_lens[row] - 1;
  } else {
    const int tile = blockIdx.x >> 7, r = blockIdx.x & 127;
    seq = p.tile_seq[tile];
    const int qi = p.tile_q0[tile] + r;
    if (qi >= p.q_lens[seq]) return;
    row = p.q_start[seq] + qi;
    pos = p.ctx_lens[seq] - p.q_lens[seq] + qi;
  }
  if (pos < 0) return;  // padding row
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  const T* qp = static_cast<const T*>(p.q) + static_cast<long long>(row) * p.q_ld;
  const T* cache = static_cast<const T*>(p.cache);
  for (int i = tid; i < HD; i += 256) {
    s_q[i] = to_f(qp[(i / D) * p.DP + i % D]);
    s_o[i] = 0.f;
  }
  for (int i = tid; i < H * H; i += 256) s_t[i] = p.talk[i];
  for (int i = tid; i < H; i += 256) {
    s_m[i] = -INFINITY;
    s_l[i] = 0.f;
  }
  const int lo = p.window > 0 && pos + 1 > p.window ? pos + 1 - p.window : 0;
  for (int base = lo; base <= pos; base += kRowKeys) {
    const int n = min(kRowKeys, pos + 1 - base);
    __syncthreads();
    if (tid < n) {
      const int j = base + tid, tok = block_of(p, bt, j >> 4) * 16 + (j & 15);
      s_tok[tid] = tok;
      s_r[tid] = p.k_rms[tok] * p.scale;
    }
    __syncthreads();
    auto key = [&](int t, int kv) { return cache + (static_cast<long long>(s_tok[t] >> 4) * p.G + kv) * 16 * p.DP + (s_tok[t] & 15) * p.DP; };
    for (int i = tid; i < H * n; i += 256) {
      const int g = i / n, t = i - g * n;
      const T* k = key(t, g / R);
      float a = 0.f;
      for (int d = 0; d < D; ++d) a = fmaf(s_q[g * D + d], to_f(k[d]), a);
      a *= s_r[t];
      s_c[g * (kRowKeys + 1) + t] = p.cap > 0.f ? p.cap * tanhf(a / p.cap) : a;
    }
    __syncthreads();
    for (int i = tid; i < H * n; i += 256) {
      const int h = i / n, t = i - h * n;
      float a = 0.f;
      for (int g = 0; g < H; ++g) a = fmaf(s_t[h * H + g], s_c[g * (kRowKeys + 1) + t], a);
      s_p[h * (kRowKeys + 1) + t] = a - p.bias[static_cast<long long>(h) * p.n_bias + min(pos - base - t, p.n_bias - 1)];
    }
    __syncthreads();
    for (int h = tid >> 5; h < H; h += 8) {
      const int lane = tid & 31;
      const float x = lane < n ? s_p[h * (kRowKeys + 1) + lane] : -INFINITY;
      const float m = fmaxf(s_m[h], warp_max(x));
      const float e = lane < n ? expf(x - m) : 0.f, sum = warp_sum(e);
      const float alpha = s_m[h] == -INFINITY ? 0.f : expf(s_m[h] - m);
      s_p[h * (kRowKeys + 1) + lane] = e;
      __syncwarp();
      if (lane == 0) {
        s_l[h] = s_l[h] * alpha + sum;
        s_m[h] = m;
        s_a[h] = alpha;
      }
    }
    __syncthreads();
    for (int i = tid; i < HD; i += 256) {
      const int h = i / D, d = i - h * D;
      float a = s_o[i] * s_a[h];
      for (int t = 0; t < n; ++t) a = fmaf(s_p[h * (kRowKeys + 1) + t], to_f(key(t, h / R)[d]), a);
      s_o[i] = a;
    }
  }
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo;
  for (int i = tid; i < HD; i += 256) out[i] = from_f<T>(s_o[i] / s_l[i / D] * gate_at(p, row, i));  // own elements, last barrier above
}

// ---------------------------------------------------------------- decoding
constexpr int kDecWarps = 16, kDecThreads = kDecWarps * 32;
constexpr int kMaxTiles = 8;     // 16 x 8 pieces of the output per warp
constexpr int kMaxHeads = 64;
constexpr int kHeadsPerWarp = kMaxHeads / kDecWarps;
constexpr int kMaxPages = 8;     // pages per block

struct DecodeLayout {
  int pages, stages, nt, cld, tld, pld;   // pages per block, ring stages, 8-head columns per key head, row pitches
  int page_bytes, stage_bytes, q, c, t, phi, plo, total;
};
__host__ __device__ inline DecodeLayout decode_layout(int H, int G, int D) {
  DecodeLayout l;
  const int R = H / G;
  l.nt = (R + 7) / 8;
  l.page_bytes = G * 16 * D * 2;
  l.pages = 32768 / l.page_bytes;
  l.pages = l.pages < 2 ? 2 : (l.pages < 4 ? l.pages : (l.pages < kMaxPages ? 4 : kMaxPages));
  l.stage_bytes = l.pages * (l.page_bytes + 64);      // a page and its 16 norm factors
  const int toks = l.pages * 16;
  l.cld = H | 1;                                      // odd: lanes are positions
  l.tld = (H + 3) / 4 * 4;
  l.pld = toks + 8;
  l.stages = 3;
  for (;; --l.stages) {
    l.q = l.stages * l.stage_bytes;
    l.c = l.q + H * (D * 2 + 16);
    l.t = (l.c + toks * l.cld * 4 + 15) / 16 * 16;
    l.phi = l.t + H * l.tld * 4;
    l.plo = l.phi + H * l.pld * 2;
    l.total = l.plo + H * l.pld * 2;
    if (l.total <= 220 * 1024 || l.stages == 2) break;
  }
  return l;
}

template <int D>
__global__ void __launch_bounds__(kDecThreads) talk_decode_kernel(const TalkParams p, const DecodeLayout L, int want_splits) {
  constexpr int CH = D / 8, MT = D / 16;   // 16-byte chunks per row, pieces of 16 dims
  extern __shared__ __align__(128) uint8_t s_raw[];
  __shared__ float s_alpha[kMaxHeads];
  __shared__ int s_ids[2][kMaxPages];
  const int H = p.H, G = p.G, R = H / G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t s_base = smem_u32(s_raw);
  float* s_c = reinterpret_cast<float*>(s_raw + L.c);
  float* s_t = reinterpret_cast<float*>(s_raw + L.t);
  __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(s_raw + L.phi);
  __nv_bfloat16* s_lo = reinterpret_cast<__nv_bfloat16*>(s_raw + L.plo);
  for (int h = warp; h < H; h += kDecWarps)
    for (int g = lane; g < L.tld; g += 32) s_t[h * L.tld + g] = g < H ? p.talk[h * H + g] * kLog2e : 0.f;
  pdl_wait();  // q and the newest cache rows come from the kernel before this one
  const int seq = blockIdx.x, split = blockIdx.y, seq_len = p.seq_lens[seq];
  const int win_start = p.window > 0 && seq_len > p.window ? seq_len - p.window : 0;
  int n_pages = (seq_len + 15) / 16;
  if (n_pages > p.max_blocks) {
    if (tid == 0) set_status_once(p.status, kStatusBadIndex);
    n_pages = p.max_blocks;
  }
  // the visible pages over `want_splits` CTAs, in whole blocks
  const int first_page = win_start / 16, n_list = n_pages - first_page;
  const int pps = ((n_list + want_splits - 1) / want_splits + L.pages - 1) / L.pages * L.pages;
  const int pg_lo = first_page + split * pps, pg_hi = min(pg_lo + pps, n_pages);
  if (pg_lo >= pg_hi || seq_len <= 0) {
    for (int h = tid; h < H; h += kDecThreads) {
      float* ml = p.part_ml + ((static_cast<long long>(seq) * H + h) * p.max_splits + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  const int n_blocks = (pg_hi - pg_lo + L.pages - 1) / L.pages;
  const int page_chunks = G * 16 * CH;
  auto fetch_ids = [&](int b) {   // block ids of page block b
    const int pg = pg_lo + b * L.pages + tid;
    if (tid < L.pages) s_ids[b & 1][tid] = pg < pg_hi ? block_of(p, bt, pg) : -1;
  };
  auto issue = [&](int b, int slot) {
    const uint32_t stage = s_base + slot * L.stage_bytes;
    for (int pg = 0; pg < L.pages; ++pg) {
      const int id = s_ids[b & 1][pg];
      const bool in = id >= 0;
      const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.cache) + static_cast<long long>(in ? id : 0) * G * 16 * D;
      const uint32_t dst = stage + pg * L.page_bytes;
#pragma unroll 4
      for (int c = tid; c < page_chunks; c += kDecThreads) {
        const int r = c / CH, ch = c % CH;
        cp_async16(dst + r * (D * 2) + ((ch ^ (r & 7)) << 4), src + c * 8, in);
      }
      if (tid < 4) cp_async16(stage + L.pages * L.page_bytes + pg * 64 + tid * 16, p.k_rms + (in ? id : 0) * 16ll + tid * 4, in);
    }
  };
  // queries of all heads, rows D * 2 + 16 bytes apart
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(seq) * p.q_ld;
  for (int c = tid; c < H * CH; c += kDecThreads)
    *reinterpret_cast<uint4*>(s_raw + L.q + (c / CH) * (D * 2 + 16) + (c % CH) * 16) = *reinterpret_cast<const uint4*>(qp + c * 8);
  fetch_ids(0);
  fetch_ids(1);
  __syncthreads();
  for (int b = 0; b < L.stages - 1; ++b) {
    if (b < n_blocks) issue(b, b);
    cp_commit();
    __syncthreads();
    fetch_ids(b + 2);
    __syncthreads();
  }
  float acc[kMaxTiles][4], m_run[kHeadsPerWarp], l_run[kHeadsPerWarp];
#pragma unroll
  for (int j = 0; j < kMaxTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
#pragma unroll
  for (int i = 0; i < kHeadsPerWarp; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  const int g8 = lane >> 2, t4 = lane & 3;
  const int n_tiles = G * L.nt * MT, per_warp = (n_tiles + kDecWarps - 1) / kDecWarps, ti0 = warp * per_warp;
  const int toks = L.pages * 16;
  const float k2 = p.cap > 0.f ? 2.f * kLog2e / p.cap : 0.f;
  // lanes' offsets in a page: rows of the key operand, rows (positions) of the transposed value operand
  const int kr = lane & 15, kc = lane >> 4, vr = ((lane >> 4) << 3) + (lane & 7), vc = (lane >> 3) & 1;
  int slot = 0;
  for (int b = 0; b < n_blocks; ++b) {
    if (L.stages == 3) cp_wait<1>();
    else cp_wait<0>();
    __syncthreads();   // block b has landed; every warp is done with the block before it
    const int nb = b + L.stages - 1, slot_new = slot == 0 ? L.stages - 1 : slot - 1;
    if (nb < n_blocks) issue(nb, slot_new);
    cp_commit();
    const uint32_t stage = s_base + slot * L.stage_bytes;
    const float* s_rms = reinterpret_cast<const float*>(s_raw + slot * L.stage_bytes + L.pages * L.page_bytes);
    // ---- scores: [16 positions x 8 heads] per page, key head and column ----
    for (int pg = 0, kv = warp; pg < L.pages;) {
      if (kv >= G) {
        kv -= G;
        ++pg;
        continue;
      }
      const uint32_t rows = stage + pg * L.page_bytes + (kv * 16 + kr) * (D * 2);
      const float r0 = s_rms[pg * 16 + g8] * p.scale, r1 = s_rms[pg * 16 + g8 + 8] * p.scale;
      for (int nt = 0; nt < L.nt; ++nt) {
        const int hq = min(kv * R + nt * 8 + g8, H - 1);
        const uint8_t* qr = s_raw + L.q + hq * (D * 2 + 16) + t4 * 4;
        float s[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < MT; ++ks) {
          uint32_t a[4];
          ldsm4(rows + (((ks * 2 + kc) ^ (kr & 7)) << 4), a);
          mma_bf16(s[ks & 1], a, *reinterpret_cast<const uint32_t*>(qr + ks * 32), *reinterpret_cast<const uint32_t*>(qr + ks * 32 + 16));
        }
        const int lh = nt * 8 + 2 * t4;
        float* c0 = s_c + (pg * 16 + g8) * L.cld + kv * R + lh;
        float* c1 = c0 + 8 * L.cld;
        if (lh < R) {
          c0[0] = capped((s[0][0] + s[1][0]) * r0, p.cap, k2);
          c1[0] = capped((s[0][2] + s[1][2]) * r1, p.cap, k2);
        }
        if (lh + 1 < R) {
          c0[1] = capped((s[0][1] + s[1][1]) * r0, p.cap, k2);
          c1[1] = capped((s[0][3] + s[1][3]) * r1, p.cap, k2);
        }
      }
      kv += kDecWarps;
    }
    __syncthreads();
    // ---- mixed scores (times log2 e) and softmax: warps take heads warp + 16 i, lanes positions ----
    const int pos0 = (pg_lo + b * L.pages) * 16;
#pragma unroll
    for (int rep = 0; rep < kHeadsPerWarp / 2; ++rep) {   // two heads at a time
      const int h0 = warp + 2 * kDecWarps * rep;
      if (h0 < H) {
        const int hs[2] = {h0, min(h0 + kDecWarps, H - 1)};
        float x[4][2], mx[2] = {-INFINITY, -INFINITY};   // [positions / 32][heads]
#pragma unroll
        for (int tc = 0; tc < 4; ++tc) {
          x[tc][0] = x[tc][1] = -INFINITY;
          if (tc * 32 < toks) {
            const int tok = tc * 32 + lane, dist = seq_len - 1 - pos0 - tok;
            const bool see = tok < toks && dist >= 0 && (p.window == 0 || dist < p.window);
            const float* c = s_c + min(tok, toks - 1) * L.cld;
            float bias[2], a[2][2] = {};
#pragma unroll
            for (int i = 0; i < 2; ++i)
              bias[i] = see ? __ldg(p.bias + static_cast<long long>(hs[i]) * p.n_bias + min(dist, p.n_bias - 1)) : 0.f;
#pragma unroll 4
            for (int g = 0; g < L.tld; g += 4) {
              float cv[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) cv[e] = g + e < H ? c[g + e] : 0.f;
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                const float4 t = *reinterpret_cast<const float4*>(s_t + hs[i] * L.tld + g);
                a[i][0] = fmaf(t.x, cv[0], fmaf(t.y, cv[1], a[i][0]));
                a[i][1] = fmaf(t.z, cv[2], fmaf(t.w, cv[3], a[i][1]));
              }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              if (see) x[tc][i] = a[i][0] + a[i][1] - kLog2e * bias[i];
              mx[i] = fmaxf(mx[i], x[tc][i]);
            }
          }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          mx[0] = fmaxf(mx[0], __shfl_xor_sync(0xffffffffu, mx[0], o));
          mx[1] = fmaxf(mx[1], __shfl_xor_sync(0xffffffffu, mx[1], o));
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int h = h0 + kDecWarps * i;
          if (h < H) {
            const float m = fmaxf(m_run[rep * 2 + i], mx[i]), ms = m == -INFINITY ? 0.f : m;
            const float alpha = ex2t(m_run[rep * 2 + i] - ms);
            float sum = 0.f;
#pragma unroll
            for (int tc = 0; tc < 4; ++tc) {
              const int tok = tc * 32 + lane;
              if (tok < toks) {
                const float e = ex2t(x[tc][i] - ms);
                const __nv_bfloat16 hi = __float2bfloat16(e);
                s_hi[h * L.pld + tok] = hi;
                s_lo[h * L.pld + tok] = __float2bfloat16(e - __bfloat162float(hi));
                sum += e;
              }
            }
            m_run[rep * 2 + i] = m;
            l_run[rep * 2 + i] = l_run[rep * 2 + i] * alpha + sum;   // of this lane's positions
            if (lane == 0) s_alpha[h] = alpha;
          }
        }
      }
    }
    fetch_ids(nb + 1);   // (the ids of block nb have been read)
    __syncthreads();
    // ---- sums: warps own tiles of [16 dims x 8 heads], one after the other ----
#pragma unroll
    for (int j = 0; j < kMaxTiles; ++j) {
      const int ti = ti0 + j;
      if (j < per_warp && ti < n_tiles) {
        const int mt = ti % MT, gn = ti / MT, kv = L.nt == 1 ? gn : gn / L.nt, nt = gn - kv * L.nt;
        const int hb = kv * R + nt * 8, left = R - nt * 8;
        const float a0 = s_alpha[min(hb + 2 * t4, H - 1)], a1 = s_alpha[min(hb + 2 * t4 + 1, H - 1)];
        acc[j][0] *= a0;
        acc[j][1] *= a1;
        acc[j][2] *= a0;
        acc[j][3] *= a1;
        const bool on = g8 < left;
        const int pr = (hb + (on ? g8 : 0)) * L.pld + 2 * t4;
        const uint32_t rows = stage + (kv * 16 + vr) * (D * 2) + (((mt * 2 + vc) ^ (vr & 7)) << 4);
        for (int pg = 0; pg < L.pages; ++pg) {
          uint32_t a[4];
          ldsm4t(rows + pg * L.page_bytes, a);
          const uint32_t* hi = reinterpret_cast<const uint32_t*>(s_hi + pr + pg * 16);
          const uint32_t* lo = reinterpret_cast<const uint32_t*>(s_lo + pr + pg * 16);
          mma_bf16(acc[j], a, on ? hi[0] : 0u, on ? hi[4] : 0u);
          mma_bf16(acc[j], a, on ? lo[0] : 0u, on ? lo[4] : 0u);
        }
      }
    }
    slot = slot + 1 == L.stages ? 0 : slot + 1;
  }
  cp_wait<0>();
  pdl_launch_dependents();
  const long long part0 = static_cast<long long>(seq) * H;
#pragma unroll
  for (int j = 0; j < kMaxTiles; ++j) {
    const int ti = ti0 + j;
    if (j < per_warp && ti < n_tiles) {
      const int mt = ti % MT, gn = ti / MT, kv = gn / L.nt, nt = gn - kv * L.nt;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int lh = nt * 8 + 2 * t4 + (e & 1), d = mt * 16 + g8 + (e >> 1) * 8;
        if (lh < R) p.part_o[((part0 + kv * R + lh) * p.max_splits + split) * D + d] = acc[j][e];
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kHeadsPerWarp; ++i) {
    const int h = warp + kDecWarps * i;
    const float l = warp_sum(l_run[i]);
    if (h < H && lane == 0) {
      float* ml = p.part_ml + ((part0 + h) * p.max_splits + split) * 2;
      ml[0] = m_run[i];
      ml[1] = l;
    }
  }
}

template <int D>
__global__ void __launch_bounds__(D) talk_merge_kernel(const TalkParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.x, head = blockIdx.y, d = threadIdx.x;
  const long long base = (static_cast<long long>(seq) * p.H + head) * p.max_splits;
  float M = -INFINITY;
  for (int s = 0; s < p.max_splits; ++s) M = fmaxf(M, p.part_ml[(base + s) * 2]);
  float acc = 0.f, L = 0.f;
  for (int s = 0; s < p.max_splits; ++s) {
    const float ms = p.part_ml[(base + s) * 2];
    if (ms == -INFINITY) continue;
    const float f = ex2t(ms - M);
    acc += f * p.part_o[(base + s) * D + d];
    L += f * p.part_ml[(base + s) * 2 + 1];
  }
  if (d >= p.D) return;
  const int col = head * p.D + d;
  static_cast<__nv_bfloat16*>(p.out)[static_cast<long long>(seq) * p.ldo + col] =
      __float2bfloat16(L > 0.f ? acc / L * gate_at(p, seq, col) : 0.f);
}

// ---------------------------------------------------------------- prompts
constexpr int kTile = 128;   // query rows of the scheduler's tiles
constexpr int kKeys = 32;    // keys of a block
constexpr int kQ = 16;       // queries of a scores CTA
constexpr int kBlocks = 4;   // blocks of keys that a scores CTA walks

// What a piece of a tile's rows sees: positions of its first and last row, first visible key.
struct Piece {
  int seq, len, pos0, pos1, row0, lo;
};
__device__ __forceinline__ Piece piece_of(const TalkParams& p, int tile, int q, int rows) {
  Piece x;
  x.seq = p.tile_seq[tile];
  x.len = p.q_lens[x.seq];
  const int off = p.ctx_lens[x.seq] - x.len, q0 = p.tile_q0[tile] + q;
  x.pos0 = off + q0;
  x.pos1 = off + min(q0 + rows, x.len) - 1;
  x.row0 = p.q_start[x.seq] + q0;
  x.lo = p.window > 0 ? max(0, x.pos0 - p.window + 1) : 0;
  return x;
}
// first key of a tile's row of scores
__device__ __forceinline__ int first_key(const TalkParams& p, int tile) { return piece_of(p, tile, 0, kTile).lo / kKeys * kKeys; }

// Row pitch of a head's scores in shared memory, and of a query's keys inside: a warp's stores (8 keys x 4 queries) and its
// reads (4 heads, two apart, x 8 keys) both touch 32 banks.
constexpr int kQPitch = kKeys + 4, kHPitch = kQ * kQPitch + 4;
static_assert(kHPitch % 16 == 4, "banks");
constexpr int kBiasPitch = 72;

// HM: heads of this instantiation, 16 or 32 (H <= HM). 8 warps = 4 sets of heads x 2 halves of the keys: a warp multiplies 16 keys
// x 16 queries for the heads of its set, operands straight from memory (16-byte pieces, the same permutation of the dimensions in q
// and k). Then the scores of all heads are mixed as a product with the matrix T: 8 keys of a query are the columns, T is bf16 and
// exact, and the fp32 scores enter as three bf16 terms that carry all their bits.
template <int D, int HM>
__global__ void __launch_bounds__(256, 2) talk_scores_kernel(const TalkParams p) {
  constexpr int CPL = D / 32;   // 16-byte pieces of a row per lane
  constexpr int HT = HM / 16;
  extern __shared__ __align__(128) uint8_t s_raw[];
  float* s_c = reinterpret_cast<float*>(s_raw);   // [HM][kQ][keys]
  float* s_b = s_c + HM * kHPitch;                // [H][distances]: bias times log2 e; +inf hides a key
  float* s_r = s_b + p.H * kBiasPitch;            // [keys] norm factors times the scale
  const int H = p.H, R = H / p.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  uint32_t ta[HT][HT][4];   // T as the left operand
#pragma unroll
  for (int m = 0; m < HT; ++m)
#pragma unroll
    for (int k = 0; k < HT; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int h = m * 16 + g8 + (i & 1) * 8, g = k * 16 + 2 * t4 + (i >> 1) * 8;
        ta[m][k][i] = pack_bf16x2(h < H && g < H ? p.talk[h * H + g] : 0.f, h < H && g + 1 < H ? p.talk[h * H + g + 1] : 0.f);
      }
  for (int i = tid; i < (HM - H) * kHPitch; i += 256) s_c[H * kHPitch + i] = 0.f;
  pdl_wait();
  const int tile = blockIdx.z, q_in = blockIdx.y * kQ;
  const Piece x = piece_of(p, tile, q_in, kQ);
  if (p.tile_q0[tile] + q_in >= x.len) return;
  const int k_start = first_key(p, tile);
  const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
  const int n_pg = (p.ctx_lens[x.seq] + 15) >> 4;
  const int n_q = x.pos1 - x.pos0 + 1;
  const int half = warp & 1, hc = (H + 3) / 4, h_lo = (warp >> 1) * hc, h_hi = min(h_lo + hc, H);
  const float k2 = p.cap > 0.f ? 2.f * kLog2e / p.cap : 0.f;
  const __nv_bfloat16* q0 = static_cast<const __nv_bfloat16*>(p.q) + (static_cast<long long>(x.row0) + min(g8, n_q - 1)) * p.q_ld + t4 * 8;
  const __nv_bfloat16* q1 = static_cast<const __nv_bfloat16*>(p.q) + (static_cast<long long>(x.row0) + min(g8 + 8, n_q - 1)) * p.q_ld + t4 * 8;
  bool first = true;
  for (int blk = 0; blk < kBlocks; ++blk) {
    const int kb = blockIdx.x * kBlocks + blk, k0 = k_start + kb * kKeys;
    if (k0 > x.pos1) break;
    if (k0 + kKeys <= x.lo) continue;
    if (!first) __syncthreads();   // every warp is done with the block before
    first = false;
    const int pg = (k0 >> 4) + half;
    const int id = pg < n_pg ? block_of(p, bt, pg) : -1;
    if (lane < 16 && (warp >> 1) == 0) s_r[half * 16 + lane] = id >= 0 ? p.k_rms[id * 16ll + lane] * p.scale : 0.f;
    const int far0 = x.pos0 - k0 - (kKeys - 1);   // distance of bias entry 0
    for (int h = warp; h < H; h += 8)
      for (int i = lane; i < kKeys + kQ - 1; i += 32) {
        const int dist = far0 + i;
        const bool see = dist >= 0 && (p.window == 0 || dist < p.window);
        s_b[h * kBiasPitch + i] = see ? kLog2e * __ldg(p.bias + static_cast<long long>(h) * p.n_bias + min(dist, p.n_bias - 1)) : INFINITY;
      }
    __syncthreads();
    // ---- scores of this warp's heads: [16 keys x 16 queries] ----
    const float r0 = s_r[half * 16 + g8], r1 = s_r[half * 16 + g8 + 8];
    uint4 ka[2][CPL];
    int kv_have = -1;
    for (int h = h_lo; h < h_hi; ++h) {
      const int kv = h / R;
      if (kv != kv_have) {
        kv_have = kv;
        const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(p.cache) + (static_cast<long long>(max(id, 0)) * p.G + kv) * 16 * D + t4 * 8;
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
          for (int c = 0; c < CPL; ++c) ka[r][c] = *reinterpret_cast<const uint4*>(kp + (g8 + 8 * r) * D + c * 32);
      }
      uint4 qb[2][CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        qb[0][c] = *reinterpret_cast<const uint4*>(q0 + h * D + c * 32);
        qb[1][c] = *reinterpret_cast<const uint4*>(q1 + h * D + c * 32);
      }
      float s[2][4] = {};
#pragma unroll
      for (int c = 0; c < CPL; ++c)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16(s[n], ka[0][c].x, ka[1][c].x, ka[0][c].y, ka[1][c].y, qb[n][c].x, qb[n][c].y);
          mma_bf16(s[n], ka[0][c].z, ka[1][c].z, ka[0][c].w, ka[1][c].w, qb[n][c].z, qb[n][c].w);
        }
      float* d = s_c + h * kHPitch + 2 * t4 * kQPitch + half * 16 + g8;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          d[(n * 8 + (e & 1)) * kQPitch + (e >> 1) * 8] = capped(s[n][e] * (e < 2 ? r0 : r1), p.cap, k2);
    }
    __syncthreads();
    // ---- mixed scores: a warp takes two queries, 8 keys at a time ----
#pragma unroll
    for (int it = 0; it < 2 * kKeys / 8; ++it) {
      const int q = warp * 2 + it / (kKeys / 8), k8 = it % (kKeys / 8) * 8;
      const float* src = s_c + 2 * t4 * kHPitch + q * kQPitch + k8 + g8;
      float o[HT][4] = {};
#pragma unroll
      for (int k = 0; k < HT; ++k) {
        const float* f = src + k * 16 * kHPitch;
        uint32_t b0[3], b1[3];
        split3(f[0], f[kHPitch], b0);
        split3(f[8 * kHPitch], f[9 * kHPitch], b1);
#pragma unroll
        for (int t = 2; t >= 0; --t)   // small terms first
#pragma unroll
          for (int m = 0; m < HT; ++m) mma_bf16(o[m], ta[m][k], b0[t], b1[t]);
      }
      const int bi = kKeys - 1 + q - k8 - 2 * t4;   // bias entry of the lane's first key; the second one is one nearer
      float* dst = p.scores + ((static_cast<long long>(tile) * H) * kTile + q_in + q) * p.span + kb * kKeys + k8 + 2 * t4;
#pragma unroll
      for (int m = 0; m < HT; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int h = m * 16 + g8 + 8 * r;
          if (h < H) {
            const float* bb = s_b + h * kBiasPitch + bi;
            *reinterpret_cast<float2*>(dst + static_cast<long long>(h) * kTile * p.span) =
                make_float2(fmaf(o[m][2 * r], kLog2e, -bb[0]), fmaf(o[m][2 * r + 1], kLog2e, -bb[-1]));
          }
        }
    }
  }
}

constexpr int kValueRows = 64;   // query rows of a values CTA: 4 warps of 16
constexpr int kValueRing = 4;

template <int D>
__global__ void __launch_bounds__(128, D == 64 ? 4 : 3) talk_values_kernel(const TalkParams p) {
  constexpr int CH = D / 8, kBlk = kKeys * D * 2, kScr = 16 * kKeys * 4, kRing = kValueRing;
  extern __shared__ __align__(128) uint8_t s_raw[];
  pdl_wait();
  const int head = blockIdx.x, tile = blockIdx.z, q_in = blockIdx.y * kValueRows, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const Piece x = piece_of(p, tile, q_in, kValueRows);
  if (p.tile_q0[tile] + q_in >= x.len) return;
  const int k_start = first_key(p, tile), H = p.H, kv = head / (H / p.G);
  const int b0 = (x.lo - k_start) / kKeys, n_blk = (x.pos1 - k_start) / kKeys + 1 - b0;   // blocks that some row sees
  const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
  const int n_pg = (p.ctx_lens[x.seq] + 15) >> 4;
  // blocks whose scores exist for this warp's rows
  const int qw = q_in + warp * 16;
  const Piece y = piece_of(p, tile, qw, 16);
  const bool rows = p.tile_q0[tile] + qw < x.len;
  const int w0 = rows ? (y.lo - k_start) / kKeys - b0 : 1 << 30, w1 = rows ? (y.pos1 - k_start) / kKeys - b0 : -1;
  const uint32_t sv = smem_u32(s_raw), ss = sv + kRing * kBlk + warp * kRing * kScr;   // values of the CTA, scores of the warp
  const float* sp = p.scores + ((static_cast<long long>(tile) * H + head) * kTile + qw) * p.span + b0 * kKeys;
  auto issue = [&](int i) {
    if (i < n_blk) {
      const int pg0 = (k_start >> 4) + (b0 + i) * 2;
      const uint32_t dst = sv + (i & (kRing - 1)) * kBlk;
      const int ids[2] = {pg0 < n_pg ? block_of(p, bt, pg0) : -1, pg0 + 1 < n_pg ? block_of(p, bt, pg0 + 1) : -1};
#pragma unroll
      for (int k = 0; k < kKeys * CH / 128; ++k) {
        const int c = tid + k * 128, r = c / CH, ch = c % CH, id = ids[k * 128 / CH >= 16 ? 1 : 0];
        cp_async16(dst + r * (D * 2) + ((ch ^ (r & 7)) << 4),
                   static_cast<const __nv_bfloat16*>(p.cache) + ((static_cast<long long>(max(id, 0)) * p.G + kv) * 16 + (r & 15)) * D + ch * 8, id >= 0);
      }
      if (i >= w0 && i <= w1) {   // 16 rows of 32 scores, 16-byte pieces
        const uint32_t d = ss + (i & (kRing - 1)) * kScr;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int r = k * 4 + (lane >> 3), ch = lane & 7;
          cp_async16(d + r * 128 + ((ch ^ (r & 7)) << 4), sp + static_cast<long long>(r) * p.span + i * kKeys + ch * 4, true);
        }
      }
    }
    cp_commit();
  };
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) issue(i);
  const int g8 = lane >> 2, t4 = lane & 3;
  float o[D / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < D / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  for (int i = 0; i < n_blk; ++i) {
    cp_wait<kRing - 2>();
    __syncthreads();
    issue(i + kRing - 1);
    if (i < w0 || i > w1) continue;
    const uint8_t* sc = s_raw + (ss - sv) + (i & (kRing - 1)) * kScr + (t4 & 1) * 8;
    uint32_t hi[2][4], lo[2][4];   // [row half][8-key group]
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float2 s[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        s[j] = *reinterpret_cast<const float2*>(sc + (g8 + 8 * r) * 128 + (((2 * j + (t4 >> 1)) ^ g8) << 4));
      float mx = fmaxf(fmaxf(fmaxf(s[0].x, s[0].y), fmaxf(s[1].x, s[1].y)), fmaxf(fmaxf(s[2].x, s[2].y), fmaxf(s[3].x, s[3].y)));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      // the reference moves only when a maximum grows by more than 2^8 (or there was none)
      alpha[r] = 1.f;
      if (mx > m[r] + 8.f || m[r] == -INFINITY) {
        const float mn = fmaxf(m[r], mx);
        alpha[r] = m[r] == -INFINITY ? 1.f : ex2t(m[r] - mn);   // (nothing has been added yet: any factor will do)
        m[r] = mn;
      }
      const float ms = m[r] == -INFINITY ? 0.f : m[r];
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float a = ex2t(s[j].x - ms), b = ex2t(s[j].y - ms);
        sum += a + b;
        hi[r][j] = pack_bf16x2(a, b);
        lo[r][j] = pack_bf16x2(a - __uint_as_float(hi[r][j] << 16), b - __uint_as_float(hi[r][j] & 0xffff0000u));
      }
      l[r] = l[r] * alpha[r] + sum;
    }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int n = 0; n < D / 8; ++n) {
        o[n][0] *= alpha[0];
        o[n][1] *= alpha[0];
        o[n][2] *= alpha[1];
        o[n][3] *= alpha[1];
      }
    }
    const uint32_t vb = sv + (i & (kRing - 1)) * kBlk;
#pragma unroll
    for (int ks = 0; ks < 2; ++ks)
#pragma unroll
      for (int n = 0; n < D / 16; ++n) {
        uint32_t v[4];
        const int r = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), ch = n * 2 + (lane >> 4);
        ldsm4t(vb + r * (D * 2) + ((ch ^ (r & 7)) << 4), v);
#pragma unroll
        for (int w = 0; w < 2; ++w)
          mma_bf16(o[2 * n + w], hi[0][2 * ks], hi[1][2 * ks], hi[0][2 * ks + 1], hi[1][2 * ks + 1], v[2 * w], v[2 * w + 1]);
#pragma unroll
        for (int w = 0; w < 2; ++w)
          mma_bf16(o[2 * n + w], lo[0][2 * ks], lo[1][2 * ks], lo[0][2 * ks + 1], lo[1][2 * ks + 1], v[2 * w], v[2 * w + 1]);
      }
  }
  cp_wait<0>();
  const bool even = (p.D & 1) == 0 && (p.ldo & 1) == 0 && (p.gate_ld & 1) == 0;   // pairs of values stay aligned
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float sum = l[r];
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    const int qr = warp * 16 + r * 8 + g8;
    if (x.pos0 + qr > x.pos1) continue;
    const float inv = sum > 0.f ? 1.f / sum : 0.f;
    const long long row = x.row0 + qr;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.ldo;
#pragma unroll
    for (int n = 0; n < D / 8; ++n) {
      const int d = n * 8 + 2 * t4, col = head * p.D + d;
      const float a = o[n][2 * r] * inv, b = o[n][2 * r + 1] * inv;
      if (even) {
        if (d < p.D) {
          const float2 z = p.gate_f32 ? *reinterpret_cast<const float2*>(static_cast<const float*>(p.gate) + row * p.gate_ld + col)
                                      : __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(static_cast<const __nv_bfloat16*>(p.gate) + row * p.gate_ld + col));
          *reinterpret_cast<uint32_t*>(out + col) = pack_bf16x2(__fdividef(a, 1.f + __expf(-z.x)), __fdividef(b, 1.f + __expf(-z.y)));
        }
      } else {
        if (d < p.D) out[col] = __float2bfloat16(a * gate_at(p, row, col));
        if (d + 1 < p.D) out[col + 1] = __float2bfloat16(b * gate_at(p, row, col + 1));
      }
    }
  }
}

template <int D, int HM>
cudaError_t launch_scores(const TalkParams& p, cudaStream_t stream) {
  auto kern = talk_scores_kernel<D, HM>;
  const size_t smem = 4ull * (HM * kHPitch + p.H * kBiasPitch + kKeys);
  ensure_dynamic_smem(kern, smem);
  const int groups = (p.span / kKeys + kBlocks - 1) / kBlocks;
  return launch_kernel(kern, dim3(groups, kTile / kQ, p.n_rows), dim3(256), smem, stream, true, false, p);
}
template <int D>
cudaError_t launch_prefill(const TalkParams& p, cudaStream_t stream) {
  const cudaError_t e = p.H <= 16 ? launch_scores<D, 16>(p, stream) : launch_scores<D, 32>(p, stream);
  if (e != cudaSuccess) return e;
  auto kern = talk_values_kernel<D>;
  const size_t smem = static_cast<size_t>(kValueRing) * (kKeys * D * 2 + 4 * 16 * kKeys * 4);
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(p.H, kTile / kValueRows, p.n_rows), dim3(128), smem, stream, true, false, p);
}
template <int D>
cudaError_t launch_decode(const TalkParams& p, cudaStream_t stream) {
  auto kern = talk_decode_kernel<D>;
  const DecodeLayout l = decode_layout(p.H, p.G, D);
  ensure_dynamic_smem(kern, l.total + 1024);
  // about as many CTAs as fit the SMs at once
  const int fit = (l.total > 100 * 1024 ? 1 : 2) * sm_count() / p.n_rows;
  const int splits = fit < 1 ? 1 : (fit < p.max_splits ? fit : p.max_splits);
  const cudaError_t e = launch_kernel(kern, dim3(p.n_rows, p.max_splits), dim3(kDecThreads), static_cast<size_t>(l.total), stream, true, false, p, l, splits);
  if (e != cudaSuccess) return e;
  return launch_kernel(talk_merge_kernel<D>, dim3(p.n_rows, p.H), dim3(D), 0, stream, true, false, p);
}

}  // namespace

size_t talk_rows_smem(int H, int D) {
  return sizeof(float) * (2ull * H * D + 2ull * H * (kRowKeys + 1) + static_cast<size_t>(H) * H + 3ull * H);
}

cudaError_t launch_talk_rows(const TalkParams& p, int dtype, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  const dim3 grid(p.tile_seq == nullptr ? p.n_rows : p.n_rows * kTile);
  const size_t smem = talk_rows_smem(p.H, p.D);
  if (smem > 226 * 1024) return cudaErrorInvalidValue;
  auto kern = dtype == 1 ? talk_rows_kernel<float> : talk_rows_kernel<__nv_bfloat16>;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, grid, dim3(256), smem, stream, true, false, p);
}

bool talk_decode_ok(int H, int G, int DP) {
  if ((DP != 64 && DP != 128) || H > kMaxHeads || H % G != 0) return false;
  const DecodeLayout l = decode_layout(H, G, DP);
  return G * l.nt * (DP / 16) <= kDecWarps * kMaxTiles && l.total <= 220 * 1024;
}

cudaError_t launch_talk_decode(const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_decode_ok(p.H, p.G, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_decode<64>(p, stream) : launch_decode<128>(p, stream);
}

bool talk_prefill_ok(int H, int DP) { return (DP == 64 || DP == 128) && H <= 32; }

int talk_span(int window, int max_ctx) {
  const int n = window > 0 && window + kTile - 1 < max_ctx ? window + kTile - 1 : max_ctx;
  return (n + 2 * kKeys - 2) / kKeys * kKeys;
}

cudaError_t launch_talk_prefill(const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_prefill_ok(p.H, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_prefill<64>(p, stream) : launch_prefill<128>(p, stream);
}

}  // namespace oxb
