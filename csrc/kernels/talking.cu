// Talking heads over keys that are values (sm_100a): the softmax of a head runs over a mix of all heads' scores, so the scores of
// all heads have to meet before any weight is known. The cache keeps one tensor, the keys before their norm (which are the
// values), and the norm's factor per token; a page is read once for both products.
//
// Decoding (talk_decode): one CTA = (sequence, KV split) walks its pages with all heads. A block of pages in shared memory is
// first the key operand (warps take page x key head), the capped scores meet in shared memory and are mixed there in fp32
// (lanes are positions), and then the same block is the value operand (warps own pieces of the output, [16 dims x 8 heads]).
//
// Prompts: the sums of all heads of a query tile do not fit an SM, the scores of a tile do. talk_scores: one CTA = 32 queries x 32
// keys; a warp keeps the scores of 8 queries x 16 keys for all heads in registers (mma.sync; the tile of one head is too small
// for a 128-row tcgen05 tile), mixes them with fp32 FMAs and writes them out. talk_values: softmax and sums per head from there.
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
constexpr int kMaxTiles = 16;    // 16 x 8 pieces of the output per warp
constexpr int kMaxHeads = 64;

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
  l.pages = l.pages < 2 ? 2 : (l.pages > 8 ? 8 : l.pages);
  l.stage_bytes = l.pages * (l.page_bytes + 64);      // a page and its 16 norm factors
  const int toks = l.pages * 16;
  l.cld = H | 1;                                      // odd: lanes are positions
  l.tld = (H + 3) / 4 * 4;
  l.pld = toks + 8;
  l.stages = 3;
  for (;; --l.stages) {
    l.q = l.stages * l.stage_bytes;
    l.c = l.q + H * (D * 2 + 16);
    l.t = l.c + toks * l.cld * 4;
    l.t = (l.t + 15) / 16 * 16;
    l.phi = l.t + H * l.tld * 4;
    l.plo = l.phi + H * l.pld * 2;
    l.total = l.plo + H * l.pld * 2;
    if (l.total <= 220 * 1024 || l.stages == 2) break;
  }
  return l;
}

template <int D>
__global__ void __launch_bounds__(256) talk_decode_kernel(const TalkParams p) {
  constexpr int CH = D / 8;   // 16-byte chunks per row
  extern __shared__ __align__(128) uint8_t s_raw[];
  __shared__ float s_alpha[kMaxHeads];
  __shared__ int s_ids[2][8];
  const int H = p.H, G = p.G, R = H / G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const DecodeLayout L = decode_layout(H, G, D);
  const uint32_t s_base = smem_u32(s_raw);
  float* s_c = reinterpret_cast<float*>(s_raw + L.c);
  float* s_t = reinterpret_cast<float*>(s_raw + L.t);
  __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(s_raw + L.phi);
  __nv_bfloat16* s_lo = reinterpret_cast<__nv_bfloat16*>(s_raw + L.plo);
  for (int i = tid; i < H * L.tld; i += 256) s_t[i] = i % L.tld < H ? p.talk[i / L.tld * H + i % L.tld] * kLog2e : 0.f;
  pdl_wait();  // q and the newest cache rows come from the kernel before this one
  const int seq = blockIdx.x, split = blockIdx.y, seq_len = p.seq_lens[seq];
  const int win_start = p.window > 0 && seq_len > p.window ? seq_len - p.window : 0;
  int n_pages = (seq_len + 15) / 16;
  if (n_pages > p.max_blocks) {
    if (tid == 0) set_status_once(p.status, kStatusBadIndex);
    n_pages = p.max_blocks;
  }
  int pps = *p.pages_per_split;
  const int first_page = win_start / 16, n_list = n_pages - first_page;
  if (first_page > 0) {   // the host sized the splits for the whole context: spread the visible pages over as many
    const int used = (n_pages + pps - 1) / pps;
    pps = ((n_list + used - 1) / used + L.pages - 1) / L.pages * L.pages;
  }
  const int pg_lo = first_page + split * pps, pg_hi = min(pg_lo + pps, n_pages);
  if (pg_lo >= pg_hi || seq_len <= 0) {
    for (int h = tid; h < H; h += 256) {
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
  auto issue = [&](int b) {
    const uint32_t stage = s_base + (b % L.stages) * L.stage_bytes;
    for (int pg = 0; pg < L.pages; ++pg) {
      const int id = s_ids[b & 1][pg];
      const bool in = id >= 0;
      const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.cache) + static_cast<long long>(in ? id : 0) * G * 16 * D;
      const uint32_t dst = stage + pg * L.page_bytes;
      for (int c = tid; c < page_chunks; c += 256) {
        const int r = c / CH, ch = c % CH;
        cp_async16(dst + r * (D * 2) + ((ch ^ (r & 7)) << 4), src + c * 8, in);
      }
      if (tid < 4) cp_async16(stage + L.pages * L.page_bytes + pg * 64 + tid * 16, p.k_rms + (in ? id : 0) * 16ll + tid * 4, in);
    }
  };
  // queries of all heads, rows D * 2 + 16 bytes apart
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(seq) * p.q_ld;
  for (int c = tid; c < H * CH; c += 256)
    *reinterpret_cast<uint4*>(s_raw + L.q + (c / CH) * (D * 2 + 16) + (c % CH) * 16) = *reinterpret_cast<const uint4*>(qp + c * 8);
  fetch_ids(0);
  fetch_ids(1);
  __syncthreads();
  for (int b = 0; b < L.stages - 1; ++b) {
    if (b < n_blocks) issue(b);
    cp_commit();
    __syncthreads();
    fetch_ids(b + 2);
    __syncthreads();
  }
  float acc[kMaxTiles][4], m_run[8], l_run[8];
#pragma unroll
  for (int j = 0; j < kMaxTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    m_run[i] = -INFINITY;
    l_run[i] = 0.f;
  }
  const int g8 = lane >> 2, t4 = lane & 3;
  const int n_tiles = G * L.nt * (D / 16), toks = L.pages * 16;
  const float k2 = p.cap > 0.f ? 2.f * kLog2e / p.cap : 0.f;
  for (int b = 0; b < n_blocks; ++b) {
    if (L.stages == 3) cp_wait<1>();
    else cp_wait<0>();
    __syncthreads();   // block b has landed; every warp is done with the block before it
    const int nb = b + L.stages - 1;
    if (nb < n_blocks) issue(nb);
    cp_commit();
    const uint32_t stage = s_base + (b % L.stages) * L.stage_bytes;
    const float* s_rms = reinterpret_cast<const float*>(s_raw + (b % L.stages) * L.stage_bytes + L.pages * L.page_bytes);
    // ---- scores: [16 positions x 8 heads] per page, key head and column ----
    for (int u = warp; u < L.pages * G; u += 8) {
      const int pg = u / G, kv = u - pg * G;
      const uint32_t rows = stage + pg * L.page_bytes + kv * (16 * D * 2);
      const float r0 = s_rms[pg * 16 + g8] * p.scale, r1 = s_rms[pg * 16 + g8 + 8] * p.scale;
      for (int nt = 0; nt < L.nt; ++nt) {
        const int hq = min(kv * R + nt * 8 + g8, H - 1);
        const uint8_t* qr = s_raw + L.q + hq * (D * 2 + 16) + t4 * 4;
        float s[4] = {};
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          uint32_t a[4];
          const int r = lane & 15, ch = ks * 2 + (lane >> 4);
          ldsm4(rows + r * (D * 2) + ((ch ^ (r & 7)) << 4), a);
          mma_bf16(s, a, *reinterpret_cast<const uint32_t*>(qr + ks * 32), *reinterpret_cast<const uint32_t*>(qr + ks * 32 + 16));
        }
        const int lh = nt * 8 + 2 * t4, h = kv * R + lh;
        float* c0 = s_c + (pg * 16 + g8) * L.cld + h;
        float* c1 = c0 + 8 * L.cld;
        if (lh < R) {
          c0[0] = capped(s[0] * r0, p.cap, k2);
          c1[0] = capped(s[2] * r1, p.cap, k2);
        }
        if (lh + 1 < R) {
          c0[1] = capped(s[1] * r0, p.cap, k2);
          c1[1] = capped(s[3] * r1, p.cap, k2);
        }
      }
    }
    __syncthreads();
    // ---- mixed scores (times log2 e) and softmax: warps take heads warp + 8 i, lanes positions ----
    const int pos0 = (pg_lo + b * L.pages) * 16;
#pragma unroll
    for (int rep = 0; rep < 2; ++rep) {
      const int hb = warp + 32 * rep;
      if (hb < H) {
        float x[4][4];   // [positions / 32][heads]
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int tc = 0; tc < 4; ++tc) {
          const int tok = tc * 32 + lane, dist = seq_len - 1 - pos0 - tok;
          const bool see = tok < toks && dist >= 0 && (p.window == 0 || dist < p.window);
#pragma unroll
          for (int i = 0; i < 4; ++i) x[tc][i] = 0.f;
          if (tc * 32 < toks) {
            const float* c = s_c + min(tok, toks - 1) * L.cld;
            for (int g = 0; g < L.tld; g += 4) {
              float cv[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) cv[e] = g + e < H ? c[g + e] : 0.f;
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const float4 t = *reinterpret_cast<const float4*>(s_t + min(hb + 8 * i, H - 1) * L.tld + g);
                x[tc][i] = fmaf(t.x, cv[0], fmaf(t.y, cv[1], fmaf(t.z, cv[2], fmaf(t.w, cv[3], x[tc][i]))));
              }
            }
          }
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int h = min(hb + 8 * i, H - 1);
            x[tc][i] = see ? x[tc][i] - kLog2e * __ldg(p.bias + static_cast<long long>(h) * p.n_bias + min(dist, p.n_bias - 1)) : -INFINITY;
            mx[i] = fmaxf(mx[i], x[tc][i]);
          }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int h = hb + 8 * i;
          if (h >= H) break;
          const float m = fmaxf(m_run[rep * 4 + i], warp_max(mx[i])), ms = m == -INFINITY ? 0.f : m;
          const float alpha = ex2t(m_run[rep * 4 + i] - ms);
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
          m_run[rep * 4 + i] = m;
          l_run[rep * 4 + i] = l_run[rep * 4 + i] * alpha + sum;   // of this lane's positions
          if (lane == 0) s_alpha[h] = alpha;
        }
      }
    }
    fetch_ids(nb + 1);   // (the ids of block nb have been read)
    __syncthreads();
    // ---- sums: warps own tiles of [16 dims x 8 heads] ----
#pragma unroll
    for (int j = 0; j < kMaxTiles; ++j) {
      const int ti = warp + 8 * j;
      if (ti < n_tiles) {
        const int mt = ti % (D / 16), gn = ti / (D / 16), kv = gn / L.nt, nt = gn - kv * L.nt;
        const int h0 = kv * R + nt * 8, left = R - nt * 8;
        const float a0 = s_alpha[min(h0 + 2 * t4, H - 1)], a1 = s_alpha[min(h0 + 2 * t4 + 1, H - 1)];
        acc[j][0] *= a0;
        acc[j][1] *= a1;
        acc[j][2] *= a0;
        acc[j][3] *= a1;
        const bool on = g8 < left;
        const int pr = (h0 + (on ? g8 : 0)) * L.pld + 2 * t4;
        for (int pg = 0; pg < L.pages; ++pg) {
          uint32_t a[4];
          const int r = ((lane >> 4) << 3) + (lane & 7), ch = mt * 2 + ((lane >> 3) & 1);
          ldsm4t(stage + pg * L.page_bytes + kv * (16 * D * 2) + r * (D * 2) + ((ch ^ (r & 7)) << 4), a);
          const uint32_t* hi = reinterpret_cast<const uint32_t*>(s_hi + pr + pg * 16);
          const uint32_t* lo = reinterpret_cast<const uint32_t*>(s_lo + pr + pg * 16);
          mma_bf16(acc[j], a, on ? hi[0] : 0u, on ? hi[4] : 0u);
          mma_bf16(acc[j], a, on ? lo[0] : 0u, on ? lo[4] : 0u);
        }
      }
    }
  }
  cp_wait<0>();
  pdl_launch_dependents();
  const long long part0 = static_cast<long long>(seq) * H;
#pragma unroll
  for (int j = 0; j < kMaxTiles; ++j) {
    const int ti = warp + 8 * j;
    if (ti < n_tiles) {
      const int mt = ti % (D / 16), gn = ti / (D / 16), kv = gn / L.nt, nt = gn - kv * L.nt;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int lh = nt * 8 + 2 * t4 + (e & 1), d = mt * 16 + g8 + (e >> 1) * 8;
        if (lh < R) p.part_o[((part0 + kv * R + lh) * p.max_splits + split) * D + d] = acc[j][e];
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int h = warp + 8 * (i & 3) + 32 * (i >> 2);
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
constexpr int kSub = 32;     // queries and keys of a scores CTA

// What a 32-query piece of a tile sees: positions of its first and last row, first visible key.
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
__device__ __forceinline__ int first_key(const TalkParams& p, int tile) { return piece_of(p, tile, 0, kTile).lo / kSub * kSub; }

__device__ __forceinline__ void fma2(float2& d, float2 a, float2 b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;"
      : "+l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
}

// HM: heads of this instantiation (H <= HM)
template <int D, int HM>
__global__ void __launch_bounds__(256, HM <= 16 ? 2 : 1) talk_scores_kernel(const TalkParams p) {
  constexpr int CH = D / 8, kBlk = kSub * D * 2;
  constexpr int kRing = 4;
  extern __shared__ __align__(128) uint8_t s_raw[];
  uint8_t* s_q = s_raw;                    // ring of heads: [32 queries x D]
  uint8_t* s_k = s_raw + kRing * kBlk;     // ring of key heads: [32 keys x D]
  float2* s_t = reinterpret_cast<float2*>(s_raw + 2 * kRing * kBlk);   // [H][HM], every factor twice, times log2 e
  float* s_b = reinterpret_cast<float*>(s_t + p.H * HM);               // [H][64]: bias by distance; +inf hides a key
  __shared__ float s_r[kSub];
  const int H = p.H, R = H / p.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < H * HM; i += 256) {
    const float t = i % HM < H ? p.talk[i / HM * H + i % HM] * kLog2e : 0.f;
    s_t[i] = make_float2(t, t);
  }
  pdl_wait();
  const int tile = blockIdx.z, q_in = blockIdx.y * kSub;
  const Piece x = piece_of(p, tile, q_in, kSub);
  if (p.tile_q0[tile] + q_in >= x.len) return;
  const int k_start = first_key(p, tile), k0 = k_start + blockIdx.x * kSub;
  if (k0 > x.pos1 || k0 + kSub <= x.lo) return;
  const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
  const int ctx = p.ctx_lens[x.seq], pg0 = k0 >> 4, n_pg = (ctx + 15) >> 4;
  const int id0 = block_of(p, bt, pg0), id1 = pg0 + 1 < n_pg ? block_of(p, bt, pg0 + 1) : -1;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(x.row0) * p.q_ld;
  const int n_q = x.pos1 - x.pos0 + 1;
  auto issue = [&](int h) {
    if (h < H) {
      const uint32_t dq = smem_u32(s_q) + (h & (kRing - 1)) * kBlk;
#pragma unroll
      for (int i = 0; i < kSub * CH / 256; ++i) {
        const int c = tid + i * 256, r = c / CH, ch = c % CH;
        const bool in = r < n_q;
        cp_async16(dq + r * (D * 2) + ((ch ^ (r & 7)) << 4), qp + (in ? r : 0) * p.q_ld + h * D + ch * 8, in);
      }
      if (h % R == 0) {
        const int kv = h / R;
        const uint32_t dk = smem_u32(s_k) + (kv & (kRing - 1)) * kBlk;
#pragma unroll
        for (int i = 0; i < kSub * CH / 256; ++i) {
          const int c = tid + i * 256, r = c / CH, ch = c % CH, id = r < 16 ? id0 : id1;
          const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.cache) + (static_cast<long long>(max(id, 0)) * p.G + kv) * 16 * D;
          cp_async16(dk + r * (D * 2) + ((ch ^ (r & 7)) << 4), src + (r & 15) * D + ch * 8, id >= 0);
        }
      }
    }
    cp_commit();
  };
#pragma unroll
  for (int h = 0; h < kRing - 1; ++h) issue(h);
  if (tid < kSub) {
    const int id = tid < 16 ? id0 : id1;
    s_r[tid] = id >= 0 ? p.k_rms[id * 16ll + (tid & 15)] * p.scale : 0.f;
  }
  const int far0 = x.pos0 - k0 - 31;   // distance of bias entry 0
  for (int i = tid; i < H * 64; i += 256) {
    const int dist = far0 + (i & 63);
    const bool see = dist >= 0 && (p.window == 0 || dist < p.window);
    s_b[i] = see ? kLog2e * __ldg(p.bias + static_cast<long long>(i >> 6) * p.n_bias + min(dist, p.n_bias - 1)) : INFINITY;
  }
  const int kh = warp & 1, qo = warp >> 1, g8 = lane >> 2, t4 = lane & 3;   // 16 keys, 8 queries of this warp
  const float k2 = p.cap > 0.f ? 2.f * kLog2e / p.cap : 0.f;
  float2 c[HM][2];   // scores: (key g8 | key g8 + 8) x (queries 2 t4, 2 t4 + 1)
  uint32_t kf[D / 16][4];
  float r0 = 0.f, r1 = 0.f;
#pragma unroll
  for (int h = 0; h < HM; ++h) {
    c[h][0] = c[h][1] = make_float2(0.f, 0.f);
    if (h < H) {
      cp_wait<kRing - 2>();
      __syncthreads();   // head h has landed; every warp is done with head h - 1
      issue(h + kRing - 1);
      if (h == 0) {
        r0 = s_r[kh * 16 + g8];
        r1 = s_r[kh * 16 + g8 + 8];
      }
      if (h % R == 0) {
        const uint32_t kb = smem_u32(s_k) + ((h / R) & (kRing - 1)) * kBlk;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          const int r = kh * 16 + (lane & 15), ch = ks * 2 + (lane >> 4);
          ldsm4(kb + r * (D * 2) + ((ch ^ (r & 7)) << 4), kf[ks]);
        }
      }
      const uint32_t qb = smem_u32(s_q) + (h & (kRing - 1)) * kBlk;
      float s[2][4] = {};
#pragma unroll
      for (int k2s = 0; k2s < D / 32; ++k2s) {
        uint32_t b[4];
        const int r = qo * 8 + (lane & 7), ch = k2s * 4 + (lane >> 3);
        ldsm4(qb + r * (D * 2) + ((ch ^ (r & 7)) << 4), b);
        mma_bf16(s[0], kf[2 * k2s], b[0], b[1]);
        mma_bf16(s[1], kf[2 * k2s + 1], b[2], b[3]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[0][e] = capped((s[0][e] + s[1][e]) * (e < 2 ? r0 : r1), p.cap, k2);
      c[h][0] = make_float2(s[0][0], s[0][1]);
      c[h][1] = make_float2(s[0][2], s[0][3]);
    }
  }
  cp_wait<0>();
  const int key = kh * 16 + g8, q = qo * 8 + 2 * t4;
  float* dst = p.scores + (static_cast<long long>(tile) * H * kTile + q_in + q) * p.span + (k0 - k_start) + key;
  const int bi = 31 + q - key;
  for (int h = 0; h < H; ++h) {
    const float4* t = reinterpret_cast<const float4*>(s_t + h * HM);
    float2 a[2][2] = {};
#pragma unroll
    for (int g = 0; g < HM; g += 2) {
      const float4 f = t[g >> 1];
      const float2 f0 = make_float2(f.x, f.y), f1 = make_float2(f.z, f.w);
      fma2(a[0][0], c[g][0], f0);
      fma2(a[0][1], c[g][1], f0);
      fma2(a[1][0], c[g + 1][0], f1);
      fma2(a[1][1], c[g + 1][1], f1);
    }
    const float* bb = s_b + h * 64 + bi;
    float* d = dst + static_cast<long long>(h) * kTile * p.span;
    d[0] = a[0][0].x + a[1][0].x - bb[0];
    d[p.span] = a[0][0].y + a[1][0].y - bb[1];
    d[8] = a[0][1].x + a[1][1].x - bb[-8];
    d[p.span + 8] = a[0][1].y + a[1][1].y - bb[-7];
  }
}

constexpr int kValueRows = 64;   // query rows of a values CTA: 4 warps of 16

template <int D>
__global__ void __launch_bounds__(128) talk_values_kernel(const TalkParams p) {
  constexpr int CH = D / 8, kBlk = kSub * D * 2, kRing = 4;
  extern __shared__ __align__(128) uint8_t s_raw[];
  pdl_wait();
  const int head = blockIdx.x, tile = blockIdx.z, q_in = blockIdx.y * kValueRows, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const Piece x = piece_of(p, tile, q_in, kValueRows);
  if (p.tile_q0[tile] + q_in >= x.len) return;
  const int k_start = first_key(p, tile), H = p.H, kv = head / (H / p.G);
  const int b0 = (x.lo - k_start) / kSub, n_blk = (x.pos1 - k_start) / kSub + 1 - b0;   // 32-key blocks that some row sees
  const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
  const int n_pg = (p.ctx_lens[x.seq] + 15) >> 4;
  auto issue = [&](int i) {
    if (i < n_blk) {
      const int pg0 = (k_start >> 4) + (b0 + i) * 2;
      const uint32_t dst = smem_u32(s_raw) + (i & (kRing - 1)) * kBlk;
#pragma unroll
      for (int k = 0; k < kSub * CH / 128; ++k) {
        const int c = tid + k * 128, r = c / CH, ch = c % CH, pg = pg0 + (r >> 4);
        const bool in = pg < n_pg;
        const int id = in ? block_of(p, bt, pg) : 0;
        cp_async16(dst + r * (D * 2) + ((ch ^ (r & 7)) << 4),
                   static_cast<const __nv_bfloat16*>(p.cache) + ((static_cast<long long>(id) * p.G + kv) * 16 + (r & 15)) * D + ch * 8, in);
      }
    }
    cp_commit();
  };
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) issue(i);
  // blocks whose scores exist for this warp's rows
  const int qw = q_in + warp * 16;
  const Piece y = piece_of(p, tile, qw / kSub * kSub, kSub);
  const bool rows = p.tile_q0[tile] + qw < x.len;
  const int w0 = rows ? (y.lo - k_start) / kSub - b0 : 1 << 30, w1 = rows ? (y.pos1 - k_start) / kSub - b0 : -1;
  const int g8 = lane >> 2, t4 = lane & 3;
  const float* sp = p.scores + ((static_cast<long long>(tile) * H + head) * kTile + qw + g8) * p.span + b0 * kSub + 2 * t4;
  float2 nxt[2][4];
  auto load = [&](int i) {
    if (i >= w0 && i <= w1) {
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int j = 0; j < 4; ++j) nxt[r][j] = __ldcs(reinterpret_cast<const float2*>(sp + r * 8ll * p.span + i * kSub + j * 8));
    }
  };
  load(0);
  float o[D / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < D / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  for (int i = 0; i < n_blk; ++i) {
    cp_wait<kRing - 2>();
    __syncthreads();
    issue(i + kRing - 1);
    if (i < w0 || i > w1) {
      load(i + 1);
      continue;
    }
    float2 s[2][4];
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[r][j] = nxt[r][j];
    load(i + 1);
    uint32_t hi[2][4], lo[2][4];   // [row half][8-key group]
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < 4; ++j) mx = fmaxf(mx, fmaxf(s[r][j].x, s[r][j].y));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m[r], mx), ms = mn == -INFINITY ? 0.f : mn;
      alpha[r] = ex2t(m[r] - ms);
      m[r] = mn;
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float a = ex2t(s[r][j].x - ms), b = ex2t(s[r][j].y - ms);
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
    const uint32_t vb = smem_u32(s_raw) + (i & (kRing - 1)) * kBlk;
#pragma unroll
    for (int ks = 0; ks < 2; ++ks)
#pragma unroll
      for (int n = 0; n < D / 16; ++n) {
        uint32_t v[4];
        const int r = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), ch = n * 2 + (lane >> 4);
        ldsm4t(vb + r * (D * 2) + ((ch ^ (r & 7)) << 4), v);
#pragma unroll
        for (int w = 0; w < 2; ++w) {
          mma_bf16(o[2 * n + w], hi[0][2 * ks], hi[1][2 * ks], hi[0][2 * ks + 1], hi[1][2 * ks + 1], v[2 * w], v[2 * w + 1]);
          mma_bf16(o[2 * n + w], lo[0][2 * ks], lo[1][2 * ks], lo[0][2 * ks + 1], lo[1][2 * ks + 1], v[2 * w], v[2 * w + 1]);
        }
      }
  }
  cp_wait<0>();
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
    for (int n = 0; n < D / 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = n * 8 + 2 * t4 + e, col = head * p.D + d;
        if (d < p.D) out[col] = __float2bfloat16(o[n][2 * r + e] * inv * gate_at(p, row, col));
      }
  }
}

template <int D, int HM>
cudaError_t launch_scores(const TalkParams& p, cudaStream_t stream) {
  auto kern = talk_scores_kernel<D, HM>;
  const size_t smem = 8ull * kSub * D * 2 + p.H * HM * 8ull + p.H * 64 * 4ull;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(p.span / kSub, kTile / kSub, p.n_rows), dim3(256), smem, stream, true, false, p);
}
template <int D>
cudaError_t launch_prefill(const TalkParams& p, cudaStream_t stream) {
  const cudaError_t e = p.H <= 8 ? launch_scores<D, 8>(p, stream) : (p.H <= 16 ? launch_scores<D, 16>(p, stream) : launch_scores<D, 32>(p, stream));
  if (e != cudaSuccess) return e;
  auto kern = talk_values_kernel<D>;
  const size_t smem = 4ull * kSub * D * 2;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(p.H, kTile / kValueRows, p.n_rows), dim3(128), smem, stream, true, false, p);
}
template <int D>
cudaError_t launch_decode(const TalkParams& p, cudaStream_t stream) {
  auto kern = talk_decode_kernel<D>;
  const size_t smem = decode_layout(p.H, p.G, D).total;
  ensure_dynamic_smem(kern, smem);
  const cudaError_t e = launch_kernel(kern, dim3(p.n_rows, p.max_splits), dim3(256), smem, stream, true, false, p);
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
  return G * l.nt * (DP / 16) <= 8 * kMaxTiles && l.total <= 220 * 1024;
}

cudaError_t launch_talk_decode(const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_decode_ok(p.H, p.G, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_decode<64>(p, stream) : launch_decode<128>(p, stream);
}

bool talk_prefill_ok(int H, int DP) { return (DP == 64 || DP == 128) && H <= 32; }

int talk_span(int window, int max_ctx) {
  const int n = window > 0 && window + kTile - 1 < max_ctx ? window + kTile - 1 : max_ctx;
  return (n + 2 * kSub - 2) / kSub * kSub;
}

cudaError_t launch_talk_prefill(const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_prefill_ok(p.H, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_prefill<64>(p, stream) : launch_prefill<128>(p, stream);
}

}  // namespace oxb
