// Talking heads over keys that are values (sm_100a): the softmax of a head runs over a mix of all heads' scores, so the scores of
// all heads have to meet before any weight is known. The cache keeps one tensor, the keys before their norm (which are the
// values), and the norm's factor per token; a page is read once for both products.
//
// Decoding (talk_decode): one CTA = (sequence, KV split) walks its pages with all heads. A block of pages (by TMA) in shared memory is
// first the key operand (warps take page x key head); the capped scores meet in shared memory and are mixed there (warps take page x
// 8 mixed heads); then the same block is the value operand (warps own pieces of the output, [16 dims x 8 heads]).
//
// Prompts: the sums of all heads of a query tile do not fit an SM, the scores of a tile do. talk_scores: one CTA = 16 queries, 32 keys
// at a time; the scores of all heads (mma.sync: a head's 16 x 32 tile is too small for a 128-row tcgen05 tile) meet in shared memory,
// are mixed as a product with the heads' matrix and written out. talk_values: softmax and sums per head from there (tcgen05).
//
// talk_rows takes any sizes in fp32 FMAs, one row per CTA.
#include "../common/device_info.h"
#include "hybrid_mma.cuh"

#include <cuda_fp16.h>

namespace oxb {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2t(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcpt(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// The score of a product x: cap tanh(x f / cap) = cap - 2 cap / (e^(2 x f / cap) + 1), good to about cap * 2^-22, or x f without a
// cap. f: factor of the key, already times 2 log2(e) / cap where there is a cap (key_factor); the result is times `unit`.
struct Cap {
  float k, top;   // 2 log2(e) / cap, cap (0: none); top and 2 top times unit
  float unit;
};
__device__ __forceinline__ Cap cap_of(float cap, float unit) { return {cap > 0.f ? 2.f * kLog2e / cap : 1.f, cap * unit, unit}; }
__device__ __forceinline__ float capped(float x, float f, const Cap& c) {
  if (c.top == 0.f) return fminf(fmaxf(x * f * c.unit, -60000.f), 60000.f);
  return fmaf(-2.f * c.top, rcpt(ex2t(x * f) + 1.f), c.top);
}
__device__ __forceinline__ float gate_at(const TalkParams& p, long long row, int col) {
  const float z = p.gate_f32 ? static_cast<const float*>(p.gate)[row * p.gate_ld + col]
                             : to_f(static_cast<const __nv_bfloat16*>(p.gate)[row * p.gate_ld + col]);
  return 1.f / (1.f + expf(-z));
}
// Block id of page pg of a sequence, as it stands in the table (loaded ahead of its use), and checked: ids outside the pool are
// recorded and replaced by 0.
__device__ __forceinline__ int raw_block(const TalkParams& p, const int* bt, int pg) { return pg < p.max_blocks ? bt[pg] : -1; }
__device__ __forceinline__ int checked_block(const TalkParams& p, int b) {
  if (static_cast<unsigned>(b) < static_cast<unsigned>(p.num_blocks)) return b;
  set_status_once(p.status, kStatusBadIndex);
  return 0;
}
__device__ __forceinline__ int block_of(const TalkParams& p, const int* bt, int pg) { return checked_block(p, raw_block(p, bt, pg)); }

// Mixing the heads' scores is a product with the heads' matrix: the scores (fp32) enter as two fp16 terms, which carry 22 bits of
// them (scores without a cap are kept inside fp16's range); the matrix holds bf16 values, exact in fp16 but for tiny ones.
__device__ __forceinline__ uint32_t pack_f16x2(float a, float b) {
  const __half2 v = __floats2half2_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void split_f16(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __half2 h = __floats2half2_rn(a, b);
  const float2 f = __half22float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_f16x2(a - f.x, b - f.y);
}
__device__ __forceinline__ void mma_f16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 "
      "{%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t x) {
  uint32_t y;
  asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
  return y;
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
constexpr int kMaxPages = 8;     // pages per block
constexpr int kMaxUnits = 4;     // (page, key head) per warp

// A block holds `pages` pages; pages * mt <= 16, so every (page, 8 mixed heads) has a warp.
struct DecodeLayout {
  int pages, stages, nt, mt, hk;     // pages per block, ring stages, 8-head columns per key head and in all, 16-head steps
  int box;                           // key heads per copy
  int tiles;                         // output pieces per warp, a power of two
  int cld, tld, pld;                 // row pitches of the scores (fp32), the matrix (fp16) and the weights (bf16)
  int page_bytes, rms, q, c, t, phi, plo, red, bar, total;
};
inline DecodeLayout decode_layout(int H, int G, int D) {
  DecodeLayout l;
  const int R = H / G;
  l.nt = (R + 7) / 8;
  l.mt = (H + 7) / 8;
  l.hk = (H + 15) / 16;
  l.box = G < 16 ? G : 16;
  while (G % l.box) --l.box;
  l.tiles = 2;
  while (l.tiles * kDecWarps < G * l.nt * (D / 16)) l.tiles *= 2;
  l.page_bytes = G * 16 * D * 2;
  l.pages = 65536 / l.page_bytes;
  if (l.pages > kMaxPages) l.pages = kMaxPages;
  if (l.pages > kDecWarps / l.mt) l.pages = kDecWarps / l.mt;
  if (l.pages * G > kDecWarps * kMaxUnits) l.pages = kDecWarps * kMaxUnits / G;
  if (l.pages < 1) l.pages = 1;
  l.cld = (l.hk * 16 + 23) / 32 * 32 + 8;             // 8 mod 32: four rows of eight 8-byte pieces touch all banks
  l.tld = l.hk * 16 + 8;
  l.pld = l.pages * 16 + 8;
  l.stages = 3;
  for (;; --l.stages) {
    l.rms = l.stages * l.pages * l.page_bytes;        // norm factors, 16 per page
    l.q = l.rms + l.stages * l.pages * 64;
    l.c = l.q + H * (D * 2 + 16);
    l.t = l.c + l.pages * 16 * l.cld * 4;
    l.phi = l.t + l.mt * 8 * l.tld * 2;
    l.plo = l.phi + l.mt * 8 * l.pld * 2;
    l.red = l.plo + l.mt * 8 * l.pld * 2;             // fp32: page maxima, then reference, factor and sum per head
    l.bar = (l.red + (l.pages + 3) * l.mt * 8 * 4 + 7) / 8 * 8;
    l.total = l.bar + 3 * 8 + 1024;
    if (l.total <= 222 * 1024 || l.stages == 2) break;
  }
  return l;
}

// TPW: output pieces per warp, all of one column of heads, or of two
template <int D, int TPW>
__global__ void __launch_bounds__(kDecThreads) talk_decode_kernel(const __grid_constant__ CUtensorMap tmC, const TalkParams p, const DecodeLayout L) {
  constexpr int CH = D / 8, MT = D / 16, HF = D / 64;          // 16-byte chunks of a row, pieces of 16 dims, 128-byte halves
  constexpr int NG = TPW > MT ? TPW / MT : 1, JG = TPW / NG;   // columns per warp, pieces of each
  extern __shared__ uint8_t s_unaligned[];
  uint8_t* s_raw = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(s_unaligned) + 1023) & ~uintptr_t(1023));
  const int H = p.H, G = p.G, R = H / G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t s_base = smem_u32(s_raw);
  float* s_c = reinterpret_cast<float*>(s_raw + L.c);
  __half* s_t = reinterpret_cast<__half*>(s_raw + L.t);
  __nv_bfloat16* s_hi = reinterpret_cast<__nv_bfloat16*>(s_raw + L.phi);
  const int lo_off = (L.plo - L.phi) / 4;                   // low terms, in pairs behind the high ones
  const int h8 = L.mt * 8;
  float* s_max = reinterpret_cast<float*>(s_raw + L.red);   // [page][head] largest score of a page
  float* s_ref = s_max + L.pages * h8;                      // reference that weights are relative to
  float* s_alpha = s_ref + h8;                              // what the sums are multiplied by when it moves
  float* s_sum = s_alpha + h8;
  uint64_t* full = reinterpret_cast<uint64_t*>(s_raw + L.bar);
  for (int h = warp; h < h8; h += kDecWarps)
    for (int g = lane; g < L.hk * 16; g += 32) s_t[h * L.tld + g] = __float2half(h < H && g < H ? p.talk[h * H + g] : 0.f);
  for (int i = tid; i < L.pages * 16 * L.cld; i += kDecThreads) s_c[i] = 0.f;   // (columns beyond the heads stay zero)
  if (tid < h8) {
    s_ref[tid] = -INFINITY;
    s_sum[tid] = 0.f;
  }
  if (tid == 0) {
    tma_prefetch_desc(&tmC);
    for (int i = 0; i < L.stages; ++i) mbar_init(&full[i], 1);
    fence_mbar_init();
  }
  pdl_wait();  // q and the newest cache rows come from the kernel before this one
  const int seq = blockIdx.x, split = blockIdx.y, seq_len = p.seq_lens[seq];
  const int win_start = p.window > 0 && seq_len > p.window ? seq_len - p.window : 0;
  int n_pages = (seq_len + 15) / 16;
  if (n_pages > p.max_blocks) {
    if (tid == 0) set_status_once(p.status, kStatusBadIndex);
    n_pages = p.max_blocks;
  }
  // the visible pages over the splits, in whole blocks
  const int first_page = win_start / 16, n_list = n_pages - first_page, n_splits = gridDim.y;
  const int pps = ((n_list + n_splits - 1) / n_splits + L.pages - 1) / L.pages * L.pages;
  const int pg_lo = first_page + split * pps, pg_hi = min(pg_lo + pps, n_pages);
  const long long part0 = static_cast<long long>(seq) * H;
  if (pg_lo >= pg_hi || seq_len <= 0) {
    for (int h = tid; h < H; h += kDecThreads) {
      float* ml = p.part_ml + ((part0 + h) * p.max_splits + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  const int n_blocks = (pg_hi - pg_lo + L.pages - 1) / L.pages;
  // copies (by the last warp, which is the likeliest to have no scores to mix): per page the boxes of its key heads and 64 dims, and
  // its norm factors; lane pg holds the block id of page pg
  constexpr int kCopyWarp = kDecWarps - 1;
  const int per_page = G / L.box * HF + 1;
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  auto id_of = [&](int b) {
    const int pg = pg_lo + b * L.pages + lane;
    return lane < L.pages && pg < pg_hi ? raw_block(p, bt, pg) : 0;
  };
  auto issue = [&](int b, int slot, int id) {
    const int n = min(L.pages, pg_hi - pg_lo - b * L.pages);
    if (lane == 0) mbar_arrive_expect_tx(&full[slot], n * (L.page_bytes + 64));
    id = checked_block(p, id);
    __syncwarp();
    for (int c0 = 0; c0 < n * per_page; c0 += 32) {
      const int c = c0 + lane, pg = c / per_page, k = c - pg * per_page;
      const int blk = __shfl_sync(0xffffffffu, id, pg & 31);
      if (pg >= n) continue;
      const int at = slot * L.pages + pg;
      if (k == per_page - 1) {
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], 64, [%2];" ::"r"(s_base + L.rms + at * 64),
                     "l"(p.k_rms + blk * 16ll), "r"(smem_u32(&full[slot]))
                     : "memory");
      } else {
        const int hf = k % HF, g0 = k / HF * L.box;
        tma_load_2d(s_raw + at * L.page_bytes + hf * (G * 2048) + g0 * 2048, &tmC, &full[slot], hf * 64, (blk * G + g0) * 16);
      }
    }
  };
  __syncthreads();   // (the barriers are set up)
  int id = 0;
  if (warp == kCopyWarp) {
    id = id_of(0);
    for (int b = 0; b < L.stages - 1; ++b) {
      if (b < n_blocks) issue(b, b, id);
      id = id_of(b + 1);
    }
  }
  // queries of all heads, rows D * 2 + 16 bytes apart
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(seq) * p.q_ld;
  for (int c = tid; c < H * CH; c += kDecThreads)
    *reinterpret_cast<uint4*>(s_raw + L.q + (c / CH) * (D * 2 + 16) + (c % CH) * 16) = *reinterpret_cast<const uint4*>(qp + c * 8);
  __syncthreads();
  float acc[TPW][4], l_run[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < TPW; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const int g8 = lane >> 2, t4 = lane & 3;
  const Cap cap = cap_of(p.cap, kLog2e);   // scores times log2 e
  const float unit = p.scale * cap.k;
  // What this warp does in every block. Scores: (page, key head) warp + 16 i.
  int k_page[kMaxUnits], k_at[kMaxUnits], k_kv[kMaxUnits];
  {
    const int r = lane & 15;
#pragma unroll
    for (int i = 0; i < kMaxUnits; ++i) {
      const int u = warp + i * kDecWarps;
      k_page[i] = u / G;
      k_kv[i] = u - k_page[i] * G;
      k_at[i] = k_page[i] * L.page_bytes + k_kv[i] * 2048 + r * 128 + (((lane >> 4) ^ (r & 7)) << 4);
    }
  }
  // Mixed scores: page m_page, heads m8 .. m8 + 7
  const int m_page = warp / L.mt, m8 = (warp - m_page * L.mt) * 8, mh = m8 + 2 * t4;
  const float* m_c = s_c + (m_page * 16 + g8) * L.cld + 2 * t4;
  const __half* m_t = s_t + (m8 + g8) * L.tld + 2 * t4;
  uint32_t* m_w = reinterpret_cast<uint32_t*>(s_hi + (m8 + g8) * L.pld + m_page * 16 + 2 * t4);
  const float* m_bias0 = p.bias + static_cast<long long>(min(mh, H - 1)) * p.n_bias;
  const float* m_bias1 = p.bias + static_cast<long long>(min(mh + 1, H - 1)) * p.n_bias;
  // Sums: pieces warp * TPW .. of the list (column of heads, 16 dims)
  int v_at[NG], v_w[NG], v_h[NG];
  bool v_on[NG];
  const int v_x = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
#pragma unroll
  for (int n = 0; n < NG; ++n) {
    const int gn = (warp * TPW + n * JG) / MT;
    v_on[n] = gn < G * L.nt;
    const int kv = min(gn / L.nt, G - 1), nt = v_on[n] ? gn - kv * L.nt : 0, row = ((lane >> 4) << 3) + (lane & 7);
    v_at[n] = kv * 2048 + row * 128 + v_x;
    v_h[n] = kv * R + nt * 8;
    v_w[n] = min(v_h[n] + g8, H - 1) * L.pld / 2 + t4;   // (what columns beyond the heads sum up is not used)
  }
  const int mt0 = (warp * TPW) % MT;
  const uint32_t* s_w = reinterpret_cast<const uint32_t*>(s_hi);
  int slot = 0, phase = 0;
  bool ok = true;
  for (int b = 0; b < n_blocks; ++b) {
    const int np = min(L.pages, pg_hi - pg_lo - b * L.pages);
    // biases of this warp's mixed scores: positions g8 and g8 + 8; +inf hides a position
    const int dist = seq_len - 1 - (pg_lo + b * L.pages + m_page) * 16 - g8;
    float x[4] = {INFINITY, INFINITY, INFINITY, INFINITY};
    if (m_page < np) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = dist - 8 * e, at = min(d, p.n_bias - 1);
        if (d >= 0 && (p.window == 0 || d < p.window)) {
          if (mh < H) x[2 * e] = __ldg(m_bias0 + at);
          if (mh + 1 < H) x[2 * e + 1] = __ldg(m_bias1 + at);
        }
      }
    }
    if (ok && !mbar_wait(&full[slot], phase)) {
      set_status_once(p.status, kStatusMbarTimeoutProducer);
      ok = false;
    }
    const uint32_t stage = s_base + slot * L.pages * L.page_bytes;
    const float* s_rms = reinterpret_cast<const float*>(s_raw + L.rms) + slot * L.pages * 16 + g8;
    // ---- scores: [16 positions x 8 heads] per page, key head and column ----
#pragma unroll
    for (int i = 0; i < kMaxUnits; ++i) {
      if (k_page[i] < np) {
        const uint32_t at = stage + k_at[i];
        const float r0 = s_rms[k_page[i] * 16] * unit, r1 = s_rms[k_page[i] * 16 + 8] * unit;
        for (int nt = 0; nt < L.nt; ++nt) {
          const int lh = nt * 8 + 2 * t4, h = k_kv[i] * R + nt * 8;
          const uint8_t* qr = s_raw + L.q + min(h + g8, H - 1) * (D * 2 + 16) + t4 * 4;
          float s[2][4] = {};
#pragma unroll
          for (int ks = 0; ks < MT; ++ks) {
            uint32_t a[4];
            ldsm4((at + (ks >> 2) * G * 2048) ^ ((ks & 3) << 5), a);
            mma_bf16(s[ks & 1], a, *reinterpret_cast<const uint32_t*>(qr + ks * 32), *reinterpret_cast<const uint32_t*>(qr + ks * 32 + 16));
          }
          float* c0 = s_c + (k_page[i] * 16 + g8) * L.cld + h + 2 * t4;
          float* c1 = c0 + 8 * L.cld;
          const float y00 = capped(s[0][0] + s[1][0], r0, cap), y01 = capped(s[0][1] + s[1][1], r0, cap);
          const float y10 = capped(s[0][2] + s[1][2], r1, cap), y11 = capped(s[0][3] + s[1][3], r1, cap);
          if (lh < R) {
            c0[0] = y00;
            c1[0] = y10;
          }
          if (lh + 1 < R) {
            c0[1] = y01;
            c1[1] = y11;
          }
        }
      }
    }
    __syncthreads();   // (and every warp is done with the sums of the block before)
    if (warp == kCopyWarp) {
      const int nb = b + L.stages - 1;
      if (nb < n_blocks) issue(nb, slot == 0 ? L.stages - 1 : slot - 1, id);
      id = id_of(nb + 1);
    }
    // ---- mixed scores and weights, relative to a reference that moves when a score is 2^8 above it ----
    float sum[2] = {0.f, 0.f};
    auto weights = [&]() {
      const float2 f = *reinterpret_cast<const float2*>(s_ref + mh);
      const float r0 = f.x == -INFINITY ? 0.f : f.x, r1 = f.y == -INFINITY ? 0.f : f.y;
      const float e00 = ex2t(x[0] - r0), e01 = ex2t(x[1] - r1), e10 = ex2t(x[2] - r0), e11 = ex2t(x[3] - r1);
      sum[0] = e00 + e10;
      sum[1] = e01 + e11;
      const uint32_t h0 = pack_bf16x2(e00, e01), h1 = pack_bf16x2(e10, e11);
      const uint32_t l0 = pack_bf16x2(e00 - __uint_as_float(h0 << 16), e01 - __uint_as_float(h0 & 0xffff0000u));
      const uint32_t l1 = pack_bf16x2(e10 - __uint_as_float(h1 << 16), e11 - __uint_as_float(h1 & 0xffff0000u));
      m_w[0] = movmatrix_trans(h0);   // transposed: head g8, positions 2 t4 and 2 t4 + 1
      m_w[4] = movmatrix_trans(h1);
      m_w[lo_off] = movmatrix_trans(l0);
      m_w[lo_off + 4] = movmatrix_trans(l1);
    };
    bool above = false;
    if (m_page < np) {
      float mixed[4] = {};
      for (int ks = 0; ks < L.hk; ++ks) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = *reinterpret_cast<const float2*>(m_c + (e & 1) * 8 * L.cld + ks * 16 + (e >> 1) * 8);
          split_f16(v.x, v.y, hi[e], lo[e]);
        }
        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(m_t + ks * 16), b1 = *reinterpret_cast<const uint32_t*>(m_t + ks * 16 + 8);
        mma_f16(mixed, lo, b0, b1);
        mma_f16(mixed, hi, b0, b1);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = fmaf(-kLog2e, x[e], mixed[e]);
      float m0 = fmaxf(x[0], x[2]), m1 = fmaxf(x[1], x[3]);
#pragma unroll
      for (int w = 4; w < 32; w <<= 1) {
        m0 = fmaxf(m0, __shfl_xor_sync(0xffffffffu, m0, w));
        m1 = fmaxf(m1, __shfl_xor_sync(0xffffffffu, m1, w));
      }
      if (g8 == 0) *reinterpret_cast<float2*>(s_max + m_page * h8 + mh) = make_float2(m0, m1);
      const float2 f = *reinterpret_cast<const float2*>(s_ref + mh);
      above = m0 > f.x + 8.f || m1 > f.y + 8.f;   // (a reference of -inf: any score)
      weights();
    }
    const int state = __syncthreads_or((above ? 1 : 0) | (ok ? 0 : 2));
    if (state & 2) {   // some thread gave up its wait: all leave together, once the copies under way have had their time
      ok = false;
      for (int k = b; k < min(b + L.stages, n_blocks); ++k) {
        mbar_wait(&full[slot], phase);
        if (++slot == L.stages) {
          slot = 0;
          phase ^= 1;
        }
      }
      break;
    }
    if (state) {
      // the reference of some head moves: new references, weights once more, sums so far rescaled
      if (tid < H) {
        const float old = s_ref[tid];
        float ref = old;
        for (int pg = 0; pg < np; ++pg) ref = fmaxf(ref, s_max[pg * h8 + tid]);
        s_ref[tid] = ref;
        s_alpha[tid] = old == -INFINITY ? 0.f : ex2t(old - ref);
      }
      __syncthreads();
      if (m_page < np) weights();
      l_run[0] *= s_alpha[min(mh, H - 1)];
      l_run[1] *= s_alpha[min(mh + 1, H - 1)];
#pragma unroll
      for (int n = 0; n < NG; ++n) {
        const float a0 = s_alpha[min(v_h[n] + 2 * t4, H - 1)], a1 = s_alpha[min(v_h[n] + 2 * t4 + 1, H - 1)];
#pragma unroll
        for (int j = n * JG; j < (n + 1) * JG; ++j) {
          acc[j][0] *= a0;
          acc[j][1] *= a1;
          acc[j][2] *= a0;
          acc[j][3] *= a1;
        }
      }
      __syncthreads();
    }
    l_run[0] += sum[0];
    l_run[1] += sum[1];
    // ---- sums: pieces of [16 dims x 8 heads] ----
#pragma unroll
    for (int n = 0; n < NG; ++n)
      if (v_on[n]) {
        uint32_t at = stage + v_at[n];
        const uint32_t* w = s_w + v_w[n];
        for (int pg = 0; pg < np; ++pg, at += L.page_bytes, w += 8) {
          const uint32_t h0 = w[0], h1 = w[4], l0 = w[lo_off], l1 = w[lo_off + 4];
#pragma unroll
          for (int j = 0; j < JG; ++j) {
            const int mt = mt0 + j;
            uint32_t a[4];
            ldsm4t((at + (mt >> 2) * G * 2048) ^ ((mt & 3) << 5), a);
            mma_bf16(acc[n * JG + j], a, h0, h1);
            mma_bf16(acc[n * JG + j], a, l0, l1);
          }
        }
      }
    if (++slot == L.stages) {
      slot = 0;
      phase ^= 1;
    }
  }
  pdl_launch_dependents();
  if (!ok) return;
#pragma unroll
  for (int j = 0; j < TPW; ++j) {
    const int n = j / JG;
    if (v_on[n]) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int lh = 2 * t4 + (e & 1), d = (mt0 + j % JG) * 16 + g8 + (e >> 1) * 8, h = v_h[n] + lh;
        if (h < (v_h[n] / R + 1) * R) p.part_o[((part0 + h) * p.max_splits + split) * D + d] = acc[j][e];
      }
    }
  }
#pragma unroll
  for (int w = 4; w < 32; w <<= 1) {
    l_run[0] += __shfl_xor_sync(0xffffffffu, l_run[0], w);
    l_run[1] += __shfl_xor_sync(0xffffffffu, l_run[1], w);
  }
  if (g8 == 0 && m_page < L.pages) {
    atomicAdd(&s_sum[mh], l_run[0]);
    atomicAdd(&s_sum[mh + 1], l_run[1]);
  }
  __syncthreads();
  if (tid < H) {
    float* ml = p.part_ml + ((part0 + tid) * p.max_splits + split) * 2;
    ml[0] = s_ref[tid];
    ml[1] = s_sum[tid];
  }
}

template <int D>
__global__ void __launch_bounds__(D) talk_merge_kernel(const TalkParams p, int n_splits) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.x, head = blockIdx.y, d = threadIdx.x;
  const long long base = (static_cast<long long>(seq) * p.H + head) * p.max_splits;
  float M = -INFINITY;
  for (int s = 0; s < n_splits; ++s) M = fmaxf(M, p.part_ml[(base + s) * 2]);
  float acc = 0.f, L = 0.f;
  for (int s = 0; s < n_splits; ++s) {
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

// Places in shared memory, so that no access of a warp meets a bank twice. Scores [head][query][key]: of 16 keys, key 4 t + 2 a + b
// lies at 8 a + 2 t + b, so a lane that mixes the places 2 t and 2 t + 1 of both eights has four neighbouring keys. Biases
// [head][distance].
constexpr int kHPitch = 580;
__device__ __forceinline__ int query_at(int q) { return q * 34 + (q >> 2) * 8; }
__device__ __forceinline__ int key_at(int k) { return (k & 16) + ((k >> 1) & 1) * 8 + ((k >> 2) & 3) * 2 + (k & 1); }
static_assert(kHPitch >= 15 * 34 + 3 * 8 + kKeys && kHPitch % 16 == 4, "banks");
constexpr int kBiasPitch = 80;
__device__ __forceinline__ int bias_at(int h) { return h * kBiasPitch + ((h >> 1) & 3); }

// HM: heads of this instantiation, 16 or 32 (H <= HM). The queries of all heads stay in shared memory while the CTA walks its
// blocks of keys. HM / 2 warps = HM / 4 sets of heads x 2 halves of a block: a warp multiplies 16 keys x 16 queries for the heads of its set,
// keys straight from memory a block ahead (16-byte pieces, the same permutation of the dimensions in q and k). Then the scores of
// all heads are mixed as a product with the heads' matrix T, 8 keys of a query as its columns.
template <int D, int HM>
__global__ void __launch_bounds__(HM * 16, HM == 16 ? 2 : 1) talk_scores_kernel(const TalkParams p, int blocks_per_cta) {
  constexpr int kThreads = HM * 16, W = HM / 2;
  constexpr int CPL = D / 32, CH = D / 8;   // 16-byte pieces of a row per lane, and in all
  constexpr int HT = HM / 16;
  extern __shared__ __align__(128) uint8_t s_raw[];
  float* s_c = reinterpret_cast<float*>(s_raw);                            // [HM][kQ][keys]
  float* s_b = s_c + HM * kHPitch;                                         // [H][distances]: bias times log2 e; +inf hides a key
  uint8_t* s_q = reinterpret_cast<uint8_t*>(s_b + (p.H + 1) / 2 * 2 * kBiasPitch);   // [H][kQ][D]
  const int H = p.H, R = H / p.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  uint32_t ta[HT][HT][4];   // T as the left operand
#pragma unroll
  for (int m = 0; m < HT; ++m)
#pragma unroll
    for (int k = 0; k < HT; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int h = m * 16 + g8 + (i & 1) * 8, g = k * 16 + 2 * t4 + (i >> 1) * 8;
        ta[m][k][i] = pack_f16x2(h < H && g < H ? p.talk[h * H + g] : 0.f, h < H && g + 1 < H ? p.talk[h * H + g + 1] : 0.f);
      }
  for (int i = tid; i < (HM - H) * kHPitch; i += kThreads) s_c[H * kHPitch + i] = 0.f;
  pdl_wait();
  const int tile = blockIdx.z, q_in = blockIdx.y * kQ;
  const Piece x = piece_of(p, tile, q_in, kQ);
  if (p.tile_q0[tile] + q_in >= x.len) return;
  const int k_start = first_key(p, tile), n_q = x.pos1 - x.pos0 + 1;
  // blocks of this CTA that some of its queries sees
  const int b_lo = max(static_cast<int>(blockIdx.x) * blocks_per_cta, (x.lo - k_start) / kKeys);
  const int b_hi = min((static_cast<int>(blockIdx.x) + 1) * blocks_per_cta, (x.pos1 - k_start) / kKeys + 1);
  if (b_lo >= b_hi) return;
  // a row's 16-byte piece c lies at c ^ swz(row): a lane's reads (row g8, piece t4 + 4 c) touch all banks
  auto swz = [](int row) { return (((row >> 1) & 3) << 1) ^ ((row & 1) << 2); };
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(x.row0) * p.q_ld;
  for (int c = tid; c < H * kQ * CH; c += kThreads) {
    const int row = c / CH, ch = c % CH, h = row / kQ, q = row % kQ;
    cp_async16(smem_u32(s_q) + row * (D * 2) + ((ch ^ swz(q)) << 4), qp + (q < n_q ? q : 0) * p.q_ld + h * D + ch * 8, q < n_q);
  }
  cp_commit();
  const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
  const int n_pg = (p.ctx_lens[x.seq] + 15) >> 4;
  const int half = warp & 1, hc = (H + W / 2 - 1) / (W / 2), h_lo = min((warp >> 1) * hc, H), h_hi = min(h_lo + hc, H), kv_lo = h_lo / R;
  const Cap cap = cap_of(p.cap, kLog2e);   // scores times log2 e
  const float unit = p.scale * cap.k;
  uint4 ka[2][CPL];
  float r0 = 0.f, r1 = 0.f;   // factors of the lane's keys
  const int c_at = query_at(2 * t4) + key_at(half * 16 + g8);
  int id = 0;
  auto page = [&](int b) { return raw_block(p, bt, min((k_start >> 4) + 2 * b + half, n_pg - 1)); };   // of this warp's half of key block b
  auto load_keys = [&](int kv) {
    const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(p.cache) + (static_cast<long long>(id) * p.G + kv) * 16 * D + t4 * 8;
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int c = 0; c < CPL; ++c) ka[r][c] = *reinterpret_cast<const uint4*>(kp + (g8 + 8 * r) * D + c * 32);
  };
  auto load_norms = [&]() {
    r0 = p.k_rms[id * 16ll + g8];
    r1 = p.k_rms[id * 16ll + g8 + 8];
  };
  // biases of key block b, two heads per warp: lanes are distances
  float bias_next[2][2];
  auto load_bias = [&](int b) {
    const int far0 = x.pos0 - (k_start + b * kKeys) - (kKeys - 1);   // distance of entry 0
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int v = 0; v < 2; ++v) {
        const int h = warp + W * u, dist = far0 + lane + 32 * v;
        const bool see = h < H && dist >= 0 && (p.window == 0 || dist < p.window);
        bias_next[u][v] = see ? __ldg(p.bias + static_cast<long long>(h) * p.n_bias + min(dist, p.n_bias - 1)) : INFINITY;
      }
  };
  id = checked_block(p, page(b_lo));
  if (h_lo < h_hi) load_keys(kv_lo);
  load_norms();
  load_bias(b_lo);
  int id_next = page(b_lo + 1);
  cp_wait<0>();
  __syncthreads();
  for (int b = b_lo; b < b_hi; ++b) {
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (warp + W * u < H) {
        float* d = s_b + bias_at(warp + W * u) + lane;
        d[0] = kLog2e * bias_next[u][0];
        if (lane < kQ - 1) d[32] = kLog2e * bias_next[u][1];
      }
    // ---- scores of this warp's heads: [16 keys x 16 queries]; positions behind the context are hidden by their bias ----
    r0 *= unit;
    r1 *= unit;
    int kv = kv_lo, left = R - (h_lo - kv_lo * R);   // heads of this key head that are still to come
    for (int h = h_lo; h < h_hi; ++h, --left) {
      if (left == 0) {
        load_keys(++kv);
        left = R;
      }
      const uint8_t* qr = s_q + (h * kQ + g8) * (D * 2);   // (rows g8 and g8 + 8 have the same swz)
      float s[2][4] = {};
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const int at = ((t4 + 4 * c) ^ swz(g8)) << 4;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const uint4 f = *reinterpret_cast<const uint4*>(qr + n * 8 * (D * 2) + at);
          mma_bf16(s[n], ka[0][c].x, ka[1][c].x, ka[0][c].y, ka[1][c].y, f.x, f.y);
          mma_bf16(s[n], ka[0][c].z, ka[1][c].z, ka[0][c].w, ka[1][c].w, f.z, f.w);
        }
      }
      float* d = s_c + h * kHPitch + c_at;   // (queries 8 and 1, and keys 8 further on are a fixed way off)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) d[n * 288 + (e & 1) * 34 + (e >> 1) * 4] = capped(s[n][e], e < 2 ? r0 : r1, cap);
    }
    id = checked_block(p, id_next);   // the next block's keys while this one's scores are mixed
    if (h_lo < h_hi) load_keys(kv_lo);
    load_norms();
    load_bias(b + 1);
    id_next = page(b + 2);
    __syncthreads();
    // ---- mixed scores: a warp takes a query, 16 keys at a time ----
#pragma unroll
    for (int q = warp; q < kQ; q += W) {
      const float* src = s_c + 2 * t4 * kHPitch + query_at(q) + g8;
      const float* bb = s_b + bias_at(g8) + kKeys - 1 + q - 4 * t4;   // bias of the lane's first key; the next ones are one nearer each
      float* dst = p.scores + ((static_cast<long long>(tile) * H + g8) * kTile + q_in + q) * p.span + b * kKeys + 4 * t4;
#pragma unroll
      for (int k16 = 0; k16 < kKeys; k16 += 16) {
        float o[2][HT][4];   // places of the lower and of the upper eight
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
          for (int m = 0; m < HT; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int h = m * 16 + 8 * (e >> 1);   // (bias_at(g8 + h) = bias_at(g8) + h * pitch)
              o[a][m][e] = h + g8 < H ? -bb[h * kBiasPitch - k16 - 2 * a - (e & 1)] : 0.f;
            }
#pragma unroll
        for (int a = 0; a < 2; ++a)
#pragma unroll
          for (int k = 0; k < HT; ++k) {
            const float* f = src + k * 16 * kHPitch + k16 + 8 * a;
            uint32_t h0, h1, l0, l1;
            split_f16(f[0], f[kHPitch], h0, l0);
            split_f16(f[8 * kHPitch], f[9 * kHPitch], h1, l1);
#pragma unroll
            for (int m = 0; m < HT; ++m) mma_f16(o[a][m], ta[m][k], l0, l1);
#pragma unroll
            for (int m = 0; m < HT; ++m) mma_f16(o[a][m], ta[m][k], h0, h1);
          }
#pragma unroll
        for (int m = 0; m < HT; ++m)
#pragma unroll
          for (int r = 0; r < 2; ++r)
            if (m * 16 + 8 * r + g8 < H)
              *reinterpret_cast<float4*>(dst + static_cast<long long>(m * 16 + 8 * r) * kTile * p.span + k16) =
                  make_float4(o[0][m][2 * r], o[0][m][2 * r + 1], o[1][m][2 * r], o[1][m][2 * r + 1]);
      }
    }
    __syncthreads();
  }
}

// Softmax and sums of a tile's 128 rows for one head, from the mixed scores. 64 keys at a time: the values by TMA through the block
// table, the weights (as hi + lo bf16 terms) by eight warps that read a row with eight lanes, the products on tcgen05 with the
// sums in TMEM. Two buffers of weights, so the products of one step run under the softmax of the next; the sums are rescaled only
// when a row's maximum grows by more than 2^8. Warp 0 copies, warp 1 issues products, 2 to 9 are softmax and epilogue: two warps
// share the 32 TMEM lanes of a quarter, 16 rows each in the softmax, half of the columns each of the sums. Every wait is bounded.
constexpr int kStep = 64;
constexpr int kValueThreads = 320;
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr),
               "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
               "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
               : "memory");
}
template <int D>
struct ValuesSmem {
  static constexpr int kSub = kStep * 128;                 // [64 keys x 64 dims]
  static constexpr int kWeights = kTile * 128;             // [128 rows x 64 keys]
  static constexpr int kV = 0;                             // 2 stages
  static constexpr int kP = kV + 2 * (D / 64) * kSub;      // 2 buffers of hi and lo
  static constexpr int kAlpha = kP + 4 * kWeights;
  static constexpr int kBar = kAlpha + 2 * kTile * 4 + 64;
  static constexpr int kTotal = kBar + 128 + 1024;
};

template <int D>
__global__ void __launch_bounds__(kValueThreads, 2) talk_values_kernel(const __grid_constant__ CUtensorMap tmV, const TalkParams p) {
  using L = ValuesSmem<D>;
  constexpr int VH = D / 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* s_v = smem + L::kV;
  uint8_t* s_p = smem + L::kP;
  float* s_alpha = reinterpret_cast<float*>(smem + L::kAlpha);   // 2 x per row: rescaling factor, at the end the sum of the weights
  int* s_grow = reinterpret_cast<int*>(s_alpha + 2 * kTile);     // 2 x per softmax warp: whether a factor is not 1
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::kBar);
  uint64_t* v_full = bars;        // 2
  uint64_t* v_empty = bars + 2;   // 2
  uint64_t* p_full = bars + 4;    // 2
  uint64_t* pv_done = bars + 6;   // 2
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmV);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&p_full[i], 8);
      mbar_init(&pv_done[i], 1);
    }
    fence_mbar_init();
  }
  pdl_wait();
  const int head = blockIdx.x, tile = blockIdx.y, H = p.H, kv = head / (H / p.G);
  const Piece x = piece_of(p, tile, 0, kTile);
  const int k_start = first_key(p, tile), n_steps = (x.pos1 - k_start) / kStep + 1;
  if (warp == 1) {
    tmem_alloc(tmem_slot, D);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_o = *tmem_slot;

  if (warp == 0) {
    const int* bt = p.block_tables + static_cast<long long>(x.seq) * p.max_blocks;
    const int n_pg = (p.ctx_lens[x.seq] + 15) >> 4;
    const int my_pg = (k_start >> 4) + lane / VH;   // lane = (page of the step, 64 dims); pages beyond the context weigh nothing
    int id = lane < 4 * VH ? raw_block(p, bt, min(my_pg, n_pg - 1)) : 0;
    for (int j = 0; j < n_steps; ++j) {
      const int s = j & 1;
      bool ok = j < 2 || mbar_wait(&v_empty[s], ((j >> 1) - 1) & 1);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) {
        if (lane == 0) set_status_once(p.status, kStatusMbarTimeoutProducer);
        break;
      }
      if (lane == 0) mbar_arrive_expect_tx(&v_full[s], VH * L::kSub);
      __syncwarp();
      if (lane < 4 * VH) {
        const int hf = lane % VH;
        tma_load_2d(s_v + (s * VH + hf) * L::kSub + lane / VH * 2048, &tmV, &v_full[s], hf * 64, (checked_block(p, id) * p.G + kv) * 16);
        id = raw_block(p, bt, min(my_pg + 4 * (j + 1), n_pg - 1));
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(kFmtBF16, kFmtBF16, kTile, D, 0, 1);   // values are MN-major
      for (int j = 0; j < n_steps; ++j) {
        const int s = j & 1;
        if (!mbar_wait(&p_full[s], (j >> 1) & 1) || !mbar_wait(&v_full[s], (j >> 1) & 1)) {
          set_status_once(p.status, kStatusMbarTimeoutMma);
          break;
        }
        tc_fence_after_sync();
        const uint32_t pa = smem_u32(s_p + s * 2 * L::kWeights), vb = smem_u32(s_v + s * VH * L::kSub);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int kk = 0; kk < kStep / 16; ++kk)
            tc_mma_f16(tmem_o, make_desc_kmajor_sw128(pa + term * L::kWeights + kk * 32), make_desc_mnmajor_sw128(vb + kk * 2048, L::kSub, 1024),
                       idesc, (j | kk | term) != 0 ? 1u : 0u);
        tc_commit(&v_empty[s]);
        tc_commit(&pv_done[s]);
      }
    }
  } else {
    // quarter of the rows, half of it; a lane's rows are q * 32 + hr * 16 + 4 lr + i, its keys 4 lc .. 4 lc + 3 of either half of a
    // step (a row's half is one line of memory; the eight-byte stores of two rows four apart touch all banks)
    const int q = warp & 3, hr = (warp - 2) >> 2, lr = lane >> 3, lc = lane & 7, row0 = q * 32 + hr * 16 + 4 * lr;
    constexpr int kRows = 4;   // rows per lane
    auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(1 + q) : "memory"); };   // the quarter's two warps
    // blocks of 32 keys whose scores exist for these 16 rows
    const Piece y = piece_of(p, tile, q * 32 + hr * 16, 16);
    const bool rows = p.tile_q0[tile] + q * 32 + hr * 16 < x.len;
    const int w0 = rows ? (y.lo - k_start) / kKeys : 1 << 30, w1 = rows ? (y.pos1 - k_start) / kKeys : -1;
    const float* sp = p.scores + ((static_cast<long long>(tile) * H + head) * kTile + row0) * p.span + lc * 4;
    float4 buf[kRows][2];
    auto load = [&](int j, int i) {
#pragma unroll
      for (int u = 0; u < 2; ++u)   // (blocks without scores are hidden when they are used; 128 spans fit an int)
        buf[i][u] = __ldcg(reinterpret_cast<const float4*>(sp + (i * p.span + min(j * kStep + u * kKeys, p.span - kKeys))));
    };
#pragma unroll
    for (int i = 0; i < kRows; ++i) load(0, i);
    float m[kRows], l[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      m[i] = -INFINITY;
      l[i] = 0.f;
    }
    const uint32_t lane_sel = static_cast<uint32_t>(q * 32) << 16;
    bool ok = true;
    for (int j = 0; j < n_steps; ++j) {
      const int b = j & 1;
      if (j >= 2 && !mbar_wait(&pv_done[b], ((j >> 1) - 1) & 1)) ok = false;   // this buffer's last products
      ok = __all_sync(0xffffffffu, ok);
      uint8_t* pb = s_p + b * 2 * L::kWeights;
      const bool in[2] = {2 * j >= w0 && 2 * j <= w1, 2 * j + 1 >= w0 && 2 * j + 1 <= w1};   // blocks with scores
      bool grow = false;
      float mx[kRows];
#pragma unroll
      for (int i = 0; i < kRows; ++i) {
        if (!in[0]) buf[i][0] = make_float4(-INFINITY, -INFINITY, -INFINITY, -INFINITY);
        if (!in[1]) buf[i][1] = make_float4(-INFINITY, -INFINITY, -INFINITY, -INFINITY);
        mx[i] = fmaxf(fmaxf(fmaxf(buf[i][0].x, buf[i][0].y), fmaxf(buf[i][0].z, buf[i][0].w)),
                      fmaxf(fmaxf(buf[i][1].x, buf[i][1].y), fmaxf(buf[i][1].z, buf[i][1].w)));
      }
#pragma unroll
      for (int o = 1; o < 8; o <<= 1)
#pragma unroll
        for (int i = 0; i < kRows; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
#pragma unroll
      for (int i = 0; i < kRows; ++i) {
        const float s[8] = {buf[i][0].x, buf[i][0].y, buf[i][0].z, buf[i][0].w, buf[i][1].x, buf[i][1].y, buf[i][1].z, buf[i][1].w};
        load(j + 1, i);
        float alpha = 1.f;
        if (mx[i] > m[i] + 8.f) {   // (of a reference of -inf: any score)
          alpha = m[i] == -INFINITY ? 0.f : ex2t(m[i] - mx[i]);
          m[i] = mx[i];
          grow = true;
        }
        const float ms = m[i] == -INFINITY ? 0.f : m[i];
        const int row = row0 + i;
        if (lc == 0) s_alpha[b * kTile + row] = alpha;
        float sum = 0.f;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float a = ex2t(s[2 * e] - ms), c = ex2t(s[2 * e + 1] - ms);
          sum += a + c;
          hi[e] = pack_bf16x2(a, c);
          lo[e] = pack_bf16x2(a - __uint_as_float(hi[e] << 16), c - __uint_as_float(hi[e] & 0xffff0000u));
        }
        l[i] = l[i] * alpha + sum;   // of this lane's keys
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          uint8_t* d = pb + (row >> 3) * 1024 + (row & 7) * 128 + (((4 * u + (lc >> 1)) ^ (row & 7)) << 4) + (lc & 1) * 8;
          *reinterpret_cast<uint2*>(d) = make_uint2(hi[2 * u], hi[2 * u + 1]);
          *reinterpret_cast<uint2*>(d + L::kWeights) = make_uint2(lo[2 * u], lo[2 * u + 1]);
        }
      }
      grow = __any_sync(0xffffffffu, grow);
      // a warp that gave up a wait tells the other one of its quarter, so both leave together
      if (lane == 0) s_grow[b * 8 + q * 2 + hr] = ok ? (grow ? 1 : 0) : 2;
      pair_sync();
      const int both = s_grow[b * 8 + q * 2] | s_grow[b * 8 + q * 2 + 1];
      if (both & 2) {
        ok = false;
        break;
      }
      if (j > 0 && both) {
        // the quarter's 32 sums, once the products before this step have been added
        if (!mbar_wait(&pv_done[b ^ 1], ((j - 1) >> 1) & 1)) ok = false;
        ok = __all_sync(0xffffffffu, ok);
        if (ok) {
          tc_fence_after_sync();
          const float alpha = s_alpha[b * kTile + q * 32 + lane];
#pragma unroll 1
          for (int c = hr * (D / 32); c < (hr + 1) * (D / 32); ++c) {   // (16 columns at a time: the next scores wait in registers)
            uint32_t v[16];
            tmem_ld_32x32b_x16(tmem_o + lane_sel + c * 16, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * alpha);
            tmem_st_32x32b_x16(tmem_o + lane_sel + c * 16, v);
          }
          tmem_st_wait();
        }
      }
      tc_fence_before_sync();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0 && ok) mbar_arrive(&p_full[b]);
    }
    if (ok && !mbar_wait(&pv_done[(n_steps - 1) & 1], ((n_steps - 1) >> 1) & 1)) ok = false;
    ok = __all_sync(0xffffffffu, ok);
    if (!ok && lane == 0) set_status_once(p.status, kStatusMbarTimeoutEpilogue);
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      float sum = l[i];
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (lc == 0) s_alpha[(n_steps & 1) * kTile + row0 + i] = sum;   // (the factors of the last step lie in the other half)
    }
    pair_sync();
    if (ok) {
      tc_fence_after_sync();
      const int r = q * 32 + lane;   // a thread has half a row of sums
      const float sum = s_alpha[(n_steps & 1) * kTile + r], inv = sum > 0.f ? 1.f / sum : 0.f;
      const bool valid = x.pos0 + r <= x.pos1;
      const long long row = x.row0 + (valid ? r : 0);
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.ldo + head * p.D;
      const bool vec = (p.D & 7) == 0 && (p.ldo & 7) == 0 && (p.gate_ld & 7) == 0 &&
                       ((reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.gate)) & 15) == 0;
#pragma unroll 1
      for (int c = hr * (D / 64); c < (hr + 1) * (D / 64); ++c) {
        uint32_t v[32];
        tmem_ld_32x32b_x32(tmem_o + lane_sel + c * 32, v);
        tmem_ld_wait();
        if (!valid) continue;
#pragma unroll
        for (int e = 0; e < 32; e += 8) {
          const int d = c * 32 + e, col = head * p.D + d;
          if (d >= p.D) break;
          if (!vec) {
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (d + k < p.D) out[d + k] = __float2bfloat16(__uint_as_float(v[e + k]) * inv * gate_at(p, row, col + k));
            continue;
          }
          float z[8];
          if (p.gate_f32) {
            const float4* g = reinterpret_cast<const float4*>(static_cast<const float*>(p.gate) + row * p.gate_ld + col);
            const float4 g0 = g[0], g1 = g[1];
            z[0] = g0.x, z[1] = g0.y, z[2] = g0.z, z[3] = g0.w, z[4] = g1.x, z[5] = g1.y, z[6] = g1.z, z[7] = g1.w;
          } else {
            const uint4 g = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.gate) + row * p.gate_ld + col);
            const uint32_t* gw = &g.x;
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              z[2 * k] = __uint_as_float(gw[k] << 16);
              z[2 * k + 1] = __uint_as_float(gw[k] & 0xffff0000u);
            }
          }
          uint4 o4;
          uint32_t* ow = &o4.x;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            ow[k] = pack_bf16x2(__fdividef(__uint_as_float(v[e + 2 * k]) * inv, 1.f + __expf(-z[2 * k])),
                                __fdividef(__uint_as_float(v[e + 2 * k + 1]) * inv, 1.f + __expf(-z[2 * k + 1])));
          *reinterpret_cast<uint4*>(out + d) = o4;
        }
      }
    }
    tc_fence_before_sync();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_o, D);
  }
}

size_t scores_smem(int H, int D) {
  return 4ull * ((H <= 16 ? 16 : 32) * kHPitch + (H + 1) / 2 * 2 * kBiasPitch) + static_cast<size_t>(H) * kQ * D * 2;
}

template <int D, int HM>
cudaError_t launch_scores(const TalkParams& p, cudaStream_t stream) {
  auto kern = talk_scores_kernel<D, HM>;
  const size_t smem = scores_smem(p.H, D);
  ensure_dynamic_smem(kern, smem);
  // parts of a piece's keys, so that the CTAs' rounds are shortest (loading the queries costs about one and a half blocks)
  const int blocks = p.span / kKeys, pieces = p.n_rows * (kTile / kQ), room = (HM == 16 ? 2 : 1) * sm_count();
  int per = blocks;
  float best = 0.f;
  for (int parts = 1; parts <= 16 && parts <= blocks; ++parts) {
    const int n = (blocks + parts - 1) / parts;
    const float cost = static_cast<float>((static_cast<long long>(pieces) * parts + room - 1) / room) * (n + 1.5f);
    if (parts == 1 || cost < best) {
      best = cost;
      per = n;
    }
  }
  return launch_kernel(kern, dim3((blocks + per - 1) / per, kTile / kQ, p.n_rows), dim3(HM * 16), smem, stream, true, false, p, per);
}
template <int D>
cudaError_t launch_prefill(const CUtensorMap& tmV, const TalkParams& p, cudaStream_t stream) {
  const cudaError_t e = p.H <= 16 ? launch_scores<D, 16>(p, stream) : launch_scores<D, 32>(p, stream);
  if (e != cudaSuccess) return e;
  auto kern = talk_values_kernel<D>;
  constexpr size_t smem = ValuesSmem<D>::kTotal;
  ensure_dynamic_smem(kern, smem);
  return launch_kernel(kern, dim3(p.H, p.n_rows), dim3(kValueThreads), smem, stream, true, false, tmV, p);
}
template <int D, int TPW>
cudaError_t launch_decode_t(const CUtensorMap& tmC, const TalkParams& p, const DecodeLayout& l, int splits, cudaStream_t stream) {
  auto kern = talk_decode_kernel<D, TPW>;
  ensure_dynamic_smem(kern, l.total);
  return launch_kernel(kern, dim3(p.n_rows, splits), dim3(kDecThreads), static_cast<size_t>(l.total), stream, true, false, tmC, p, l);
}
template <int D>
cudaError_t launch_decode(const CUtensorMap& tmC, const TalkParams& p, cudaStream_t stream) {
  const DecodeLayout l = decode_layout(p.H, p.G, D);
  // about as many CTAs as the SMs take at once
  const int fit = sm_count() / p.n_rows, splits = fit < 1 ? 1 : (fit < p.max_splits ? fit : p.max_splits);
  const cudaError_t e = l.tiles == 2 ? launch_decode_t<D, 2>(tmC, p, l, splits, stream)
                                     : (l.tiles == 4 ? launch_decode_t<D, 4>(tmC, p, l, splits, stream) : launch_decode_t<D, kMaxTiles>(tmC, p, l, splits, stream));
  if (e != cudaSuccess) return e;
  return launch_kernel(talk_merge_kernel<D>, dim3(p.n_rows, p.H), dim3(D), 0, stream, true, false, p, splits);
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
  return l.tiles <= kMaxTiles && l.pages * G <= kDecWarps * kMaxUnits && l.total <= 226 * 1024;
}
int talk_decode_box(int H, int G, int DP) { return decode_layout(H, G, DP).box * 16; }

cudaError_t launch_talk_decode(const CUtensorMap& tmC, const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_decode_ok(p.H, p.G, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_decode<64>(tmC, p, stream) : launch_decode<128>(tmC, p, stream);
}

bool talk_prefill_ok(int H, int DP) { return (DP == 64 || DP == 128) && H <= 32; }   // (scores_smem is at most 212 KB then)

int talk_span(int window, int max_ctx) {
  const int n = window > 0 && window + kTile - 1 < max_ctx ? window + kTile - 1 : max_ctx;
  return (n + 2 * kKeys - 2) / kKeys * kKeys;
}

cudaError_t launch_talk_prefill(const CUtensorMap& tmV, const TalkParams& p, cudaStream_t stream) {
  if (p.n_rows <= 0) return cudaSuccess;
  if (!talk_prefill_ok(p.H, p.DP)) return cudaErrorInvalidValue;
  return p.DP == 64 ? launch_prefill<64>(tmV, p, stream) : launch_prefill<128>(tmV, p, stream);
}

}  // namespace oxb
