// Decode rows of latent attention against the cached latents themselves (sm_100a, tcgen05).
//
// With the key expansion moved to the query (q' = W_uk^T q) and the value expansion behind the sum, all heads of a row
// share one key, which is also the value: a cache row is read once for scores and sums. One CTA = (row, up to 64 heads, KV
// split); tiles of 64 positions (4 pages) come by TMA straight from the paged cache into 128B-swizzled shared memory. The
// positions are the M dimension, so a handful of heads does not leave the tensor core's rows empty:
//     S^T = K Q^T          [64 positions x heads], fp32 in TMEM
//     P   = exp2(S - m)    as two bf16 terms, [2 heads x positions] in shared memory
//     O^T += V^T P^T       [128 value columns x 2 heads] per block of columns, fp32 in TMEM: the tile of keys is the
//                          operand once more, now M-major; both terms in one product, added up at the end
// A tile lies in units of 128 columns with full and empty barriers of their own: scores start with the units that are
// there, a unit is free for a later tile as soon as its block of sums is done. The reference m of a head is moved only when
// a score exceeds it by more than 2^8.
// Warp roles: warps 0..3 = softmax + epilogue, warp 4 = MMA issuer (scores of a tile or sums of the one before, whichever
// can go), warps 5 and 6 = TMA producers, 8 lanes per unit and one copy per lane (the rate of copies grows with the threads
// that issue them). Every wait is bounded.
// A second kernel merges the splits.
#include <cuda.h>

#include "../common/device_info.h"
#include "hybrid_dev.cuh"

namespace oxb {

namespace {

constexpr int kThreads = 224, kMmaWarp = 4, kLoadWarp = 5;
constexpr int kKeys = 64;                     // positions per tile
constexpr int kSub = kKeys * 128;             // [64 positions x 64 columns] (8 KB)
constexpr int kMaxUnits = 6, kMaxBufs = 4;
constexpr int kBarBytes = 512;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
      "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// softmax_sync and the OR of a predicate over its threads
__device__ __forceinline__ bool softmax_any(bool x) {
  uint32_t any;
  asm volatile(
      "{\n\t"
      ".reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, 128, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t"
      "}\n"
      : "=r"(any)
      : "r"(static_cast<uint32_t>(x))
      : "memory");
  return any != 0;
}
// Whether the phase is complete, without waiting
__device__ __forceinline__ bool mbar_test(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}

// Shared memory of a CTA of HN heads: tile buffers, queries, weights (two terms), barriers and small tables.
struct Layout {
  int subs, units, blocks, bufs, tile, q, p, bar, table, total;
  uint32_t cols;
  __host__ __device__ Layout(int HN, int R, int CP) {
    subs = (CP + 63) / 64;
    blocks = (R + 127) / 128;
    units = (subs + 1) / 2;
    tile = (subs > 2 * blocks ? subs : 2 * blocks) * kSub;
    const int rest = HN * 128 * subs + HN * 512 + kBarBytes + HN * 32 + 1024;
    bufs = (227 * 1024 - rest) / tile;
    if (bufs > kMaxBufs) bufs = kMaxBufs;
    q = bufs * tile;
    p = q + HN * 128 * subs;
    bar = p + HN * 512;   // two buffers of weights
    table = bar + kBarBytes;
    total = table + HN * 32 + 1024;
    cols = 32;
    while (cols < static_cast<uint32_t>((2 + 2 * blocks) * HN)) cols *= 2;
  }
  __host__ __device__ bool fits() const { return bufs >= 1 && cols <= 512 && units <= kMaxUnits; }
};

template <int HN>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const Layout L(HN, p.R, p.CP);
  constexpr int kMine = HN / 2;               // heads per thread: two threads share a position
  uint8_t* sQ = smem + L.q;
  uint8_t* sP = smem + L.p;
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + L.bar);   // [bufs][units]
  uint64_t* empty = full + kMaxBufs * kMaxUnits;
  uint64_t* q_full = empty + kMaxBufs * kMaxUnits;
  uint64_t* s_full = q_full + 1;              // [2]
  uint64_t* p_full = s_full + 2;              // [2]
  uint64_t* pv_done = p_full + 2;             // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
  int* s_flag = reinterpret_cast<int*>(tmem_slot + 2);          // [4]
  float* s_ref = reinterpret_cast<float*>(smem + L.table);      // reference of every head (log2 units)
  float* s_alpha = s_ref + HN;
  float* s_warp = s_alpha + HN;                                 // [4][HN]

  const int row = blockIdx.x, h0 = blockIdx.y * HN, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();   // queries and the newest cache rows come from the kernels before this one
  const int seq_len = p.seq_lens[row];
  int n_pages = (seq_len + 15) / 16;
  if (n_pages > p.max_blocks) {
    if (threadIdx.x == 0) set_status_once(p.status, kStatusBadIndex);
    n_pages = p.max_blocks;
  }
  // even shares of whole tiles
  const int tiles = (n_pages + 3) / 4, share = (tiles + p.n_splits - 1) / p.n_splits;
  const int t_lo = split * share, n_tiles = min(share, tiles - t_lo);
  const long long part0 = (static_cast<long long>(row) * p.H + h0) * p.max_splits + split;
  if (n_tiles <= 0) {
    for (int h = threadIdx.x; h < HN && h0 + h < p.H; h += kThreads) {
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2] = -INFINITY;
      p.part_ml[(part0 + static_cast<long long>(h) * p.max_splits) * 2 + 1] = 0.f;
    }
    return;
  }
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmC);
    for (int i = 0; i < kMaxBufs * kMaxUnits; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&pv_done[i], 1);
    }
    fence_mbar_init();
  }
  if (warp == kMmaWarp) {
    tmem_alloc(tmem_slot, L.cols);
    tmem_relinquish();
  }
  for (int h = threadIdx.x; h < HN; h += kThreads) s_ref[h] = -INFINITY;
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_s = *tmem_slot;          // two buffers of HN columns
  const uint32_t tmem_o = tmem_s + 2 * HN;     // blocks of 2 HN columns
  const int bufs = L.bufs, units = L.units, subs = L.subs, blocks = L.blocks;

  if (warp >= kLoadWarp) {
    // ------------------------------ TMA producers -----------------------------
    if (warp == kLoadWarp) {
      if (lane == 0) mbar_arrive_expect_tx(q_full, subs * HN * 128);
      __syncwarp();
      if (lane < subs) tma_load_3d(sQ + lane * HN * 128, &tmQ, q_full, lane * 64, h0, row);
    }
    const int* bt = p.block_tables + static_cast<long long>(row) * p.max_blocks;
    // lane -> (unit, sub-tile of the unit, page)
    const int u = 4 * (warp - kLoadWarp) + (lane >> 3), half = (lane >> 2) & 1, pg = lane & 3;
    const unsigned mates = 0xffu << (lane & 24);
    const int n = min(2, subs - 2 * u);
    if (u < units) {
      for (int j = 0; j < n_tiles; ++j) {
        const int page = (t_lo + j) * 4 + pg;
        int blk = page < n_pages ? bt[page] : 0;   // (positions past the end weigh nothing)
        if (static_cast<unsigned>(blk) >= static_cast<unsigned>(p.num_blocks)) {
          set_status_once(p.status, kStatusBadIndex);
          blk = 0;
        }
        const int buf = j % bufs, use = j / bufs;
        uint64_t* bar = &full[buf * kMaxUnits + u];
        const bool ok = use == 0 || mbar_wait(&empty[buf * kMaxUnits + u], (use - 1) & 1);
        if (!__all_sync(mates, ok)) {
          if ((lane & 7) == 0) set_status_once(p.status, kStatusMbarTimeoutProducer);
          break;
        }
        if ((lane & 7) == 0) mbar_arrive_expect_tx(bar, n * kSub);
        __syncwarp(mates);
        if (half < n) tma_load_2d(smem + buf * L.tile + (2 * u + half) * kSub + pg * 2048, &tmC, bar, (2 * u + half) * 64, blk * 16);
      }
    }
  } else if (warp == kMmaWarp) {
    // ------------------------------ MMA issuer --------------------------------
    // The whole warp walks through the loop with uniform values, one elected thread issues: operands then come from uniform
    // registers, which is what the rate of such small products hangs on.
    constexpr uint32_t idesc_s = make_idesc(kFmtBF16, kFmtBF16, 64, HN);
    constexpr uint32_t idesc_o = make_idesc(kFmtBF16, kFmtBF16, 128, 2 * HN, 1, 0);   // the tile is M-major here
    const bool ok = __all_sync(0xffffffffu, mbar_wait(q_full, 0));
    const uint32_t base = __shfl_sync(0xffffffffu, smem_u32(smem), 0);
    const uint32_t ts = __shfl_sync(0xffffffffu, tmem_s, 0), to = __shfl_sync(0xffffffffu, tmem_o, 0);
    const int n_t = __shfl_sync(0xffffffffu, n_tiles, 0);
    // (descriptors count 16-byte steps, so a step is an addition)
    const uint64_t dq = make_desc_kmajor_sw128(base + L.q), dp = make_desc_kmajor_sw128(base + L.p);
    const uint32_t leader = elect_one_sync();
    int js = 0, u = 0, jp = 0, bs = 0, bp = 0;   // next unit of scores, next tile of sums, their buffers
    uint32_t use = 0;                            // parity of the buffer's use
    const uint32_t limit = spin_budget(0);
    uint32_t idle = ok ? 0 : limit + 1;
    while (jp < n_t && idle <= limit) {
      if (jp < js && __all_sync(0xffffffffu, mbar_test(&p_full[jp & 1], (jp >> 1) & 1))) {
        tc_fence_after_sync();
        const uint64_t da = make_desc_mnmajor_sw128(base + bp * L.tile, kSub, 1024), db = dp + (jp & 1) * (HN * 16);
        if (leader) {
          for (int b = 0; b < blocks; ++b) {
#pragma unroll
            for (int kk = 0; kk < kKeys / 16; ++kk)
              tc_mma_f16(to + b * 2 * HN, da + b * (2 * kSub / 16) + kk * 128, db + kk * 2, idesc_o, (jp | kk) != 0 ? 1u : 0u);
            tc_commit(&empty[bp * kMaxUnits + b]);
          }
          tc_commit(&pv_done[jp & 1]);
        }
        __syncwarp();
        ++jp;
        if (++bp == bufs) bp = 0;
        idle = 0;
      } else if (js < n_t && js - jp < 2 && __all_sync(0xffffffffu, mbar_test(&full[bs * kMaxUnits + u], use))) {
        tc_fence_after_sync();
        const uint64_t da = make_desc_kmajor_sw128(base + bs * L.tile) + u * (2 * kSub / 16), db = dq + u * (2 * HN * 8);
        const uint32_t d = ts + (js & 1) * HN;
        const bool two = 2 * u + 1 < subs, last = u + 1 == units;
        if (leader) {
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) tc_mma_f16(d, da + kk * 2, db + kk * 2, idesc_s, (u | kk) != 0 ? 1u : 0u);
          if (two) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) tc_mma_f16(d, da + (kSub / 16 + kk * 2), db + (HN * 8 + kk * 2), idesc_s, 1u);
          }
          if (u >= blocks) tc_commit(&empty[bs * kMaxUnits + u]);   // no values in it
          if (last) tc_commit(&s_full[js & 1]);
        }
        __syncwarp();
        if (last) {
          u = 0;
          ++js;
          if (++bs == bufs) {
            bs = 0;
            use ^= 1;
          }
        } else {
          ++u;
        }
        idle = 0;
      } else {
        ++idle;
      }
    }
    if (idle > limit && leader) set_status_once(p.status, kStatusMbarTimeoutMma);
  } else {
    // ------------------------------ softmax + epilogue ------------------------
    // A warp owns 16 positions (scores in the first 16 lanes of its TMEM quarter); thread lane + 16 takes the second half
    // of a position's heads.
    const int q = warp & 3, r = q * 32 + lane, key = q * 16 + (lane & 15), hsel = (lane >> 4) * kMine;
    const uint32_t lane_sel = static_cast<uint32_t>(q * 32) << 16;
    float l[kMine];
#pragma unroll
    for (int h = 0; h < kMine; ++h) l[h] = 0.f;
    // this position's column of the weights, 16-byte pieces swizzled by the row
    uint8_t* pcol = sP + hsel * 128 + (key & 7) * 2;
    const int piece = key >> 3;
    const float* ref = s_ref + hsel;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      if (ok && !mbar_wait(&s_full[j & 1], (j >> 1) & 1)) ok = false;
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after_sync();
      const bool seen = (t_lo + j) * kKeys + key < seq_len;
      float x[kMine];   // scores in log2 units
      {
        uint32_t v[HN];
#pragma unroll
        for (int c = 0; c < HN; c += 16) tmem_ld_32x32b_x16(tmem_s + (j & 1) * HN + lane_sel + c, *reinterpret_cast<uint32_t(*)[16]>(v + c));
        tmem_ld_wait();
#pragma unroll
        for (int h = 0; h < kMine; ++h) {
          const uint32_t up = __shfl_sync(0xffffffffu, v[kMine + h], lane & 15);
          x[h] = seen ? __uint_as_float(lane < 16 ? v[h] : up) * p.scale_log2 : -INFINITY;
        }
      }
      // ---- does a score exceed its head's reference? ----
      float over = -INFINITY;
#pragma unroll
      for (int h = 0; h < kMine; ++h) over = fmaxf(over, x[h] - ref[h]);
      const bool grow = softmax_any((seen && over > 8.f) || !ok);
      // the weights' buffer has been read by the sums of two tiles before
      if (j >= 2 && ok && !mbar_wait(&pv_done[j & 1], ((j - 2) >> 1) & 1)) ok = false;
      ok = __all_sync(0xffffffffu, ok);   // (a warp whose wait ran out says so at the next tile)
      tc_fence_after_sync();
      if (grow) {
        // sums of the tile before are complete before they are scaled
        if (j >= 1 && ok && !mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1)) ok = false;
        ok = __all_sync(0xffffffffu, ok);
        if (lane == 0) s_flag[q] = ok ? 0 : 1;
        tc_fence_after_sync();
#pragma unroll
        for (int h = 0; h < kMine; ++h) {
          float m = x[h];
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
          if ((lane & 15) == 0) s_warp[q * HN + hsel + h] = m;
        }
        softmax_sync();
        if ((s_flag[0] | s_flag[1] | s_flag[2] | s_flag[3]) != 0) {   // a wait ran out in some warp: all four leave here
          ok = false;
          break;
        }
        if (r < HN) {
          const float old = s_ref[r];
          const float m = fmaxf(fmaxf(fmaxf(s_warp[r], s_warp[HN + r]), fmaxf(s_warp[2 * HN + r], s_warp[3 * HN + r])), old);
          s_alpha[r] = old == -INFINITY ? 0.f : ex2(old - m);
          s_ref[r] = m;
        }
        softmax_sync();
#pragma unroll
        for (int h = 0; h < kMine; ++h) l[h] *= s_alpha[hsel + h];
        if (j > 0) {
          for (int b = 0; b < 2 * blocks; ++b)
#pragma unroll
            for (int c = 0; c < HN; c += 16) {
              uint32_t v[16];
              const uint32_t at = tmem_o + b * HN + c + lane_sel;
              tmem_ld_32x32b_x16(at, v);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * s_alpha[c + i]);
              tmem_st_32x32b_x16(at, v);
            }
          tmem_st_wait();
        }
      }
      // ---- weights ----
      {
        float w[kMine];   // all references are read before the first store
#pragma unroll
        for (int h = 0; h < kMine; h += 4) load4<float>(ref + h, *reinterpret_cast<float(*)[4]>(w + h));
#pragma unroll
        for (int h = 0; h < kMine; ++h) {
          w[h] = ex2(x[h] - w[h]);
          l[h] += w[h];
        }
#pragma unroll
        for (int h = 0; h < kMine; ++h) {
          const __nv_bfloat16 hi = __float2bfloat16(w[h]);
          uint8_t* d = pcol + (j & 1) * (HN * 256) + h * 128 + ((piece ^ (h & 7)) << 4);
          *reinterpret_cast<__nv_bfloat16*>(d) = hi;
          *reinterpret_cast<__nv_bfloat16*>(d + HN * 128) = __float2bfloat16(w[h] - __bfloat162float(hi));
        }
      }
      tc_fence_before_sync();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    pdl_launch_dependents();
    if (ok && !mbar_wait(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1)) ok = false;
    ok = __all_sync(0xffffffffu, ok);
    if (!ok && lane == 0) set_status_once(p.status, kStatusMbarTimeoutEpilogue);
    tc_fence_after_sync();
#pragma unroll
    for (int h = 0; h < kMine; ++h) {
      float a = l[h];
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
      if ((lane & 15) == 0) s_warp[q * HN + hsel + h] = a;
    }
    for (int b = 0; b < blocks && ok; ++b) {
      const int d = b * 128 + r;
#pragma unroll
      for (int c = 0; c < HN; c += 16) {
        uint32_t v[16], lo[16];
        tmem_ld_32x32b_x16(tmem_o + b * 2 * HN + c + lane_sel, v);
        tmem_ld_32x32b_x16(tmem_o + b * 2 * HN + HN + c + lane_sel, lo);
        tmem_ld_wait();
        if (d < p.R) {
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (h0 + c + i < p.H)
              p.part_o[(part0 + static_cast<long long>(c + i) * p.max_splits) * p.R + d] = __uint_as_float(v[i]) + __uint_as_float(lo[i]);
        }
      }
    }
    softmax_sync();   // (every warp comes here once, whatever its waits said)
    if (r < HN && h0 + r < p.H) {
      float* ml = p.part_ml + (part0 + static_cast<long long>(r) * p.max_splits) * 2;
      ml[0] = s_ref[r];
      ml[1] = s_warp[r] + s_warp[HN + r] + s_warp[2 * HN + r] + s_warp[3 * HN + r];
    }
    tc_fence_before_sync();
  }
  __syncthreads();
  if (warp == kMmaWarp) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_s, L.cols);
  }
}

// out[row, head] = sum_s w_s O_s / sum_s w_s l_s with w_s = 2^(m_s - max m). grid (rows, heads)
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentDecodeParams p) {
  __shared__ float s_w[64];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, head = blockIdx.y;
  const long long base = (static_cast<long long>(row) * p.H + head) * p.max_splits;
  if (threadIdx.x < 32) {
    const int s0 = threadIdx.x, s1 = threadIdx.x + 32;
    const float m0 = s0 < p.n_splits ? p.part_ml[(base + s0) * 2] : -INFINITY, m1 = s1 < p.n_splits ? p.part_ml[(base + s1) * 2] : -INFINITY;
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
    for (int s = 0; s < p.n_splits; ++s) {
      const float w = s_w[s];
      if (w > 0.f) a = fmaf(w, p.part_o[(base + s) * p.R + c], a);
    }
    out[c] = __float2bfloat16(a);
  }
}

}  // namespace

int latent_decode_heads(int H, int R, int CP) {
  for (int top = 64; top > 0; top -= 16) {
    if (!Layout(top, R, CP).fits()) continue;
    const int groups = (H + top - 1) / top;
    return ((H + groups - 1) / groups + 15) / 16 * 16;
  }
  return 0;
}

cudaError_t launch_latent_decode(const CUtensorMap& tmQ, const CUtensorMap& tmC, const LatentDecodeParams& p, cudaStream_t stream) {
  if (p.rows <= 0) return cudaSuccess;
  const int hn = latent_decode_heads(p.H, p.R, p.CP);
  if (hn == 0 || p.max_splits > 64) return cudaErrorInvalidValue;
  const Layout L(hn, p.R, p.CP);
  auto kern = hn == 16 ? latent_decode_kernel<16> : (hn == 32 ? latent_decode_kernel<32> : (hn == 48 ? latent_decode_kernel<48> : latent_decode_kernel<64>));
  ensure_dynamic_smem(kern, static_cast<size_t>(L.total));
  // splits: few waves of CTAs, each with a share of a sequence beside a fixed cost
  const int groups = (p.H + hn - 1) / hn;
  int per_sm = 227 * 1024 / (L.total + 1024);
  if (per_sm > static_cast<int>(512 / L.cols)) per_sm = static_cast<int>(512 / L.cols);
  const int slots = sm_count() * (per_sm < 1 ? 1 : per_sm);
  LatentDecodeParams q = p;
  float best = 0.f;
  for (int z = 1; z <= p.max_splits; ++z) {
    const float cost = static_cast<float>((p.rows * groups * z + slots - 1) / slots) * (1.f / static_cast<float>(z) + 0.03f);
    if (z == 1 || cost < best) {
      best = cost;
      q.n_splits = z;
    }
  }
  const cudaError_t e = launch_kernel(kern, dim3(p.rows, groups, q.n_splits), dim3(kThreads), static_cast<size_t>(L.total), stream, true, false,
                                      tmQ, tmC, q);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_merge_kernel, dim3(p.rows, p.H), dim3(128), 0, stream, true, false, q);
}

}  // namespace oxb
