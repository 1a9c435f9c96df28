// Prompts of attention over keys that are the values, on the 5th-generation tensor cores (tcgen05 + TMEM), bf16.
//
// A CTA has 128 rows: the (token, query head) pairs of a KV head's group and 128 / group tokens, or one query head's 128 tokens where the
// group does not divide 128.  One shared-memory block of keys serves both products, as in latent_attention_tc.cu:
//
//   warp 0    : TMA producer.  The queries once; then every 16-token page, 64 columns at a time (2 KB boxes, 128-byte swizzle), so a
//               block is [column chunk][token][64 values]: the K-major operand of S = Q K^T and, read along the other axis, the
//               MN-major operand of O += P K.  The pages' factors follow as bulk copies.
//   warp 1    : one elected lane issues S_j (smem x smem) and O_g += P_j K_j (TMEM x smem) in the order S_j, PV_{j-1}, S_{j+1}
//   warps 2-5, 6-9 : two softmax groups on alternate key blocks, each with its own scores, running maximum, sum and accumulator; a
//               thread owns a row.  The cap's tanh is a polynomial where the scores of 32 columns of a warp are small, which leaves the
//               exponential unit to the softmax.  Blocks that need a mask or a new maximum put their scores back into tensor memory
//               and take the exponentials from there.
//   epilogue  : the groups merge through shared memory, the sink joins the sums, the head's gate is applied, bf16 rows are stored
//
// Keys wider than 128 columns: a CTA produces 128 of the output columns (blockIdx.y) and computes all scores.  Every wait is bounded
// and watches an abort flag.
#include <algorithm>

#include "attention_tc.cuh"
#include "tied_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

int encode_tmap_bf16_3d(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint64_t planes, uint64_t row_stride, uint64_t plane_stride,
                        uint32_t box_cols, uint32_t box_rows, uint32_t box_planes);

constexpr int kTtBM = 128;
constexpr int kTtSoftmaxWarp = 2;
constexpr int kTtThreads = (kTtSoftmaxWarp + 8) * 32;
constexpr float kTtRecentre = 24.f;      // the running maximum may lag by this many powers of two
constexpr float kLog2e = 1.4426950408889634f;

template <int R, int OC, int BN, int ST>
struct TtCfg {
  static constexpr int kChunks = R / 64;
  static constexpr int kQBytes = kTtBM * R * 2;
  static constexpr int kKBytes = BN * R * 2;
  static constexpr int kStageBytes = kKBytes + 1024;       // keys, BN factors
  static constexpr int kSmemBytes = kQBytes + ST * kStageBytes + 1024 /*alignment*/ + 512 /*barriers*/ + 2 * kTtBM * 8 /*(m, l)*/;
  static constexpr int kColS = 2 * OC;
  static constexpr int kTmemCols = 2 * OC + 2 * BN <= 256 ? 256 : 512;
  static constexpr int kXPitch = (OC / 2 + 4) * 4;
  static_assert(R % 64 == 0 && R >= OC && (OC == 64 || OC == 128) && BN % 32 == 0 && BN <= 256, "tile shape");
  static_assert(2 * OC + 2 * BN <= 512, "TMEM budget");
  static_assert(2 * kTtBM * kXPitch <= kQBytes + ST * kStageBytes, "the exchange slab reuses the operand buffers");
  static_assert(kSmemBytes <= 227 * 1024, "shared memory");
};

template <int ST>
struct TtBars {
  uint64_t q_full, k_full[ST], k_empty[ST], s_full[2], p_full[2], pv_done[2];
};

struct TtShape {                         // how a tile's rows are dealt out
  int group, tokens, span, per_tile;     // query heads of a CTA, its tokens, tokens of its tiles, CTAs they take
};

struct TtRows {                          // the query rows of a CTA
  int entry, tok0, rows, pos_first, pos_last, ctx;
};

OGB_DEVICE bool tt_rows(const TiedParams& p, const TtShape& sh, TtRows& o) {
  const int tile = blockIdx.x / sh.per_tile, rb = blockIdx.x % sh.per_tile;
  o.entry = p.tile_seq[tile];
  const int len = p.cu_q[o.entry + 1] - p.cu_q[o.entry], q0 = p.tile_q0[tile], first = q0 + rb * sh.tokens;
  if (q0 % sh.span != 0) return false;   // a pair's second tile belongs to the first one's CTA
  const int n = min(min(sh.span, len - q0) - rb * sh.tokens, sh.tokens);
  o.ctx = p.ctx_len[o.entry];
  if (o.ctx <= 0 || n <= 0) return false;
  o.tok0 = p.cu_q[o.entry] + first;
  o.rows = n * sh.group;
  o.pos_first = o.ctx - len + first;
  o.pos_last = o.pos_first + n - 1;
  return true;
}

OGB_DEVICE float tt_ex2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// tanh(x) for |x| <= kTtSmall: a polynomial in x^2 fitted at Chebyshev nodes, good to 7e-8
constexpr float kTtSmall = 0.75f;
OGB_DEVICE float tt_tanh_small(float x) {
  const float u = x * x;
  float a = fmaf(u, -0.004723952151834965f, 0.01959378644824028f);
  a = fmaf(u, a, -0.053349819034338f);
  a = fmaf(u, a, 0.13325515389442444f);
  a = fmaf(u, a, -0.3333296775817871f);
  return fmaf(x * u, a, x);
}
// tanh(x) = 1 - 2 / (exp(2 |x|) + 1) with the sign of x
OGB_DEVICE float tt_tanh(float x) {
  const float e = tt_ex2(2.f * kLog2e * fabsf(x));
  return copysignf(1.f - __fdividef(2.f, e + 1.f), x);
}
// 32 products to scores (log2 domain, less `base` + slope * column)
OGB_DEVICE void tt_scores(uint32_t (&a)[32], const float* factor, float cap2, float slope, float base, float (&z)[32]) {
  float top = 0.f;
#pragma unroll
  for (int v = 0; v < 8; ++v) {
    const float4 f = *reinterpret_cast<const float4*>(factor + 4 * v);
    z[4 * v] = __uint_as_float(a[4 * v]) * f.x;
    z[4 * v + 1] = __uint_as_float(a[4 * v + 1]) * f.y;
    z[4 * v + 2] = __uint_as_float(a[4 * v + 2]) * f.z;
    z[4 * v + 3] = __uint_as_float(a[4 * v + 3]) * f.w;
  }
  if (cap2 > 0.f) {
#pragma unroll
    for (int j = 0; j < 32; ++j) top = fmaxf(top, fabsf(z[j]));
    if (__any_sync(0xffffffffu, top > kTtSmall)) {
#pragma unroll
      for (int j = 0; j < 32; ++j) z[j] = tt_tanh(z[j]);
    } else {
#pragma unroll
      for (int j = 0; j < 32; ++j) z[j] = tt_tanh_small(z[j]);
    }
  }
  const float f = cap2 > 0.f ? cap2 : kLog2e;
#pragma unroll
  for (int j = 0; j < 32; ++j) z[j] = fmaf(z[j], f, fmaf(slope, static_cast<float>(j), base));
}

template <int R, int OC, int BN, int ST>
__global__ void __launch_bounds__(kTtThreads, 1)
tied_attention_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const TiedParams p, const TtShape sh) {
  using Cfg = TtCfg<R, OC, BN, ST>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + Cfg::kQBytes;
  TtBars<ST>* bars = reinterpret_cast<TtBars<ST>*>(sK + ST * Cfg::kStageBytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float2* x_ml = reinterpret_cast<float2*>(reinterpret_cast<uint8_t*>(bars) + 512);

  TtRows rw;
  if (!tt_rows(p, sh, rw)) return;
  const int units = p.hq / sh.group, head0 = blockIdx.y % units * sh.group, kvh = head0 / (p.hq / p.hkv);
  const int col0 = blockIdx.y / units * OC;             // output columns of this CTA
  const int kv_lo = p.window > 0 ? max(0, rw.pos_first - p.window + 1) : 0;
  const int b_begin = kv_lo / BN, nblk = (rw.pos_last + BN) / BN - b_begin;  // last visible key is pos_last

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    for (int i = 0; i < ST; ++i) { mbar_init(&bars->k_full[i], 1); mbar_init(&bars->k_empty[i], 1); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_full[i], 4);
      mbar_init(&bars->pv_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&k_map);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    // ------------------------------ TMA producer ------------------------------
    if (lane == 0) {
      bool ok = true;
      mbar_expect_tx(&bars->q_full, Cfg::kChunks * sh.tokens * sh.group * 128);
#pragma unroll
      for (int h = 0; h < Cfg::kChunks; ++h) tma_load_3d(sQ + h * kTtBM * 128, &q_map, &bars->q_full, h * 64, head0, rw.tok0);
      const int n_pages = (rw.ctx + kTaPage - 1) / kTaPage;
      const int* table = p.page_table + static_cast<size_t>(rw.entry) * p.max_pages;
      const __nv_bfloat16* factors = static_cast<const __nv_bfloat16*>(p.pool) + static_cast<size_t>(p.hkv) * kTaPage * p.dp;
      for (int it = 0; it < nblk && ok; ++it) {
        const int st = it % ST;
        int page_of[BN / kTaPage];
#pragma unroll
        for (int i = 0; i < BN / kTaPage; ++i) {
          // outside the visible pages (masked below): re-read a visible one, the others may have been released
          int64_t page = table[ta_page_index(p, (b_begin + it) * (BN / kTaPage) + i, n_pages, kv_lo)];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          page_of[i] = static_cast<int>(page);
        }
        if (!fa_wait(&bars->k_empty[st], ((it / ST) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_expect_tx(&bars->k_full[st], Cfg::kKBytes + BN * 4);
        uint8_t* dst = sK + st * Cfg::kStageBytes;
#pragma unroll
        for (int i = 0; i < BN / kTaPage; ++i) {
#pragma unroll
          for (int h = 0; h < Cfg::kChunks; ++h)
            tma_load_3d(dst + h * BN * 128 + i * 2048, &k_map, &bars->k_full[st], h * 64, kvh * kTaPage, page_of[i]);
          bulk_load(dst + Cfg::kKBytes + i * 64, factors + page_of[i] * p.page_elems, 64, &bars->k_full[st]);
        }
      }
      if (!ok) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    }
  } else if (warp == 1) {
    // ------------------------------ MMA issuer ------------------------------
    // MMAs of one thread execute in issue order: S_{j+2}, issued after PV_j, cannot overwrite the P_j it has yet to read.
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(kTtBM, BN);
      constexpr uint32_t idesc_o = make_idesc_bf16(kTtBM, OC) | (1u << 16);   // B is MN-major
      bool ok = fa_wait(&bars->q_full, 0, abort_flag);
      auto issue_pv = [&](int t) -> bool {
        const int buf = t & 1, st = t % ST;
        if (!fa_wait(&bars->p_full[buf], (t >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t sv = smem_u32(sK + st * Cfg::kStageBytes + (col0 / 64) * BN * 128);
#pragma unroll
        for (int k = 0; k < BN / 16; ++k)
          umma_f16_ts(tmem_base + buf * OC, tmem_base + Cfg::kColS + buf * BN + k * 8, make_mnmajor_sw128_desc(sv + k * 2048, BN * 128), idesc_o,
                      (t >= 2 || k > 0) ? 1u : 0u);
        umma_commit(&bars->k_empty[st]);
        umma_commit(&bars->pv_done[buf]);
        return true;
      };
      for (int it = 0; it < nblk && ok; ++it) {
        const int st = it % ST, buf = it & 1;
        if (!fa_wait(&bars->k_full[st], (it / ST) & 1, abort_flag)) { ok = false; break; }
        tc_fence_after();
        const uint32_t sq = smem_u32(sQ), sk = smem_u32(sK + st * Cfg::kStageBytes);
#pragma unroll
        for (int h = 0; h < Cfg::kChunks; ++h) {
          const uint64_t da = make_kmajor_sw128_desc(sq + h * kTtBM * 128), db = make_kmajor_sw128_desc(sk + h * BN * 128);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(tmem_base + Cfg::kColS + buf * BN, da + 2 * k, db + 2 * k, idesc_s, (h | k) != 0 ? 1u : 0u);
        }
        umma_commit(&bars->s_full[buf]);
        if (it >= 1 && !issue_pv(it - 1)) ok = false;
      }
      if (ok && !issue_pv(nblk - 1)) ok = false;
      if (!ok) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    }
  } else {
    // ------------------------------ softmax groups / epilogue ------------------------------
    const int q = warp & 3;                              // TMEM lane quarter
    const int g = (warp - kTtSoftmaxWarp) >> 2;          // softmax group: even key blocks, odd key blocks
    const int row = q * 32 + lane;
    const uint32_t lane_base = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
    const uint32_t s_addr = lane_base + Cfg::kColS + g * BN;
    const uint32_t o_addr = lane_base + g * OC;
    const int tok = row / sh.group, head = head0 + row - tok * sh.group;
    const int pos = rw.pos_first + tok;                  // rows past the last are computed and dropped
    const int hi_abs = min(pos, rw.ctx - 1);
    const int lo_abs = p.window > 0 ? pos - p.window + 1 : 0;
    const float slope = ta_slope(p, head) * kLog2e, cap2 = p.cap > 0.f ? p.cap * kLog2e : 0.f;
    float m_run = -INFINITY, l_run = 0.f;                // running maximum in the log2 domain
    bool ok = true;
    for (int it = g; it < nblk && ok; it += 2) {
      ok = __all_sync(0xffffffffu, fa_wait(&bars->s_full[g], (it >> 1) & 1, abort_flag));
      if (!ok) break;
      tc_fence_after();
      // the factors came with the keys: the barrier that the product waited for makes them visible here too
      ok = __all_sync(0xffffffffu, fa_wait(&bars->k_full[it % ST], (it / ST) & 1, abort_flag));
      if (!ok) break;
      const float* factor = reinterpret_cast<const float*>(sK + (it % ST) * Cfg::kStageBytes + Cfg::kKBytes);
      const int k0 = (b_begin + it) * BN;
      const float base = slope * static_cast<float>(k0 - pos);
      // every column visible to every row of the CTA: no mask
      const bool plain = k0 + BN - 1 <= rw.pos_first && (p.window <= 0 || k0 > rw.pos_last - p.window);
      uint32_t pk[BN / 2];
      bool done = false;
      if (plain && it >= 2) {
        // one pass against the current maximum; kept unless some row's maximum has outgrown it
        const float neg_m = m_run == -INFINITY ? 0.f : -m_run;
        float mx = -INFINITY, sum = 0.f;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          float z[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
          tt_scores(a, factor + 32 * c, cap2, slope, base + slope * (32 * c) + neg_m, z);
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            mx = fmaxf(mx, fmaxf(z[2 * j], z[2 * j + 1]));
            const float e0 = tt_ex2(z[2 * j]), e1 = tt_ex2(z[2 * j + 1]);
            sum += e0 + e1;
            pk[16 * c + j] = pack_bf16(e0, e1);
          }
        }
        if (!__any_sync(0xffffffffu, mx > kTtRecentre || (m_run == -INFINITY && mx > -INFINITY))) {
          l_run += sum;
          done = true;
        }
      }
      if (!done) {
        float mx = -INFINITY;
#pragma unroll 1
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          float z[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
          tt_scores(a, factor + 32 * c, cap2, slope, base + slope * (32 * c), z);
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const int k = k0 + 32 * c + j;
            const float v = k <= hi_abs && k >= lo_abs ? z[j] : -INFINITY;
            mx = fmaxf(mx, v);
            a[j] = __float_as_uint(v);
          }
          tmem_st_32x32(s_addr + 32 * c, a);
        }
        tmem_st_wait();
        const float m_new = fmaxf(m_run, mx);
        const bool raise = m_new > m_run + kTtRecentre || (m_run == -INFINITY && m_new > -INFINITY);
        if (it < 2) {
          m_run = m_new;
        } else if (__any_sync(0xffffffffu, raise)) {
          // the accumulator must hold every earlier block of this group before it is rescaled
          ok = __all_sync(0xffffffffu, fa_wait(&bars->pv_done[g], ((it - 2) >> 1) & 1, abort_flag));
          if (!ok) break;
          tc_fence_after();
          float alpha = 1.f;
          if (raise) {
            alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_new);
            m_run = m_new;
            l_run *= alpha;
          }
#pragma unroll 1
          for (int c = 0; c < OC / 32; ++c) {
            uint32_t o[32];
            tmem_ld_32x32(o_addr + 32 * c, o);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
            tmem_st_32x32(o_addr + 32 * c, o);
          }
          tmem_st_wait();
        }
        const float neg_m = m_run == -INFINITY ? 0.f : -m_run;
        float sum = 0.f;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float e0 = tt_ex2(__uint_as_float(a[2 * j]) + neg_m), e1 = tt_ex2(__uint_as_float(a[2 * j + 1]) + neg_m);
            sum += e0 + e1;
            pk[16 * c + j] = pack_bf16(e0, e1);
          }
        }
        l_run += sum;
      }
      // P overwrites the first half of the scores it came from
#pragma unroll
      for (int c = 0; c < BN / 32; ++c) tmem_st_32x16(s_addr + 16 * c, *reinterpret_cast<uint32_t(*)[16]>(&pk[16 * c]));
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_full[g]);
    }
    int last = nblk - 1;
    if ((last & 1) != g) --last;
    if (ok && last >= 0) ok = __all_sync(0xffffffffu, fa_wait(&bars->pv_done[g], (last >> 1) & 1, abort_flag));
    if (!ok && lane == 0) {
      atomicOr(p.status, kStatusWaitTimeout);
      *abort_flag = 1;
    }
    // ---- merge the groups: each finishes one half of the CTA's columns ----
    constexpr int HC = OC / 2;
    uint8_t* xo = sQ;                                    // the operands are idle once both groups' last products have landed
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const bool live = ok && last >= 0;
    if (live) {
      tc_fence_after();
      float* dst = reinterpret_cast<float*>(xo + (static_cast<size_t>(g) * kTtBM + row) * Cfg::kXPitch);
#pragma unroll
      for (int c = 0; c < HC / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(o_addr + (g ^ 1) * HC + 32 * c, o);
        tmem_ld_wait();
#pragma unroll
        for (int v = 0; v < 8; ++v)
          *reinterpret_cast<uint4*>(dst + 32 * c + 4 * v) = make_uint4(o[4 * v], o[4 * v + 1], o[4 * v + 2], o[4 * v + 3]);
      }
    }
    const float m_mine = live ? m_run : -INFINITY, l_mine = live ? l_run : 0.f;
    x_ml[g * kTtBM + row] = make_float2(m_mine, l_mine);
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float2 other = x_ml[(g ^ 1) * kTtBM + row];
    const bool stores = row < rw.rows;
    const float sink = stores ? ta_sink(p, head) * kLog2e : -INFINITY;
    const float m_all = fmaxf(fmaxf(m_mine, other.x), sink);
    float a = m_mine == -INFINITY ? 0.f : exp2f(m_mine - m_all), b = other.x == -INFINITY ? 0.f : exp2f(other.x - m_all);
    const float l_all = l_mine * a + other.y * b + (sink == -INFINITY ? 0.f : exp2f(sink - m_all));
    const int64_t trow = static_cast<int64_t>(rw.tok0) + tok;
    const float inv = stores && l_all > 0.f ? ta_gate<__nv_bfloat16>(p, trow, head) / l_all : 0.f;
    a *= inv; b *= inv;
    const float* src = reinterpret_cast<const float*>(xo + (static_cast<size_t>(g ^ 1) * kTtBM + row) * Cfg::kXPitch);
#pragma unroll
    for (int c = 0; c < HC / 32; ++c) {
      uint32_t o[32];
      __syncwarp();
      tmem_ld_32x32(o_addr + g * HC + 32 * c, o);
      tmem_ld_wait();
      if (!stores) continue;
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        const int col = col0 + g * HC + 32 * c + 8 * v;
        if (col >= p.dp) continue;                       // a multiple of 8
        float r[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          // a group without blocks holds an uninitialised accumulator: select, never multiply by zero
          const float mine = a > 0.f ? __uint_as_float(o[8 * v + j]) * a : 0.f;
          r[j] = mine + (b > 0.f ? src[32 * c + 8 * v + j] * b : 0.f);
        }
        *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + trow * p.ldo + static_cast<int64_t>(head) * p.dp + col) =
            make_uint4(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3]), pack_bf16(r[4], r[5]), pack_bf16(r[6], r[7]));
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag != 0 && threadIdx.x == 0) {
    // a wait ran out: give copies that may still be in flight a bounded time to land
    const uint64_t t0 = global_timer_ns();
    while (global_timer_ns() - t0 < 200000ull) { __nanosleep(1000); }
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, Cfg::kTmemCols);
  }
}

template <int R, int OC, int BN, int ST>
static int launch_tt(const TiedParams& p, cudaStream_t stream) {
  using Cfg = TtCfg<R, OC, BN, ST>;
  TtShape sh;
  const int group = p.hq / p.hkv;
  sh.group = kTtBM % group == 0 ? group : 1;
  sh.span = sh.group == 1 ? 128 : 64;
  sh.tokens = kTtBM / sh.group;
  sh.per_tile = sh.span / sh.tokens;
  CUtensorMap q_map, k_map;
  int rc = encode_tmap_bf16_3d(&q_map, p.q, p.dp, p.hq, p.rows, p.dp, p.ldq, 64, sh.group, sh.tokens);
  if (rc != 0) return rc;
  rc = encode_tmap_bf16_3d(&k_map, p.pool, p.dp, static_cast<uint64_t>(p.hkv) * kTaPage, static_cast<uint64_t>(p.num_pages), p.dp, p.page_elems, 64, kTaPage, 1);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(tied_attention_tc_kernel<R, OC, BN, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    attr_set = true;
  }
  const dim3 grid(p.num_tiles * sh.per_tile, p.hq / sh.group * ((p.dp + OC - 1) / OC));
  tied_attention_tc_kernel<R, OC, BN, ST><<<grid, kTtThreads, Cfg::kSmemBytes, stream>>>(q_map, k_map, p, sh);
  return static_cast<int>(cudaGetLastError());
}

int launch_tied_prefill_tc(const TiedParams& p, cudaStream_t stream) {
  if (p.dp > 256 || ((p.dp | p.ldq | p.ldo | p.page_elems) & 7) != 0) return -2;
  if ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.pool)) & 15) return -2;
  if (p.dp <= 64) return launch_tt<64, 64, 128, 4>(p, stream);
  if (p.dp <= 128) return launch_tt<128, 128, 128, 4>(p, stream);
  if (p.dp <= 192) return launch_tt<192, 128, 128, 3>(p, stream);
  return launch_tt<256, 128, 64, 4>(p, stream);
}

}  // namespace ogb
