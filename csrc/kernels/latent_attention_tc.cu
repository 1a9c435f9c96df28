// Latent attention on the 5th-generation tensor cores (tcgen05 + TMEM): bf16 query rows (token, head) over paged latents.
//
// All heads of a layer read the same latents, so the rows of a CTA are 128 consecutive (token, head) pairs -- several
// tokens of a prefill tile, or the heads of one decode row -- and one shared-memory block of latents serves both products:
//
//   warp 0    : TMA producer.  Q' once; then every 16-token page, 64 columns at a time (2 KB boxes, 128-byte swizzle), so a
//               block is [column chunk][token][64 values]: the K-major operand of S = Q' C^T and, read along the other
//               axis, the MN-major operand of O += P C.  A latent crosses HBM once for both.
//   warp 1    : one elected lane issues S_j (smem x smem) and O_g += P_j C_j (TMEM x smem) in the order S_j, PV_{j-1}, S_{j+1}
//   warps 2-5, 6-9 : two softmax groups on alternate key blocks, each with its own scores, running maximum, sum and
//               accumulator (the scheme of attention_tc.cu; a thread owns one row)
//   epilogue  : the groups merge through shared memory and store bf16 rows, or fp32 partials when the keys are split
//
// A CTA produces OC of the output columns (blockIdx.y picks them; the values are the first columns of a key), so two accumulators and two score buffers fit tensor
// memory for every R; for R > OC the scores are computed once per column chunk.  Ranks that are no multiple of 64 are
// rounded up: the tensor maps fill the missing columns with zeros.  Every wait is bounded and watches an abort flag.
#include <algorithm>

#include "attention_tc.cuh"
#include "latent_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows, uint32_t box_cols);

constexpr int kLtBM = 128;
constexpr int kLtSoftmaxWarp = 2;
constexpr int kLtThreads = (kLtSoftmaxWarp + 8) * 32;
constexpr float kLtRecentre = 24.f;      // see attention_tc.cu: the running maximum may lag by this many powers of two

template <int R, int OC, int BN, int ST>
struct LtCfg {
  static constexpr int kChunks = R / 64;
  static constexpr int kQBytes = kLtBM * R * 2;
  static constexpr int kKBytes = BN * R * 2;
  static constexpr int kSmemBytes = kQBytes + ST * kKBytes + 1024 /*alignment*/ + 512 /*barriers*/ + 2 * kLtBM * 8 /*(m, l)*/;
  static constexpr int kColS = 2 * OC;
  static constexpr int kTmemCols = 512;
  static constexpr int kXPitch = (OC / 2 + 4) * 4;
  static_assert(R % 64 == 0 && R >= OC && (OC == 64 || OC == 128) && BN % 32 == 0, "tile shape");
  static_assert(2 * OC + 2 * BN <= 512, "TMEM budget");
  static_assert(2 * kLtBM * kXPitch <= kQBytes + ST * kKBytes, "the exchange slab reuses the operand buffers");
  static_assert(kSmemBytes <= 227 * 1024, "shared memory");
};

template <int ST>
struct LtBars {
  uint64_t q_full, k_full[ST], k_empty[ST], s_full[2], p_full[2], pv_done[2];
};

struct LtRows {                          // the query rows of a CTA
  int entry, row0, rows, pos_first, pos_last, ctx;
};

OGB_DEVICE bool lt_rows(const LatParams& p, int q_per_tile, LtRows& o) {
  const int tile = blockIdx.x / q_per_tile, rb = blockIdx.x % q_per_tile;
  int base, n, start;
  if (p.cu_q == nullptr) {
    o.entry = tile;
    o.ctx = p.ctx_len[tile];
    base = tile; n = 1; start = o.ctx - 1;
  } else {
    o.entry = p.tile_seq[tile];
    const int len = p.cu_q[o.entry + 1] - p.cu_q[o.entry], q0 = p.tile_q0[tile];
    o.ctx = p.ctx_len[o.entry];
    base = p.cu_q[o.entry] + q0; n = min(64, len - q0); start = o.ctx - len + q0;
  }
  if (o.ctx <= 0 || n <= 0) return false;
  o.rows = min(kLtBM, n * p.heads - rb * kLtBM);
  if (o.rows <= 0) return false;
  o.row0 = base * p.heads + rb * kLtBM;
  o.pos_first = start + (rb * kLtBM) / p.heads;
  o.pos_last = start + (rb * kLtBM + o.rows - 1) / p.heads;
  return true;
}

template <int R, int OC, int BN, int ST>
__global__ void __launch_bounds__(kLtThreads, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap c_map, const LatParams p,
                           const int q_per_tile) {
  using Cfg = LtCfg<R, OC, BN, ST>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + Cfg::kQBytes;
  LtBars<ST>* bars = reinterpret_cast<LtBars<ST>*>(sK + ST * Cfg::kKBytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float2* x_ml = reinterpret_cast<float2*>(reinterpret_cast<uint8_t*>(bars) + 512);

  LtRows rw;
  if (!lt_rows(p, q_per_tile, rw)) return;
  const int heads_in = rw.row0 % p.heads;               // head of the CTA's first row
  const int col0 = blockIdx.y * OC;                     // output columns of this CTA
  const int kv_lo = p.window > 0 ? max(0, rw.pos_first - p.window + 1) : 0;
  int b_begin = kv_lo / BN, b_end = (rw.pos_last + BN) / BN;   // last visible key is pos_last
  if (p.num_splits > 1) {
    const int per = (b_end - b_begin + p.num_splits - 1) / p.num_splits;
    b_begin += static_cast<int>(blockIdx.z) * per;
    b_end = min(b_end, b_begin + per);
  }
  const int nblk = b_end - b_begin;
  if (nblk <= 0) {                                      // a split without keys
    if (blockIdx.y == 0 && static_cast<int>(threadIdx.x) < rw.rows) {
      const size_t pr = static_cast<size_t>(rw.row0 + threadIdx.x) * p.num_splits + blockIdx.z;
      p.part_ml[2 * pr] = -INFINITY;
      p.part_ml[2 * pr + 1] = 0.f;
    }
    return;
  }

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
    tma_prefetch_desc(&c_map);
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
      mbar_expect_tx(&bars->q_full, Cfg::kQBytes);
#pragma unroll
      for (int h = 0; h < Cfg::kChunks; ++h) tma_load_2d(sQ + h * kLtBM * 128, &q_map, &bars->q_full, h * 64, rw.row0);
      const int n_pages = (rw.ctx + kLatPage - 1) / kLatPage;
      const int* table = p.page_table + static_cast<size_t>(rw.entry) * p.max_pages;
      for (int it = 0; it < nblk && ok; ++it) {
        const int st = it % ST;
        int row_of_page[BN / kLatPage];
#pragma unroll
        for (int i = 0; i < BN / kLatPage; ++i) {
          // outside the visible pages (masked below): re-read a visible one, the others may have been released
          int pi = min(max((b_begin + it) * (BN / kLatPage) + i, kv_lo / kLatPage), min(n_pages, p.max_pages) - 1);
          int64_t page = table[pi];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          row_of_page[i] = static_cast<int>(page) * kLatPage;
        }
        if (!fa_wait(&bars->k_empty[st], ((it / ST) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_expect_tx(&bars->k_full[st], Cfg::kKBytes);
        uint8_t* dst = sK + st * Cfg::kKBytes;
#pragma unroll
        for (int i = 0; i < BN / kLatPage; ++i)
#pragma unroll
          for (int h = 0; h < Cfg::kChunks; ++h)
            tma_load_2d(dst + h * BN * 128 + i * 2048, &c_map, &bars->k_full[st], h * 64, row_of_page[i]);
      }
      if (!ok) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    }
  } else if (warp == 1) {
    // ------------------------------ MMA issuer ------------------------------
    // MMAs of one thread execute in issue order: S_{j+2}, issued after PV_j, cannot overwrite the P_j it has yet to read.
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(kLtBM, BN);
      constexpr uint32_t idesc_o = make_idesc_bf16(kLtBM, OC) | (1u << 16);   // B is MN-major
      bool ok = fa_wait(&bars->q_full, 0, abort_flag);
      auto issue_pv = [&](int t) -> bool {
        const int buf = t & 1, st = t % ST;
        if (!fa_wait(&bars->p_full[buf], (t >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t sv = smem_u32(sK + st * Cfg::kKBytes + (col0 / 64) * BN * 128);
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
        const uint32_t sq = smem_u32(sQ), sk = smem_u32(sK + st * Cfg::kKBytes);
#pragma unroll
        for (int h = 0; h < Cfg::kChunks; ++h) {
          const uint64_t da = make_kmajor_sw128_desc(sq + h * kLtBM * 128), db = make_kmajor_sw128_desc(sk + h * BN * 128);
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
    const int g = (warp - kLtSoftmaxWarp) >> 2;          // group: even key blocks, odd key blocks
    const int row = q * 32 + lane;
    const uint32_t lane_base = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
    const uint32_t s_addr = lane_base + Cfg::kColS + g * BN;
    const uint32_t o_addr = lane_base + g * OC;
    const float scale = p.scale * 1.4426950408889634f;
    const int pos = rw.pos_first + (heads_in + row) / p.heads;     // rows past the last are computed and dropped
    const int hi_abs = min(pos, rw.ctx - 1);
    const int lo_abs = p.window > 0 ? pos - p.window + 1 : 0;
    float m_run = -INFINITY, l_run = 0.f;                // running maximum in the scaled log2 domain
    bool ok = true;
    for (int it = g; it < nblk && ok; it += 2) {
      ok = __all_sync(0xffffffffu, fa_wait(&bars->s_full[g], (it >> 1) & 1, abort_flag));
      if (!ok) break;
      tc_fence_after();
      const int k0 = (b_begin + it) * BN;
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
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float v0 = __uint_as_float(a[2 * j]), v1 = __uint_as_float(a[2 * j + 1]);
            mx = fmaxf(mx, fmaxf(v0, v1));
            const float e0 = exp2f(fmaf(v0, scale, neg_m)), e1 = exp2f(fmaf(v1, scale, neg_m));
            sum += e0 + e1;
            pk[16 * c + j] = pack_bf16(e0, e1);
          }
        }
        if (!__any_sync(0xffffffffu, mx * scale > m_run + kLtRecentre)) {
          l_run += sum;
          done = true;
        }
      }
      if (!done) {
        float mx = -INFINITY;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const int k = k0 + 32 * c + j;
            mx = fmaxf(mx, k <= hi_abs && k >= lo_abs ? __uint_as_float(a[j]) * scale : -INFINITY);
          }
        }
        const float m_new = fmaxf(m_run, mx);
        const bool raise = m_new > m_run + kLtRecentre || (m_run == -INFINITY && m_new > -INFINITY);
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
            const int k = k0 + 32 * c + 2 * j;
            const float v0 = k <= hi_abs && k >= lo_abs ? __uint_as_float(a[2 * j]) : -INFINITY;
            const float v1 = k + 1 <= hi_abs && k + 1 >= lo_abs ? __uint_as_float(a[2 * j + 1]) : -INFINITY;
            const float e0 = exp2f(fmaf(v0, scale, neg_m)), e1 = exp2f(fmaf(v1, scale, neg_m));
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
      float* dst = reinterpret_cast<float*>(xo + (static_cast<size_t>(g) * kLtBM + row) * Cfg::kXPitch);
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
    x_ml[g * kLtBM + row] = make_float2(m_mine, l_mine);
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float2 other = x_ml[(g ^ 1) * kLtBM + row];
    const float m_all = fmaxf(m_mine, other.x);
    float a = m_mine == -INFINITY ? 0.f : exp2f(m_mine - m_all), b = other.x == -INFINITY ? 0.f : exp2f(other.x - m_all);
    const float l_all = l_mine * a + other.y * b;
    const bool split = p.num_splits > 1;
    if (!split) {
      const float inv = l_all > 0.f && row < rw.rows ? latent_gate<__nv_bfloat16>(p, static_cast<int64_t>(rw.row0) + row) / l_all : 0.f;
      a *= inv; b *= inv;
    }
    const float* src = reinterpret_cast<const float*>(xo + (static_cast<size_t>(g ^ 1) * kLtBM + row) * Cfg::kXPitch);
    const size_t orow = static_cast<size_t>(rw.row0) + row;
    const size_t pr = split ? orow * p.num_splits + blockIdx.z : 0;
    if (split && g == 0 && blockIdx.y == 0 && row < rw.rows) {
      p.part_ml[2 * pr] = m_all * 0.6931471805599453f;   // the combine kernel works with natural exponentials
      p.part_ml[2 * pr + 1] = l_all;
    }
#pragma unroll
    for (int c = 0; c < HC / 32; ++c) {
      uint32_t o[32];
      __syncwarp();
      tmem_ld_32x32(o_addr + g * HC + 32 * c, o);
      tmem_ld_wait();
      if (row >= rw.rows) continue;
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        const int col = col0 + g * HC + 32 * c + 8 * v;
        if (col >= p.vrank) continue;                    // a multiple of 8
        float r[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          // a group without blocks holds an uninitialised accumulator: select, never multiply by zero
          const float mine = a > 0.f ? __uint_as_float(o[8 * v + j]) * a : 0.f;
          r[j] = mine + (b > 0.f ? src[32 * c + 8 * v + j] * b : 0.f);
        }
        if (split) {
          float4* po = reinterpret_cast<float4*>(p.part_o + pr * p.vrank + col);
          po[0] = make_float4(r[0], r[1], r[2], r[3]);
          po[1] = make_float4(r[4], r[5], r[6], r[7]);
        } else {
          *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + orow * p.ldo + col) =
              make_uint4(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3]), pack_bf16(r[4], r[5]), pack_bf16(r[6], r[7]));
        }
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
static int launch_lt(const LatParams& p, cudaStream_t stream) {
  using Cfg = LtCfg<R, OC, BN, ST>;
  CUtensorMap q_map, c_map;
  int rc = make_tmap_bf16_2d(&q_map, p.q, static_cast<uint64_t>(p.rows) * p.heads, p.rank, p.ldq, kLtBM, 64);
  if (rc != 0) return rc;
  rc = make_tmap_bf16_2d(&c_map, p.pool, static_cast<uint64_t>(p.num_pages) * kLatPage, p.rank, p.ldp, kLatPage, 64);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(latent_attention_tc_kernel<R, OC, BN, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    attr_set = true;
  }
  const int q_per_tile = ((p.cu_q == nullptr ? 1 : 64) * p.heads + kLtBM - 1) / kLtBM;
  const dim3 grid((p.cu_q == nullptr ? p.rows : p.num_tiles) * q_per_tile, (p.vrank + OC - 1) / OC, p.num_splits);
  latent_attention_tc_kernel<R, OC, BN, ST><<<grid, kLtThreads, Cfg::kSmemBytes, stream>>>(q_map, c_map, p, q_per_tile);
  return static_cast<int>(cudaGetLastError());
}

int launch_latent_tc(const LatParams& p, cudaStream_t stream) {
  if (p.rank > 576 || p.vrank > 512 || (p.rank | p.vrank | p.ldo) % 8 != 0 || p.ldq % 8 != 0 || p.ldp % 8 != 0 || p.num_pages <= 0) return -2;
  if ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.pool) |
       reinterpret_cast<uintptr_t>(p.part_o)) & 15) return -2;
  if (p.cu_q == nullptr) return launch_latent_decode(p, stream);
  if (p.scale <= 0.f) return -2;           // the row maximum is taken before scaling
  if (p.rank <= 64) return launch_lt<64, 64, 128, 4>(p, stream);
  if (p.rank <= 128) return launch_lt<128, 128, 128, 4>(p, stream);
  if (p.rank <= 192) return p.vrank <= 128 ? launch_lt<192, 128, 128, 3>(p, stream) : launch_lt<192, 64, 128, 3>(p, stream);
  if (p.rank <= 256) return launch_lt<256, 128, 64, 4>(p, stream);
  if (p.rank <= 320 && p.vrank <= 256) return launch_lt<320, 128, 64, 3>(p, stream);
  if (p.rank <= 384) return launch_lt<384, 128, 64, 2>(p, stream);
  if (p.rank <= 512) return launch_lt<512, 128, 32, 2>(p, stream);
  return launch_lt<576, 128, 32, 2>(p, stream);
}

}  // namespace ogb
