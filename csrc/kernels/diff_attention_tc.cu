// Differential attention over prompts on the 5th-generation tensor cores (tcgen05 + TMEM), bf16.
//
//   one CTA   = 128 query rows of one head (two of the scheduler's 64-row tiles), both maps, against the sequence's keys in blocks
//               of BN tokens: first the blocks of the kept tokens, then those of the window
//   warp 0    : TMA producer of the two maps' queries (once) and of K1 | K2 blocks, warp 1: of V blocks.  A 16-token page half is
//               one 2 KB box per 64 columns, 128-byte swizzled; columns past a head's size are filled with zeros
//   warp 2    : one elected lane issues  S_m = Q_m K_m^T  (smem x smem -> TMEM) and  O_m += P_m V  (TMEM x smem -> TMEM): both maps
//               read one V block.  Order: P1 V_j, S1_{j+1}, P2 V_j, S2_{j+1} -- while one map's softmax works the other's products run
//   warps 3-6 : softmax of map 1, warps 7-10: of map 2 (the scheme of attention_tc.cu: a thread owns a row, P over the scores it
//               came from, the running maximum may lag by 2^24)
//   epilogue  : each softmax group hands half of its normalised accumulator to the other through shared memory; o = a1 - lambda a2,
//               its root mean square over the head (halves summed through shared memory), bf16 rows out
//
// Every wait is bounded and watches an abort flag; page ids are bounds-checked.
#include "attention_tc.cuh"
#include "diff_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

int encode_tmap_bf16_3d(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint64_t planes, uint64_t row_stride, uint64_t plane_stride,
                        uint32_t box_cols, uint32_t box_rows, uint32_t box_planes);

constexpr int kDtBM = 128;
constexpr int kDtSoftmaxWarp = 3;
constexpr int kDtThreads = (kDtSoftmaxWarp + 8) * 32;
constexpr float kDtRecentre = 24.f;

template <int DP, int VP, int BN, int ST>
struct DtCfg {
  static constexpr int kChunksD = DP / 64, kChunksV = VP / 64;
  static constexpr int kQBytes = 2 * kDtBM * DP * 2;            // both maps
  static constexpr int kKBytes = 2 * BN * DP * 2;               // both maps
  static constexpr int kVBytes = BN * VP * 2;
  static constexpr int kRing = kQBytes + ST * (kKBytes + kVBytes);
  static constexpr int kSmemBytes = kRing + 1024 /*alignment*/ + 512 /*barriers*/ + 2 * kDtBM * 4 /*sums of squares*/;
  static constexpr int kColS = 2 * VP;
  static constexpr int kTmemCols = 512;
  static constexpr int kXPitch = (VP / 2 + 4) * 4;
  static_assert(2 * VP + 2 * BN <= 512, "TMEM budget");
  static_assert(2 * kDtBM * kXPitch <= kRing, "the exchange slab reuses the operand buffers");
  static_assert(kSmemBytes <= 227 * 1024, "shared memory");
};

template <int ST>
struct DtBars {
  uint64_t q_full, k_full[ST], k_empty[ST], v_full[ST], v_empty[ST], s_full[2], p_full[2], pv_done[2];
};

template <int DP, int VP, int BN, int ST>
__global__ void __launch_bounds__(kDtThreads, 1)
diff_prefill_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                       const DiffParams p) {
  using Cfg = DtCfg<DP, VP, BN, ST>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;                                   // [map][column chunk][128 rows][128 bytes]
  uint8_t* sK = sQ + Cfg::kQBytes;                      // [stage][map][column chunk][BN][128 bytes]
  uint8_t* sV = sK + ST * Cfg::kKBytes;                 // [stage][column chunk][BN][128 bytes]
  DtBars<ST>* bars = reinterpret_cast<DtBars<ST>*>(sV + ST * Cfg::kVBytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* x_ss = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 512);      // [half][row]

  const int tile = blockIdx.x;
  if (tile >= p.num_tiles) return;
  const int q0 = p.tile_q0[tile];
  if ((q0 & 127) != 0) return;                          // the odd 64-row tiles are served by their 128-row neighbours
  const int head = blockIdx.y, kvh = head / (p.hq / p.hkv);
  const int seq = p.tile_seq[tile];
  const int q_begin = p.cu_q[seq], q_len = p.cu_q[seq + 1] - q_begin, ctx = p.ctx_len[seq];
  const int rows = min(kDtBM, q_len - q0), pos0 = ctx - q_len + q0;
  if (rows <= 0 || ctx <= 0 || pos0 < 0) return;
  const int kv_end = pos0 + rows;
  // the key blocks of this tile: those of the kept tokens, then from the window's first key on
  const int kv_lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
  int nsink = p.window > 0 && p.keep > 0 ? (min(p.keep, kv_end) + BN - 1) / BN : 0, first = kv_lo / BN;
  if (first <= nsink) { first = 0; nsink = 0; }
  const int nblk = nsink + (kv_end + BN - 1) / BN - first;
  auto block_at = [&](int j) { return j < nsink ? j : first + j - nsink; };

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    for (int i = 0; i < ST; ++i) {
      mbar_init(&bars->k_full[i], 1);
      mbar_init(&bars->k_empty[i], 1);
      mbar_init(&bars->v_full[i], 1);
      mbar_init(&bars->v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_full[i], 4);
      mbar_init(&bars->pv_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
  }
  if (warp == 2) {
    tmem_alloc(tmem_slot, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp < 2) {
    // ------------------------------ TMA producers ------------------------------
    if (lane == 0) {
      bool ok = true;
      const bool is_v = warp == 1;
      if (!is_v) {
        mbar_expect_tx(&bars->q_full, Cfg::kQBytes);
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int h = 0; h < Cfg::kChunksD; ++h)
            tma_load_3d(sQ + (m * Cfg::kChunksD + h) * kDtBM * 128, &q_map, &bars->q_full, h * 64, 2 * head + m, q_begin + q0);
      }
      const int n_pages = (ctx + kDaPage - 1) / kDaPage;
      const int* table = p.page_table + static_cast<size_t>(seq) * p.max_pages;
      uint64_t* full = is_v ? bars->v_full : bars->k_full;
      uint64_t* empty = is_v ? bars->v_empty : bars->k_empty;
      for (int it = 0; it < nblk && ok; ++it) {
        const int st = it % ST, b = block_at(it);
        int page_of[BN / kDaPage];
#pragma unroll
        for (int i = 0; i < BN / kDaPage; ++i) {
          int64_t page = table[da_page_index(p, b * (BN / kDaPage) + i, n_pages, kv_lo)];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          page_of[i] = static_cast<int>(page);
        }
        if (!fa_wait(&empty[st], ((it / ST) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_expect_tx(&full[st], is_v ? Cfg::kVBytes : Cfg::kKBytes);
        if (is_v) {
          uint8_t* dst = sV + st * Cfg::kVBytes;
#pragma unroll
          for (int i = 0; i < BN / kDaPage; ++i)
#pragma unroll
            for (int h = 0; h < Cfg::kChunksV; ++h)
              tma_load_3d(dst + h * BN * 128 + i * 2048, &v_map, &full[st], h * 64, kvh * kDaPage, page_of[i]);
        } else {
          uint8_t* dst = sK + st * Cfg::kKBytes;
#pragma unroll
          for (int i = 0; i < BN / kDaPage; ++i)
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
              for (int h = 0; h < Cfg::kChunksD; ++h)
                tma_load_3d(dst + (m * Cfg::kChunksD + h) * BN * 128 + i * 2048, &k_map, &full[st], h * 64, (2 * kvh + m) * kDaPage, page_of[i]);
        }
      }
      if (!ok) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    }
  } else if (warp == 2) {
    // ------------------------------ MMA issuer ------------------------------
    // MMAs of one thread execute in issue order: S_m of the next block, issued after P_m V, cannot overwrite the P_m it has yet to
    // read, and a commit covers everything issued before it.
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(kDtBM, BN);
      constexpr uint32_t idesc_o = make_idesc_bf16(kDtBM, VP) | (1u << 16);   // V is MN-major
      bool ok = fa_wait(&bars->q_full, 0, abort_flag);
      auto scores = [&](int m, int j) {
        const uint32_t sq = smem_u32(sQ + m * Cfg::kChunksD * kDtBM * 128);
        const uint32_t sk = smem_u32(sK + (j % ST) * Cfg::kKBytes + m * Cfg::kChunksD * BN * 128);
#pragma unroll
        for (int h = 0; h < Cfg::kChunksD; ++h) {
          const uint64_t da = make_kmajor_sw128_desc(sq + h * kDtBM * 128), db = make_kmajor_sw128_desc(sk + h * BN * 128);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(tmem_base + Cfg::kColS + m * BN, da + 2 * k, db + 2 * k, idesc_s, (h | k) != 0 ? 1u : 0u);
        }
        if (m == 1) umma_commit(&bars->k_empty[j % ST]);
        umma_commit(&bars->s_full[m]);
      };
      auto outputs = [&](int m, int j) -> bool {
        if (!fa_wait(&bars->p_full[m], j & 1, abort_flag)) return false;
        if (m == 0 && !fa_wait(&bars->v_full[j % ST], (j / ST) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t sv = smem_u32(sV + (j % ST) * Cfg::kVBytes);
#pragma unroll
        for (int k = 0; k < BN / 16; ++k)
          umma_f16_ts(tmem_base + m * VP, tmem_base + Cfg::kColS + m * BN + k * 8, make_mnmajor_sw128_desc(sv + k * 2048, BN * 128), idesc_o,
                      (j > 0 || k > 0) ? 1u : 0u);
        if (m == 1) umma_commit(&bars->v_empty[j % ST]);
        if (j == nblk - 1) umma_commit(&bars->pv_done[m]);
        return true;
      };
      if (ok) ok = fa_wait(&bars->k_full[0], 0, abort_flag);
      if (ok) {
        tc_fence_after();
        scores(0, 0);
        scores(1, 0);
      }
      for (int j = 0; j < nblk && ok; ++j) {
        ok = outputs(0, j);
        if (ok && j + 1 < nblk) {
          ok = fa_wait(&bars->k_full[(j + 1) % ST], ((j + 1) / ST) & 1, abort_flag);
          if (ok) {
            tc_fence_after();
            scores(0, j + 1);
          }
        }
        if (ok) ok = outputs(1, j);
        if (ok && j + 1 < nblk) scores(1, j + 1);
      }
      if (!ok) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    }
  } else {
    // ------------------------------ softmax of one map, epilogue ------------------------------
    const int q = warp & 3;                              // TMEM lane quarter
    const int g = (warp - kDtSoftmaxWarp) >> 2;          // map
    const int row = q * 32 + lane;
    const uint32_t lane_base = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
    const uint32_t s_addr = lane_base + Cfg::kColS + g * BN, o_addr = lane_base + g * VP;
    const float scale = p.scale * 1.4426950408889634f;
    const int pos = pos0 + row;
    const int hi = min(pos, ctx - 1), lo = p.window > 0 ? pos - p.window + 1 : 0;
    const int keep = p.window > 0 ? p.keep : 0;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int it = 0; it < nblk && ok; ++it) {
      ok = __all_sync(0xffffffffu, fa_wait(&bars->s_full[g], it & 1, abort_flag));
      if (!ok) break;
      tc_fence_after();
      const int k0 = block_at(it) * BN;
      // every column visible to every row of the tile: no mask
      const bool plain = k0 + BN - 1 <= pos0 && (p.window <= 0 || k0 > pos0 + kDtBM - 1 - p.window || k0 + BN <= keep);
      uint32_t pk[BN / 2];
      bool done = false;
      if (plain && it >= 1) {
        // one pass against the current maximum; kept unless some row's maximum has outgrown it
        const float neg_m = m_run == -INFINITY ? 0.f : -m_run;
        float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float v0 = __uint_as_float(a[2 * j]), v1 = __uint_as_float(a[2 * j + 1]);
            mx[0] = fmaxf(mx[0], v0);
            mx[1] = fmaxf(mx[1], v1);
            const float e0 = exp2f(fmaf(v0, scale, neg_m)), e1 = exp2f(fmaf(v1, scale, neg_m));
            sum[j & 1] += e0 + e1;
            pk[16 * c + j] = pack_bf16(e0, e1);
          }
        }
        if (!__any_sync(0xffffffffu, fmaxf(mx[0], mx[1]) * scale > m_run + kDtRecentre)) {
          l_run += sum[0] + sum[1];
          done = true;
        }
      }
      if (!done) {
        auto seen = [&](int k) { return k <= hi && (k >= lo || k < keep); };
        float mx = -INFINITY;
#pragma unroll
        for (int c = 0; c < BN / 32; ++c) {
          uint32_t a[32];
          tmem_ld_32x32(s_addr + 32 * c, a);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) mx = fmaxf(mx, seen(k0 + 32 * c + j) ? __uint_as_float(a[j]) * scale : -INFINITY);
        }
        const float m_new = fmaxf(m_run, mx);
        const bool raise = m_new > m_run + kDtRecentre || (m_run == -INFINITY && m_new > -INFINITY);
        if (it == 0) {
          m_run = m_new;
        } else if (__any_sync(0xffffffffu, raise)) {
          // the scores of this block were committed after the last product into the accumulator: it is complete
          float alpha = 1.f;
          if (raise) {
            alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_new);
            m_run = m_new;
            l_run *= alpha;
          }
#pragma unroll 1
          for (int c = 0; c < VP / 32; ++c) {
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
            const float e0 = exp2f(fmaf(seen(k) ? __uint_as_float(a[2 * j]) : -INFINITY, scale, neg_m));
            const float e1 = exp2f(fmaf(seen(k + 1) ? __uint_as_float(a[2 * j + 1]) : -INFINITY, scale, neg_m));
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
    if (ok) ok = __all_sync(0xffffffffu, fa_wait(&bars->pv_done[g], 0, abort_flag));
    if (!ok && lane == 0) {
      atomicOr(p.status, kStatusWaitTimeout);
      *abort_flag = 1;
    }
    // ---- o = a1 - lambda a2: each group finishes one half of the columns ----
    constexpr int HC = VP / 2;
    uint8_t* xo = sQ;
    asm volatile("bar.sync 1, 256;" ::: "memory");       // both groups' last products have landed: the operands are idle
    tc_fence_after();
    const float f = l_run > 0.f ? (g == 0 ? 1.f : -p.lambda) / l_run : 0.f;
    {
      float* dst = reinterpret_cast<float*>(xo + (static_cast<size_t>(g) * kDtBM + row) * Cfg::kXPitch);
#pragma unroll
      for (int c = 0; c < HC / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(o_addr + (g ^ 1) * HC + 32 * c, o);
        tmem_ld_wait();
#pragma unroll
        for (int v = 0; v < 8; ++v)
          *reinterpret_cast<float4*>(dst + 32 * c + 4 * v) = make_float4(__uint_as_float(o[4 * v]) * f, __uint_as_float(o[4 * v + 1]) * f,
                                                                        __uint_as_float(o[4 * v + 2]) * f, __uint_as_float(o[4 * v + 3]) * f);
      }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float* src = reinterpret_cast<const float*>(xo + (static_cast<size_t>(g ^ 1) * kDtBM + row) * Cfg::kXPitch);
    float o[HC], ss = 0.f;
#pragma unroll
    for (int c = 0; c < HC / 32; ++c) {
      uint32_t mine[32];
      tmem_ld_32x32(o_addr + g * HC + 32 * c, mine);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; j += 4) {
        const float4 other = *reinterpret_cast<const float4*>(src + 32 * c + j);
        o[32 * c + j] = fmaf(__uint_as_float(mine[j]), f, other.x);
        o[32 * c + j + 1] = fmaf(__uint_as_float(mine[j + 1]), f, other.y);
        o[32 * c + j + 2] = fmaf(__uint_as_float(mine[j + 2]), f, other.z);
        o[32 * c + j + 3] = fmaf(__uint_as_float(mine[j + 3]), f, other.w);
      }
    }
#pragma unroll
    for (int c = 0; c < HC; ++c) ss = fmaf(o[c], o[c], ss);
    x_ss[g * kDtBM + row] = ss;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    const float inv = p.gain / sqrtf((ss + x_ss[(g ^ 1) * kDtBM + row]) / static_cast<float>(p.dv) + p.eps);
    if (row < rows) {
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + static_cast<size_t>(q_begin + q0 + row) * p.ldo + head * p.vp + g * HC;
#pragma unroll
      for (int c = 0; c < HC; c += 8)
        if (g * HC + c < p.vp)
          *reinterpret_cast<uint4*>(out + c) = make_uint4(pack_bf16(o[c] * inv, o[c + 1] * inv), pack_bf16(o[c + 2] * inv, o[c + 3] * inv),
                                                          pack_bf16(o[c + 4] * inv, o[c + 5] * inv), pack_bf16(o[c + 6] * inv, o[c + 7] * inv));
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
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem_base, Cfg::kTmemCols);
  }
}

template <int DP, int VP, int BN, int ST>
static int launch_dt(const DiffParams& p, cudaStream_t stream) {
  using Cfg = DtCfg<DP, VP, BN, ST>;
  CUtensorMap q_map, k_map, v_map;
  const uint64_t pages = static_cast<uint64_t>(p.num_pages);
  int rc = encode_tmap_bf16_3d(&q_map, p.q, p.dp, 2 * p.hq, p.rows, p.dp, p.ldq, 64, 1, kDtBM);
  if (rc == 0) rc = encode_tmap_bf16_3d(&k_map, p.pool, p.dp, static_cast<uint64_t>(2 * p.hkv) * kDaPage, pages, p.dp, p.page_elems, 64, kDaPage, 1);
  if (rc == 0)
    rc = encode_tmap_bf16_3d(&v_map, static_cast<const __nv_bfloat16*>(p.pool) + static_cast<size_t>(2 * p.hkv) * kDaPage * p.dp, p.vp,
                             static_cast<uint64_t>(p.hkv) * kDaPage, pages, p.vp, p.page_elems, 64, kDaPage, 1);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(diff_prefill_tc_kernel<DP, VP, BN, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    attr_set = true;
  }
  diff_prefill_tc_kernel<DP, VP, BN, ST><<<dim3(p.num_tiles, p.hq), kDtThreads, Cfg::kSmemBytes, stream>>>(q_map, k_map, v_map, p);
  return static_cast<int>(cudaGetLastError());
}

int launch_diff_prefill_tc(const DiffParams& p, cudaStream_t stream) {
  if (p.d > 128 || p.dv > 192 || p.scale <= 0.f) return -2;          // the row maximum is taken before scaling
  if ((p.dp | p.vp | p.ldq | p.ldo) & 7 || (p.page_elems & 7)) return -2;
  if ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.pool)) & 15) return -2;
  if (p.d <= 64) {
    if (p.dv <= 64) return launch_dt<64, 64, 128, 2>(p, stream);
    if (p.dv <= 128) return launch_dt<64, 128, 128, 2>(p, stream);
    return launch_dt<64, 192, 64, 3>(p, stream);
  }
  if (p.dv <= 64) return launch_dt<128, 64, 64, 3>(p, stream);
  if (p.dv <= 128) return launch_dt<128, 128, 64, 3>(p, stream);
  return launch_dt<128, 192, 64, 2>(p, stream);
}

}  // namespace ogb
