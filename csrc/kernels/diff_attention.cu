// Differential attention over paged keys and values: the kernel for any size and both activation types, the decode kernel, and
// the entry point.  Prompts of the bf16 engine run in diff_attention_tc.cu.
#include "attention_common.cuh"
#include "diff_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

// ------------------------------------------------------------------------------------------------------
// any size, fp32 or bf16: one warp per (token, head).  32 keys at a time, a lane per key for the scores of both maps, a lane per
// value column for the products; all fp32.
// ------------------------------------------------------------------------------------------------------
constexpr int kDwWarps = 4, kDwMaxV = 512;

template <typename T, int NV>
__global__ void __launch_bounds__(kDwWarps * 32) diff_attention_warp_kernel(DiffParams p) {
  extern __shared__ float dw_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sq = dw_smem + warp * 2 * p.d;
  int entry, row, pos;
  if (p.cu_q == nullptr) {
    row = blockIdx.x * kDwWarps + warp;
    if (row >= p.rows) return;
    entry = row;
    pos = p.ctx_len[entry] - 1;
  } else {
    const int tile = blockIdx.x / (64 / kDwWarps), j = p.tile_q0[tile] + (blockIdx.x % (64 / kDwWarps)) * kDwWarps + warp;
    entry = p.tile_seq[tile];
    const int len = p.cu_q[entry + 1] - p.cu_q[entry];
    if (j >= len) return;
    row = p.cu_q[entry] + j;
    pos = p.ctx_len[entry] - len + j;
  }
  if (pos < 0 || p.ctx_len[entry] <= 0) return;
  const int head = blockIdx.y, kvh = head / (p.hq / p.hkv);
  const T* q = static_cast<const T*>(p.q) + static_cast<size_t>(row) * p.ldq + 2 * head * p.dp;
  for (int i = lane; i < 2 * p.d; i += 32) sq[i] = to_f32<T>(q[i < p.d ? i : p.dp + i - p.d]);
  __syncwarp();
  const int kv_lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, n_pages = (p.ctx_len[entry] + kDaPage - 1) / kDaPage;
  const int* table = p.page_table + static_cast<size_t>(entry) * p.max_pages;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[2][NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[0][i] = o[1][i] = 0.f;
  const int keep_end = (p.keep + 31) / 32 * 32;
  for (int k0 = 0; k0 <= pos; k0 += 32) {
    if (p.window > 0 && k0 >= keep_end && k0 + 32 <= kv_lo) k0 = kv_lo / 32 * 32;      // over the gap
    const int key = k0 + lane;
    const bool seen = da_visible(p, key, pos);
    const T* page = nullptr;
    float s[2] = {-INFINITY, -INFINITY};
    if (seen) {
      int64_t pg = table[da_page_index(p, key / kDaPage, n_pages, kv_lo)];
      if (pg < 0 || pg >= p.num_pages) { atomicOr(p.status, kStatusIndexOutOfRange); pg = 0; }
      page = static_cast<const T*>(p.pool) + pg * p.page_elems;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const T* k = page + ((2 * kvh + i) * kDaPage + key % kDaPage) * p.dp;
        float a[4] = {};
        int d = 0;
        for (; d + 4 <= p.d; d += 4)
#pragma unroll
          for (int j = 0; j < 4; ++j) a[j] = fmaf(sq[i * p.d + d + j], to_f32<T>(k[d + j]), a[j]);
        for (; d < p.d; ++d) a[0] = fmaf(sq[i * p.d + d], to_f32<T>(k[d]), a[0]);
        s[i] = ((a[0] + a[1]) + (a[2] + a[3])) * p.scale;
      }
    }
    const T* v = page != nullptr ? page + 2 * p.hkv * kDaPage * p.dp + (kvh * kDaPage + key % kDaPage) * p.vp : nullptr;
    float e[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float mn = fmaxf(m[i], warp_max(s[i]));
      const float c = mn == -INFINITY ? 1.f : expf(m[i] - mn);
      e[i] = seen ? expf(s[i] - mn) : 0.f;
      l[i] = l[i] * c + warp_sum(e[i]);
      m[i] = mn;
#pragma unroll
      for (int n = 0; n < NV; ++n) o[i][n] *= c;
    }
    const unsigned live = __ballot_sync(0xffffffffu, seen);
    for (int j = 0; j < 32; ++j) {
      if (!((live >> j) & 1u)) continue;
      const float e0 = __shfl_sync(0xffffffffu, e[0], j), e1 = __shfl_sync(0xffffffffu, e[1], j);
      const T* vj = reinterpret_cast<const T*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(v), j));
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int c = n * 32 + lane;
        const float x = c < p.dv ? to_f32<T>(vj[c]) : 0.f;
        o[0][n] = fmaf(e0, x, o[0][n]);
        o[1][n] = fmaf(e1, x, o[1][n]);
      }
    }
  }
  const float i0 = 1.f / l[0], i1 = p.lambda / l[1];
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    o[0][n] = o[0][n] * i0 - o[1][n] * i1;
    ss = fmaf(o[0][n], o[0][n], ss);
  }
  const float inv = p.gain / sqrtf(warp_sum(ss) / static_cast<float>(p.dv) + p.eps);
  T* dst = static_cast<T*>(p.out) + static_cast<size_t>(row) * p.ldo + head * p.vp;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int c = n * 32 + lane;
    if (c < p.vp) dst[c] = from_f32<T>(c < p.dv ? o[0][n] * inv : 0.f);
  }
}

template <typename T, int NV>
static int launch_diff_warp(const DiffParams& p, cudaStream_t stream) {
  const int smem = kDwWarps * 2 * p.d * 4;
  if (smem > 48 * 1024) return -3;
  const dim3 grid(p.cu_q == nullptr ? (p.rows + kDwWarps - 1) / kDwWarps : p.num_tiles * (64 / kDwWarps), p.hq);
  diff_attention_warp_kernel<T, NV><<<grid, kDwWarps * 32, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T>
static int dispatch_diff_warp(const DiffParams& p, cudaStream_t stream) {
  if (p.dv <= 64) return launch_diff_warp<T, 2>(p, stream);
  if (p.dv <= 128) return launch_diff_warp<T, 4>(p, stream);
  if (p.dv <= 256) return launch_diff_warp<T, 8>(p, stream);
  return launch_diff_warp<T, kDwMaxV / 32>(p, stream);
}

// ------------------------------------------------------------------------------------------------------
// decode, bf16.  One CTA = (sequence, 8 query heads of one KV head, split of the keys).  Rows 0 - 7 of the mma.sync tile are the
// heads' first maps, rows 8 - 15 their second maps: the scores of a fragment's upper rows come from the product with K1, of its
// lower rows from the one with K2, and one product with V serves both.  Warp 4 streams 64-token blocks (4 pages of K1 | K2 | V)
// by TMA; each of the warps 0 - 3 takes one page of a block, and they merge at the end.  The last split of a row to finish merges
// the splits.  Difference, norm and scaling follow in the CTA that holds the merged rows.
// ------------------------------------------------------------------------------------------------------
int encode_tmap_bf16_3d(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint64_t planes, uint64_t row_stride, uint64_t plane_stride,
                        uint32_t box_cols, uint32_t box_rows, uint32_t box_planes);

constexpr int kDdHeads = 8;

template <int DP, int VP>
struct DdCfg {
  static constexpr int kKBytes = kKvBlock * DP * 2, kVBytes = kKvBlock * VP * 2;
  static constexpr int kStageBytes = 2 * kKBytes + kVBytes;
  static constexpr int kStages = 100 * 1024 / kStageBytes < 2 ? 2 : 100 * 1024 / kStageBytes > 4 ? 4 : 100 * 1024 / kStageBytes;
  static constexpr int kQBytes = 16 * DP * 2;
  static constexpr int kSmemBytes = kStages * kStageBytes + kQBytes + 1024 /*alignment*/ + 1024 /*barriers, merge statistics*/;
  static_assert(4 * 16 * VP * 4 <= kStages * kStageBytes, "the merge slab reuses the ring");
};

template <int DP, int VP>
__global__ void __launch_bounds__(kAttnThreads) diff_decode_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                                                                  const DiffParams p) {
  using Cfg = DdCfg<DP, VP>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* stages = smem;
  uint8_t* sq = smem + Cfg::kStages * Cfg::kStageBytes;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(sq + Cfg::kQBytes);
  uint64_t* empty_bar = full_bar + Cfg::kStages;
  float* sm_ml = reinterpret_cast<float*>(empty_bar + Cfg::kStages);   // [4 warps][16 rows][2]
  int* sm_last = reinterpret_cast<int*>(sm_ml + 4 * 16 * 2);

  const int seq = blockIdx.x / p.num_splits, split = blockIdx.x % p.num_splits;
  const int group = p.hq / p.hkv, chunks = (group + kDdHeads - 1) / kDdHeads;
  const int kvh = blockIdx.y / chunks, h0 = (blockIdx.y % chunks) * kDdHeads;     // first head of this CTA within its group
  const int nh = min(kDdHeads, group - h0);
  const int ctx = p.ctx_len[seq];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (ctx <= 0) return;                          // padding row
  const int kv_lo = p.window > 0 ? max(0, ctx - p.window) : 0, keep = p.window > 0 ? p.keep : 0;
  const KvBlocks blocks = make_kv_blocks(p.window, keep, kv_lo, ctx, kKvBlock);
  const int per = (blocks.count + p.num_splits - 1) / p.num_splits;
  const int b_begin = split * per, b_end = min(b_begin + per, blocks.count);

  if (threadIdx.x == 0) {
    for (int i = 0; i < Cfg::kStages; ++i) { mbar_init(&full_bar[i], 1); mbar_init(&empty_bar[i], 4); }
    mbar_fence_init();
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
  }
  __syncthreads();

  if (warp == 4) {
    if (lane == 0) {
      const int n_pages = (ctx + kDaPage - 1) / kDaPage;
      const int* table = p.page_table + static_cast<size_t>(seq) * p.max_pages;
      int stage = 0;
      uint32_t phase = 0;
      for (int j = b_begin; j < b_end; ++j) {
        const int b = blocks.phys(j);
        int page_of[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          int64_t page = table[da_page_index(p, b * 4 + i, n_pages, kv_lo)];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          page_of[i] = static_cast<int>(page);
        }
        if (!mbar_wait(&empty_bar[stage], phase ^ 1)) { atomicOr(p.status, kStatusWaitTimeout); break; }
        uint8_t* dst = stages + stage * Cfg::kStageBytes;
        mbar_expect_tx(&full_bar[stage], Cfg::kStageBytes);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int h = 0; h < DP / 64; ++h)
              tma_load_3d(dst + m * Cfg::kKBytes + ((i * (DP / 64) + h) << 11), &k_map, &full_bar[stage], h * 64, (2 * kvh + m) * kDaPage, page_of[i]);
#pragma unroll
          for (int h = 0; h < VP / 64; ++h)
            tma_load_3d(dst + 2 * Cfg::kKBytes + ((i * (VP / 64) + h) << 11), &v_map, &full_bar[stage], h * 64, kvh * kDaPage, page_of[i]);
        }
        if (++stage == Cfg::kStages) { stage = 0; phase ^= 1; }
      }
    }
    return;
  }

  {
    const __nv_bfloat16* qsrc = static_cast<const __nv_bfloat16*>(p.q) + static_cast<size_t>(seq) * p.ldq;
    for (int idx = threadIdx.x; idx < 16 * (DP / 8); idx += 128) {
      const int row = idx / (DP / 8), ch = idx % (DP / 8), h = row & 7;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (h < nh && ch * 8 < p.dp) v = *reinterpret_cast<const uint4*>(qsrc + (2 * (kvh * group + h0 + h) + (row >> 3)) * p.dp + ch * 8);
      *reinterpret_cast<uint4*>(sq + q_tile_off<16>(row, ch * 8)) = v;
    }
  }
  compute_bar_sync();
  uint32_t qf[DP / 16][4];
  {
    const uint32_t sq_u = smem_u32(sq);
#pragma unroll
    for (int kk = 0; kk < DP / 16; ++kk)
      ldsm_x4(sq_u + q_tile_off<16>(lane & 15, 16 * kk + 8 * (lane >> 4)), qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3]);
  }
  float o[VP / 8][4];
#pragma unroll
  for (int j = 0; j < VP / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const float scale = p.scale * 1.4426950408889634f;
  const int mi = lane >> 3;

  int stage = 0;
  uint32_t phase = 0;
  bool ok = true;
  for (int jb = b_begin; jb < b_end; ++jb) {
    const int b = blocks.phys(jb);
    if (!__all_sync(0xffffffffu, mbar_wait(&full_bar[stage], phase))) { ok = false; break; }
    const int tok0 = b * kKvBlock + 16 * warp;   // first token of this warp's page in the block
    if (tok0 < ctx && (tok0 + 16 > kv_lo || tok0 < keep)) {
      const uint32_t sk = smem_u32(stages + stage * Cfg::kStageBytes), sv = sk + 2 * Cfg::kKBytes;
      float s[2][2][4] = {};                     // [map][8 keys]
#pragma unroll
      for (int kk = 0; kk < DP / 16; ++kk) {
        const uint32_t off = kv_tile_off<DP>(16 * warp + 8 * (mi >> 1) + (lane & 7), 16 * kk + 8 * (mi & 1));
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(sk + m * Cfg::kKBytes + off, b0, b1, b2, b3);
          mma_bf16_16816(s[m][0], qf[kk], b0, b1);
          mma_bf16_16816(s[m][1], qf[kk], b2, b3);
        }
      }
      float e[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int col = tok0 + 8 * j + 2 * (lane & 3) + (x & 1);
          e[j][x] = col < ctx && (col >= kv_lo || col < keep) ? s[x >> 1][j][x] * scale : -INFINITY;
        }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = fmaxf(fmaxf(e[0][2 * r], e[0][2 * r + 1]), fmaxf(e[1][2 * r], e[1][2 * r + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m_run[r], mx), m_use = m_new == -INFINITY ? 0.f : m_new;
        const float alpha = exp2f(m_run[r] - m_use);
        m_run[r] = m_new;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          e[j][2 * r] = exp2f(e[j][2 * r] - m_use);
          e[j][2 * r + 1] = exp2f(e[j][2 * r + 1] - m_use);
          sum += e[j][2 * r] + e[j][2 * r + 1];
        }
        l_run[r] = l_run[r] * alpha + sum;
#pragma unroll
        for (int j = 0; j < VP / 8; ++j) { o[j][2 * r] *= alpha; o[j][2 * r + 1] *= alpha; }
      }
      const uint32_t a[4] = {pack_bf16(e[0][0], e[0][1]), pack_bf16(e[0][2], e[0][3]), pack_bf16(e[1][0], e[1][1]), pack_bf16(e[1][2], e[1][3])};
#pragma unroll
      for (int jd = 0; jd < VP / 16; ++jd) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(sv + kv_tile_off<VP>(16 * warp + 8 * (mi & 1) + (lane & 7), 16 * jd + 8 * (mi >> 1)), b0, b1, b2, b3);
        mma_bf16_16816(o[2 * jd], a, b0, b1);
        mma_bf16_16816(o[2 * jd + 1], a, b2, b3);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty_bar[stage]);
    if (++stage == Cfg::kStages) { stage = 0; phase ^= 1; }
  }
  if (!ok && lane == 0) atomicOr(p.status, kStatusWaitTimeout);

  // ---- merge the four warps (each saw a disjoint quarter of the keys) ----
  compute_bar_sync();                            // every stage has been consumed: the ring is scratch now
  float* sm_o = reinterpret_cast<float*>(stages);      // [4][16][VP]
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const int row = (lane >> 2) + 8 * r;
    if ((lane & 3) == 0) {
      sm_ml[(warp * 16 + row) * 2] = m_run[r];
      sm_ml[(warp * 16 + row) * 2 + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < VP / 8; ++j)
      *reinterpret_cast<float2*>(sm_o + (warp * 16 + row) * VP + 8 * j + 2 * (lane & 3)) = make_float2(o[j][2 * r], o[j][2 * r + 1]);
  }
  compute_bar_sync();
  // a warp finishes the heads warp, warp + 4: values of n parts with (maximum, sum) each
  auto finish = [&](int n, auto ml, auto val) {
    for (int h = warp; h < nh; h += 4) {
      float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        for (int i = 0; i < n; ++i) m[r] = fmaxf(m[r], ml(i, h + 8 * r).x);
        for (int i = 0; i < n; ++i) { const float2 x = ml(i, h + 8 * r); l[r] += x.y * (x.x == -INFINITY ? 0.f : exp2f(x.x - m[r])); }
      }
      float x[VP / 32], ss = 0.f;
#pragma unroll
      for (int c = 0; c < VP / 32; ++c) x[c] = 0.f;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float f = l[r] > 0.f ? (r == 0 ? 1.f : -p.lambda) / l[r] : 0.f;
        for (int i = 0; i < n; ++i) {
          const float mx = ml(i, h + 8 * r).x;
          if (mx == -INFINITY) continue;
          const float w = f * exp2f(mx - m[r]);
#pragma unroll
          for (int c = 0; c < VP / 32; ++c) x[c] = fmaf(w, val(i, h + 8 * r, c * 32 + lane), x[c]);
        }
      }
#pragma unroll
      for (int c = 0; c < VP / 32; ++c) ss = fmaf(x[c], x[c], ss);
      const float inv = p.gain / sqrtf(warp_sum(ss) / static_cast<float>(p.dv) + p.eps);
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + static_cast<size_t>(seq) * p.ldo + (kvh * group + h0 + h) * p.vp;
#pragma unroll
      for (int c = 0; c < VP / 32; ++c)
        if (c * 32 + lane < p.vp) dst[c * 32 + lane] = __float2bfloat16(x[c] * inv);
    }
  };
  if (p.num_splits == 1) {
    finish(4, [&](int i, int row) { return make_float2(sm_ml[(i * 16 + row) * 2], sm_ml[(i * 16 + row) * 2 + 1]); },
           [&](int i, int row, int c) { return sm_o[(i * 16 + row) * VP + c]; });
    return;
  }
  // ---- publish this split; the last one merges them all ----
  const size_t unit = static_cast<size_t>(seq) * gridDim.y + blockIdx.y;
  for (int row = warp; row < 16; row += 4) {
    if ((row & 7) >= nh) continue;
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, sm_ml[(w * 16 + row) * 2]);
    float f[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = sm_ml[(w * 16 + row) * 2];
      f[w] = mw == -INFINITY ? 0.f : exp2f(mw - m);
      l += f[w] * sm_ml[(w * 16 + row) * 2 + 1];
    }
    const size_t at = (unit * 16 + row) * p.num_splits + split;
    if (lane == 0) *reinterpret_cast<float2*>(p.part_ml + 2 * at) = make_float2(m, l);
    for (int c = lane; c < p.vp; c += 32) {
      float x = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) x = fmaf(f[w], sm_o[(w * 16 + row) * VP + c], x);
      p.part_o[at * p.vp + c] = x;
    }
  }
  __threadfence();
  compute_bar_sync();
  if (threadIdx.x == 0) *sm_last = atomicAdd(p.counters + unit, 1) == p.num_splits - 1;
  compute_bar_sync();
  if (*sm_last == 0) return;
  __threadfence();
  if (threadIdx.x == 0) p.counters[unit] = 0;
  finish(p.num_splits, [&](int i, int row) { return __ldcg(reinterpret_cast<const float2*>(p.part_ml) + (unit * 16 + row) * p.num_splits + i); },
         [&](int i, int row, int c) { return c < p.vp ? __ldcg(p.part_o + ((unit * 16 + row) * p.num_splits + i) * p.vp + c) : 0.f; });
}

template <int DP, int VP>
static int launch_dd(DiffParams p, cudaStream_t stream) {
  using Cfg = DdCfg<DP, VP>;
  CUtensorMap k_map, v_map;
  const uint64_t pages = static_cast<uint64_t>(p.num_pages);
  int rc = encode_tmap_bf16_3d(&k_map, p.pool, p.dp, static_cast<uint64_t>(2 * p.hkv) * kDaPage, pages, p.dp, p.page_elems, 64, kDaPage, 1);
  if (rc == 0)
    rc = encode_tmap_bf16_3d(&v_map, static_cast<const __nv_bfloat16*>(p.pool) + static_cast<size_t>(2 * p.hkv) * kDaPage * p.dp, p.vp,
                             static_cast<uint64_t>(p.hkv) * kDaPage, pages, p.vp, p.page_elems, 64, kDaPage, 1);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(diff_decode_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(diff_decode_kernel<DP, VP>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
    attr_set = true;
  }
  if (p.part_o == nullptr || p.part_ml == nullptr || p.counters == nullptr) p.num_splits = 1;
  const int chunks = (p.hq / p.hkv + kDdHeads - 1) / kDdHeads;
  diff_decode_kernel<DP, VP><<<dim3(p.rows * p.num_splits, p.hkv * chunks), kAttnThreads, Cfg::kSmemBytes, stream>>>(k_map, v_map, p);
  return static_cast<int>(cudaGetLastError());
}

int launch_diff_decode(const DiffParams& p, cudaStream_t stream) {
  if (p.d > 128 || p.dv > 256) return -2;
  if ((p.dp | p.vp | p.ldq) & 7 || (p.page_elems & 7)) return -2;
  if ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.pool)) & 15) return -2;
  if (p.d <= 64) {
    if (p.dv <= 64) return launch_dd<64, 64>(p, stream);
    if (p.dv <= 128) return launch_dd<64, 128>(p, stream);
    return launch_dd<64, 256>(p, stream);
  }
  if (p.dv <= 64) return launch_dd<128, 64>(p, stream);
  if (p.dv <= 128) return launch_dd<128, 128>(p, stream);
  return launch_dd<128, 256>(p, stream);
}

}  // namespace ogb

using namespace ogb;

static int g_diff_tc = 1;
// 0 keeps the bf16 engine on the kernel for any size as well (comparison runs); returns the old setting.
extern "C" int ogb_diff_set_tc(int on) {
  const int old = g_diff_tc;
  g_diff_tc = on != 0;
  return old;
}

extern "C" int ogb_diff_attention(const void* q, void* out, const void* pool, const int* page_table, const int* ctx_len, const int* cu_q,
                                  const int* tile_seq, const int* tile_q0, int rows, int num_tiles, int max_pages, int64_t num_pages,
                                  int64_t page_elems, int hq, int hkv, int d, int dv, int dp, int vp, int ldq, int ldo, int window, int keep,
                                  float scale, float lambda, float eps, float gain, int num_splits, float* part_o, float* part_ml, int* counters,
                                  int elem, int* status, void* stream) {
  if (rows <= 0 || (cu_q != nullptr && num_tiles <= 0)) return 0;
  if (hkv <= 0 || hq % hkv != 0 || d < 1 || dv < 1 || dv > kDwMaxV || dp < d || vp < dv || max_pages < 1 || num_pages < 1) return -3;
  if (page_elems < static_cast<int64_t>(hkv) * kDaPage * (2 * dp + vp)) return -3;
  DiffParams p{q, out, pool, page_table, ctx_len, cu_q, tile_seq, tile_q0, rows, num_tiles, max_pages, num_pages, page_elems, hq, hkv, d, dv, dp, vp,
               ldq, ldo, window, window > 0 ? keep : 0, scale, lambda, eps, gain, num_splits < 1 ? 1 : num_splits, part_o, part_ml, counters, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) {
    if (g_diff_tc) {
      const int rc = cu_q == nullptr ? launch_diff_decode(p, s) : launch_diff_prefill_tc(p, s);
      if (rc != -2) return rc;
    }
    return dispatch_diff_warp<__nv_bfloat16>(p, s);
  }
  if (elem == kElemF32) return dispatch_diff_warp<float>(p, s);
  return -3;
}
