// Attention over paged keys that are the values too: pages and norms (tied_append), the kernel for any size and both activation types,
// the decode kernel, and the entry point.  Prompts of the bf16 engine run in tied_attention_tc.cu.
#include "attention_common.cuh"
#include "tied_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

// ------------------------------------------------------------------------------------------------------
// One block per token: biases, the root mean square of all its queries and of all its keys, queries times their gain, keys to their slot
// with `factor` over their root mean square.
// ------------------------------------------------------------------------------------------------------
struct TiedAppendParams {
  const void* row;         // [tokens, ldr]: hq d queries | hkv d keys
  const float *q_bias, *k_bias, *q_gain;       // biases may be null
  void* q;                 // [tokens, ldq]: head at column head * dp
  void* pool;
  const int* slots;
  int64_t num_slots, page_elems;
  float eps, factor;
  int ldr, ldq, hq, hkv, d, dp;
  int* status;
};

template <typename T, int V>
__global__ void __launch_bounds__(256) tied_append_kernel(TiedAppendParams p) {
  extern __shared__ float ta_row[];            // the row with its biases
  __shared__ float red[2][8];
  const int t = blockIdx.x, nq = p.hq * p.d, n = nq + p.hkv * p.d, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* src = static_cast<const T*>(p.row) + static_cast<size_t>(t) * p.ldr;
  float ss[2] = {0.f, 0.f};
  for (int c = threadIdx.x * V; c < n; c += 256 * V) {
    const bool key = c >= nq;                  // V divides d
    const float* bias = key ? p.k_bias : p.q_bias;
    float x[V], b[V];
    load_vec<V>(src + c, x);
    if (bias != nullptr) {
      load_vec<V>(bias + (key ? c - nq : c), b);
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] += b[v];
    }
    float a = 0.f;
#pragma unroll
    for (int v = 0; v < V; ++v) a = fmaf(x[v], x[v], a);
    ss[key] += a;
    store_vec<V>(ta_row + c, x);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    ss[i] = warp_sum(ss[i]);
    if (lane == 0) red[i][warp] = ss[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float a = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) a += red[i][w];
    ss[i] = 1.f / sqrtf(a / static_cast<float>(i == 0 ? nq : n - nq) + p.eps);
  }
  T* q = static_cast<T*>(p.q) + static_cast<size_t>(t) * p.ldq;
  for (int c = threadIdx.x * V; c < p.hq * p.dp; c += 256 * V) {
    const int h = c / p.dp, e = c - h * p.dp;
    float x[V], g[V];
#pragma unroll
    for (int v = 0; v < V; ++v) x[v] = 0.f;
    if (e < p.d) {
      load_vec<V>(ta_row + h * p.d + e, x);
      load_vec<V>(p.q_gain + h * p.d + e, g);
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] *= ss[0] * g[v];
    }
    store_vec<V>(q + c, x);
  }
  const int64_t slot = p.slots[t];
  if (slot < 0) return;                        // padding row
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    return;
  }
  T* page = static_cast<T*>(p.pool) + slot / kTaPage * p.page_elems;
  const int off = static_cast<int>(slot % kTaPage);
  for (int c = threadIdx.x * V; c < p.hkv * p.dp; c += 256 * V) {
    const int h = c / p.dp, e = c - h * p.dp;
    float x[V];
#pragma unroll
    for (int v = 0; v < V; ++v) x[v] = 0.f;
    if (e < p.d) load_vec<V>(ta_row + nq + h * p.d + e, x);
    store_vec<V>(page + (static_cast<size_t>(h) * kTaPage + off) * p.dp + e, x);
  }
  if (threadIdx.x == 0) reinterpret_cast<float*>(page + static_cast<size_t>(p.hkv) * kTaPage * p.dp)[off] = ss[1] * p.factor;
}

template <typename T>
static int launch_tied_append(const TiedAppendParams& p, int tokens, cudaStream_t s) {
  const int smem = (p.hq + p.hkv) * p.d * 4;
  const uintptr_t act = reinterpret_cast<uintptr_t>(p.row) | reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.pool);
  const uintptr_t f32 = reinterpret_cast<uintptr_t>(p.q_bias) | reinterpret_cast<uintptr_t>(p.k_bias) | reinterpret_cast<uintptr_t>(p.q_gain);
  const bool vec = ((p.d | p.dp | p.ldr | p.ldq | p.page_elems) & 3) == 0 && (f32 & 15) == 0 && (act & (4 * sizeof(T) - 1)) == 0;
  if (smem > 160 * 1024) return -3;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(tied_append_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(tied_append_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr_set = true;
  }
  if (vec) tied_append_kernel<T, 4><<<tokens, 256, smem, s>>>(p);
  else tied_append_kernel<T, 1><<<tokens, 256, smem, s>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------------
// any size, fp32 or bf16: one warp per (token, head).  32 keys at a time, a lane per key for the scores, a lane per column for the
// products; all fp32.
// ------------------------------------------------------------------------------------------------------
constexpr int kTwWarps = 4, kTwMaxD = 512;

template <typename T, int NV>
__global__ void __launch_bounds__(kTwWarps * 32) tied_attention_warp_kernel(TiedParams p) {
  extern __shared__ float tw_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sq = tw_smem + warp * p.d;
  int entry, row, pos;
  if (p.cu_q == nullptr) {
    row = blockIdx.x * kTwWarps + warp;
    if (row >= p.rows) return;
    entry = row;
    pos = p.ctx_len[entry] - 1;
  } else {
    const int tile = blockIdx.x / (64 / kTwWarps), j = p.tile_q0[tile] + (blockIdx.x % (64 / kTwWarps)) * kTwWarps + warp;
    entry = p.tile_seq[tile];
    const int len = p.cu_q[entry + 1] - p.cu_q[entry];
    if (j >= len) return;
    row = p.cu_q[entry] + j;
    pos = p.ctx_len[entry] - len + j;
  }
  if (pos < 0 || p.ctx_len[entry] <= 0) return;
  const int head = blockIdx.y, kvh = head / (p.hq / p.hkv);
  const T* q = static_cast<const T*>(p.q) + static_cast<size_t>(row) * p.ldq + static_cast<size_t>(head) * p.dp;
  for (int i = lane; i < p.d; i += 32) sq[i] = to_f32<T>(q[i]);
  __syncwarp();
  const int kv_lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, n_pages = (p.ctx_len[entry] + kTaPage - 1) / kTaPage;
  const int* table = p.page_table + static_cast<size_t>(entry) * p.max_pages;
  const float slope = ta_slope(p, head);
  float m = ta_sink(p, head), l = m == -INFINITY ? 0.f : 1.f, o[NV];   // the sink counts once
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i] = 0.f;
  for (int k0 = kv_lo / 32 * 32; k0 <= pos; k0 += 32) {
    const int key = k0 + lane;
    const bool seen = key >= kv_lo && key <= pos;
    const T* k = nullptr;
    float s = -INFINITY;
    if (seen) {
      int64_t pg = table[ta_page_index(p, key / kTaPage, n_pages, kv_lo)];
      if (pg < 0 || pg >= p.num_pages) { atomicOr(p.status, kStatusIndexOutOfRange); pg = 0; }
      const T* page = static_cast<const T*>(p.pool) + pg * p.page_elems;
      k = page + (static_cast<size_t>(kvh) * kTaPage + key % kTaPage) * p.dp;
      float a[4] = {};
      int d = 0;
      for (; d + 4 <= p.d; d += 4)
#pragma unroll
        for (int j = 0; j < 4; ++j) a[j] = fmaf(sq[d + j], to_f32<T>(k[d + j]), a[j]);
      for (; d < p.d; ++d) a[0] = fmaf(sq[d], to_f32<T>(k[d]), a[0]);
      s = ((a[0] + a[1]) + (a[2] + a[3])) * reinterpret_cast<const float*>(page + static_cast<size_t>(p.hkv) * kTaPage * p.dp)[key % kTaPage];
      if (p.cap > 0.f) s = p.cap * tanhf(s);
      s -= slope * static_cast<float>(pos - key);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float c = mn == -INFINITY ? 1.f : expf(m - mn);
    const float e = seen ? expf(s - mn) : 0.f;
    l = l * c + warp_sum(e);
    m = mn;
#pragma unroll
    for (int n = 0; n < NV; ++n) o[n] *= c;
    const unsigned live = __ballot_sync(0xffffffffu, seen);
    for (int j = 0; j < 32; ++j) {
      if (!((live >> j) & 1u)) continue;
      const float ej = __shfl_sync(0xffffffffu, e, j);
      const T* v = reinterpret_cast<const T*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(k), j));
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int c0 = n * 32 + lane;
        if (c0 < p.d) o[n] = fmaf(ej, to_f32<T>(v[c0]), o[n]);
      }
    }
  }
  const float f = ta_gate<T>(p, row, head) / l;
  T* dst = static_cast<T*>(p.out) + static_cast<size_t>(row) * p.ldo + static_cast<size_t>(head) * p.dp;
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const int c = n * 32 + lane;
    if (c < p.dp) dst[c] = from_f32<T>(c < p.d ? o[n] * f : 0.f);
  }
}

template <typename T, int NV>
static int launch_tied_warp(const TiedParams& p, cudaStream_t stream) {
  const dim3 grid(p.cu_q == nullptr ? (p.rows + kTwWarps - 1) / kTwWarps : p.num_tiles * (64 / kTwWarps), p.hq);
  tied_attention_warp_kernel<T, NV><<<grid, kTwWarps * 32, kTwWarps * p.d * 4, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T>
static int dispatch_tied_warp(const TiedParams& p, cudaStream_t stream) {
  if (p.dp <= 64) return launch_tied_warp<T, 2>(p, stream);
  if (p.dp <= 128) return launch_tied_warp<T, 4>(p, stream);
  if (p.dp <= 256) return launch_tied_warp<T, 8>(p, stream);
  return launch_tied_warp<T, kTwMaxD / 32>(p, stream);
}

// ------------------------------------------------------------------------------------------------------
// decode, bf16.  One CTA = (sequence, up to 16 query heads of one KV head, split of the keys); the heads are the rows of the mma.sync
// tile.  Warp 4 streams 64-token blocks (4 pages of keys, and their factors) by TMA; each of the warps 0 - 3 takes one page of a block,
// once as the keys and once as the values, and they merge at the end.  The last split of a row to finish merges the splits.
// ------------------------------------------------------------------------------------------------------
int encode_tmap_bf16_3d(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint64_t planes, uint64_t row_stride, uint64_t plane_stride,
                        uint32_t box_cols, uint32_t box_rows, uint32_t box_planes);

constexpr int kTdHeads = 16;

template <int DP>
struct TdCfg {
  static constexpr int kKBytes = kKvBlock * DP * 2;
  static constexpr int kStageBytes = kKBytes + 1024;   // keys, 4 x 16 factors (stages stay 1024-byte aligned)
  static constexpr int kStages = DP <= 128 ? 5 : 2;
  static constexpr int kQBytes = 16 * DP * 2;
  static constexpr int kSmemBytes = kStages * kStageBytes + kQBytes + 1024 /*alignment*/ + 1024 /*barriers, merge statistics*/;
  static_assert(4 * 16 * DP * 4 <= kStages * kStageBytes, "the merge slab reuses the ring");
};

template <int DP>
__global__ void __launch_bounds__(kAttnThreads) tied_decode_kernel(const __grid_constant__ CUtensorMap k_map, const TiedParams p) {
  using Cfg = TdCfg<DP>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* stages = smem;
  uint8_t* sq = smem + Cfg::kStages * Cfg::kStageBytes;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(sq + Cfg::kQBytes);
  uint64_t* empty_bar = full_bar + Cfg::kStages;
  float* sm_ml = reinterpret_cast<float*>(empty_bar + Cfg::kStages);   // [4 warps][16 rows][2]
  int* sm_last = reinterpret_cast<int*>(sm_ml + 4 * 16 * 2);

  const int seq = blockIdx.x / p.num_splits, split = blockIdx.x % p.num_splits;
  const int group = p.hq / p.hkv, chunks = (group + kTdHeads - 1) / kTdHeads;
  const int kvh = blockIdx.y / chunks, h0 = (blockIdx.y % chunks) * kTdHeads;     // first head of this CTA within its group
  const int nh = min(kTdHeads, group - h0), head0 = kvh * group + h0;
  const int ctx = p.ctx_len[seq];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (ctx <= 0) return;                          // padding row
  const int kv_lo = p.window > 0 ? max(0, ctx - p.window) : 0;
  const int b_first = kv_lo / kKvBlock, count = (ctx + kKvBlock - 1) / kKvBlock - b_first;
  const int per = (count + p.num_splits - 1) / p.num_splits;
  const int b_begin = b_first + split * per, b_end = min(b_begin + per, b_first + count);

  if (threadIdx.x == 0) {
    for (int i = 0; i < Cfg::kStages; ++i) { mbar_init(&full_bar[i], 1); mbar_init(&empty_bar[i], 4); }
    mbar_fence_init();
    tma_prefetch_desc(&k_map);
  }
  __syncthreads();

  if (warp == 4) {
    if (lane == 0) {
      const int n_pages = (ctx + kTaPage - 1) / kTaPage;
      const int* table = p.page_table + static_cast<size_t>(seq) * p.max_pages;
      const __nv_bfloat16* factors = static_cast<const __nv_bfloat16*>(p.pool) + static_cast<size_t>(p.hkv) * kTaPage * p.dp;
      int stage = 0;
      uint32_t phase = 0;
      for (int b = b_begin; b < b_end; ++b) {
        int page_of[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          int64_t page = table[ta_page_index(p, b * 4 + i, n_pages, kv_lo)];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          page_of[i] = static_cast<int>(page);
        }
        if (!mbar_wait(&empty_bar[stage], phase ^ 1)) { atomicOr(p.status, kStatusWaitTimeout); break; }
        uint8_t* dst = stages + stage * Cfg::kStageBytes;
        mbar_expect_tx(&full_bar[stage], Cfg::kKBytes + 4 * 64);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
#pragma unroll
          for (int h = 0; h < DP / 64; ++h)
            tma_load_3d(dst + ((i * (DP / 64) + h) << 11), &k_map, &full_bar[stage], h * 64, kvh * kTaPage, page_of[i]);
          bulk_load(dst + Cfg::kKBytes + i * 64, factors + page_of[i] * p.page_elems, 64, &full_bar[stage]);
        }
        if (++stage == Cfg::kStages) { stage = 0; phase ^= 1; }
      }
    }
    return;
  }

  {
    const __nv_bfloat16* qsrc = static_cast<const __nv_bfloat16*>(p.q) + static_cast<size_t>(seq) * p.ldq;
    for (int idx = threadIdx.x; idx < 16 * (DP / 8); idx += 128) {
      const int row = idx / (DP / 8), ch = idx % (DP / 8);
      uint4 v = make_uint4(0, 0, 0, 0);
      if (row < nh && ch * 8 < p.dp) v = *reinterpret_cast<const uint4*>(qsrc + static_cast<size_t>(head0 + row) * p.dp + ch * 8);
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
  constexpr float kLog2e = 1.4426950408889634f;
  float o[DP / 8][4];
#pragma unroll
  for (int j = 0; j < DP / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f}, slope[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) slope[r] = (lane >> 2) + 8 * r < nh ? ta_slope(p, head0 + (lane >> 2) + 8 * r) * kLog2e : 0.f;
  const float cap = p.cap * kLog2e;
  const int mi = lane >> 3;
  const bool low_rows = nh <= 8;                 // rows 8 - 15 are empty

  int stage = 0;
  uint32_t phase = 0;
  bool ok = true;
  for (int b = b_begin; b < b_end; ++b) {
    if (!__all_sync(0xffffffffu, mbar_wait(&full_bar[stage], phase))) { ok = false; break; }
    const int tok0 = b * kKvBlock + 16 * warp;   // first token of this warp's page in the block
    if (tok0 < ctx && tok0 + 16 > kv_lo) {
      const uint32_t sk = smem_u32(stages + stage * Cfg::kStageBytes);
      const float* factor = reinterpret_cast<const float*>(stages + stage * Cfg::kStageBytes + Cfg::kKBytes) + 16 * warp;
      float s[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < DP / 16; ++kk) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(sk + kv_tile_off<DP>(16 * warp + 8 * (mi >> 1) + (lane & 7), 16 * kk + 8 * (mi & 1)), b0, b1, b2, b3);
        mma_bf16_16816(s[0], qf[kk], b0, b1);
        mma_bf16_16816(s[1], qf[kk], b2, b3);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int c = 8 * j + 2 * (lane & 3) + (x & 1), key = tok0 + c;
          if ((x >> 1) == 1 && low_rows) { s[j][x] = -INFINITY; continue; }
          float y = s[j][x] * factor[c];
          y = p.cap > 0.f ? cap * tanhf(y) : y * kLog2e;
          s[j][x] = key < ctx && key >= kv_lo ? y - slope[x >> 1] * static_cast<float>(ctx - 1 - key) : -INFINITY;
        }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = fmaxf(fmaxf(s[0][2 * r], s[0][2 * r + 1]), fmaxf(s[1][2 * r], s[1][2 * r + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m_run[r], mx), m_use = m_new == -INFINITY ? 0.f : m_new;
        const float alpha = exp2f(m_run[r] - m_use);
        m_run[r] = m_new;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          s[j][2 * r] = exp2f(s[j][2 * r] - m_use);
          s[j][2 * r + 1] = exp2f(s[j][2 * r + 1] - m_use);
          sum += s[j][2 * r] + s[j][2 * r + 1];
        }
        l_run[r] = l_run[r] * alpha + sum;
        if (__any_sync(0xffffffffu, alpha != 1.f)) {       // some row has a new maximum
#pragma unroll
          for (int j = 0; j < DP / 8; ++j) { o[j][2 * r] *= alpha; o[j][2 * r + 1] *= alpha; }
        }
      }
      const uint32_t a[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
#pragma unroll
      for (int jd = 0; jd < DP / 16; ++jd) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(sk + kv_tile_off<DP>(16 * warp + 8 * (mi & 1) + (lane & 7), 16 * jd + 8 * (mi >> 1)), b0, b1, b2, b3);
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
  float* sm_o = reinterpret_cast<float*>(stages);      // [4][16][DP]
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const int row = (lane >> 2) + 8 * r;
    if (row >= nh) continue;
    if ((lane & 3) == 0) {
      sm_ml[(warp * 16 + row) * 2] = m_run[r];
      sm_ml[(warp * 16 + row) * 2 + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < DP / 8; ++j)
      *reinterpret_cast<float2*>(sm_o + (warp * 16 + row) * DP + 8 * j + 2 * (lane & 3)) = make_float2(o[j][2 * r], o[j][2 * r + 1]);
  }
  compute_bar_sync();
  // a warp finishes the heads warp, warp + 4, ..: values of n parts with (maximum, sum) each, and the sink
  auto finish = [&](int n, auto ml, auto val) {
    for (int h = warp; h < nh; h += 4) {
      const float sink = ta_sink(p, head0 + h) * kLog2e;
      float m = sink, l = 0.f;
      for (int i = 0; i < n; ++i) m = fmaxf(m, ml(i, h).x);
      if (sink != -INFINITY) l = exp2f(sink - m);
      for (int i = 0; i < n; ++i) { const float2 x = ml(i, h); l += x.y * (x.x == -INFINITY ? 0.f : exp2f(x.x - m)); }
      const float f = l > 0.f ? ta_gate<__nv_bfloat16>(p, seq, head0 + h) / l : 0.f;
      float x[DP / 32];
#pragma unroll
      for (int c = 0; c < DP / 32; ++c) x[c] = 0.f;
      for (int i = 0; i < n; ++i) {
        const float mx = ml(i, h).x;
        if (mx == -INFINITY) continue;
        const float w = f * exp2f(mx - m);
#pragma unroll
        for (int c = 0; c < DP / 32; ++c) x[c] = fmaf(w, val(i, h, c * 32 + lane), x[c]);
      }
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + static_cast<size_t>(seq) * p.ldo + static_cast<size_t>(head0 + h) * p.dp;
#pragma unroll
      for (int c = 0; c < DP / 32; ++c)
        if (c * 32 + lane < p.dp) dst[c * 32 + lane] = __float2bfloat16(x[c]);
    }
  };
  if (p.num_splits == 1) {
    finish(4, [&](int i, int row) { return make_float2(sm_ml[(i * 16 + row) * 2], sm_ml[(i * 16 + row) * 2 + 1]); },
           [&](int i, int row, int c) { return sm_o[(i * 16 + row) * DP + c]; });
    return;
  }
  // ---- publish this split; the last one merges them all ----
  const size_t unit = static_cast<size_t>(seq) * gridDim.y + blockIdx.y;
  for (int row = warp; row < nh; row += 4) {
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
    for (int c = lane; c < p.dp; c += 32) {
      float x = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) x = fmaf(f[w], sm_o[(w * 16 + row) * DP + c], x);
      p.part_o[at * p.dp + c] = x;
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
         [&](int i, int row, int c) { return c < p.dp ? __ldcg(p.part_o + ((unit * 16 + row) * p.num_splits + i) * p.dp + c) : 0.f; });
}

template <int DP>
static int launch_td(TiedParams p, cudaStream_t stream) {
  using Cfg = TdCfg<DP>;
  CUtensorMap k_map;
  const int rc = encode_tmap_bf16_3d(&k_map, p.pool, p.dp, static_cast<uint64_t>(p.hkv) * kTaPage, static_cast<uint64_t>(p.num_pages), p.dp, p.page_elems, 64,
                                     kTaPage, 1);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(tied_decode_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(tied_decode_kernel<DP>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
    attr_set = true;
  }
  if (p.part_o == nullptr || p.part_ml == nullptr || p.counters == nullptr) p.num_splits = 1;
  const int chunks = (p.hq / p.hkv + kTdHeads - 1) / kTdHeads;
  tied_decode_kernel<DP><<<dim3(p.rows * p.num_splits, p.hkv * chunks), kAttnThreads, Cfg::kSmemBytes, stream>>>(k_map, p);
  return static_cast<int>(cudaGetLastError());
}

int launch_tied_decode(const TiedParams& p, cudaStream_t stream) {
  if (p.dp > 256 || ((p.dp | p.ldq | p.page_elems) & 7) != 0) return -2;
  if ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.pool)) & 15) return -2;
  if (p.dp <= 64) return launch_td<64>(p, stream);
  if (p.dp <= 128) return launch_td<128>(p, stream);
  return launch_td<256>(p, stream);
}

}  // namespace ogb

using namespace ogb;

extern "C" int ogb_tied_append(const void* row, int ldr, const float* q_bias, const float* k_bias, const float* q_gain, float eps, float factor, void* q,
                               int ldq, void* pool, const int* slots, int64_t num_slots, int64_t page_elems, int tokens, int hq, int hkv, int d, int dp,
                               int elem, int* status, void* stream) {
  if (tokens <= 0) return 0;
  if (hq < 1 || hkv < 1 || d < 1 || dp < d || dp % 8 != 0 || ldq < hq * dp || page_elems < static_cast<int64_t>(hkv) * kTaPage * dp + 2 * kTaPage ||
      (page_elems & 1)) return -3;
  TiedAppendParams p{row, q_bias, k_bias, q_gain, q, pool, slots, num_slots, page_elems, eps, factor, ldr, ldq, hq, hkv, d, dp, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return launch_tied_append<__nv_bfloat16>(p, tokens, s);
  if (elem == kElemF32) return launch_tied_append<float>(p, tokens, s);
  return -3;
}

static int g_tied_tc = 1;
// 0 keeps the bf16 engine on the kernel for any size as well (comparison runs); returns the old setting.
extern "C" int ogb_tied_set_tc(int on) {
  const int old = g_tied_tc;
  g_tied_tc = on != 0;
  return old;
}

extern "C" int ogb_tied_attention(const void* q, void* out, const void* pool, const int* page_table, const int* ctx_len, const int* cu_q,
                                  const int* tile_seq, const int* tile_q0, const void* gate, const float* slope, const float* sink, int rows,
                                  int num_tiles, int max_pages, int64_t num_pages, int64_t page_elems, int hq, int hkv, int d, int dp, int ldq, int ldo,
                                  int ldg, int window, float cap, int num_splits, float* part_o, float* part_ml, int* counters, int elem, int* status,
                                  void* stream) {
  if (rows <= 0 || (cu_q != nullptr && num_tiles <= 0)) return 0;
  if (hkv <= 0 || hq % hkv != 0 || d < 1 || dp < d || dp > kTwMaxD || max_pages < 1 || num_pages < 1) return -3;
  if (page_elems < static_cast<int64_t>(hkv) * kTaPage * dp + 2 * kTaPage) return -3;
  TiedParams p{q, out, pool, page_table, ctx_len, cu_q, tile_seq, tile_q0, gate, slope, sink, rows, num_tiles, max_pages, num_pages, page_elems, hq, hkv,
               d, dp, ldq, ldo, ldg, window, cap, num_splits < 1 ? 1 : num_splits, part_o, part_ml, counters, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) {
    if (g_tied_tc) {
      const int rc = cu_q == nullptr ? launch_tied_decode(p, s) : launch_tied_prefill_tc(p, s);
      if (rc != -2) return rc;
    }
    return dispatch_tied_warp<__nv_bfloat16>(p, s);
  }
  if (elem == kElemF32) return dispatch_tied_warp<float>(p, s);
  return -3;
}
