// Attention over paged latents: every head of a layer reads the same cached row c_j as key and, in its first kv_rank values, as value.
// The per-head expansions are folded into the query and the output by matrix products outside this file
// (q' = W_uk^T q before, W_uv o after), so a query row is (token, head) with as many values as a cached row -- kv_rank, and
// behind them those of a rotated part that all heads share, where there is one --, score = q' . c * scale, and the result is the
// softmax-weighted sum of the visible c_j, times the sigmoid of the head's gate where there is one.  A token at position i sees j with 0 <= i - j < window
// (window <= 0: every earlier token).
//
// bf16 rows of up to 576 values run on the tensor cores (latent_attention_tc.cu).  latent_attention_warp_kernel takes any rank
// and both activation types: one warp per query row, four keys at a time, online softmax in fp32.  Decode rows can split
// their keys `num_splits` ways (combined by a second kernel).
#include <stdlib.h>

#include "latent_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kLatWarps = 4;

template <typename T, int PER>
__global__ void __launch_bounds__(kLatWarps * 32) latent_attention_warp_kernel(LatParams p) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int entry, token, head, pos;
  if (p.cu_q == nullptr) {
    const int item = blockIdx.x * kLatWarps + warp;
    if (item >= p.rows * p.heads) return;
    token = item / p.heads; head = item % p.heads; entry = token;
    pos = p.ctx_len[entry] - 1;
    if (pos < 0) return;                          // padding row
  } else {
    const int per_tile = (64 * p.heads + kLatWarps - 1) / kLatWarps;
    const int tile = blockIdx.x / per_tile;
    const int item = (blockIdx.x % per_tile) * kLatWarps + warp;
    if (item >= 64 * p.heads) return;
    entry = p.tile_seq[tile];
    const int n = p.cu_q[entry + 1] - p.cu_q[entry];
    const int j = p.tile_q0[tile] + item / p.heads;
    if (j >= n) return;
    token = p.cu_q[entry] + j; head = item % p.heads;
    pos = p.ctx_len[entry] - n + j;
  }
  int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0, hi = pos + 1;
  if (p.num_splits > 1) {                         // split the visible keys in whole pages
    const int p0 = lo / kLatPage, pages = (hi + kLatPage - 1) / kLatPage - p0;
    const int per = (pages + p.num_splits - 1) / p.num_splits;
    const int b = (p0 + static_cast<int>(blockIdx.y) * per) * kLatPage;
    lo = max(lo, b);
    hi = min(hi, b + per * kLatPage);
  }
  const size_t row = static_cast<size_t>(token) * p.heads + head;
  const T* qp = static_cast<const T*>(p.q) + row * p.ldq;
  float q[PER], acc[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = lane + 32 * e;
    q[e] = i < p.rank ? to_f32<T>(qp[i]) : 0.f;
    acc[e] = 0.f;
  }
  const int* table = p.page_table + static_cast<size_t>(entry) * p.max_pages;
  float m = -INFINITY, l = 0.f;
  for (int j0 = lo; j0 < hi; j0 += 4) {
    float c[4][PER], d[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int j = j0 + u;
      const T* src = nullptr;
      if (j < hi) {
        const int pi = j / kLatPage;
        const int page = pi < p.max_pages ? table[pi] : -1;
        if (page < 0 || page >= p.num_pages) {
          if (lane == 0) atomicOr(p.status, kStatusIndexOutOfRange);
        } else {
          src = static_cast<const T*>(p.pool) + (static_cast<size_t>(page) * kLatPage + j % kLatPage) * p.ldp;
        }
      }
      d[u] = 0.f;
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        const int i = lane + 32 * e;
        c[u][e] = (src != nullptr && i < p.rank) ? to_f32<T>(src[i]) : 0.f;
        d[u] = fmaf(q[e], c[u][e], d[u]);
      }
      d[u] = warp_sum(d[u]) * p.scale;
      if (src == nullptr) d[u] = -INFINITY;
    }
    const float mb = fmaxf(fmaxf(d[0], d[1]), fmaxf(d[2], d[3]));
    if (mb == -INFINITY) continue;
    const float mn = fmaxf(m, mb);
    const float corr = expf(m - mn);              // exp(-inf) = 0 at the first live key
    l *= corr;
#pragma unroll
    for (int e = 0; e < PER; ++e) acc[e] *= corr;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float w = expf(d[u] - mn);
      l += w;
#pragma unroll
      for (int e = 0; e < PER; ++e) acc[e] = fmaf(w, c[u][e], acc[e]);
    }
    m = mn;
  }
  if (p.num_splits > 1) {
    const size_t pr = row * p.num_splits + blockIdx.y;
#pragma unroll
    for (int e = 0; e < PER; ++e)
      if (lane + 32 * e < p.vrank) p.part_o[pr * p.vrank + lane + 32 * e] = acc[e];
    if (lane == 0) { p.part_ml[2 * pr] = m; p.part_ml[2 * pr + 1] = l; }
    return;
  }
  const float inv = (l > 0.f ? 1.f / l : 0.f) * latent_gate<T>(p, row);
  T* op = static_cast<T*>(p.out) + row * p.ldo;
#pragma unroll
  for (int e = 0; e < PER; ++e)
    if (lane + 32 * e < p.vrank) op[lane + 32 * e] = from_f32<T>(acc[e] * inv);
}

// combine the partial results of split keys: one warp per query row
template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(LatParams p) {
  const int lane = threadIdx.x & 31, splits = p.num_splits;
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (row >= p.rows * p.heads || p.ctx_len[row / p.heads] <= 0) return;
  float m = -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, p.part_ml[2 * (static_cast<size_t>(row) * splits + s)]);
  float l = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float* ml = p.part_ml + 2 * (static_cast<size_t>(row) * splits + s);
    l += ml[0] == -INFINITY ? 0.f : ml[1] * expf(ml[0] - m);
  }
  const float inv = (l > 0.f ? 1.f / l : 0.f) * latent_gate<T>(p, row);
  for (int i = lane; i < p.vrank; i += 32) {
    float a = 0.f;
    for (int s = 0; s < splits; ++s) {
      const size_t pr = static_cast<size_t>(row) * splits + s;
      const float ms = p.part_ml[2 * pr];
      if (ms != -INFINITY) a = fmaf(p.part_o[pr * p.vrank + i], expf(ms - m), a);
    }
    static_cast<T*>(p.out)[static_cast<size_t>(row) * p.ldo + i] = from_f32<T>(a * inv);
  }
}

// Visible latents of every prefill entry, packed page by page: block b copies one 16-token page to dense rows 16 b .. 16 b + 15
// and enters b into the entry's scratch page table.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* __restrict__ pool, const int* __restrict__ page_table,
                                                            const int* __restrict__ ctx_len, const int* __restrict__ cu_q, int entries, int max_pages,
                                                            int64_t num_pages, int window, int vecs, uint4* __restrict__ out,
                                                            int* __restrict__ scratch_table, int* status) {
  int b = blockIdx.x, e = 0, pi = -1;
  for (; e < entries; ++e) {
    const int ctx = ctx_len[e], start = ctx - (cu_q[e + 1] - cu_q[e]);
    const int lo = (window > 0 ? max(0, start - window + 1) : 0) / kLatPage, n = (ctx + kLatPage - 1) / kLatPage - lo;
    if (b < n) { pi = lo + b; break; }
    b -= n;
  }
  if (pi < 0 || pi >= max_pages) return;
  int64_t page = page_table[static_cast<size_t>(e) * max_pages + pi];
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, kStatusIndexOutOfRange);
    page = 0;
  }
  if (threadIdx.x == 0) scratch_table[static_cast<size_t>(e) * max_pages + pi] = blockIdx.x;
  const uint4* src = pool + static_cast<size_t>(page) * kLatPage * vecs;
  uint4* dst = out + static_cast<size_t>(blockIdx.x) * kLatPage * vecs;
  for (int i = threadIdx.x; i < kLatPage * vecs; i += blockDim.x) dst[i] = src[i];
}

template <typename T>
static int launch_warp(const LatParams& p, cudaStream_t stream) {
  const long long blocks = p.cu_q == nullptr ? (static_cast<long long>(p.rows) * p.heads + kLatWarps - 1) / kLatWarps
                                             : static_cast<long long>(p.num_tiles) * ((64 * p.heads + kLatWarps - 1) / kLatWarps);
  const dim3 grid(static_cast<unsigned>(blocks), p.num_splits);
  if (p.rank <= 64) latent_attention_warp_kernel<T, 2><<<grid, kLatWarps * 32, 0, stream>>>(p);
  else if (p.rank <= 128) latent_attention_warp_kernel<T, 4><<<grid, kLatWarps * 32, 0, stream>>>(p);
  else if (p.rank <= 256) latent_attention_warp_kernel<T, 8><<<grid, kLatWarps * 32, 0, stream>>>(p);
  else if (p.rank <= 512) latent_attention_warp_kernel<T, 16><<<grid, kLatWarps * 32, 0, stream>>>(p);
  else if (p.rank <= 1024) latent_attention_warp_kernel<T, 32><<<grid, kLatWarps * 32, 0, stream>>>(p);
  else return -2;
  return static_cast<int>(cudaGetLastError());
}

}  // namespace ogb

using namespace ogb;

static int g_latent_tc = -1;    // -1: read OGB_LATENT_TC once (default on)
static bool use_tensor_cores() {
  if (g_latent_tc < 0) {
    const char* e = getenv("OGB_LATENT_TC");
    g_latent_tc = (e != nullptr && e[0] == '0') ? 0 : 1;
  }
  return g_latent_tc == 1;
}

// 1 / 0: bf16 latent attention on the tensor cores or on the warp kernel (comparisons); returns the old setting.
extern "C" int ogb_latent_set_tc(int on) {
  const int old = use_tensor_cores() ? 1 : 0;
  g_latent_tc = on ? 1 : 0;
  return old;
}

extern "C" int ogb_latent_attention(const void* q, void* out, const void* pool, const int* page_table, const int* ctx_len, const int* cu_q,
                                    const int* tile_seq, const int* tile_q0, const void* gate, int rows, int heads, int rank, int vrank, int ldq,
                                    int ldo, int ldp, int ldg, int max_pages, int num_tiles, int64_t num_pages, int window, float scale,
                                    int num_splits, float* part_o, float* part_ml, int* counters, int elem, int* status, void* stream) {
  if (rows <= 0 || (cu_q != nullptr && num_tiles <= 0)) return 0;
  if (heads <= 0 || rank <= 0 || rank > ldq || rank > ldp || vrank <= 0 || vrank > rank || vrank > ldo) return -3;
  if (cu_q != nullptr) num_splits = 1;
  if (num_splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -3;
  LatParams p{q, out, pool, page_table, ctx_len, cu_q, tile_seq, tile_q0, gate, rows, heads, rank, vrank, ldq, ldo, ldp, ldg, max_pages, num_tiles, window,
              num_splits < 1 ? 1 : num_splits, num_pages, scale, part_o, part_ml, counters, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int rc = -2;                                    // the tensor-core kernel declines what it cannot take
  if (elem == kElemBF16 && use_tensor_cores()) {
    rc = launch_latent_tc(p, s);
    if (rc == 0 && counters != nullptr) return 0;
  }
  if (rc == -2) rc = elem == kElemBF16 ? launch_warp<__nv_bfloat16>(p, s) : elem == kElemF32 ? launch_warp<float>(p, s) : -3;
  if (rc != 0 || p.num_splits == 1) return rc;
  const int blocks = (rows * heads + 3) / 4;
  if (elem == kElemBF16) latent_combine_kernel<__nv_bfloat16><<<blocks, 128, 0, s>>>(p);
  else latent_combine_kernel<float><<<blocks, 128, 0, s>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// Packs the visible latents (bf16, rows of ldp values, ldp a multiple of 8) of the prefill entries for an expansion to keys and
// values; `blocks` = their pages in total.
extern "C" int ogb_latent_gather(const void* pool, const int* page_table, const int* ctx_len, const int* cu_q, int entries, int max_pages,
                                 int64_t num_pages, int window, int ldp, int blocks, void* out, int* scratch_table, int* status, void* stream) {
  if (blocks <= 0 || entries <= 0) return 0;
  if (ldp % 8 != 0) return -3;
  latent_gather_kernel<<<blocks, 128, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const uint4*>(pool), page_table, ctx_len, cu_q, entries,
                                                                             max_pages, num_pages, window, ldp / 8, static_cast<uint4*>(out),
                                                                             scratch_table, status);
  return static_cast<int>(cudaGetLastError());
}
