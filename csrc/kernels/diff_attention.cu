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

namespace ogb {
int launch_diff_decode(const DiffParams&, cudaStream_t) { return -2; }
int launch_diff_prefill_tc(const DiffParams&, cudaStream_t) { return -2; }
}
