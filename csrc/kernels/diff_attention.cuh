// Parameters and output step shared by the differential attention kernels (diff_attention.cu, diff_attention_tc.cu).
//
// A head is two softmax maps over the same values: queries and keys come in pairs (map 1, map 2), o = a1 - lambda a2, and o is
// divided by its root mean square over the head's vdim values and scaled.  A KV page holds [2 * hkv][16][dp] keys (map fastest
// within a head), then [hkv][16][vp] values; dp and vp are the sizes padded to 8.
#pragma once
#include "hybrid.cuh"

namespace ogb {

constexpr int kDaPage = 16;

struct DiffParams {
  const void* q;           // [rows, ldq]: (head, map) at column (2 head + map) * dp
  void* out;               // [rows, ldo]: head at column head * vp
  const void* pool;
  const int* page_table;
  const int* ctx_len;
  const int* cu_q;         // null: every row is a decode row of its own
  const int* tile_seq;
  const int* tile_q0;
  int rows, num_tiles, max_pages;
  int64_t num_pages, page_elems;
  int hq, hkv, d, dv, dp, vp, ldq, ldo;
  int window, keep;        // window > 0: the last `window` keys and the first `keep`
  float scale, lambda, eps, gain;
  int num_splits;
  float* part_o;           // [rows][hkv chunks of 16 (map, head) rows][16][splits][vp]
  float* part_ml;
  int* counters;
  int* status;
};

OGB_DEVICE bool da_visible(const DiffParams& p, int key, int pos) {
  return key <= pos && (p.window <= 0 || key > pos - p.window || key < p.keep);
}
// first key of the gap between the kept tokens and the window whose page may be gone: pages [lo, hi) are never looked up
OGB_DEVICE int da_page_index(const DiffParams& p, int pi, int n_pages, int kv_lo) {
  pi = min(min(pi, n_pages - 1), p.max_pages - 1);
  if (p.window > 0) {
    const int lo = (p.keep + kDaPage - 1) / kDaPage, hi = kv_lo / kDaPage;
    if (pi >= lo && pi < hi) pi = hi;
  }
  return pi;
}

int launch_diff_decode(const DiffParams& p, cudaStream_t stream);      // -2: sizes it does not serve
int launch_diff_prefill_tc(const DiffParams& p, cudaStream_t stream);  // -2: sizes it does not serve

}  // namespace ogb
