// Parameters and scores shared by the kernels of attention over keys that are the values too (tied_attention.cu, tied_attention_tc.cu).
//
// A KV page holds [hkv][16][dp] keys as projected, which are the values as they are, then 16 fp32 factors, one per token: what is left
// of the keys' norm (its weight is folded into the queries) times the scale of the scores.  A score is
//
//   s = (q . k) factor,  cap tanh(s) where there is a cap (the factor then has 1 / cap in it),  less slope[head] times the distance
//
// and the softmax's denominator also holds exp(sink[head]).
#pragma once
#include "hybrid.cuh"

namespace ogb {

constexpr int kTaPage = 16;

struct TiedParams {
  const void* q;           // [rows, ldq]: head at column head * dp
  void* out;               // [rows, ldo]: head at column head * dp
  const void* pool;
  const int* page_table;
  const int* ctx_len;
  const int* cu_q;         // null: every row is a decode row of its own
  const int* tile_seq;
  const int* tile_q0;
  const void* gate;        // [rows, ldg] or null: a head's output is multiplied by the sigmoid of its column
  const float* slope;      // [hq] or null
  const float* sink;       // [hq] or null
  int rows, num_tiles, max_pages;
  int64_t num_pages, page_elems;
  int hq, hkv, d, dp, ldq, ldo, ldg, window;
  float cap;
  int num_splits;
  float* part_o;           // [rows][hkv chunks of 16 heads][16][splits][dp]
  float* part_ml;
  int* counters;
  int* status;
};

// page index of a sequence: pages the window has passed may be gone, pages behind the last do not exist
OGB_DEVICE int ta_page_index(const TiedParams& p, int pi, int n_pages, int kv_lo) {
  return max(min(min(pi, n_pages - 1), p.max_pages - 1), kv_lo / kTaPage);
}
OGB_DEVICE float ta_sink(const TiedParams& p, int head) { return p.sink != nullptr ? p.sink[head] : -INFINITY; }
OGB_DEVICE float ta_slope(const TiedParams& p, int head) { return p.slope != nullptr ? p.slope[head] : 0.f; }
template <typename T>
OGB_DEVICE float ta_gate(const TiedParams& p, int64_t row, int head) {
  if (p.gate == nullptr) return 1.f;
  return 1.f / (1.f + expf(-to_f32<T>(static_cast<const T*>(p.gate)[row * p.ldg + head])));
}

int launch_tied_decode(const TiedParams& p, cudaStream_t stream);      // -2: sizes it does not serve
int launch_tied_prefill_tc(const TiedParams& p, cudaStream_t stream);  // -2: sizes it does not serve

}  // namespace ogb
