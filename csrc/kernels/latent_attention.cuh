// Parameter block shared by the latent-attention kernels.
#pragma once
#include "hybrid.cuh"

namespace ogb {

constexpr int kLatPage = 16;

struct LatParams {
  const void* q;          // [rows * heads, ldq]: rows of the launch's region (decode rows, or the packed prefill rows)
  void* out;              // [rows * heads, ldo]
  const void* pool;       // [pages, 16, ldp]: the first `rank` values of a row are the key, the first `vrank` of them the value
  const int* page_table;  // [entries, max_pages]
  const int* ctx_len;
  const int* cu_q;        // null: decode (entry = row)
  const int* tile_seq;
  const int* tile_q0;
  const void* gate;       // [rows, ldg] or null: a head's output is multiplied by the sigmoid of its column
  int rows, heads, rank, vrank, ldq, ldo, ldp, ldg, max_pages, num_tiles, window, num_splits;
  int64_t num_pages;
  float scale;
  float *part_o, *part_ml;
  int* counters;          // zeroed words, one per (decode row, 16 heads): the last split of a row merges them (null: a second kernel does)
  int* status;
};

// Factor of row (token, head) `row` of the launch's region.
template <typename T>
OGB_DEVICE float latent_gate(const LatParams& p, int64_t row) {
  if (p.gate == nullptr) return 1.f;
  return 1.f / (1.f + expf(-to_f32<T>(static_cast<const T*>(p.gate)[row / p.heads * p.ldg + row % p.heads])));
}

// Tensor-core launch; -2 when it does not take the call (keys above 576 or values above 512 columns, alignment).
int launch_latent_tc(const LatParams& p, cudaStream_t stream);
// Decode rows (latent_decode.cu); launch_latent_tc hands them over.  It merges split keys itself when it has counters.
int launch_latent_decode(const LatParams& p, cudaStream_t stream);

}  // namespace ogb
