// Parameter block shared by the latent-attention kernels.
#pragma once
#include "hybrid.cuh"

namespace ogb {

constexpr int kLatPage = 16;

struct LatParams {
  const void* q;          // [rows * heads, ldq]: rows of the launch's region (decode rows, or the packed prefill rows)
  void* out;              // same shape
  const void* pool;       // [pages, 16, ldp]
  const int* page_table;  // [entries, max_pages]
  const int* ctx_len;
  const int* cu_q;        // null: decode (entry = row)
  const int* tile_seq;
  const int* tile_q0;
  int rows, heads, rank, ldq, ldp, max_pages, num_tiles, window, num_splits;
  int64_t num_pages;
  float scale;
  float *part_o, *part_ml;
  int* counters;          // zeroed words, one per (decode row, 16 heads): the last split of a row merges them (null: a second kernel does)
  int* status;
};

// Tensor-core launch; -2 when it does not take the call (rank above 512, alignment).
int launch_latent_tc(const LatParams& p, cudaStream_t stream);
// Decode rows (latent_decode.cu); launch_latent_tc hands them over.  It merges split keys itself when it has counters.
int launch_latent_decode(const LatParams& p, cudaStream_t stream);

}  // namespace ogb
