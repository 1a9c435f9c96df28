// Mixture-of-experts routing and data movement around the grouped tcgen05 GEMM.
//
// Reference counterparts: qmoe_route (one CTA per token row, k rounds of block-wide argmax on
// total-order keys, crates/onnx-runtime-ep-cuda/src/kernels/qmoe.rs:56-120), qmoe_group_{init,count,
// prefix,assign} and qmoe_gather_* (qmoe_grouping.rs), qmoe_combine_* (qmoe.rs:22-47).  Router
// semantics follow the metadata's MixtureOfExpertsSpec (score_function softmax, selection top_k,
// normalize_weights; crates/onnx-genai-metadata/src/schema/hardware.rs:64-98).
//   moe_route_topk   one warp per token: softmax over the expert logits, k rounds of warp argmax with
//                    lowest-index tie break, optional renormalisation over the chosen k
//   moe_count / moe_plan / moe_assign   routes -> per-expert counts -> offsets, the 128-row tile table
//                    the grouped GEMM walks, and each route's row in the expert-sorted order
//   moe_gather_rows  activations copied into expert-sorted order
//   moe_combine      out[t] (+)= sum_j w[t,j] * y[row of route (t,j)], j in fixed order (deterministic)
// All routing state stays on the device; nothing here synchronises with the host.
#include "common.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kMaxExperts = 256;

// Softmax scores: `bias` (fp32, or null) is added to the logits, and the choice compares logits, which order experts as their scores do.
// Sigmoid scores: the choice compares scores plus `bias`, the weights are the scores (over their sum + 1e-20 when renormalised).
// `groups` > 1: experts form that many equal groups of neighbours, a group scores as its best expert (`group_best` 2: as the sum of its
// best two), and only the `keep` best groups can be chosen from.
template <typename T>
__global__ void __launch_bounds__(256) moe_route_topk_kernel(const T* __restrict__ logits, const float* __restrict__ bias, int* __restrict__ topk_ids,
                                                             float* __restrict__ topk_w,
                                                             int tokens, int experts, int k, int renormalize, int ld, int groups, int keep, bool sigmoid,
                                                             int group_best) {
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  __shared__ float s_group[8][kMaxExperts];
  if (warp >= tokens) return;
  constexpr int PER = kMaxExperts / 32;
  float v[PER];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    v[i] = -INFINITY;
    if (e < experts) {
      const float z = static_cast<float>(logits[static_cast<size_t>(warp) * ld + e]);
      v[i] = (sigmoid ? 1.f / (1.f + expf(-z)) : z) + (bias != nullptr ? bias[e] : 0.f);
    }
    mx = fmaxf(mx, v[i]);
  }
  float inv = 1.f;
  if (!sigmoid) {
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) sum += (i * 32 + lane < experts) ? expf(v[i] - mx) : 0.f;
    sum = warp_sum(sum);
    inv = 1.f / sum;
  }
  // the largest of a set of values with the lowest index among equals (-inf: not a candidate)
  auto best_of = [&](const float (&x)[PER], int count, float& best, int& at) {
    best = -INFINITY;
    at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = i * 32 + lane;
      if (e < count && x[i] > best) { best = x[i]; at = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oe < at)) { best = ob; at = oe; }
    }
  };
  if (groups > 1 && keep < groups) {
    float* s = s_group[threadIdx.x >> 5];
    const int size = experts / groups;
#pragma unroll
    for (int i = 0; i < PER; ++i) s[i * 32 + lane] = v[i];
    __syncwarp();
    float gs[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int g = i * 32 + lane;
      gs[i] = -INFINITY;
      if (g < groups) {
        float second = -INFINITY;
        for (int e = 0; e < size; ++e) {
          const float x = s[g * size + e];
          second = fmaxf(second, fminf(gs[i], x));
          gs[i] = fmaxf(gs[i], x);
        }
        if (group_best > 1 && size > 1) gs[i] += second;
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < PER; ++i) s[i * 32 + lane] = 0.f;      // 1: the group stays
    __syncwarp();
    for (int r = 0; r < keep; ++r) {
      float best;
      int at;
      best_of(gs, groups, best, at);
      if (lane == 0 && at < groups) s[at] = 1.f;
#pragma unroll
      for (int i = 0; i < PER; ++i)
        if (i * 32 + lane == at) gs[i] = -INFINITY;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = i * 32 + lane;
      if (e < experts && s[e / size] == 0.f) v[i] = -INFINITY;
    }
  }
  float chosen_sum = 0.f;
  float my_w = 0.f;
  int my_id = 0;
  for (int r = 0; r < k; ++r) {
    float best;
    int best_e;
    best_of(v, experts, best, best_e);
    if (sigmoid) {
      const float z = best_e < experts ? static_cast<float>(logits[static_cast<size_t>(warp) * ld + best_e]) : -INFINITY;
      best = 1.f / (1.f + expf(-z));
    } else {
      best = expf(best - mx);
    }
    if (lane == r) { my_w = best; my_id = best_e; }
    chosen_sum += best;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (i * 32 + lane == best_e) v[i] = -INFINITY;           // remove the winner
  }
  if (lane < k) {
    topk_ids[static_cast<size_t>(warp) * k + lane] = my_id;
    topk_w[static_cast<size_t>(warp) * k + lane] = renormalize ? my_w / (chosen_sum + (sigmoid ? 1e-20f : 0.f)) : my_w * inv;
  }
}

// counts[e] = routes to local expert e (ids outside [e0, e0 + experts) are other ranks' experts)
__global__ void moe_count_kernel(const int* __restrict__ topk_ids, int* __restrict__ counts, int routes, int e0, int experts) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= routes) return;
  const int e = topk_ids[i] - e0;
  if (e >= 0 && e < experts) atomicAdd(&counts[e], 1);
}

// One CTA: offsets[e] (exclusive prefix), tile table {e, first row, end row, 0} per 128 rows, number of
// tiles, and cursor reset.  meta = {num_mtiles, total_rows}.
__global__ void moe_plan_kernel(const int* __restrict__ counts, int* __restrict__ offsets, int* __restrict__ cursor,
                                int* __restrict__ tile_tab, int* __restrict__ meta, int experts, int max_mtiles) {
  __shared__ int s_off[kMaxExperts + 1];
  __shared__ int s_tile[kMaxExperts + 1];
  if (threadIdx.x == 0) {
    int o = 0, t = 0;
    for (int e = 0; e < experts; ++e) {
      s_off[e] = o;
      s_tile[e] = t;
      o += counts[e];
      t += (counts[e] + 127) / 128;
    }
    s_off[experts] = o;
    s_tile[experts] = t;
    meta[0] = min(t, max_mtiles);
    meta[1] = o;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += blockDim.x) {
    offsets[e] = s_off[e];
    cursor[e] = 0;
    const int end = s_off[e + 1];
    int t = s_tile[e];
    for (int r = s_off[e]; r < end && t < max_mtiles; r += 128, ++t) {
      tile_tab[4 * t] = e;
      tile_tab[4 * t + 1] = r;
      tile_tab[4 * t + 2] = end;
      tile_tab[4 * t + 3] = 0;
    }
  }
  if (threadIdx.x == 0) offsets[experts] = s_off[experts];
}

__global__ void moe_assign_kernel(const int* __restrict__ topk_ids, const int* __restrict__ offsets, int* __restrict__ cursor,
                                  int* __restrict__ sorted_route, int* __restrict__ route_pos, int routes, int e0, int experts) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= routes) return;
  const int e = topk_ids[i] - e0;
  if (e < 0 || e >= experts) { route_pos[i] = -1; return; }
  const int pos = offsets[e] + atomicAdd(&cursor[e], 1);
  sorted_route[pos] = i;
  route_pos[i] = pos;
}

__global__ void moe_gather_rows_kernel(const uint4* __restrict__ x, const int* __restrict__ sorted_route, const int* __restrict__ meta,
                                       uint4* __restrict__ xs, int k, int vecs) {
  const int pos = blockIdx.x;
  if (pos >= meta[1]) return;
  const int token = sorted_route[pos] / k;
  const uint4* src = x + static_cast<size_t>(token) * vecs;
  uint4* dst = xs + static_cast<size_t>(pos) * vecs;
  for (int i = threadIdx.x; i < vecs; i += blockDim.x) dst[i] = src[i];
}

__global__ void moe_combine_kernel(const __nv_bfloat16* __restrict__ ys, const int* __restrict__ route_pos,
                                   const float* __restrict__ topk_w, __nv_bfloat16* __restrict__ out, int k, int hidden,
                                   int accumulate) {
  const int t = blockIdx.x;
  for (int i = threadIdx.x; i < hidden / 8; i += blockDim.x) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (accumulate) {
      const uint4 v = reinterpret_cast<const uint4*>(out + static_cast<size_t>(t) * hidden)[i];
      float2 f;
      f = unpack_bf16(v.x); acc[0] = f.x; acc[1] = f.y;
      f = unpack_bf16(v.y); acc[2] = f.x; acc[3] = f.y;
      f = unpack_bf16(v.z); acc[4] = f.x; acc[5] = f.y;
      f = unpack_bf16(v.w); acc[6] = f.x; acc[7] = f.y;
    }
    for (int j = 0; j < k; ++j) {
      const int pos = route_pos[static_cast<size_t>(t) * k + j];
      if (pos < 0) continue;   // the route's expert lives on another rank
      const float w = topk_w[static_cast<size_t>(t) * k + j];
      const uint4 v = reinterpret_cast<const uint4*>(ys + static_cast<size_t>(pos) * hidden)[i];
      float2 f;
      f = unpack_bf16(v.x); acc[0] += w * f.x; acc[1] += w * f.y;
      f = unpack_bf16(v.y); acc[2] += w * f.x; acc[3] += w * f.y;
      f = unpack_bf16(v.z); acc[4] += w * f.x; acc[5] += w * f.y;
      f = unpack_bf16(v.w); acc[6] += w * f.x; acc[7] += w * f.y;
    }
    reinterpret_cast<uint4*>(out + static_cast<size_t>(t) * hidden)[i] =
        make_uint4(pack_bf16(acc[0], acc[1]), pack_bf16(acc[2], acc[3]), pack_bf16(acc[4], acc[5]), pack_bf16(acc[6], acc[7]));
  }
}

}  // namespace ogb

using namespace ogb;

template <typename T>
static int route_topk(const T* logits, const float* bias, int* topk_ids, float* topk_w, int tokens, int experts, int k, int renormalize, int ld, int groups, int keep,
                      bool sigmoid, int group_best, void* stream) {
  if (tokens <= 0) return 0;
  if (experts > kMaxExperts || k > 32 || k > experts) return -3;
  if (groups < 1 || experts % groups != 0 || keep < 1 || keep > groups || k > keep * (experts / groups)) return -3;
  const int warps_per_block = 8;
  const int blocks = (tokens + warps_per_block - 1) / warps_per_block;
  moe_route_topk_kernel<T><<<blocks, warps_per_block * 32, 0, static_cast<cudaStream_t>(stream)>>>(logits, bias, topk_ids, topk_w, tokens,
                                                                                                 experts, k, renormalize, ld, groups, keep, sigmoid,
                                                                                                 group_best);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int ogb_moe_route_topk(const void* router_logits, int* topk_ids, float* topk_w, int tokens, int experts, int k,
                                  int renormalize, int ld, void* stream) {
  return route_topk(static_cast<const __nv_bfloat16*>(router_logits), nullptr, topk_ids, topk_w, tokens, experts, k, renormalize, ld, 1, 1, false, 1, stream);
}

// fp32 logits and bias (or null); `groups` equal groups of experts of which the `keep` best can be chosen from (1, 1: all).  sigmoid,
// group_best: how experts and groups score (moe_route_topk_kernel).
extern "C" int ogb_moe_route_grouped(const float* router_logits, const float* bias, int* topk_ids, float* topk_w, int tokens, int experts, int k, int renormalize,
                                     int ld, int groups, int keep, int sigmoid, int group_best, void* stream) {
  if (group_best < 1 || group_best > 2) return -3;
  return route_topk(router_logits, bias, topk_ids, topk_w, tokens, experts, k, renormalize, ld, groups, keep, sigmoid != 0, group_best, stream);
}

// counts must be zero on entry (the caller clears it); e0 = first expert owned by this rank.
extern "C" int ogb_moe_permute(const int* topk_ids, int* counts, int* offsets, int* cursor, int* sorted_route, int* route_pos,
                               int* tile_tab, int* meta, int tokens, int k, int e0, int experts, int max_mtiles, void* stream) {
  if (tokens <= 0) return 0;
  if (experts > kMaxExperts) return -3;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int routes = tokens * k;
  OGB_CUDA_CHECK(cudaMemsetAsync(counts, 0, sizeof(int) * experts, st));
  moe_count_kernel<<<(routes + 255) / 256, 256, 0, st>>>(topk_ids, counts, routes, e0, experts);
  moe_plan_kernel<<<1, 256, 0, st>>>(counts, offsets, cursor, tile_tab, meta, experts, max_mtiles);
  moe_assign_kernel<<<(routes + 255) / 256, 256, 0, st>>>(topk_ids, offsets, cursor, sorted_route, route_pos, routes, e0, experts);
  return static_cast<int>(cudaGetLastError());
}

static int gather_rows(const void* x, const int* sorted_route, const int* meta, void* xs, int max_routes, int k, int row_bytes, void* stream) {
  if (max_routes <= 0) return 0;
  if (row_bytes % 16) return -3;
  const int vecs = row_bytes / 16;
  moe_gather_rows_kernel<<<max_routes, vecs < 128 ? (vecs + 31) / 32 * 32 : 128, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(x), sorted_route, meta, static_cast<uint4*>(xs), k, vecs);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int ogb_moe_gather_rows(const void* x, const int* sorted_route, const int* meta, void* xs, int max_routes, int k,
                                   int hidden, void* stream) {
  return gather_rows(x, sorted_route, meta, xs, max_routes, k, 2 * hidden, stream);
}
// Rows of any type, row_bytes a multiple of 16.
extern "C" int ogb_moe_gather_bytes(const void* x, const int* sorted_route, const int* meta, void* xs, int max_routes, int k, int row_bytes,
                                    void* stream) {
  return gather_rows(x, sorted_route, meta, xs, max_routes, k, row_bytes, stream);
}

extern "C" int ogb_moe_combine(const void* ys, const int* route_pos, const float* topk_w, void* out, int tokens, int k,
                               int hidden, int accumulate, void* stream) {
  if (tokens <= 0) return 0;
  if (hidden % 8) return -3;
  moe_combine_kernel<<<tokens, 128, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const __nv_bfloat16*>(ys), route_pos, topk_w, static_cast<__nv_bfloat16*>(out), k, hidden, accumulate);
  return static_cast<int>(cudaGetLastError());
}
