// Row-wise kernels of models with a mixer per layer: hyper-connected residual streams with Dynamic-Tanh norms and token shift, one
// residual stream with RMS norms and input convolutions, embeddings, latent KV pages; plus the fp32 matrix product of the 32-bit
// engine.
//
// hyper_step is the one pass between two matrix products: it folds a sublayer's output y into the residual streams
// (x_t <- sum_s mix[s][t] x_s + out[t] y), reads the next sublayer's input (u = sum_s in[s] x_s), applies the
// Dynamic-Tanh norm (tanh(alpha u) w + b) and, where the mixer wants it, the token shift (h + (h_before - h) amount).
// Everything is elementwise in the column, so a thread keeps its columns and walks a few tokens; the row before its
// first token is computed again from the streams the pass reads (the streams are double buffered), or comes from the
// sequence's state.  Streams, norm and shift are fp32 whatever the activation type.
#include <algorithm>

#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kHsThreads = 256;
constexpr int kHsRows = 16;                   // tokens a thread walks (a 64-row scheduler tile is four such groups)

struct HyperParams {
  const float* x_in;       // [rows, S, W]
  float* x_out;            // [rows, S, W] or null (nothing to write back)
  const void* y;           // [rows, ldy] or null (no update)
  const float *mix, *out_w, *in_w;             // [S, S] (from, to), [S], [S] (null: ones)
  const float *alpha, *w, *b;                  // Dynamic-Tanh norm (alpha null: none)
  const float* shift;      // [W] or null
  float* prev;             // [slots, W] state of the shift: h of the sequence's last computed token
  void* h;                 // [rows, ldh] or null
  const int* gather;       // row r of h comes from row gather[r] (final norm of the rows that sample)
  int rows, total_rows, S, W, ldy, ldh;
  int rows_per_block;      // without the shift
  StepRows sr;
  int* status;
};

template <typename T, int SMAX, int V>
struct HyperCol {
  const HyperParams& p;
  int c;                                       // first column of this thread
  float mix[SMAX][SMAX], out_w[SMAX], in_w[SMAX];
  float alpha, w[V], b[V];

  OGB_DEVICE HyperCol(const HyperParams& p_, int c_) : p(p_), c(c_) {
#pragma unroll
    for (int s = 0; s < SMAX; ++s) {
      const bool live = s < p.S;
      in_w[s] = live ? (p.in_w != nullptr ? p.in_w[s] : 1.f) : 0.f;
      out_w[s] = (live && p.y != nullptr) ? p.out_w[s] : 0.f;
#pragma unroll
      for (int t = 0; t < SMAX; ++t) mix[s][t] = (live && t < p.S && p.y != nullptr) ? p.mix[s * p.S + t] : 0.f;
    }
    alpha = p.alpha != nullptr ? *p.alpha : 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      w[i] = p.alpha != nullptr ? p.w[c + i] : 1.f;
      b[i] = p.alpha != nullptr ? p.b[c + i] : 0.f;
    }
  }

  // streams of row t after the update, normed read-out in hv
  OGB_DEVICE void row(int t, bool write, float (&hv)[V]) const {
    float x[SMAX][V], y[V], u[V];
    const float* src = p.x_in + static_cast<size_t>(t) * p.S * p.W + c;
#pragma unroll
    for (int s = 0; s < SMAX; ++s)
      if (s < p.S) load_vec<V>(src + static_cast<size_t>(s) * p.W, x[s]);
    if (p.y != nullptr) {
      load_vec<V>(static_cast<const T*>(p.y) + static_cast<size_t>(t) * p.ldy + c, y);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float n[SMAX];
#pragma unroll
        for (int q = 0; q < SMAX; ++q) {
          n[q] = out_w[q] * y[i];
#pragma unroll
          for (int s = 0; s < SMAX; ++s)
            if (s < p.S) n[q] = fmaf(mix[s][q], x[s][i], n[q]);
        }
#pragma unroll
        for (int q = 0; q < SMAX; ++q) x[q][i] = n[q];
      }
      if (write && p.x_out != nullptr) {
        float* dst = p.x_out + static_cast<size_t>(t) * p.S * p.W + c;
#pragma unroll
        for (int s = 0; s < SMAX; ++s)
          if (s < p.S) store_vec<V>(dst + static_cast<size_t>(s) * p.W, x[s]);
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      u[i] = 0.f;
#pragma unroll
      for (int s = 0; s < SMAX; ++s)
        if (s < p.S) u[i] = fmaf(in_w[s], x[s][i], u[i]);
      hv[i] = p.alpha != nullptr ? fmaf(tanhf(alpha * u[i]), w[i], b[i]) : u[i];
    }
  }
};

// rows are independent: no shift
template <typename T, int SMAX, int V>
__global__ void __launch_bounds__(kHsThreads) hyper_rows_kernel(HyperParams p) {
  const int c = (blockIdx.y * kHsThreads + threadIdx.x) * V;
  if (c >= p.W) return;
  HyperCol<T, SMAX, V> col(p, c);
  const int r0 = blockIdx.x * p.rows_per_block;
#pragma unroll 2
  for (int j = 0; j < p.rows_per_block; ++j) {
    const int r = r0 + j;
    if (r >= p.rows) return;
    int t = r;
    if (p.gather != nullptr) {
      t = p.gather[r];
      if (t < 0 || t >= p.total_rows) {
        if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
        t = 0;
      }
    }
    float hv[V];
    col.row(t, true, hv);
    if (p.h != nullptr) store_vec<V>(static_cast<T*>(p.h) + static_cast<size_t>(r) * p.ldh + c, hv);
  }
}

// with the token shift: a block is one decode row or kHsRows rows of one prefill chunk
template <typename T, int SMAX, int V>
__global__ void __launch_bounds__(kHsThreads) hyper_shift_kernel(HyperParams p) {
  const int c = (blockIdx.y * kHsThreads + threadIdx.x) * V;
  if (c >= p.W) return;
  const StepRows& sr = p.sr;
  int entry, base, n, j0;                      // sequence entry, its first row, its rows, first row of this block within them
  if (static_cast<int>(blockIdx.x) < sr.num_decode) {
    entry = blockIdx.x; base = blockIdx.x; n = 1; j0 = 0;
  } else {
    const int g = blockIdx.x - sr.num_decode;
    const int tile = g / (64 / kHsRows);
    const int s = sr.tile_seq[tile];
    entry = sr.num_decode + s;
    base = sr.num_decode + sr.cu_q[s];
    n = sr.cu_q[s + 1] - sr.cu_q[s];
    j0 = sr.tile_q0[tile] + (g % (64 / kHsRows)) * kHsRows;
    if (j0 >= n) return;
  }
  int slot = sr.state_slot[entry];
  if (slot >= sr.num_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    slot = -1;
  }
  HyperCol<T, SMAX, V> col(p, c);
  float amount[V], before[V], hv[V], o[V];
  load_vec<V>(p.shift + c, amount);
  float* state = slot >= 0 ? p.prev + static_cast<size_t>(slot) * p.W + c : nullptr;
#pragma unroll
  for (int i = 0; i < V; ++i) before[i] = 0.f;
  if (j0 > 0) {
    col.row(base + j0 - 1, false, before);
  } else {
    if (state != nullptr && sr.ctx_len[entry] > n) load_vec<V>(state, before);
    // this block also leaves the chunk's last h behind: it is the only one that reads the slot, so the order is safe
    if (state != nullptr && n > kHsRows) {
      col.row(base + n - 1, false, hv);
      store_vec<V>(state, hv);
    }
  }
  const int j1 = min(j0 + kHsRows, n);
#pragma unroll 2
  for (int j = j0; j < j1; ++j) {
    col.row(base + j, true, hv);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      o[i] = fmaf(before[i] - hv[i], amount[i], hv[i]);
      before[i] = hv[i];
    }
    store_vec<V>(static_cast<T*>(p.h) + static_cast<size_t>(base + j) * p.ldh + c, o);
  }
  if (state != nullptr && j0 == 0 && n <= kHsRows) store_vec<V>(state, before);
}

template <typename T, int SMAX, int V>
static int launch_hyper(const HyperParams& p, cudaStream_t stream) {
  const int cols = (p.W + V * kHsThreads - 1) / (V * kHsThreads);
  if (p.shift != nullptr) {
    const int blocks = p.sr.num_decode + p.sr.num_tiles * (64 / kHsRows);
    hyper_shift_kernel<T, SMAX, V><<<dim3(blocks, cols), kHsThreads, 0, stream>>>(p);
  } else {
    hyper_rows_kernel<T, SMAX, V><<<dim3((p.rows + p.rows_per_block - 1) / p.rows_per_block, cols), kHsThreads, 0, stream>>>(p);
  }
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int V>
static int dispatch_hyper(const HyperParams& p, cudaStream_t stream) {
  if (p.S <= 2) return launch_hyper<T, 2, V>(p, stream);
  if (p.S <= 4) return launch_hyper<T, 4, V>(p, stream);
  return launch_hyper<T, 8, V>(p, stream);
}

// ------------------------------------------------------------------------------------------------------
// What a sublayer left for the residual: a row per token, or -- behind routed experts -- the weighted sum of the token's expert rows
// (sum_j weight[t][j] y[pos[t][j]]) and of a shared expert's row times the sigmoid of its gate, taken here so that it never
// exists in memory.  With res_gate the output reaches the residual as (output + y_bias) sigmoid(res_gate + res_bias).
// ------------------------------------------------------------------------------------------------------
struct SublayerOut {
  const void* y;           // [rows, ldy], or the expert rows; null: nothing
  const int* pos;          // [rows, k] or null
  const float* weight;     // [rows, k]
  const void* shared;      // [rows, lds] or null
  const float* gate;       // [rows, ldg]: logits
  const float* y_bias;     // [W] or null
  const void* res_gate;    // [rows, ldr] or null
  const float* res_bias;   // [W]
  int k, ldy, lds, ldg, ldr;
  int64_t y_rows;
};

// Outputs of rows t0 .. t0 + n - 1 (n <= NB) at this thread's columns (i * blockDim.x + threadIdx.x) * V of W.
template <typename T, int NB, int N, int V>
OGB_DEVICE void sublayer_rows(const SublayerOut& o, int t0, int n, int W, float (&y)[NB][N][V], int* status) {
#pragma unroll
  for (int b = 0; b < NB; ++b)
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) y[b][i][v] = 0.f;
  if (o.y == nullptr) return;
  auto add = [&](const void* base, int64_t row, int ld, float f, float (&acc)[N][V]) {
    const T* src = static_cast<const T*>(base) + row * ld;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) {
        float z[V];
        load_vec<V>(src + c, z);
#pragma unroll
        for (int v = 0; v < V; ++v) acc[i][v] = fmaf(f, z[v], acc[i][v]);
      }
    }
  };
  auto gate = [&]() {
    if (o.res_gate == nullptr) return;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c >= W) continue;
      float bias[V], yb[V];
      load_vec<V>(o.res_bias + c, bias);
#pragma unroll
      for (int v = 0; v < V; ++v) yb[v] = 0.f;
      if (o.y_bias != nullptr) load_vec<V>(o.y_bias + c, yb);
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        if (b >= n) continue;
        float z[V];
        load_vec<V>(static_cast<const T*>(o.res_gate) + static_cast<size_t>(t0 + b) * o.ldr + c, z);
#pragma unroll
        for (int v = 0; v < V; ++v) y[b][i][v] = (y[b][i][v] + yb[v]) / (1.f + expf(-(z[v] + bias[v])));
      }
    }
  };
  if (o.pos == nullptr) {
#pragma unroll
    for (int b = 0; b < NB; ++b)
      if (b < n) add(o.y, t0 + b, o.ldy, 1.f, y[b]);
    gate();
    return;
  }
  for (int j = 0; j < o.k; ++j) {
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      if (b >= n) continue;
      const size_t at = static_cast<size_t>(t0 + b) * o.k + j;
      const int row = o.pos[at];
      if (row < 0 || row >= o.y_rows) {
        if (threadIdx.x == 0) atomicOr(status, kStatusIndexOutOfRange);
        continue;
      }
      add(o.y, row, o.ldy, o.weight[at], y[b]);
    }
  }
  if (o.shared != nullptr) {
#pragma unroll
    for (int b = 0; b < NB; ++b)
      if (b < n) add(o.shared, t0 + b, o.lds, 1.f / (1.f + expf(-o.gate[static_cast<size_t>(t0 + b) * o.ldg])), y[b]);
  }
  gate();
}

// sums over the block of NB values a thread; `red` [2][NB][32] alternates with `parity`, so one barrier a call is enough
template <int NB>
OGB_DEVICE void block_sums(float (&v)[NB], float (&red)[2][NB][32], int parity) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
#pragma unroll
  for (int b = 0; b < NB; ++b) {
    v[b] = warp_sum(v[b]);
    if (lane == 0) red[parity][b][warp] = v[b];
  }
  __syncthreads();
#pragma unroll
  for (int b = 0; b < NB; ++b) v[b] = warp_sum(lane < warps ? red[parity][b][lane] : 0.f);
}

// 1 / root mean square of every one of `groups` equal parts of a row of W columns, V of which a thread holds at (i * blockDim.x +
// threadIdx.x) * V: `part` [W / V] and `inv` [groups] are shared memory, in which the thread finds the factors of its columns
// (group_of) after the call.  A part is a multiple of V.
template <int N, int V>
OGB_DEVICE void group_factors(const float (&x)[N][V], int W, int groups, float eps, float* part, float* inv) {
  const int units = W / V, per = units / groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  __syncthreads();                             // the arrays may still be read from the call before
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int u = i * blockDim.x + threadIdx.x;
    float ss = 0.f;
#pragma unroll
    for (int v = 0; v < V; ++v) ss = fmaf(x[i][v], x[i][v], ss);
    if (u < units) part[u] = ss;
  }
  __syncthreads();
  for (int g = warp; g < groups; g += warps) {
    float a = 0.f;
    for (int u = lane; u < per; u += 32) a += part[g * per + u];
    a = warp_sum(a);
    if (lane == 0) inv[g] = 1.f / sqrtf(a / static_cast<float>(per * V) + eps);
  }
  __syncthreads();
}
// shared memory of group_factors: part and inv of `rows` rows
inline size_t group_bytes(int W, int V, int groups, int rows) { return groups > 1 ? static_cast<size_t>(rows) * (W / V + groups) * sizeof(float) : 0; }

// ------------------------------------------------------------------------------------------------------
// norm_step is the pass between two products for designs with one residual stream:
//
//   x <- x + rms(y) post        h = rms(x) w
//
// Without `post` the output is added as it is, without `w` h is the residual itself.  The residual may come from elsewhere (x_in), and a
// vector may be added to it.  `groups` > 1: that many equal parts of x have a root mean square each.  One block per row, the row in
// registers; all fp32.
// ------------------------------------------------------------------------------------------------------
struct NormStepParams {
  const float* x_in;       // [rows, ldx]
  float* x;                // [rows, W], or null where nothing is added
  SublayerOut out;
  const float* add;        // [W] or null
  const float *post, *w;   // norm weights or null
  void* h;                 // [rows, ldh] or null
  float* factor;           // [rows, groups] or null: gets 1 / root mean square of x
  const int* gather;       // row r of h comes from row gather[r]; x is then left alone
  float eps;
  int rows, total_rows, W, groups, ldx, ldh;
  int* status;
};

template <typename T, int V, int N>
__global__ void __launch_bounds__(1024) norm_step_kernel(NormStepParams p) {
  __shared__ float red[2][1][32];
  extern __shared__ float ns_groups[];         // groups > 1: [W / V] sums, [groups] factors
  const int r = blockIdx.x;
  int t = r;
  if (p.gather != nullptr) {
    t = p.gather[r];
    if (t < 0 || t >= p.total_rows) {
      if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
      t = 0;
    }
  }
  float x[N][V];
  const float* xr = p.x_in + static_cast<size_t>(t) * p.ldx;
  float* xw = p.gather == nullptr ? p.x + static_cast<size_t>(t) * p.W : nullptr;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
#pragma unroll
    for (int v = 0; v < V; ++v) x[i][v] = 0.f;
    if (c < p.W) {
      load_vec<V>(xr + c, x[i]);
      if (p.add != nullptr) {
        float a[V];
        load_vec<V>(p.add + c, a);
#pragma unroll
        for (int v = 0; v < V; ++v) x[i][v] += a[v];
        if (p.out.y == nullptr && xw != nullptr) store_vec<V>(xw + c, x[i]);
      }
    }
  }
  if (p.out.y != nullptr) {
    float y[1][N][V], inv[1] = {0.f};
    sublayer_rows<T, 1>(p.out, t, 1, p.W, y, p.status);
    if (p.post != nullptr) {
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) inv[0] = fmaf(y[0][i][v], y[0][i][v], inv[0]);
      block_sums<1>(inv, red, 0);
      inv[0] = 1.f / sqrtf(inv[0] / static_cast<float>(p.W) + p.eps);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < p.W) {
        float g[V];
        if (p.post != nullptr) load_vec<V>(p.post + c, g);
#pragma unroll
        for (int v = 0; v < V; ++v) x[i][v] = p.post != nullptr ? fmaf(y[0][i][v] * inv[0], g[v], x[i][v]) : x[i][v] + y[0][i][v];
        if (xw != nullptr) store_vec<V>(xw + c, x[i]);
      }
    }
  }
  if (p.h == nullptr && p.factor == nullptr) return;
  float inv[1] = {0.f};
  float* ginv = ns_groups + p.W / V;
  if (p.groups > 1 && (p.w != nullptr || p.factor != nullptr)) {
    group_factors<N, V>(x, p.W, p.groups, p.eps, ns_groups, ginv);
    if (p.factor != nullptr)
      for (int g = threadIdx.x; g < p.groups; g += blockDim.x) p.factor[static_cast<size_t>(r) * p.groups + g] = ginv[g];
  } else if (p.w != nullptr || p.factor != nullptr) {
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) inv[0] = fmaf(x[i][v], x[i][v], inv[0]);
    block_sums<1>(inv, red, 1);
    inv[0] = 1.f / sqrtf(inv[0] / static_cast<float>(p.W) + p.eps);
    if (p.factor != nullptr && threadIdx.x == 0) p.factor[r] = inv[0];
  }
  if (p.h == nullptr) return;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
    if (c < p.W) {
      if (p.w != nullptr) {
        float g[V];
        load_vec<V>(p.w + c, g);
        const float f = p.groups > 1 ? ginv[c / (p.W / p.groups)] : inv[0];
#pragma unroll
        for (int v = 0; v < V; ++v) x[i][v] *= f * g[v];
      }
      store_vec<V>(static_cast<T*>(p.h) + static_cast<size_t>(r) * p.ldh + c, x[i]);
    }
  }
}

template <typename T, int V>
static int launch_norm_step(const NormStepParams& p, cudaStream_t s) {
  const int units = (p.W + V - 1) / V;
  const int threads = units >= 4096 ? 1024 : units >= 256 ? 256 : (units + 31) / 32 * 32;
  const int n = (units + threads - 1) / threads;
  const size_t smem = group_bytes(p.W, V, p.groups, 1);
  if (smem > 40 * 1024) return -2;
  if (n <= 1) norm_step_kernel<T, V, 1><<<p.rows, threads, smem, s>>>(p);
  else if (n <= 2) norm_step_kernel<T, V, 2><<<p.rows, threads, smem, s>>>(p);
  else if (n <= 4) norm_step_kernel<T, V, 4><<<p.rows, threads, smem, s>>>(p);
  else if (n <= 16) norm_step_kernel<T, V, 16><<<p.rows, threads, smem, s>>>(p);
  else return -2;
  return static_cast<int>(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------------
// norm_conv_step is that pass for designs whose sublayers read a short causal convolution of the normed residual:
//
//   x_out <- x_in + y + add        h = rms(x_out) w        u_t = sum_j conv[j] h_(t - taps + 1 + j)
//
// A block is one decode row or kNcRows rows of one prefill chunk.  A thread keeps its columns' last taps - 1 values of h and walks the
// rows, NB at a time (their loads and sums are under way together).  The rows before the block's first are normed once more -- x_in and
// x_out are different buffers, so what they need is still there -- or come from the sequence's slot ([slots][taps - 1][W], oldest
// first); only the block with a chunk's first row reads a slot, so it also leaves the chunk's last values there.
// ------------------------------------------------------------------------------------------------------
constexpr int kNcRows = 16;                   // divides the scheduler's 64-row tiles

struct NormConvParams {
  const float* x_in;       // [rows, ldx]
  float* x_out;            // [rows, W], or null: nothing is added
  SublayerOut out;
  const float* add;        // [W] or null
  const float* w;          // [W]
  const float* conv;       // [taps, W]
  float* state;            // [slots, taps - 1, W]
  void* h;                 // [rows, ldh]
  void* plain;             // [rows, ldp] or null: gets the normed rows
  float eps;
  int W, groups, ldx, ldh, ldp, taps;
  StepRows sr;
  int* status;
};

template <typename T, int V, int N, int NB, int TM>
__global__ void __launch_bounds__(512) norm_conv_kernel(NormConvParams p) {
  __shared__ float red[2][NB][32];
  extern __shared__ float nc_groups[];         // groups > 1: [NB][W / V] sums, [NB][groups] factors
  RowSpan<kNcRows> r;
  if (!r.set(p.sr, blockIdx.x, p.status)) return;
  const int base = r.base, n = r.n, j0 = r.j0, j1 = r.j1, start = r.start, slot = r.slot;
  float conv[TM][N][V], w[N][V], h[TM > 1 ? TM - 1 : 1][N][V];    // filters aligned to their last tap; h: the last values, oldest first
  const int col0 = threadIdx.x * V, step = blockDim.x * V, off = TM - p.taps;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = col0 + i * step;
#pragma unroll
    for (int k = 0; k < TM; ++k) {
#pragma unroll
      for (int v = 0; v < V; ++v) conv[k][i][v] = 0.f;
      if (c < p.W && k >= off) load_vec<V>(p.conv + static_cast<size_t>(k - off) * p.W + c, conv[k][i]);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) w[i][v] = 0.f;
    if (c < p.W) load_vec<V>(p.w + c, w[i]);
  }
  int parity = 0;
  // normed rows j .. j + m - 1 of the chunk (m <= NB)
  auto normed = [&](int j, int m, bool write, float (&o)[NB][N][V]) {
    float x[NB][N][V], ss[NB];
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
      for (int i = 0; i < N; ++i) {
#pragma unroll
        for (int v = 0; v < V; ++v) x[b][i][v] = 0.f;
        if (b < m && col0 + i * step < p.W) load_vec<V>(p.x_in + static_cast<size_t>(base + j + b) * p.ldx + col0 + i * step, x[b][i]);
      }
    sublayer_rows<T, NB>(p.out, base + j, m, p.W, o, p.status);
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      ss[b] = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = col0 + i * step;
        if (p.add != nullptr && c < p.W) {
          float a[V];
          load_vec<V>(p.add + c, a);
#pragma unroll
          for (int v = 0; v < V; ++v) o[b][i][v] += a[v];
        }
#pragma unroll
        for (int v = 0; v < V; ++v) {
          x[b][i][v] += o[b][i][v];
          ss[b] = c < p.W ? fmaf(x[b][i][v], x[b][i][v], ss[b]) : ss[b];
        }
        if (write && p.x_out != nullptr && b < m && c < p.W) store_vec<V>(p.x_out + static_cast<size_t>(base + j + b) * p.W + c, x[b][i]);
      }
    }
    if (p.groups > 1) {
      const int units = p.W / V, per = units / p.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
      float* ginv = nc_groups + NB * units;
      __syncthreads();
#pragma unroll
      for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int u = i * blockDim.x + threadIdx.x;
          float a = 0.f;
#pragma unroll
          for (int v = 0; v < V; ++v) a = fmaf(x[b][i][v], x[b][i][v], a);
          if (u < units) nc_groups[b * units + u] = a;
        }
      __syncthreads();
      for (int g = warp; g < NB * p.groups; g += warps) {       // groups of the NB rows one after the other
        float a = 0.f;
        for (int u = lane; u < per; u += 32) a += nc_groups[(g / p.groups) * units + (g % p.groups) * per + u];
        a = warp_sum(a);
        if (lane == 0) ginv[g] = 1.f / sqrtf(a / static_cast<float>(per * V) + p.eps);
      }
      __syncthreads();
#pragma unroll
      for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int c = col0 + i * step;
          const float f = c < p.W ? ginv[b * p.groups + c / (p.W / p.groups)] : 0.f;
#pragma unroll
          for (int v = 0; v < V; ++v) o[b][i][v] = x[b][i][v] * (f * w[i][v]);
        }
    } else {
      block_sums<NB>(ss, red, parity);
      parity ^= 1;
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const float inv = 1.f / sqrtf(ss[b] / static_cast<float>(p.W) + p.eps);
#pragma unroll
        for (int i = 0; i < N; ++i)
#pragma unroll
          for (int v = 0; v < V; ++v) o[b][i][v] = x[b][i][v] * (inv * w[i][v]);
      }
    }
    if (write && p.plain != nullptr) {
#pragma unroll
      for (int b = 0; b < NB; ++b)
#pragma unroll
        for (int i = 0; i < N; ++i)
          if (b < m && col0 + i * step < p.W) store_vec<V>(static_cast<T*>(p.plain) + static_cast<size_t>(base + j + b) * p.ldp + col0 + i * step, o[b][i]);
    }
  };
  auto shift_in = [&](const float (&o)[N][V]) {
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) {
#pragma unroll
        for (int k = 0; k + 1 < TM - 1; ++k) h[k][i][v] = h[k + 1][i][v];
        h[TM > 1 ? TM - 2 : 0][i][v] = o[i][v];
      }
  };
  float* st = slot >= 0 ? p.state + static_cast<size_t>(slot) * (p.taps - 1) * p.W : nullptr;
  auto keep = [&]() {                          // the chunk's last values to the slot
    if (st == nullptr) return;
#pragma unroll
    for (int k = 0; k < TM - 1; ++k)
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (k >= off && col0 + i * step < p.W) store_vec<V>(st + static_cast<size_t>(k - off) * p.W + col0 + i * step, h[k][i]);
  };
  float o[NB][N][V];
  // rows from..from + m - 1 of the chunk into the last values
  auto recompute = [&](int from, int m) {
    for (int j = 0; j < m; j += NB) {
      const int c = min(NB, m - j);
      normed(from + j, c, false, o);
#pragma unroll
      for (int b = 0; b < NB; ++b)
        if (b < c) shift_in(o[b]);
    }
  };
#pragma unroll
  for (int k = 0; k < (TM > 1 ? TM - 1 : 1); ++k)
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) h[k][i][v] = 0.f;
  if (p.taps > 1) {
    if (j0 == 0) {
      if (n > kNcRows) {                       // other blocks finish the chunk
        float old[TM > 1 ? TM - 1 : 1][N][V];
#pragma unroll
        for (int k = 0; k < TM - 1; ++k)
#pragma unroll
          for (int i = 0; i < N; ++i) {
#pragma unroll
            for (int v = 0; v < V; ++v) old[k][i][v] = 0.f;
            const int t = start - (TM - 1) + k;
            if (st != nullptr && k >= off && t >= 0 && col0 + i * step < p.W) load_vec<V>(st + static_cast<size_t>(k - off) * p.W + col0 + i * step, old[k][i]);
          }
        recompute(n - (p.taps - 1), p.taps - 1);
        keep();
#pragma unroll
        for (int k = 0; k < TM - 1; ++k)
#pragma unroll
          for (int i = 0; i < N; ++i)
#pragma unroll
            for (int v = 0; v < V; ++v) h[k][i][v] = old[k][i][v];
      } else {
#pragma unroll
        for (int k = 0; k < TM - 1; ++k)
#pragma unroll
          for (int i = 0; i < N; ++i) {
            const int t = start - (TM - 1) + k;
            if (st != nullptr && k >= off && t >= 0 && col0 + i * step < p.W) load_vec<V>(st + static_cast<size_t>(k - off) * p.W + col0 + i * step, h[k][i]);
          }
      }
    } else {
      recompute(j0 - (p.taps - 1), p.taps - 1);
    }
  }
  for (int j = j0; j < j1; j += NB) {
    const int m = min(NB, j1 - j);
    normed(j, m, true, o);
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      if (b >= m) continue;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        float u[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
          u[v] = conv[TM - 1][i][v] * o[b][i][v];
#pragma unroll
          for (int k = 0; k < TM - 1; ++k) u[v] = fmaf(conv[k][i][v], h[k][i][v], u[v]);
        }
        if (col0 + i * step < p.W) store_vec<V>(static_cast<T*>(p.h) + static_cast<size_t>(base + j + b) * p.ldh + col0 + i * step, u);
      }
      shift_in(o[b]);
    }
  }
  if (p.taps > 1 && j0 == 0 && n <= kNcRows) keep();
}

template <typename T, int V, int TM>
static int launch_norm_conv(const NormConvParams& p, cudaStream_t s) {
  const int units = (p.W + V - 1) / V, blocks = span_blocks<kNcRows>(p.sr);
  const int n = units <= 256 ? 1 : units <= 1024 ? 2 : units <= 2048 ? 4 : 8;
  const int threads = ((units + n - 1) / n + 31) / 32 * 32;
  if (threads > 512 || n * V > 16) return -2;
  auto smem = [&](int nb) { return group_bytes(p.W, V, p.groups, nb); };
  if (n == 1) norm_conv_kernel<T, V, 1, 4, TM><<<blocks, threads, smem(4), s>>>(p);
  else if (n == 2) norm_conv_kernel<T, V, 2, V == 1 ? 4 : 2, TM><<<blocks, threads, smem(V == 1 ? 4 : 2), s>>>(p);
  else if (n == 4) norm_conv_kernel<T, V, 4, V == 1 ? 4 : 1, TM><<<blocks, threads, smem(V == 1 ? 4 : 1), s>>>(p);
  else if constexpr (V == 1) norm_conv_kernel<T, V, 8, 2, TM><<<blocks, threads, smem(2), s>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------------
// input_conv is the second half of that pass for steps of many rows: norm_step has left the residual and its rows' factors, and the
// convolution is elementwise in the column.  A thread loads V columns of a block's rows at once; slots as above.
// ------------------------------------------------------------------------------------------------------
constexpr int kIcRows = 8;                    // rows of a block (before them taps - 1 more are read)
struct InputConvParams {
  const float* x;          // [rows, W]
  const float* factor;     // [rows, groups]
  const float* w;          // [W]
  const float* conv;       // [taps, W]
  float* state;            // [slots, taps - 1, W]
  void* h;                 // [rows, ldh]
  void* plain;             // [rows, ldp] or null: gets the normed rows
  int W, groups, ldh, ldp, taps;
  StepRows sr;
  int* status;
};

template <typename T, int V, int TM>
__global__ void __launch_bounds__(128) input_conv_kernel(InputConvParams p) {
  RowSpan<kIcRows> r;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V, off = TM - p.taps;
  if (!r.set(p.sr, blockIdx.x, p.status) || c >= p.W) return;
  float conv[TM][V], w[V], h[TM > 1 ? TM - 1 : 1][V];        // filters aligned to their last tap; h: the last values, oldest first
  load_vec<V>(p.w + c, w);
#pragma unroll
  for (int k = 0; k < TM; ++k) {
#pragma unroll
    for (int v = 0; v < V; ++v) conv[k][v] = 0.f;
    if (k >= off) load_vec<V>(p.conv + static_cast<size_t>(k - off) * p.W + c, conv[k]);
  }
  const int group = p.groups > 1 ? c / (p.W / p.groups) : 0;
  auto normed = [&](int t, float (&o)[V]) {
    load_vec<V>(p.x + static_cast<size_t>(r.base + t) * p.W + c, o);
    const float f = p.factor[static_cast<size_t>(r.base + t) * p.groups + group];
#pragma unroll
    for (int v = 0; v < V; ++v) o[v] *= f * w[v];
  };
  float* st = r.slot >= 0 ? p.state + static_cast<size_t>(r.slot) * (p.taps - 1) * p.W + c : nullptr;
#pragma unroll
  for (int k = 0; k < (TM > 1 ? TM - 1 : 1); ++k) {
    const int t = r.j0 - (TM - 1) + k;                       // within the chunk
#pragma unroll
    for (int v = 0; v < V; ++v) h[k][v] = 0.f;
    if (k < off || TM == 1) continue;
    if (t >= 0) normed(t, h[k]);
    else if (st != nullptr && r.start + t >= 0) load_vec<V>(st + static_cast<size_t>(k - off) * p.W, h[k]);
  }
  float o[kIcRows][V];
#pragma unroll
  for (int b = 0; b < kIcRows; ++b) {
#pragma unroll
    for (int v = 0; v < V; ++v) o[b][v] = 0.f;
    if (r.j0 + b < r.j1) normed(r.j0 + b, o[b]);
  }
  if (p.plain != nullptr) {
#pragma unroll
    for (int b = 0; b < kIcRows; ++b)
      if (r.j0 + b < r.j1) store_vec<V>(static_cast<T*>(p.plain) + static_cast<size_t>(r.base + r.j0 + b) * p.ldp + c, o[b]);
  }
  if (r.j0 == 0 && st != nullptr) {
#pragma unroll
    for (int k = 0; k < TM - 1; ++k) {
      if (k < off) continue;
      const int t = r.n - (TM - 1) + k;
      float last[V];
#pragma unroll
      for (int q = 0; q < TM - 1; ++q)                       // fewer rows than taps: older values move up
#pragma unroll
        for (int v = 0; v < V; ++v) last[v] = (q == 0 || q == k + r.n) ? h[q][v] : last[v];
      if (t >= 0) normed(t, last);
      store_vec<V>(st + static_cast<size_t>(k - off) * p.W, last);
    }
  }
#pragma unroll
  for (int b = 0; b < kIcRows; ++b) {
    if (r.j0 + b >= r.j1) continue;
    float u[V];
#pragma unroll
    for (int v = 0; v < V; ++v) {
      u[v] = conv[TM - 1][v] * o[b][v];
#pragma unroll
      for (int k = 0; k < TM - 1; ++k) u[v] = fmaf(conv[k][v], b + k < TM - 1 ? h[b + k < TM - 1 ? b + k : 0][v] : o[b + k < TM - 1 ? 0 : b + k - (TM - 1)][v], u[v]);
    }
    store_vec<V>(static_cast<T*>(p.h) + static_cast<size_t>(r.base + r.j0 + b) * p.ldh + c, u);
  }
}

template <typename T, int V, int TM>
static int launch_input_conv(const InputConvParams& p, cudaStream_t s) {
  const dim3 grid(span_blocks<kIcRows>(p.sr), (p.W + 128 * V - 1) / (128 * V));
  input_conv_kernel<T, V, TM><<<grid, 128, 0, s>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------------
// all streams of a row start as the token's embedding times `scale`, normed where `w` is given; `copy` gets it too (read again by later layers)
// ------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) embed_streams_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                                                            int S, int W, int vocab, const float* __restrict__ w, float eps, float scale,
                                                            T* __restrict__ copy, int ldc, int* status) {
  __shared__ float red[2][1][32];
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicOr(status, kStatusIndexOutOfRange);
    id = 0;
  }
  const T* src = table + static_cast<size_t>(id) * W;
  float* dst = x + static_cast<size_t>(t) * S * W;
  float inv[1] = {0.f};
  if (w != nullptr) {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = to_f32<T>(src[c]) * scale;
      inv[0] = fmaf(v, v, inv[0]);
    }
    block_sums<1>(inv, red, 0);
    inv[0] = 1.f / sqrtf(inv[0] / static_cast<float>(W) + eps);
  }
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = to_f32<T>(src[c]) * scale;
    if (w != nullptr) v *= inv[0] * w[c];
    for (int s = 0; s < S; ++s) dst[static_cast<size_t>(s) * W + c] = v;
    if (copy != nullptr) copy[static_cast<size_t>(t) * ldc + c] = from_f32<T>(v);
  }
}

// ------------------------------------------------------------------------------------------------------
// latent pages [pages, 16, ldp]: a row is the normed latent (rank values, zeros up to a multiple of 8) and the rotated key part that
// all heads share (rot values).  A projected row holds the queries of `heads` heads (dim values, zeros up to a multiple of 8, and rot
// values each), the latent and the key part.  Neighbours 2i, 2i + 1 of a rotated part turn by position * freq[i].  Rotated query parts
// go to column `q_col` of a head's row of q_out for tokens below `split`, and back to where they came from for the others.
// One block per token: warp 0 has the latent.  rot 0: the latent alone (one warp per token).
// ------------------------------------------------------------------------------------------------------
struct LatentAppendParams {
  void* row;               // [tokens, ldr], queries first
  const float* w;          // [rank]
  const int* slots;
  void* pool;
  const double* freq;      // [rot / 2]
  const int* positions;
  void* q_out;             // [tokens * heads, ldq]
  float eps;
  int tokens, ldr, latent, rank, ldp, heads, dim, rot, ldq, q_col, split;
  int64_t num_slots;
  int* status;
};

template <typename T>
OGB_DEVICE void append_latent(const LatentAppendParams& p, int t, int lane) {
  const int64_t slot = p.slots[t];
  if (slot < 0) return;                        // padding row
  if (slot >= p.num_slots) {
    if (lane == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    return;
  }
  const T* src = static_cast<const T*>(p.row) + static_cast<size_t>(t) * p.ldr + p.latent;
  float ss = 0.f;
  for (int i = lane; i < p.rank; i += 32) { const float v = to_f32<T>(src[i]); ss = fmaf(v, v, ss); }
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.rank) + p.eps);
  T* dst = static_cast<T*>(p.pool) + slot * p.ldp;
  for (int i = lane; i < p.rank; i += 32) dst[i] = from_f32<T>(to_f32<T>(src[i]) * inv * p.w[i]);
}

template <typename T>
__global__ void __launch_bounds__(128) latent_append_kernel(LatentAppendParams p) {
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (t < p.tokens) append_latent<T>(p, t, threadIdx.x & 31);
}

template <typename T>
__global__ void __launch_bounds__(128) latent_rope_append_kernel(LatentAppendParams p) {
  extern __shared__ float2 s_turn[];           // [rot / 2] cos, sin
  const int t = blockIdx.x, half = p.rot / 2, dp = (p.dim + 7) / 8 * 8, rp = (p.rot + 7) / 8 * 8;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    // the angle is reduced in double, so that it is good to fp32 at every position
    const double a = static_cast<double>(p.positions[t]) * p.freq[i] * 0.15915494309189535;
    float s, c;
    sincospif(static_cast<float>(2.0 * (a - rint(a))), &s, &c);
    s_turn[i] = make_float2(c, s);
  }
  if (threadIdx.x < 32) append_latent<T>(p, t, threadIdx.x);
  __syncthreads();
  T* row = static_cast<T*>(p.row) + static_cast<size_t>(t) * p.ldr;
  const int64_t slot = p.slots[t];
  for (int i = threadIdx.x; i < (p.heads + 1) * half; i += blockDim.x) {
    const int head = i / half, e = i - head * half;
    const bool key = head == p.heads;
    T* src = row + (key ? p.latent + (p.rank + 7) / 8 * 8 : head * (dp + rp) + dp) + 2 * e;      // parts start on 8 elements
    float x[2];
    load_vec<2>(src, x);
    const float2 cs = s_turn[e];
    T* dst = src;
    if (key) {
      if (slot < 0 || slot >= p.num_slots) continue;
      dst = static_cast<T*>(p.pool) + slot * p.ldp + (p.rank + 7) / 8 * 8 + 2 * e;
    } else if (t < p.split) {
      dst = static_cast<T*>(p.q_out) + (static_cast<size_t>(t) * p.heads + head) * p.ldq + p.q_col + 2 * e;
    }
    const float o[2] = {x[0] * cs.x - x[1] * cs.y, x[1] * cs.x + x[0] * cs.y};
    store_vec<2>(dst, o);
  }
}

// ------------------------------------------------------------------------------------------------------
// RMS norm of every group of `n` columns (a head) with a weight (null: none; head h's begins at h * wstep: 0 is one for all), times silu
// or sigmoid of a gate of the same layout where there is one: fp32 in, activation type out; one warp per group
// ------------------------------------------------------------------------------------------------------
OGB_DEVICE float silu_f32(float z) { return z / (1.f + expf(-z)); }
OGB_DEVICE float gate_f32(float z, bool sigmoid) { return sigmoid ? 1.f / (1.f + expf(-z)) : silu_f32(z); }

template <typename T>
__global__ void __launch_bounds__(256) head_rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ w, int wstep, float eps,
                                                           T* __restrict__ out, int rows, int heads, int n, int ldx, int ldo, const T* __restrict__ gate,
                                                           int ldg, bool sigmoid, bool vec) {
  const int lane = threadIdx.x & 31;
  const long long g = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (g >= static_cast<long long>(rows) * heads) return;
  const int t = static_cast<int>(g / heads), h = static_cast<int>(g % heads);
  const float* src = x + static_cast<size_t>(t) * ldx + static_cast<size_t>(h) * n;
  T* dst = out + static_cast<size_t>(t) * ldo + static_cast<size_t>(h) * n;
  if (w != nullptr) w += static_cast<size_t>(h) * wstep;
  const T* gt = gate != nullptr ? gate + static_cast<size_t>(t) * ldg + static_cast<size_t>(h) * n : nullptr;
  float ss = 0.f;
  if (vec) {                                   // rows and heads of x, out and gate start on four elements; n is 128 .. 512 in steps of 128
    float v[4][4];
    const int per = n >> 7;
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k < per) {
        load_vec<4>(src + k * 128 + lane * 4, v[k]);
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(v[k][i], v[k][i], ss);
      }
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(n) + eps);
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k < per) {
        float wv[4] = {1.f, 1.f, 1.f, 1.f};
        if (w != nullptr) load_vec<4>(w + k * 128 + lane * 4, wv);
#pragma unroll
        for (int i = 0; i < 4; ++i) v[k][i] *= inv * wv[i];
        if (gt != nullptr) {
          load_vec<4>(gt + k * 128 + lane * 4, wv);
#pragma unroll
          for (int i = 0; i < 4; ++i) v[k][i] *= gate_f32(wv[i], sigmoid);
        }
        store_vec<4>(dst + k * 128 + lane * 4, v[k]);
      }
    return;
  }
  for (int i = lane; i < n; i += 32) ss = fmaf(src[i], src[i], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(n) + eps);
  for (int i = lane; i < n; i += 32) dst[i] = from_f32<T>(src[i] * inv * (w != nullptr ? w[i] : 1.f) * (gt != nullptr ? gate_f32(to_f32<T>(gt[i]), sigmoid) : 1.f));
}

// ------------------------------------------------------------------------------------------------------
// gated activation over tile-interleaved gate | up columns (ops.pack_gate_up), and an activation of every value (common.cuh Act)
// ------------------------------------------------------------------------------------------------------
OGB_DEVICE float gated_act_f32(const ActArgs& act, float g, float u) {
  if (act.kind == kActGeluTanh) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  if (act.kind == kActClampGlu) {
    g = fminf(g, act.a);
    u = fminf(fmaxf(u, -act.a), act.a);
    return g / (1.f + expf(-kClampGluSlope * g)) * (u + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}
OGB_DEVICE float plain_act_f32(const ActArgs& act, float v) {
  if (act.kind == kActRelu2) return fmaxf(v, 0.f) * fmaxf(v, 0.f);
  if (act.kind == kActXielu) return fmaf(0.5f, v, v > 0.f ? act.a * v * v : act.b * (expm1f(v) - v));
  return v;
}

template <typename T>
__global__ void __launch_bounds__(256) act_mul_packed_kernel(const T* __restrict__ gu, T* __restrict__ out, int rows, int inter, int half, ActArgs act) {
  const long long total = static_cast<long long>(rows) * inter;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const int t = static_cast<int>(i / inter), j = static_cast<int>(i % inter);
    const T* row = gu + static_cast<size_t>(t) * 2 * inter + static_cast<size_t>(j / half) * 2 * half + j % half;
    const float g = to_f32<T>(row[0]), u = to_f32<T>(row[half]);
    out[i] = from_f32<T>(gated_act_f32(act, g, u));
  }
}

// ------------------------------------------------------------------------------------------------------
// fp32 matrix product (no reduced-precision mode): C[M,N] = A[M,K] W[N,K]^T for `batch` problems whose operands start at
// column offsets of A and C and at row offsets of W.  64 x 64 tile, 4 x 4 results per thread.  Grouped: rows of A are sorted by
// expert, `tab` / `mtiles` are the 128-row tile table of moe.cu, and W holds one matrix per expert.
// ------------------------------------------------------------------------------------------------------
constexpr int kF32Tile = 64, kF32K = 16;
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ W, float* __restrict__ C, int M,
                                                       int N, int K, int lda, int ldw, int ldc, int a_step, int c_step, const int* __restrict__ tab,
                                                       const int* __restrict__ mtiles, ActArgs act) {
  __shared__ float sa[kF32K][kF32Tile + 4], sw[kF32K][kF32Tile + 4];
  A += static_cast<size_t>(blockIdx.z) * a_step;
  W += static_cast<size_t>(blockIdx.z) * N * ldw;
  C += static_cast<size_t>(blockIdx.z) * c_step;
  const int n0 = blockIdx.x * kF32Tile;
  int m0 = blockIdx.y * kF32Tile;
  if (tab != nullptr) {
    const int mt = blockIdx.y / 2;
    if (mt >= *mtiles) return;
    W += static_cast<size_t>(tab[4 * mt]) * N * ldw;
    m0 = tab[4 * mt + 1] + (blockIdx.y & 1) * kF32Tile;
    M = min(M, tab[4 * mt + 2]);
    if (m0 >= M) return;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kF32K) {
    for (int i = threadIdx.x; i < kF32Tile * kF32K; i += 256) {
      const int r = i / kF32K, k = i % kF32K;
      sa[k][r] = (m0 + r < M && k0 + k < K) ? A[static_cast<size_t>(m0 + r) * lda + k0 + k] : 0.f;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? W[static_cast<size_t>(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; b[i] = sw[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r < M && c < N) C[static_cast<size_t>(r) * ldc + c] = plain_act_f32(act, acc[i][j]);
    }
}

}  // namespace ogb

using namespace ogb;

extern "C" int ogb_hyper_step(const float* x_in, float* x_out, const void* y, const float* mix, const float* out_w, const float* in_w,
                              const float* alpha, const float* w, const float* b, const float* shift, float* prev, void* h,
                              const int* gather, int rows, int total_rows, int S, int W, int ldy, int ldh, const int* ctx_len,
                              const int* state_slot, const int* cu_q, const int* tile_seq, const int* tile_q0, int num_decode,
                              int num_tiles, int num_slots, int elem, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (S < 1 || S > 8 || W < 1 || x_in == x_out) return -3;
  if (shift != nullptr && (prev == nullptr || h == nullptr || gather != nullptr)) return -3;
  if (y != nullptr && (mix == nullptr || out_w == nullptr)) return -3;
  HyperParams p{x_in, x_out, y, mix, out_w, in_w, alpha, w, b, shift, prev, h, gather, rows, total_rows, S, W, ldy, ldh, rows <= 1024 ? 1 : kHsRows,
                StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, num_slots}, status};
  const bool vec = W % 4 == 0 && ldy % 4 == 0 && ldh % 4 == 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return vec ? dispatch_hyper<__nv_bfloat16, 4>(p, s) : dispatch_hyper<__nv_bfloat16, 1>(p, s);
  if (elem == kElemF32) return vec ? dispatch_hyper<float, 4>(p, s) : dispatch_hyper<float, 1>(p, s);
  return -3;
}

// pos / weight (null: y has one row per token): y holds y_rows expert rows, of which token t sums k; shared / gate: a row of every
// token, times the sigmoid of its gate.
static bool sublayer_ok(const SublayerOut& o) {
  return (o.pos == nullptr || (o.weight != nullptr && o.k >= 1)) && (o.shared == nullptr || (o.pos != nullptr && o.gate != nullptr)) &&
         (o.res_gate != nullptr ? o.y != nullptr && o.res_bias != nullptr : o.y_bias == nullptr);
}
// four elements at a time need rows that start on them, and pointers too
static bool sublayer_vec(const SublayerOut& o, int elem) {
  const uintptr_t act = reinterpret_cast<uintptr_t>(o.y) | reinterpret_cast<uintptr_t>(o.shared) | reinterpret_cast<uintptr_t>(o.res_gate);
  const uintptr_t f32 = reinterpret_cast<uintptr_t>(o.y_bias) | reinterpret_cast<uintptr_t>(o.res_bias);
  return ((o.ldy | o.lds | o.ldr) & 3) == 0 && (f32 & 15) == 0 && (act & (elem == kElemBF16 ? 7 : 15)) == 0;
}

// post null: y as it is; w null: h is the residual; h null: no read-out.  A gathered row's gate is the one of the row it comes from.
extern "C" int ogb_norm_step(float* x, const void* y, const int* pos, const float* weight, const void* shared, const float* gate, const float* y_bias,
                             const void* res_gate, const float* res_bias, const float* post, const float* w, void* h, const int* gather, float eps, int rows,
                             int total_rows, int W, int groups, int k, int ldy, int lds, int ldg, int ldr, int ldh, int64_t y_rows, int elem, int* status,
                             void* stream) {
  if (rows <= 0) return 0;
  NormStepParams p{x, x, SublayerOut{y, pos, weight, shared, gate, y_bias, res_gate, res_bias, k, ldy, lds, ldg, ldr, y_rows}, nullptr, post, w, h, nullptr,
                   gather, eps, rows, total_rows, W, groups, W, ldh, status};
  if (W < 1 || groups < 1 || W % groups != 0 || !sublayer_ok(p.out)) return -3;
  const uintptr_t f32 = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(post) | reinterpret_cast<uintptr_t>(w);
  const bool vec = ((W | ldh) & 3) == 0 && (groups == 1 || (W / groups & 3) == 0) && (f32 & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(h) & (elem == kElemBF16 ? 7 : 15)) == 0 && sublayer_vec(p.out, elem);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return vec ? launch_norm_step<__nv_bfloat16, 4>(p, s) : launch_norm_step<__nv_bfloat16, 1>(p, s);
  if (elem == kElemF32) return vec ? launch_norm_step<float, 4>(p, s) : launch_norm_step<float, 1>(p, s);
  return -3;
}

// x_out null: nothing is added (y and add null).  At most 8 taps.  factor null: one kernel, for few rows (of up to 8192 columns, 4096
// where they do not start on four elements); else [rows, groups] of scratch, norm_step and input_conv.
template <typename T>
static int norm_conv(const NormConvParams& p, float* factor, int rows, bool vec, cudaStream_t s) {
  if (factor == nullptr)
    return vec ? (p.taps <= 4 ? launch_norm_conv<T, 4, 4>(p, s) : launch_norm_conv<T, 4, 8>(p, s))
               : (p.taps <= 4 ? launch_norm_conv<T, 1, 4>(p, s) : launch_norm_conv<T, 1, 8>(p, s));
  const NormStepParams n{p.x_in, p.x_out, p.out, p.add, nullptr, nullptr, nullptr, factor, nullptr, p.eps, rows, rows, p.W, p.groups, p.ldx, 0, p.status};
  const int rc = vec ? launch_norm_step<T, 4>(n, s) : launch_norm_step<T, 1>(n, s);
  if (rc != 0) return rc;
  const InputConvParams q{p.x_out != nullptr ? p.x_out : p.x_in, factor, p.w, p.conv, p.state, p.h, p.plain, p.W, p.groups, p.ldh, p.ldp, p.taps, p.sr,
                         p.status};
  return vec ? (p.taps <= 4 ? launch_input_conv<T, 4, 4>(q, s) : launch_input_conv<T, 4, 8>(q, s))
             : (p.taps <= 4 ? launch_input_conv<T, 1, 4>(q, s) : launch_input_conv<T, 1, 8>(q, s));
}

extern "C" int ogb_norm_conv_step(const float* x_in, float* x_out, const void* y, const int* pos, const float* weight, const void* shared,
                                  const float* gate, const float* y_bias, const void* res_gate, const float* res_bias, const float* add, const float* w,
                                  const float* conv, float* state, void* h, void* plain, float* factor, float eps, int rows, int W, int groups, int taps,
                                  int k, int ldx, int ldy, int lds, int ldg, int ldr, int ldh, int ldp, int64_t y_rows,
                                  const int* ctx_len, const int* state_slot, const int* cu_q, const int* tile_seq, const int* tile_q0, int num_decode,
                                  int num_tiles, int num_slots, int elem, int* status, void* stream) {
  if (num_decode + num_tiles <= 0) return 0;
  NormConvParams p{x_in, x_out, SublayerOut{y, pos, weight, shared, gate, y_bias, res_gate, res_bias, k, ldy, lds, ldg, ldr, y_rows}, add, w, conv, state,
                   h, plain, eps, W, groups, ldx, ldh, ldp, taps,
                   StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, num_slots}, status};
  if (groups < 1 || W % groups != 0) return -3;
  if (W < 1 || taps < 1 || taps > 8 || x_in == x_out || !sublayer_ok(p.out) || w == nullptr || conv == nullptr || h == nullptr) return -3;
  if ((taps > 1 && state == nullptr) || ((y != nullptr || add != nullptr) && x_out == nullptr) || (x_out == nullptr && ldx != W)) return -3;
  const uintptr_t act = reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(plain);
  const uintptr_t f32 = reinterpret_cast<uintptr_t>(x_in) | reinterpret_cast<uintptr_t>(x_out) | reinterpret_cast<uintptr_t>(add) |
                        reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(conv) | reinterpret_cast<uintptr_t>(state);
  const bool vec = ((W | ldx | ldh | ldp) & 3) == 0 && (groups == 1 || (W / groups & 3) == 0) && (f32 & 15) == 0 &&
                   (act & (elem == kElemBF16 ? 7 : 15)) == 0 && sublayer_vec(p.out, elem);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return norm_conv<__nv_bfloat16>(p, factor, rows, vec, s);
  if (elem == kElemF32) return norm_conv<float>(p, factor, rows, vec, s);
  return -3;
}

extern "C" int ogb_embed_streams(const int* ids, const void* table, float* x, int tokens, int S, int W, int vocab, const float* w, float eps, float scale,
                                 void* copy, int ldc, int elem, int* status, void* stream) {
  if (tokens <= 0) return 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16)
    embed_streams_kernel<<<tokens, 256, 0, s>>>(ids, static_cast<const __nv_bfloat16*>(table), x, S, W, vocab, w, eps, scale,
                                                static_cast<__nv_bfloat16*>(copy), ldc, status);
  else if (elem == kElemF32)
    embed_streams_kernel<<<tokens, 256, 0, s>>>(ids, static_cast<const float*>(table), x, S, W, vocab, w, eps, scale, static_cast<float*>(copy), ldc, status);
  else return -3;
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int launch_latent_append(const LatentAppendParams& p, cudaStream_t s) {
  if (p.rot == 0) latent_append_kernel<T><<<(p.tokens + 3) / 4, 128, 0, s>>>(p);
  else latent_rope_append_kernel<T><<<p.tokens, 128, p.rot / 2 * sizeof(float2), s>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// `latent`: column of the latent in a projected row.
extern "C" int ogb_latent_append(void* row, int ldr, int latent, const float* w, float eps, const int* slots, void* pool, int tokens, int rank, int ldp,
                                 int64_t num_slots, const double* freq, const int* positions, void* q_out, int heads, int dim, int rot, int ldq,
                                 int q_col, int split, int elem, int* status, void* stream) {
  if (tokens <= 0) return 0;
  if (rank > ldp || rot < 0 || (rot & 1) || rot > 4096) return -3;
  if (rot > 0 && (freq == nullptr || positions == nullptr || (rank + 7) / 8 * 8 + rot > ldp || (split > 0 && (q_out == nullptr || q_col + rot > ldq)))) return -3;
  LatentAppendParams p{row, w, slots, pool, freq, positions, q_out, eps, tokens, ldr, latent, rank, ldp, heads, dim, rot, ldq, q_col, split, num_slots,
                       status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return launch_latent_append<__nv_bfloat16>(p, s);
  if (elem == kElemF32) return launch_latent_append<float>(p, s);
  return -3;
}

extern "C" int ogb_head_rmsnorm(const float* x, const float* w, int wstep, float eps, void* out, int rows, int heads, int n, int ldx, int ldo,
                                const void* gate, int ldg, int sigmoid, int elem, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(rows) * heads + 7) / 8);
  const uintptr_t unaligned = ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) |
                              ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(gate)) & (elem == kElemBF16 ? 7 : 15));
  const bool vec = (n & 127) == 0 && n <= 512 && ((ldx | ldo | ldg | wstep) & 3) == 0 && unaligned == 0;
  if (elem == kElemBF16)
    head_rmsnorm_kernel<<<blocks, 256, 0, s>>>(x, w, wstep, eps, static_cast<__nv_bfloat16*>(out), rows, heads, n, ldx, ldo,
                                               static_cast<const __nv_bfloat16*>(gate), ldg, sigmoid != 0, vec);
  else if (elem == kElemF32)
    head_rmsnorm_kernel<<<blocks, 256, 0, s>>>(x, w, wstep, eps, static_cast<float*>(out), rows, heads, n, ldx, ldo, static_cast<const float*>(gate), ldg,
                                               sigmoid != 0, vec);
  else return -3;
  return static_cast<int>(cudaGetLastError());
}

extern "C" int ogb_act_mul_packed(const void* gate_up, void* out, int rows, int inter, int half, int kind, float act_a, float act_b, int elem,
                                  void* stream) {
  if (rows <= 0) return 0;
  if (half <= 0 || inter % half != 0 || !act_gated(kind)) return -3;
  const ActArgs act{kind, act_a, act_b};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int blocks = static_cast<int>(std::min<long long>((static_cast<long long>(rows) * inter + 255) / 256, 148 * 16));
  if (elem == kElemBF16)
    act_mul_packed_kernel<<<blocks, 256, 0, s>>>(static_cast<const __nv_bfloat16*>(gate_up), static_cast<__nv_bfloat16*>(out), rows, inter, half, act);
  else if (elem == kElemF32)
    act_mul_packed_kernel<<<blocks, 256, 0, s>>>(static_cast<const float*>(gate_up), static_cast<float*>(out), rows, inter, half, act);
  else return -3;
  return static_cast<int>(cudaGetLastError());
}

extern "C" int ogb_gemm_f32(const float* A, const float* W, float* C, int M, int N, int K, int lda, int ldw, int ldc, int batch, int a_step,
                            int c_step, void* stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  const dim3 grid((N + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile, batch);
  gemm_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(A, W, C, M, N, K, lda, ldw, ldc, a_step, c_step, nullptr, nullptr, ActArgs());
  return static_cast<int>(cudaGetLastError());
}

// With an activation of every result (not a gated one).
extern "C" int ogb_gemm_f32_act(const float* A, const float* W, float* C, int M, int N, int K, int lda, int ldw, int ldc, int act, float act_a, float act_b,
                                void* stream) {
  if (M <= 0 || N <= 0) return 0;
  if (act_gated(act)) return -7;
  const dim3 grid((N + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile);
  gemm_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(A, W, C, M, N, K, lda, ldw, ldc, 0, 0, nullptr, nullptr, ActArgs{act, act_a, act_b});
  return static_cast<int>(cudaGetLastError());
}

// Products over experts (see ogb_grouped_gemm_act), with an activation of every result.
extern "C" int ogb_grouped_gemm_f32(const float* A, const float* W, float* C, const int* group_tab, const int* group_mtiles, int max_rows,
                                    int max_mtiles, int N, int K, int lda, int ldw, int ldc, int act, float act_a, float act_b, void* stream) {
  if (max_rows <= 0 || max_mtiles <= 0 || N <= 0) return 0;
  if (act_gated(act)) return -7;
  const dim3 grid((N + kF32Tile - 1) / kF32Tile, 2 * max_mtiles);
  gemm_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(A, W, C, max_rows, N, K, lda, ldw, ldc, 0, 0, group_tab, group_mtiles,
                                                                       ActArgs{act, act_a, act_b});
  return static_cast<int>(cudaGetLastError());
}
