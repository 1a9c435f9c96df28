// Short causal convolutions over time, one filter per channel, over the rows of a step:
//
//   y_t = sum_j w[j] (u_(t - taps + 1 + j) + bias)      zeros stand before the sequence's first token
//
// together with what follows the convolution, so that a projected row is read once and its results land where the next kernel
// wants them:
//
//   conv_rope_append   attention: rotate queries and keys (the first rot_dims of every head), queries to a dense buffer, keys and
//                      values to their page
//   conv_unit_gates    delta rule: silu, queries and keys to unit length per head, decay and step size of every head
//
// A block is one decode row or kCvRows rows of one prefill chunk; a thread keeps its channels' filter and the last taps - 1 inputs
// in registers and walks the rows.  Inputs from before the chunk come from the sequence's slot ([slots][taps - 1][channels],
// oldest first); only the block with the chunk's first row reads a slot, so it also leaves the chunk's last inputs there.
#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kCvRows = 16;                    // divides the scheduler's 64-row tiles

struct ConvIn {
  const void* u;           // [rows, ldu] projected channels
  const float* w;          // [taps, C]
  const float* bias;       // [C] or null
  float* state;            // [slots, taps - 1, C]
  int ldu, C, taps;
  StepRows sr;
  int* status;
};

// the rows of this block and the sequence they belong to
struct ConvRows {
  int base, n, j0, j1, start, slot;            // first row of the entry, its rows, this block's rows within them, tokens before, slot
  OGB_DEVICE bool set(const ConvIn& p) {
    const StepRows& sr = p.sr;
    int entry;
    if (static_cast<int>(blockIdx.x) < sr.num_decode) {
      entry = blockIdx.x; base = entry; n = 1; j0 = 0;
    } else {
      const int g = blockIdx.x - sr.num_decode, tile = g / (64 / kCvRows), s = sr.tile_seq[tile];
      entry = sr.num_decode + s;
      base = sr.num_decode + sr.cu_q[s];
      n = sr.cu_q[s + 1] - sr.cu_q[s];
      j0 = sr.tile_q0[tile] + (g % (64 / kCvRows)) * kCvRows;
    }
    if (j0 >= n) return false;
    j1 = min(j0 + kCvRows, n);
    const int ctx = sr.ctx_len[entry];
    start = ctx - n;
    slot = sr.state_slot[entry];
    if (slot >= sr.num_slots) {
      if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
      slot = -1;
    }
    return ctx > 0 && start >= 0;              // padding rows have no tokens
  }
};

// V neighbouring channels of one thread.  TM >= taps: the filter is aligned to its last tap.
template <typename T, int V, int TM>
struct ConvWalk {
  float w[TM][V], h[TM > 1 ? TM - 1 : 1][V], b[V];
  const T* u;
  int ldu;

  OGB_DEVICE void init(const ConvIn& p, const ConvRows& r, int c) {
    u = static_cast<const T*>(p.u) + static_cast<size_t>(r.base) * p.ldu + c;
    ldu = p.ldu;
#pragma unroll
    for (int v = 0; v < V; ++v) b[v] = 0.f;
    if (p.bias != nullptr) load_vec<V>(p.bias + c, b);
#pragma unroll
    for (int i = 0; i < TM; ++i) {
      const int tap = i - (TM - p.taps);
#pragma unroll
      for (int v = 0; v < V; ++v) w[i][v] = 0.f;
      if (tap >= 0) load_vec<V>(p.w + static_cast<size_t>(tap) * p.C + c, w[i]);
    }
    float* st = r.slot >= 0 ? p.state + static_cast<size_t>(r.slot) * (p.taps - 1) * p.C + c : nullptr;
#pragma unroll
    for (int i = 0; i < TM - 1; ++i) {
      const int t = r.j0 - (TM - 1) + i, row = i - (TM - p.taps);     // time within the chunk, row of the slot
#pragma unroll
      for (int v = 0; v < V; ++v) h[i][v] = 0.f;
      if (row >= 0) {
        if (t >= 0) load(t, h[i]);
        else if (st != nullptr && r.start + t >= 0 && p.taps - 1 + t >= 0) load_vec<V>(st + static_cast<size_t>(p.taps - 1 + t) * p.C, h[i]);
      }
    }
    if (r.j0 == 0 && st != nullptr) {
#pragma unroll
      for (int i = 0; i < TM - 1; ++i) {
        const int t = r.n - (TM - 1) + i, row = i - (TM - p.taps);
        float s[V];
#pragma unroll
        for (int k = 0; k < TM - 1; ++k)       // fewer rows than taps: the older inputs move up
#pragma unroll
          for (int v = 0; v < V; ++v) s[v] = (k == 0 || k == i + r.n) ? h[k][v] : s[v];
        if (t >= 0) load(t, s);
        if (row >= 0) store_vec<V>(st + static_cast<size_t>(row) * p.C, s);
      }
    }
  }
  OGB_DEVICE void load(int t, float (&x)[V]) const {
    load_vec<V>(u + static_cast<size_t>(t) * ldu, x);
#pragma unroll
    for (int v = 0; v < V; ++v) x[v] += b[v];
  }
  OGB_DEVICE void next(int t, float (&y)[V]) {
    float x[V];
    load(t, x);
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float a = w[TM - 1][v] * x[v];
#pragma unroll
      for (int i = 0; i < TM - 1; ++i) a = fmaf(w[i][v], h[i][v], a);
      y[v] = a;
#pragma unroll
      for (int i = 0; i + 1 < TM - 1; ++i) h[i][v] = h[i + 1][v];
      if (TM > 1) h[TM > 1 ? TM - 2 : 0][v] = x[v];
    }
  }
};

// ------------------------------------------------------------------------------------------------------
// attention.  Channels of a row: q (nq heads of d) | k (nk heads of d) | v (nv heads of dv).  A page holds
// [nk][16][dp] keys, then [nv][16][vp] values.
// ------------------------------------------------------------------------------------------------------
struct RopeParams {
  ConvIn in;
  void* q;                 // [rows, ldq], head h at column h * dp
  void* pool;
  const int* slots;
  const double* freq;      // [rot_dims / 2]
  int64_t num_slots, page_elems;
  int nq, nk, nv, d, dv, dp, vp, rot, ldq;
};

template <typename T, int V, int TM>
__global__ void __launch_bounds__(128) conv_rope_append_kernel(RopeParams p) {
  extern __shared__ float2 s_rot[];            // [kCvRows][rot / 2] cos, sin
  ConvRows r;
  if (!r.set(p.in)) return;
  const int half = p.rot / 2;
  for (int i = threadIdx.x; i < (r.j1 - r.j0) * half; i += blockDim.x) {
    // the angle is reduced in double, so that it is good to fp32 at every position
    const double a = static_cast<double>(r.start + r.j0 + i / half) * p.freq[i % half] * 0.15915494309189535;
    float s, c;
    sincospif(static_cast<float>(2.0 * (a - rint(a))), &s, &c);
    s_rot[i] = make_float2(c, s);
  }
  __syncthreads();
  const int pairs = half / V, per = pairs + (p.d - p.rot) / V, perv = p.dv / V;
  const int nqk = p.nq + p.nk, total = nqk * per + p.nv * perv;
  const int item = blockIdx.y * blockDim.x + threadIdx.x;
  if (item >= total) return;
  const int v0 = nqk * p.d;                    // first value channel
  if (item < nqk * per) {
    const int head = item / per, e = item - head * per;
    const bool pair = e < pairs, is_q = head < p.nq;
    const int c = pair ? e * V : p.rot + (e - pairs) * V;
    ConvWalk<T, V, TM> a, b;
    a.init(p.in, r, head * p.d + c);
    if (pair) b.init(p.in, r, head * p.d + c + half);
    for (int t = r.j0; t < r.j1; ++t) {
      float x[V], y[V];
      a.next(t, x);
      if (pair) {
        b.next(t, y);
#pragma unroll
        for (int v = 0; v < V; ++v) {
          const float2 cs = s_rot[(t - r.j0) * half + c + v];
          const float xr = x[v] * cs.x - y[v] * cs.y;
          y[v] = y[v] * cs.x + x[v] * cs.y;
          x[v] = xr;
        }
      }
      T* dst;
      if (is_q) {
        dst = static_cast<T*>(p.q) + static_cast<size_t>(r.base + t) * p.ldq + head * p.dp + c;
      } else {
        const int64_t slot = p.slots[r.base + t];
        if (slot < 0) continue;
        if (slot >= p.num_slots) { atomicOr(p.in.status, kStatusIndexOutOfRange); continue; }
        dst = static_cast<T*>(p.pool) + (slot >> 4) * p.page_elems + ((head - p.nq) * 16 + (slot & 15)) * p.dp + c;
      }
      store_vec<V>(dst, x);
      if (pair) store_vec<V>(dst + half, y);
    }
  } else {
    const int e = item - nqk * per, head = e / perv, c = (e - head * perv) * V;
    ConvWalk<T, V, TM> a;
    a.init(p.in, r, v0 + head * p.dv + c);
    for (int t = r.j0; t < r.j1; ++t) {
      float x[V];
      a.next(t, x);
      const int64_t slot = p.slots[r.base + t];
      if (slot < 0 || slot >= p.num_slots) continue;
      store_vec<V>(static_cast<T*>(p.pool) + (slot >> 4) * p.page_elems + static_cast<int64_t>(p.nk) * 16 * p.dp +
                       (head * 16 + (slot & 15)) * p.vp + c, x);
    }
  }
}

// ------------------------------------------------------------------------------------------------------
// delta rule.  Channels of a row: q (nk heads of d) | k (nk heads of d) | v (nv heads of dv).  One warp per head and block.
// ------------------------------------------------------------------------------------------------------
struct UnitParams {
  ConvIn in;
  const float* ab;         // [rows, ldab]: decay projection (nv) | step-size projection (nv)
  const float* a_log;      // [nv]
  const float* dt_bias;    // [nv]
  float* qk;               // [rows, 2 * nk * d] unit vectors, q times d^(-1/2)
  void* v;                 // [rows, nv * dv]
  float2* gates;           // [rows, nv]: log of the decay, step size
  int nk, nv, d, dv, ldab;
};

template <typename T, int V, int TM, int NC>
__global__ void __launch_bounds__(128) conv_unit_gates_kernel(UnitParams p) {
  ConvRows r;
  if (!r.set(p.in)) return;
  const int lane = threadIdx.x & 31;
  int item = blockIdx.y * 4 + (threadIdx.x >> 5);
  constexpr int kSpan = 32 * V * NC;           // channels a warp covers
  if (item < 2 * p.nk) {
    ConvWalk<T, V, TM> walk[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if ((i * 32 + lane) * V < p.d) walk[i].init(p.in, r, item * p.d + (i * 32 + lane) * V);
    const float scale = item < p.nk ? 1.f / sqrtf(static_cast<float>(p.d)) : 1.f;
    for (int t = r.j0; t < r.j1; ++t) {
      float y[NC][V], ss = 0.f;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if ((i * 32 + lane) * V < p.d) {
          walk[i].next(t, y[i]);
#pragma unroll
          for (int v = 0; v < V; ++v) {
            y[i][v] = y[i][v] / (1.f + expf(-y[i][v]));
            ss = fmaf(y[i][v], y[i][v], ss);
          }
        }
      const float inv = scale / sqrtf(warp_sum(ss) + 1e-6f);
      float* dst = p.qk + static_cast<size_t>(r.base + t) * (2 * p.nk * p.d) + item * p.d;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if ((i * 32 + lane) * V < p.d) {
#pragma unroll
          for (int v = 0; v < V; ++v) y[i][v] *= inv;
          store_vec<V>(dst + (i * 32 + lane) * V, y[i]);
        }
    }
    return;
  }
  item -= 2 * p.nk;
  const int segs = (p.dv + kSpan - 1) / kSpan;
  if (item < p.nv * segs) {
    const int head = item / segs, c0 = (item % segs) * kSpan;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = c0 + (i * 32 + lane) * V;
      if (c >= p.dv) continue;
      ConvWalk<T, V, TM> walk;
      walk.init(p.in, r, 2 * p.nk * p.d + head * p.dv + c);
      for (int t = r.j0; t < r.j1; ++t) {
        float y[V];
        walk.next(t, y);
#pragma unroll
        for (int v = 0; v < V; ++v) y[v] = y[v] / (1.f + expf(-y[v]));
        store_vec<V>(static_cast<T*>(p.v) + static_cast<size_t>(r.base + t) * (p.nv * p.dv) + head * p.dv + c, y);
      }
    }
    return;
  }
  if (item > p.nv * segs) return;
  for (int i = lane; i < (r.j1 - r.j0) * p.nv; i += 32) {
    const int row = r.base + r.j0 + i / p.nv, h = i % p.nv;
    const float* src = p.ab + static_cast<size_t>(row) * p.ldab;
    const float z = src[h] + p.dt_bias[h];
    const float soft = z > 20.f ? z : log1pf(expf(z));
    p.gates[static_cast<size_t>(row) * p.nv + h] = make_float2(-expf(p.a_log[h]) * soft, 1.f / (1.f + expf(-src[p.nv + h])));
  }
}

template <typename T, int V, int TM>
static int launch_rope(const RopeParams& p, cudaStream_t stream) {
  const int per = p.rot / 2 / V + (p.d - p.rot) / V, total = (p.nq + p.nk) * per + p.nv * (p.dv / V);
  const int threads = total < 128 ? (total + 31) / 32 * 32 : 128;
  const dim3 grid(p.in.sr.num_decode + p.in.sr.num_tiles * (64 / kCvRows), (total + threads - 1) / threads);
  conv_rope_append_kernel<T, V, TM><<<grid, threads, kCvRows * (p.rot / 2) * sizeof(float2), stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int V, int TM, int NC>
static int launch_unit(const UnitParams& p, cudaStream_t stream) {
  const int items = 2 * p.nk + p.nv * ((p.dv + 32 * V * NC - 1) / (32 * V * NC)) + 1;
  const dim3 grid(p.in.sr.num_decode + p.in.sr.num_tiles * (64 / kCvRows), (items + 3) / 4);
  conv_unit_gates_kernel<T, V, TM, NC><<<grid, 128, 0, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// four channels at a time: their places in the projected row, the filters and the outputs start on four elements
template <typename T>
static bool conv_aligned(const ConvIn& in, const void* out0, const void* out1, int sizes) {
  const uintptr_t act = reinterpret_cast<uintptr_t>(in.u) | reinterpret_cast<uintptr_t>(out0) | reinterpret_cast<uintptr_t>(out1);
  const uintptr_t f32 = reinterpret_cast<uintptr_t>(in.w) | reinterpret_cast<uintptr_t>(in.bias) | reinterpret_cast<uintptr_t>(in.state);
  return ((sizes | in.ldu) & 3) == 0 && (f32 & 15) == 0 && (act & (4 * sizeof(T) - 1)) == 0;
}

template <typename T>
static int dispatch_rope(const RopeParams& p, cudaStream_t s) {
  const int half = p.rot / 2;
  const bool vec = conv_aligned<T>(p.in, p.q, p.pool, half | p.d | p.dv);
  if (p.in.taps <= 4) return vec ? launch_rope<T, 4, 4>(p, s) : launch_rope<T, 1, 4>(p, s);
  return vec ? launch_rope<T, 4, 8>(p, s) : launch_rope<T, 1, 8>(p, s);
}
template <typename T>
static int dispatch_unit(const UnitParams& p, cudaStream_t s) {
  const bool vec = conv_aligned<T>(p.in, p.v, nullptr, p.d | p.dv) && (reinterpret_cast<uintptr_t>(p.qk) & 15) == 0;
  if (p.in.taps <= 4) {
    if (!vec) return launch_unit<T, 1, 4, 8>(p, s);
    return p.d <= 128 ? launch_unit<T, 4, 4, 1>(p, s) : launch_unit<T, 4, 4, 2>(p, s);
  }
  if (!vec) return launch_unit<T, 1, 8, 8>(p, s);
  return p.d <= 128 ? launch_unit<T, 4, 8, 1>(p, s) : launch_unit<T, 4, 8, 2>(p, s);
}

}  // namespace ogb

using namespace ogb;

extern "C" int ogb_conv_rope_append(const void* u, int ldu, const float* w, const float* bias, float* state, int taps, void* q, int ldq, void* pool,
                                    const int* slots, const double* freq, int64_t num_slots, int64_t page_elems, int nq, int nk, int nv, int d, int dv,
                                    int dp, int vp, int rot, const int* ctx_len, const int* state_slot, const int* cu_q, const int* tile_seq,
                                    const int* tile_q0, int num_decode, int num_tiles, int state_slots, int elem, int* status, void* stream) {
  if (num_decode + num_tiles <= 0) return 0;
  if (taps < 1 || taps > 8 || rot < 0 || rot > d || (rot & 1) || rot > 512 || dp < d || vp < dv || (ldq & 3) || (dp & 3) || (vp & 3) || (page_elems & 3))
    return -3;
  if (taps > 1 && state == nullptr) return -3;
  RopeParams p{ConvIn{u, w, bias, state, ldu, (nq + nk) * d + nv * dv, taps,
                      StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, state_slots}, status},
               q, pool, slots, freq, num_slots, page_elems, nq, nk, nv, d, dv, dp, vp, rot, ldq};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return dispatch_rope<__nv_bfloat16>(p, s);
  if (elem == kElemF32) return dispatch_rope<float>(p, s);
  return -3;
}

extern "C" int ogb_conv_unit_gates(const void* u, int ldu, const float* w, float* state, int taps, const float* ab, int ldab, const float* a_log,
                                   const float* dt_bias, float* qk, void* v, void* gates, int nk, int nv, int d, int dv, const int* ctx_len,
                                   const int* state_slot, const int* cu_q, const int* tile_seq, const int* tile_q0, int num_decode, int num_tiles,
                                   int state_slots, int elem, int* status, void* stream) {
  if (num_decode + num_tiles <= 0) return 0;
  if (taps < 1 || taps > 8 || d < 1 || d > 256) return -3;
  if (taps > 1 && state == nullptr) return -3;
  UnitParams p{ConvIn{u, w, nullptr, state, ldu, 2 * nk * d + nv * dv, taps,
                      StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, state_slots}, status},
               ab, a_log, dt_bias, qk, v, static_cast<float2*>(gates), nk, nv, d, dv, ldab};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return dispatch_unit<__nv_bfloat16>(p, s);
  if (elem == kElemF32) return dispatch_unit<float>(p, s);
  return -3;
}
