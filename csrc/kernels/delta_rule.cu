// Gated delta rule over per-sequence state.  Per head, with decay g, step size beta, unit key k and query q:
//
//   S <- g S      u = beta (v - S^T k)      S <- S + k u^T      o = S^T q
//
// delta_step_kernel walks the rows of one (head, sequence) with the state in registers, laid out as in hgrn2_kernel: a warp owns
// 16 value columns (8 for states of 256 rows), its 16 lane pairs own every sixteenth quad of state rows.  S^T k and S^T q are
// taken from the state before the write in one exchange between the lanes -- the read-out after it is g S^T q + (k . q) u -- so a
// token costs one halving exchange and one broadcast of u.  The state is stored [slot][head][column][row], fp32 like all
// arithmetic here.  The gated norm of the read-out follows in head_rmsnorm_kernel.
#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

struct DeltaParams {
  const float* qk;         // [rows, 2 * groups * D]: queries | keys
  const void* v;           // [rows, heads * V]
  const float2* gates;     // [rows, heads]: log decay, step size
  float* state;            // [slots, heads, V, DP]
  float* out;              // [rows, heads * V]
  int heads, groups, D, V, z0;
  StepRows sr;
  int* status;
};

// rows of work item z: a decode row or a whole prefill chunk
struct DeltaItem {
  int entry, base, n, slot;
  bool fresh;
  OGB_DEVICE bool set(const DeltaParams& p, int z) {
    const StepRows& sr = p.sr;
    entry = z;
    base = z; n = 1;
    if (z >= sr.num_decode) {
      const int s = z - sr.num_decode;
      base = sr.num_decode + sr.cu_q[s];
      n = sr.cu_q[s + 1] - sr.cu_q[s];
    }
    const int ctx = sr.ctx_len[entry];
    slot = sr.state_slot[entry];
    if (ctx <= 0 || slot < 0 || n <= 0) return false;
    if (slot >= sr.num_slots) {
      if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
      return false;
    }
    fresh = ctx <= n;
    return true;
  }
};

constexpr int kDeltaTok = 8;

template <typename T, int DP, int CPT>
__global__ void __launch_bounds__(256, 2) delta_step_kernel(DeltaParams p) {
  constexpr int QPT = DP / 64, kMaxCols = 16 * CPT, NV = 2 * CPT;
  __shared__ __align__(16) float sq[kDeltaTok][DP], sk[kDeltaTok][DP], sv[kDeltaTok][kMaxCols];
  __shared__ float sg[kDeltaTok], sb[kDeltaTok], skq[kDeltaTok];
  const int threads = blockDim.x, ncols = threads / 32 * 2 * CPT, head = blockIdx.y, col0 = blockIdx.x * ncols;
  DeltaItem it;
  if (!it.set(p, blockIdx.z + p.z0)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 15;
  const int lc = (warp * 2 + (lane >> 4)) * CPT;
  const int group = head / (p.heads / p.groups);
  float* own = p.state + (static_cast<size_t>(it.slot) * p.heads + head) * p.V * DP;
  f32x2 s[CPT][QPT][2];
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int i = 0; i < QPT; ++i) {
      ulonglong2 x = make_ulonglong2(0ull, 0ull);
      if (!it.fresh && col0 + lc + c < p.V) x = *reinterpret_cast<const ulonglong2*>(own + static_cast<size_t>(col0 + lc + c) * DP + (i * 16 + g) * 4);
      s[c][i][0] = x.x;
      s[c][i][1] = x.y;
    }
  for (int t0 = 0; t0 < it.n; t0 += kDeltaTok) {
    const int nt = min(kDeltaTok, it.n - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * DP; i += threads) {
      const int t = i / DP, d = i % DP;
      const float* src = p.qk + static_cast<size_t>(it.base + t0 + t) * (2 * p.groups * p.D) + group * p.D + d;
      sq[t][d] = d < p.D ? src[0] : 0.f;
      sk[t][d] = d < p.D ? src[p.groups * p.D] : 0.f;
    }
    for (int i = threadIdx.x; i < nt * ncols; i += threads) {
      const int t = i / ncols, c = i - t * ncols;
      sv[t][c] = col0 + c < p.V ? to_f32<T>(static_cast<const T*>(p.v)[static_cast<size_t>(it.base + t0 + t) * (p.heads * p.V) + head * p.V + col0 + c]) : 0.f;
    }
    if (static_cast<int>(threadIdx.x) < nt) {
      const float2 x = p.gates[static_cast<size_t>(it.base + t0 + threadIdx.x) * p.heads + head];
      sg[threadIdx.x] = expf(x.x);
      sb[threadIdx.x] = x.y;
    }
    __syncthreads();
    for (int t = warp; t < nt; t += threads / 32) {
      float a = 0.f;
      for (int d = lane; d < DP; d += 32) a = fmaf(sq[t][d], sk[t][d], a);
      a = warp_sum(a);
      if (lane == 0) skq[t] = a;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      f32x2 k[QPT][2], q[QPT][2];
#pragma unroll
      for (int i = 0; i < QPT; ++i) {
        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(&sk[t][(i * 16 + g) * 4]);
        const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&sq[t][(i * 16 + g) * 4]);
        k[i][0] = a.x; k[i][1] = a.y;
        q[i][0] = b.x; q[i][1] = b.y;
      }
      float r[NV];                             // S^T k of the CPT columns, then S^T q
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        f32x2 a = f2_mul(k[0][0], s[c][0][0]), b = f2_mul(q[0][0], s[c][0][0]);
#pragma unroll
        for (int i = 0; i < QPT; ++i)
#pragma unroll
          for (int h = 0; h < 2; ++h)
            if ((i | h) != 0) {
              a = f2_fma(k[i][h], s[c][i][h], a);
              b = f2_fma(q[i][h], s[c][i][h], b);
            }
        r[c] = f2_sum(a);
        r[CPT + c] = f2_sum(b);
      }
      // lanes halve the values they carry: lane g ends with the sum of value `mine`
      int mine = 0;
#pragma unroll
      for (int w = CPT, bit = 1; w >= 1; w >>= 1, bit <<= 1) {
        const bool up = (g & bit) != 0;
#pragma unroll
        for (int c = 0; c < w; ++c) {
          const float send = up ? r[c] : r[c + w], keep = up ? r[c + w] : r[c];
          r[c] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
        mine += up ? w : 0;
      }
#pragma unroll
      for (int bit = NV; bit < 16; bit <<= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], bit);
      const float decay = sg[t], beta = sb[t];
      float u[CPT], mu = 0.f;                  // u of every column of the lane group, and of the column of `mine`
      const float du = mine < CPT ? beta * (sv[t][lc + mine] - decay * r[0]) : 0.f;
      f32x2 dec;
      asm("mov.b64 %0, {%1, %1};" : "=l"(dec) : "f"(decay));
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        int src = 0;                           // the lane whose `mine` is c
#pragma unroll
        for (int w = CPT / 2, bit = 2; w >= 1; w >>= 1, bit <<= 1) src |= (c & w) != 0 ? bit : 0;
        u[c] = __shfl_sync(0xffffffffu, du, (lane & 16) | src);
        if (mine == CPT + c) mu = u[c];
        f32x2 uu;
        asm("mov.b64 %0, {%1, %1};" : "=l"(uu) : "f"(u[c]));
#pragma unroll
        for (int i = 0; i < QPT; ++i)
#pragma unroll
          for (int h = 0; h < 2; ++h) s[c][i][h] = f2_fma(k[i][h], uu, f2_mul(dec, s[c][i][h]));
      }
      if (mine >= CPT && g < NV && col0 + lc + mine - CPT < p.V)
        p.out[static_cast<size_t>(it.base + t0 + t) * (p.heads * p.V) + head * p.V + col0 + lc + mine - CPT] = fmaf(decay, r[0], skq[t] * mu);
    }
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int i = 0; i < QPT; ++i)
      if (col0 + lc + c < p.V)
        *reinterpret_cast<ulonglong2*>(own + static_cast<size_t>(col0 + lc + c) * DP + (i * 16 + g) * 4) = make_ulonglong2(s[c][i][0], s[c][i][1]);
}

template <typename T, int DP, int CPT>
static int launch_delta_step(const DeltaParams& p, int items, cudaStream_t stream) {
  if (items <= 0) return 0;
  int warps = (p.V + 2 * CPT - 1) / (2 * CPT);
  if (warps > 8) warps = 8;
  const dim3 grid((p.V + warps * 2 * CPT - 1) / (warps * 2 * CPT), p.heads, items);
  delta_step_kernel<T, DP, CPT><<<grid, warps * 32, 0, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}
template <typename T>
static int dispatch_delta_step(const DeltaParams& p, int items, cudaStream_t s) {
  if (p.D <= 64) return launch_delta_step<T, 64, 8>(p, items, s);
  if (p.D <= 128) return launch_delta_step<T, 128, 8>(p, items, s);
  return launch_delta_step<T, 256, 4>(p, items, s);
}

}  // namespace ogb

using namespace ogb;

extern "C" int ogb_delta_rule(const float* qk, const void* v, const void* gates, float* state, float* out, int heads, int groups, int D, int V,
                              const int* ctx_len, const int* state_slot, const int* cu_q, int num_decode, int num_prefill, int num_slots, int elem,
                              int* status, void* stream) {
  if (num_decode + num_prefill <= 0 || heads <= 0 || V <= 0) return 0;
  if (D < 1 || D > 256 || groups < 1 || heads % groups != 0) return -3;
  DeltaParams p{qk, v, static_cast<const float2*>(gates), state, out, heads, groups, D, V, 0,
                StepRows{ctx_len, state_slot, cu_q, nullptr, nullptr, num_decode, 0, num_slots}, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (elem == kElemBF16) return dispatch_delta_step<__nv_bfloat16>(p, num_decode + num_prefill, s);
  if (elem == kElemF32) return dispatch_delta_step<float>(p, num_decode + num_prefill, s);
  return -3;
}
