// Gated linear recurrences over per-sequence state: HGRN2 (per-channel forget gate, the gate's complement is the key).
//
//   f = low + (1 - low) sigmoid(z + bias)      S <- diag(f) S + (1 - f) v^T      o = S^T silu(q)
//
// One CTA owns 32 value columns of one head of one sequence and walks the sequence's rows of the step, decode rows and
// prefill chunks alike.  A warp owns 4 columns; its 8 lane groups own every eighth quad of state rows, so a thread keeps
// D / 8 fp32 state values of one column in registers, the state is stored with the row index contiguous ([slot][head][column]
// [row]) and moves as coalesced 16-byte vectors, and a token costs two fused multiply-adds per state value plus a
// three-step lane reduction.  Gates and activations of the next tokens are fetched while the current ones run.
// All arithmetic is fp32.  The per-head norm and the cast follow in head_rmsnorm_kernel.
#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kRecThreads = 256;
constexpr int kRecCols = 32;       // value columns per CTA

struct RecParams {
  const float* qfv;       // [rows, ld]: q (heads * D) | z (heads * D) | v (heads * V)
  const float* bias;      // [heads * D] gate bias
  const float* low;       // [heads * D] lower bound of the gate
  float* state;           // [slots, heads, V, DP]
  float* out;             // [rows, ldo] raw head outputs (heads * V)
  int ld, ldo, heads, D, V;
  StepRows sr;
  int* status;
};

template <int DP>          // key channels, padded to 64, 128 or 256
__global__ void __launch_bounds__(kRecThreads) hgrn2_kernel(RecParams p) {
  constexpr int kRecTok = DP == 256 ? 8 : 16;    // tokens staged at a time
  constexpr int RPT = DP / 8;                    // state rows per thread
  constexpr int QPT = RPT / 4;                   // quads of rows
  constexpr int LPT = kRecTok * DP / kRecThreads;  // staged q (and z) values per thread
  __shared__ __align__(16) float sq[kRecTok][DP];
  __shared__ __align__(16) float sf[kRecTok][DP];
  __shared__ __align__(16) float sk[kRecTok][DP];
  __shared__ float sv[kRecTok][kRecCols];
  __shared__ float so[kRecTok][kRecCols];
  const int head = blockIdx.y, entry = blockIdx.z, col0 = blockIdx.x * kRecCols;
  const StepRows& sr = p.sr;
  int base, n;
  if (entry < sr.num_decode) {
    base = entry; n = 1;
  } else {
    const int s = entry - sr.num_decode;
    base = sr.num_decode + sr.cu_q[s];
    n = sr.cu_q[s + 1] - sr.cu_q[s];
  }
  const int ctx = sr.ctx_len[entry];
  const int slot = sr.state_slot[entry];
  if (n <= 0 || ctx <= 0 || slot < 0) return;    // padding row
  if (slot >= sr.num_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2;                       // row group
  const int lc = warp * 4 + (lane & 3);          // column within the CTA
  const int col = col0 + lc;
  const bool live = col < p.V;
  float4* st = reinterpret_cast<float4*>(p.state + ((static_cast<size_t>(slot) * p.heads + head) * p.V + (live ? col : 0)) * DP);
  float s[RPT];
#pragma unroll
  for (int i = 0; i < QPT; ++i) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ctx > n && live) v = st[i * 8 + g];
    s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
  }
  const int HD = p.heads * p.D;
  constexpr int VPT = kRecTok * kRecCols / kRecThreads;
  float rq[LPT], rz[LPT], rv[VPT];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int e = 0; e < LPT; ++e) {
      const int i = threadIdx.x + e * kRecThreads, t = t0 + i / DP, d = i % DP;
      const bool in = t < n && d < p.D;
      const float* row = p.qfv + static_cast<size_t>(base + t) * p.ld + head * p.D + d;
      rq[e] = in ? row[0] : 0.f;
      rz[e] = in ? row[HD] : 0.f;
    }
#pragma unroll
    for (int e = 0; e < VPT; ++e) {
      const int i = threadIdx.x + e * kRecThreads, t = t0 + i / kRecCols, c = col0 + i % kRecCols;
      rv[e] = (t < n && c < p.V) ? p.qfv[static_cast<size_t>(base + t) * p.ld + 2 * HD + head * p.V + c] : 0.f;
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < n; t0 += kRecTok) {
    __syncthreads();
#pragma unroll
    for (int e = 0; e < LPT; ++e) {
      const int i = threadIdx.x + e * kRecThreads, t = i / DP, d = i % DP;
      float q = 0.f, f = 0.f, k = 0.f;
      if (t0 + t < n && d < p.D) {
        const float low = p.low[head * p.D + d];
        const float z = rz[e] + p.bias[head * p.D + d];
        const float ez = expf(-fabsf(z));        // sigmoid of both signs from one exponential that cannot overflow
        const float small = ez / (1.f + ez), big = 1.f / (1.f + ez);
        f = fmaf(1.f - low, z >= 0.f ? big : small, low);
        k = (1.f - low) * (z >= 0.f ? small : big);   // 1 - f without the cancellation
        q = rq[e] / (1.f + expf(-rq[e]));
      }
      sq[t][d] = q; sf[t][d] = f; sk[t][d] = k;
    }
#pragma unroll
    for (int e = 0; e < VPT; ++e) {
      const int i = threadIdx.x + e * kRecThreads;
      sv[i / kRecCols][i % kRecCols] = rv[e];
    }
    __syncthreads();
    if (t0 + kRecTok < n) fetch(t0 + kRecTok);
    const int nt = min(kRecTok, n - t0);
    for (int t = 0; t < nt; ++t) {
      const float v = sv[t][lc];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < QPT; ++i) {
        const float4 f4 = *reinterpret_cast<const float4*>(&sf[t][(i * 8 + g) * 4]);
        const float4 k4 = *reinterpret_cast<const float4*>(&sk[t][(i * 8 + g) * 4]);
        const float4 q4 = *reinterpret_cast<const float4*>(&sq[t][(i * 8 + g) * 4]);
        s[4 * i] = fmaf(f4.x, s[4 * i], k4.x * v);
        s[4 * i + 1] = fmaf(f4.y, s[4 * i + 1], k4.y * v);
        s[4 * i + 2] = fmaf(f4.z, s[4 * i + 2], k4.z * v);
        s[4 * i + 3] = fmaf(f4.w, s[4 * i + 3], k4.w * v);
        o = fmaf(q4.x, s[4 * i], o);
        o = fmaf(q4.y, s[4 * i + 1], o);
        o = fmaf(q4.z, s[4 * i + 2], o);
        o = fmaf(q4.w, s[4 * i + 3], o);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 4);
      o += __shfl_xor_sync(0xffffffffu, o, 8);
      o += __shfl_xor_sync(0xffffffffu, o, 16);
      if (g == 0) so[t][lc] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * kRecCols; i += kRecThreads) {
      const int t = i / kRecCols, c = col0 + i % kRecCols;
      if (c < p.V) p.out[static_cast<size_t>(base + t0 + t) * p.ldo + head * p.V + c] = so[t][i % kRecCols];
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < QPT; ++i) st[i * 8 + g] = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
  }
}

}  // namespace ogb

using namespace ogb;

// Row width of the stored state for D key channels (0: not supported).
extern "C" int ogb_hgrn2_state_rows(int D) { return D <= 0 ? 0 : D <= 64 ? 64 : D <= 128 ? 128 : D <= 256 ? 256 : 0; }

extern "C" int ogb_hgrn2(const float* qfv, const float* bias, const float* low, float* state, float* out, int ld, int ldo, int heads, int D,
                         int V, const int* ctx_len, const int* state_slot, const int* cu_q, int num_decode, int num_prefill, int num_slots,
                         int* status, void* stream) {
  const int entries = num_decode + num_prefill;
  if (entries <= 0 || heads <= 0 || V <= 0) return 0;
  const int dp = ogb_hgrn2_state_rows(D);
  if (dp == 0) return -2;
  RecParams p{qfv, bias, low, state, out, ld, ldo, heads, D, V, StepRows{ctx_len, state_slot, cu_q, nullptr, nullptr, num_decode, 0, num_slots}, status};
  const dim3 grid((V + kRecCols - 1) / kRecCols, heads, entries);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dp == 64) hgrn2_kernel<64><<<grid, kRecThreads, 0, s>>>(p);
  else if (dp == 128) hgrn2_kernel<128><<<grid, kRecThreads, 0, s>>>(p);
  else hgrn2_kernel<256><<<grid, kRecThreads, 0, s>>>(p);
  return static_cast<int>(cudaGetLastError());
}
