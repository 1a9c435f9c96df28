// Gated linear recurrences over per-sequence state: HGRN2 (per-channel forget gate, the gate's complement is the key).
//
//   f = low + (1 - low) sigmoid(z + bias)      S <- diag(f) S + (1 - f) v^T      o = S^T silu(q)
//
// One CTA walks the rows of one (head, sequence) -- decode rows and prefill chunks alike -- with the state in registers: a warp
// owns 16 value columns (8 when the state is 256 rows high), its 16 lane pairs own every sixteenth quad of state rows, so a
// thread holds a block of rows x columns and three 16-byte shared-memory reads (gate, key, query of four rows) serve all
// its columns.  The arithmetic is packed fp32 (two rows per instruction); a row's outputs are summed over the lanes by a
// halving exchange.  Gates and activations of the next tokens are fetched while the current ones run.  The state is stored
// with the row index contiguous ([slot][head][column][row]) and moves as 16-byte vectors.  All arithmetic is fp32.
//
// Long prompts with few (head, sequence) pairs are cut into segments that run side by side: every segment first runs from a
// zero state (MODE kLocal) and leaves its state and the product of its gates, hgrn2_chain_kernel turns those into the state
// at each segment's start, and the second pass (MODE kFull) produces the outputs from there.
//
// The per-head norm and the cast follow in head_rmsnorm_kernel.
#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

struct RecParams {
  const float* qfv;       // [rows, ld]: q (heads * D) | z (heads * D) | v (heads * V)
  const float* bias;      // [heads * D] gate bias
  const float* low;       // [heads * D] lower bound of the gate
  float* state;           // [slots, heads, V, DP]
  float* out;             // [rows, ldo] raw head outputs (heads * V)
  float* seg_state;       // [segments, heads, V, DP] (segmented runs)
  float* seg_gate;        // [segments, heads, DP]
  int ld, ldo, heads, D, V, num_prefill, seg_len;   // seg_len 0: not segmented
  int z0;                 // first work item of the launch (decode rows come first)
  StepRows sr;
  int* status;
};

enum RecMode : int { kFull = 0, kLocal = 1 };

// Rows of work item z: a decode row, or a (segment of a) prefill chunk.
struct RecItem {
  int entry, base, n, first, seg;        // first: tokens of the chunk before this segment; seg: global segment index
  bool last;                             // the item ends its chunk
};
OGB_DEVICE bool rec_item(const RecParams& p, int z, RecItem& it) {
  const StepRows& sr = p.sr;
  it.seg = -1; it.first = 0; it.last = true;
  if (z < sr.num_decode) {
    it.entry = z; it.base = z; it.n = 1;
    return true;
  }
  z -= sr.num_decode;
  for (int s = 0, before = 0; s < p.num_prefill; ++s) {
    const int len = sr.cu_q[s + 1] - sr.cu_q[s];
    const int segs = p.seg_len > 0 ? (len + p.seg_len - 1) / p.seg_len : 1;
    if (z < before + segs) {
      it.entry = sr.num_decode + s;
      it.seg = z;
      it.first = p.seg_len > 0 ? (z - before) * p.seg_len : 0;
      it.n = p.seg_len > 0 ? min(p.seg_len, len - it.first) : len;
      it.last = z - before == segs - 1;
      it.base = sr.num_decode + sr.cu_q[s] + it.first;
      return it.n > 0;
    }
    before += segs;
  }
  return false;
}

// State at a segment's start: the end of the segment before, or -- for the first one -- the sequence's state, which the chain
// kernel has put into the place of the last segment (whose own end state goes straight to the sequence).
OGB_DEVICE const float* rec_segment_start(const RecParams& p, const RecItem& it, int head, size_t head_state) {
  int seg = it.seg - 1;
  if (it.first == 0) {
    const int s = it.entry - p.sr.num_decode, len = p.sr.cu_q[s + 1] - p.sr.cu_q[s];
    seg = it.seg + (len + p.seg_len - 1) / p.seg_len - 1;
  }
  return p.seg_state + (static_cast<size_t>(seg) * p.heads + head) * head_state;
}

template <int DP, int CPT>
struct RecCfg {
  static constexpr int kTok = DP == 256 ? 8 : 16;       // tokens staged at a time
  static constexpr int kMaxCols = 8 * 2 * CPT;          // columns of a CTA of eight warps
  static constexpr int kSmemBytes = 4 * (kTok * (3 * DP + 3 * kMaxCols) + 2 * DP + 2 * kTok * (2 * DP + kMaxCols));
};

template <int DP, int CPT, int MODE>
__global__ void __launch_bounds__(256, 2) hgrn2_kernel(RecParams p) {
  constexpr int QPT = DP / 64;                   // quads of state rows per thread
  constexpr int kTok = RecCfg<DP, CPT>::kTok, kMaxCols = RecCfg<DP, CPT>::kMaxCols;
  extern __shared__ __align__(16) uint8_t rec_smem[];
  typedef float Row[DP];
  Row* sq = reinterpret_cast<Row*>(rec_smem);                                    // [kTok][DP]: query, gate, key
  Row* sf = sq + kTok;
  Row* sk = sf + kTok;
  typedef float2 VRow[kMaxCols];
  VRow* sv = reinterpret_cast<VRow*>(sk + kTok);                                 // every value twice: the packed operand of its column
  typedef float ORow[kMaxCols];
  ORow* so = reinterpret_cast<ORow*>(sv + kTok);
  float* slow = reinterpret_cast<float*>(so + kTok);                             // [DP] lower bound, bias
  float* sbias = slow + DP;
  float* raw = sbias + DP;                                                       // [2][kTok][2 * DP + kMaxCols]: the rows as they come
  constexpr int kRaw = 2 * DP + kMaxCols;
  const int threads = blockDim.x, ncols = threads / 32 * 2 * CPT;
  const int head = blockIdx.y, col0 = blockIdx.x * ncols;
  RecItem it;
  if (!rec_item(p, blockIdx.z + p.z0, it)) return;
  if (MODE == kLocal && it.last) return;         // nothing follows this segment: its end state comes out of the second pass
  const StepRows& sr = p.sr;
  const int ctx = sr.ctx_len[it.entry];
  const int slot = sr.state_slot[it.entry];
  if (ctx <= 0 || slot < 0) return;              // padding row
  if (slot >= sr.num_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane & 15;                       // row group
  const int lc = (warp * 2 + (lane >> 4)) * CPT; // first column within the CTA
  const size_t head_state = static_cast<size_t>(p.V) * DP;
  float* own = p.state + (static_cast<size_t>(slot) * p.heads + head) * head_state;
  float* segs = it.seg >= 0 && p.seg_len > 0 ? p.seg_state + (static_cast<size_t>(it.seg) * p.heads + head) * head_state : nullptr;
  // where the run starts: zero, the sequence's slot, or the chained state of the segment before
  const float* init = nullptr;
  if (MODE == kFull) {
    if (segs != nullptr && (it.first > 0 || !it.last)) init = rec_segment_start(p, it, head, head_state);
    else if (ctx - (sr.num_decode > it.entry ? 1 : sr.cu_q[it.entry - sr.num_decode + 1] - sr.cu_q[it.entry - sr.num_decode]) > 0) init = own;
  }
  f32x2 s[CPT][QPT][2];
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int i = 0; i < QPT; ++i) {
      ulonglong2 v = make_ulonglong2(0ull, 0ull);
      if (init != nullptr && col0 + lc + c < p.V) v = *reinterpret_cast<const ulonglong2*>(init + static_cast<size_t>(col0 + lc + c) * DP + (i * 16 + g) * 4);
      s[c][i][0] = v.x;
      s[c][i][1] = v.y;
    }
  float gate = 1.f;                              // MODE kLocal: product of the gates of row threadIdx.x
  const int HD = p.heads * p.D;
  for (int d = threadIdx.x; d < p.D; d += threads) { slow[d] = p.low[head * p.D + d]; sbias[d] = p.bias[head * p.D + d]; }
  // rows of the next tokens on their way while the current ones run: q, z, v side by side
  const bool vec = ((p.D | p.V | p.ld) & 3) == 0;
  auto fetch = [&](int t0, int buf) {
    const int nt = min(kTok, it.n - t0), nv = min(ncols, p.V - col0);
    const int step = vec ? 4 : 1, per = (2 * p.D + nv + step - 1) / step;
    for (int i = threadIdx.x; i < nt * per; i += threads) {
      const int t = i / per, e = (i - t * per) * step;
      const float* src = p.qfv + static_cast<size_t>(it.base + t0 + t) * p.ld;
      float* dst = raw + (buf * kTok + t) * kRaw;
      if (e < p.D) { src += head * p.D + e; dst += e; }
      else if (e < 2 * p.D) { src += HD + head * p.D + e - p.D; dst += DP + e - p.D; }
      else { src += 2 * HD + head * p.V + col0 + e - 2 * p.D; dst += 2 * DP + e - 2 * p.D; }
      if (vec) cp_async<16>(dst, src); else cp_async<4>(dst, src);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  for (int t0 = 0, buf = 0; t0 < it.n; t0 += kTok, buf ^= 1) {
    const int nt = min(kTok, it.n - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t0 + kTok < it.n) fetch(t0 + kTok, buf ^ 1);
    for (int i = threadIdx.x; i < nt * DP; i += threads) {
      const int t = i / DP, d = i % DP;
      const float* row = raw + (buf * kTok + t) * kRaw;
      float q = 0.f, f = 0.f, k = 0.f;
      if (d < p.D) {
        const float low = slow[d], z = row[DP + d] + sbias[d];
        const float ez = __expf(-fabsf(z));      // sigmoid of both signs from one exponential that cannot overflow
        const float r = __fdividef(1.f, 1.f + ez), small = ez * r;
        f = fmaf(1.f - low, z >= 0.f ? r : small, low);
        k = (1.f - low) * (z >= 0.f ? small : r);     // 1 - f without the cancellation
        if (MODE == kFull) { const float x = row[d]; q = __fdividef(x, 1.f + __expf(fminf(-x, 80.f))); }
      }
      if (MODE == kFull) sq[t][d] = q;
      sf[t][d] = f; sk[t][d] = k;
    }
    for (int i = threadIdx.x; i < nt * ncols; i += threads) {
      const int t = i / ncols, c = i - t * ncols;
      const float v = col0 + c < p.V ? raw[(buf * kTok + t) * kRaw + 2 * DP + c] : 0.f;
      sv[t][c] = make_float2(v, v);
    }
    __syncthreads();
    if (MODE == kLocal && blockIdx.x == 0) {
      if (static_cast<int>(threadIdx.x) < DP)
        for (int t = 0; t < nt; ++t) gate *= sf[t][threadIdx.x];
    }
    // two tokens at a time, so that their lane sums share the steps of one exchange
    for (int t = 0; t < nt; t += 2) {
      f32x2 o[2][CPT];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        if (u == 1 && t + 1 >= nt) {
#pragma unroll
          for (int c = 0; c < CPT; ++c) o[1][c] = 0ull;
          break;
        }
        f32x2 f[QPT][2], k[QPT][2], q[QPT][2];
#pragma unroll
        for (int i = 0; i < QPT; ++i) {
          const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(&sf[t + u][(i * 16 + g) * 4]);
          const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&sk[t + u][(i * 16 + g) * 4]);
          f[i][0] = a.x; f[i][1] = a.y;
          k[i][0] = b.x; k[i][1] = b.y;
          if (MODE == kFull) {
            const ulonglong2 c = *reinterpret_cast<const ulonglong2*>(&sq[t + u][(i * 16 + g) * 4]);
            q[i][0] = c.x; q[i][1] = c.y;
          }
        }
#pragma unroll
        for (int c2 = 0; c2 < CPT / 2; ++c2) {
          const ulonglong2 v2 = *reinterpret_cast<const ulonglong2*>(&sv[t + u][lc + 2 * c2]);
#pragma unroll
          for (int cc = 0; cc < 2; ++cc) {
            const int c = 2 * c2 + cc;
            const f32x2 v = cc == 0 ? v2.x : v2.y;
#pragma unroll
            for (int i = 0; i < QPT; ++i)
#pragma unroll
              for (int h = 0; h < 2; ++h) {
                s[c][i][h] = f2_fma(f[i][h], s[c][i][h], f2_mul(k[i][h], v));
                if (MODE == kFull) o[u][c] = (i | h) == 0 ? f2_mul(q[i][h], s[c][i][h]) : f2_fma(q[i][h], s[c][i][h], o[u][c]);
              }
          }
        }
      }
      if (MODE == kFull) {
        // sums over the 16 row groups: lanes halve the (token, column) values they carry, then plain steps
        float r[2 * CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) { r[c] = f2_sum(o[0][c]); r[CPT + c] = f2_sum(o[1][c]); }
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
        for (int bit = 2 * CPT; bit < 16; bit <<= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], bit);
        if (g < 2 * CPT) so[t + mine / CPT][lc + mine % CPT] = r[0];
      }
    }
    if (MODE == kFull) {
      __syncthreads();
      for (int i = threadIdx.x; i < nt * ncols; i += threads) {
        const int t = i / ncols, c = i % ncols;
        if (col0 + c < p.V) p.out[static_cast<size_t>(it.base + t0 + t) * p.ldo + head * p.V + col0 + c] = so[t][c];
      }
    }
  }
  float* dst = MODE == kLocal ? segs : (it.last ? own : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
      for (int i = 0; i < QPT; ++i)
        if (col0 + lc + c < p.V)
          *reinterpret_cast<ulonglong2*>(dst + static_cast<size_t>(col0 + lc + c) * DP + (i * 16 + g) * 4) = make_ulonglong2(s[c][i][0], s[c][i][1]);
  }
  if (MODE == kLocal && blockIdx.x == 0 && static_cast<int>(threadIdx.x) < DP)
    p.seg_gate[(static_cast<size_t>(it.seg) * p.heads + head) * DP + threadIdx.x] = gate;
}

// ------------------------------------------------------------------------------------------------------
// The same recurrence on the tensor cores, 16 tokens at a time, for prompts of the bf16 engine.  With P_t the product of the
// gates up to token t of the block, G = P_15 and X_s the product of the gates after token s,
//
//   o_t = (q_t P_t) S + sum_{s <= t} A[t][s] v_s,     A[t][s] = sum_d q_t k_s prod_{s < r <= t} f_r,     S <- G S + (k_s X_s)^T v_s
//
// so every factor is a product of gates (at most 1): nothing is divided by a decay and nothing overflows.  A is formed on the
// fp32 units by running products; the three products with S and v run on mma.sync tf32 with their fp32 factors split in two
// (S, q P, k X, A: about 21 bits; v, a projection, is rounded to tf32).  The transposed state [column][row] sits in a warp's
// accumulators, 16 columns a warp, and is read as the A operand of the next product without moving: the contraction index is
// relabelled so that accumulator and operand fragments agree.
// ------------------------------------------------------------------------------------------------------
constexpr int kMbTok = 16;

template <int DP>
struct MbCfg {
  static constexpr int kRaw = 2 * DP + 128 + 8;                  // floats per raw row: q, z, v
  static constexpr int kQp = 2 * DP + 16, kKp = 2 * DP + 8, kAp = 2 * kMbTok + 8;
  static constexpr int kSmemBytes = 4 * (2 * kMbTok * kRaw + 3 * kMbTok * DP + kMbTok * (kQp + kKp + kAp) + 3 * DP);
};

template <int DP, int MODE>
__global__ void __launch_bounds__(256, 2) hgrn2_mma_kernel(RecParams p) {
  using Cfg = MbCfg<DP>;
  constexpr int NT = DP / 8;                     // 8-row tiles of the state
  constexpr int EP = DP / 32;                    // gate channels per lane in the running products
  extern __shared__ __align__(16) uint8_t rec_smem[];
  float* raw = reinterpret_cast<float*>(rec_smem);                // [2][16][kRaw]
  float* sf = raw + 2 * kMbTok * Cfg::kRaw;                       // [16][DP] gate, key, query
  float* sk = sf + kMbTok * DP;
  float* sq = sk + kMbTok * DP;
  float* qp = sq + kMbTok * DP;                                   // [16][kQp]: (hi, hi, lo, lo) of two channels
  float* kx = qp + kMbTok * Cfg::kQp;                             // [16][kKp]: (hi, lo)
  float* sA = kx + kMbTok * Cfg::kKp;                             // [16][kAp]: (hi, lo)
  float* sG = sA + kMbTok * Cfg::kAp;                             // [DP] gate product of the block, lower bound, bias
  float* slow = sG + DP;
  float* sbias = slow + DP;
  const int threads = blockDim.x, warps = threads >> 5, ncols = warps * 16;
  const int head = blockIdx.y, col0 = blockIdx.x * ncols;
  RecItem it;
  if (!rec_item(p, blockIdx.z + p.z0, it)) return;
  if (MODE == kLocal && it.last) return;
  const StepRows& sr = p.sr;
  const int ctx = sr.ctx_len[it.entry], slot = sr.state_slot[it.entry];
  if (ctx <= 0 || slot < 0) return;
  if (slot >= sr.num_slots) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const size_t head_state = static_cast<size_t>(p.V) * DP;
  float* own = p.state + (static_cast<size_t>(slot) * p.heads + head) * head_state;
  float* segs = p.seg_len > 0 ? p.seg_state + (static_cast<size_t>(it.seg) * p.heads + head) * head_state : nullptr;
  const float* init = nullptr;
  if (MODE == kFull) {
    const int s = it.entry - sr.num_decode;
    if (segs != nullptr && (it.first > 0 || !it.last)) init = rec_segment_start(p, it, head, head_state);
    else if (ctx > sr.cu_q[s + 1] - sr.cu_q[s]) init = own;
  }
  const int vr = col0 + warp * 16 + g;           // state columns of this thread: vr, vr + 8
  float S[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float2 v = make_float2(0.f, 0.f);
      if (init != nullptr && vr + 8 * h < p.V) v = *reinterpret_cast<const float2*>(init + static_cast<size_t>(vr + 8 * h) * DP + 8 * j + 2 * tq);
      S[j][2 * h] = v.x; S[j][2 * h + 1] = v.y;
    }
  const int HD = p.heads * p.D;
  for (int d = threadIdx.x; d < DP; d += threads) {
    slow[d] = d < p.D ? p.low[head * p.D + d] : 0.f;
    sbias[d] = d < p.D ? p.bias[head * p.D + d] : 0.f;
  }
  for (int i = threadIdx.x; i < kMbTok * kMbTok; i += threads)     // A stays zero above the diagonal
    *reinterpret_cast<float2*>(sA + (i / kMbTok) * Cfg::kAp + 2 * (i % kMbTok)) = make_float2(0.f, 0.f);
  const bool vec = ((p.D | p.V | p.ld) & 3) == 0;
  auto fetch = [&](int t0, int buf) {
    const int nt = min(kMbTok, it.n - t0), nv = min(ncols, p.V - col0);
    const int step = vec ? 4 : 1, per = (2 * p.D + nv + step - 1) / step;
    for (int i = threadIdx.x; i < nt * per; i += threads) {
      const int t = i / per, e = (i - t * per) * step;
      const float* src = p.qfv + static_cast<size_t>(it.base + t0 + t) * p.ld;
      float* dst = raw + (buf * kMbTok + t) * Cfg::kRaw;
      if (e < p.D) { src += head * p.D + e; dst += e; }
      else if (e < 2 * p.D) { src += HD + head * p.D + e - p.D; dst += DP + e - p.D; }
      else { src += 2 * HD + head * p.V + col0 + e - 2 * p.D; dst += 2 * DP + e - 2 * p.D; }
      if (vec) cp_async<16>(dst, src); else cp_async<4>(dst, src);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  float seg_gate = 1.f;
  for (int t0 = 0, buf = 0; t0 < it.n; t0 += kMbTok, buf ^= 1) {
    const int nt = min(kMbTok, it.n - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t0 + kMbTok < it.n) fetch(t0 + kMbTok, buf ^ 1);
    // ---- gates (tokens past the end: gate 1, key and query 0) ----
    for (int i = threadIdx.x; i < kMbTok * DP; i += threads) {
      const int t = i / DP, d = i % DP;
      const float* row = raw + (buf * kMbTok + t) * Cfg::kRaw;
      float q = 0.f, f = 1.f, k = 0.f;
      if (t < nt && d < p.D) {
        const float low = slow[d], z = row[DP + d] + sbias[d];
        const float ez = __expf(-fabsf(z));
        const float r = __fdividef(1.f, 1.f + ez), small = ez * r;
        f = fmaf(1.f - low, z >= 0.f ? r : small, low);
        k = (1.f - low) * (z >= 0.f ? small : r);
        if (MODE == kFull) { const float x = row[d]; q = __fdividef(x, 1.f + __expf(fminf(-x, 80.f))); }
      }
      if (MODE == kFull) sq[i] = q;
      sf[i] = f; sk[i] = k;
    }
    __syncthreads();
    // ---- products of gates from the block's start and to its end ----
    for (int i = threadIdx.x; i < 2 * DP; i += threads) {
      const int d = i % DP;
      float x = 1.f;
      if (i < DP) {
        float* dst = qp + (d >> 1) * 4 + (d & 1);
#pragma unroll
        for (int t = 0; t < kMbTok; ++t) {
          x *= sf[t * DP + d];
          if (MODE == kFull) {
            const float2 h = tf32_split(sq[t * DP + d] * x);
            dst[t * Cfg::kQp] = h.x; dst[t * Cfg::kQp + 2] = h.y;
          }
        }
        sG[d] = x;
        if (MODE == kLocal && blockIdx.x == 0) seg_gate *= x;      // channel threadIdx.x: segmented launches have DP threads or more
      } else {
#pragma unroll
        for (int t = kMbTok - 1; t >= 0; --t) {
          *reinterpret_cast<float2*>(kx + t * Cfg::kKp + 2 * d) = tf32_split(sk[t * DP + d] * x);
          x *= sf[t * DP + d];
        }
      }
    }
    // ---- A: running products from key s to every later query ----
    if (MODE == kFull) {
      for (int i = warp; i < kMbTok / 2; i += warps) {
        // keys i and 15 - i at a time (they share the loads); a lane holds EP neighbouring channels
        float x[2][EP], a[kMbTok];
        float f[EP], q[EP];
        load_vec<EP>(sk + i * DP + lane * EP, x[0]);
        load_vec<EP>(sk + (kMbTok - 1 - i) * DP + lane * EP, x[1]);
        float a2[kMbTok / 2];                                      // key 15 - i starts in the upper half
#pragma unroll
        for (int t = 0; t < kMbTok; ++t) {
          load_vec<EP>(sf + t * DP + lane * EP, f);
          load_vec<EP>(sq + t * DP + lane * EP, q);
          float u = 0.f, w = 0.f;
#pragma unroll
          for (int e = 0; e < EP; ++e) {
            if (t > i) x[0][e] *= f[e];
            u = fmaf(q[e], x[0][e], u);
            if (t >= kMbTok / 2) {
              if (t > kMbTok - 1 - i) x[1][e] *= f[e];
              w = fmaf(q[e], x[1][e], w);
            }
          }
          a[t] = u;
          if (t >= kMbTok / 2) a2[t - kMbTok / 2] = w;
        }
        // lane sums by halving: lane L ends with a[L mod 16 bit-reversed] and a2[L mod 8 bit-reversed]
        int ta = 0, tb = 0;
#pragma unroll
        for (int w = kMbTok / 2, bit = 1; w >= 1; w >>= 1, bit <<= 1) {
          const bool up = (lane & bit) != 0;
#pragma unroll
          for (int c = 0; c < w; ++c) {
            const float send = up ? a[c] : a[c + w], keep = up ? a[c + w] : a[c];
            a[c] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
          }
          ta += up ? w : 0;
        }
        a[0] += __shfl_xor_sync(0xffffffffu, a[0], 16);
#pragma unroll
        for (int w = kMbTok / 4, bit = 1; w >= 1; w >>= 1, bit <<= 1) {
          const bool up = (lane & bit) != 0;
#pragma unroll
          for (int c = 0; c < w; ++c) {
            const float send = up ? a2[c] : a2[c + w], keep = up ? a2[c + w] : a2[c];
            a2[c] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
          }
          tb += up ? w : 0;
        }
        a2[0] += __shfl_xor_sync(0xffffffffu, a2[0], 8);
        a2[0] += __shfl_xor_sync(0xffffffffu, a2[0], 16);
        if (lane < 16 && ta >= i) *reinterpret_cast<float2*>(sA + ta * Cfg::kAp + 2 * i) = tf32_split(a[0]);
        tb += kMbTok / 2;
        if (lane < 8 && tb >= kMbTok - 1 - i)
          *reinterpret_cast<float2*>(sA + tb * Cfg::kAp + 2 * (kMbTok - 1 - i)) = tf32_split(a2[0]);
      }
    }
    __syncthreads();
    // ---- v^T as the A operand of both products with v ----
    float v[2][4];
#pragma unroll
    for (int k = 0; k < 2; ++k)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int t = 8 * k + tq + (x >> 1) * 4, c = warp * 16 + g + (x & 1) * 8;
        v[k][x] = t < nt && col0 + c < p.V ? tf32_round(raw[(buf * kMbTok + t) * Cfg::kRaw + 2 * DP + c]) : 0.f;
      }
    if (MODE == kFull) {
      float o[2][4] = {}, oc[2][4] = {};                           // leading products and corrections: four chains of accumulation
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        float hi[4], lo[4];
        const int at[4] = {0, 2, 1, 3};                            // accumulator -> operand: (g, 2 tq) is index tq, (g, 2 tq + 1) is tq + 4
#pragma unroll
        for (int x = 0; x < 4; ++x) { const float2 h = tf32_split(S[j][at[x]]); hi[x] = h.x; lo[x] = h.y; }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float4 b = *reinterpret_cast<const float4*>(qp + (8 * n + g) * Cfg::kQp + (4 * j + tq) * 4);
          mma_tf32(o[n], hi, b.x, b.y);
          mma_tf32(oc[n], lo, b.x, b.y);
          mma_tf32(oc[n], hi, b.z, b.w);
        }
      }
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float2 b0 = *reinterpret_cast<const float2*>(sA + (8 * n + g) * Cfg::kAp + 2 * (8 * k + tq));
          const float2 b1 = *reinterpret_cast<const float2*>(sA + (8 * n + g) * Cfg::kAp + 2 * (8 * k + tq + 4));
          mma_tf32(o[n], v[k], b0.x, b1.x);
          mma_tf32(oc[n], v[k], b0.y, b1.y);
        }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int t = 8 * n + 2 * tq + (x & 1), c = vr + (x >> 1) * 8;
          if (t < nt && c < p.V) p.out[static_cast<size_t>(it.base + t0 + t) * p.ldo + head * p.V + c] = o[n][x] + oc[n][x];
        }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const float2 gm = *reinterpret_cast<const float2*>(sG + 8 * j + 2 * tq);
      S[j][0] *= gm.x; S[j][1] *= gm.y; S[j][2] *= gm.x; S[j][3] *= gm.y;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float2 b0 = *reinterpret_cast<const float2*>(kx + (8 * k + tq) * Cfg::kKp + 2 * (8 * j + g));
        const float2 b1 = *reinterpret_cast<const float2*>(kx + (8 * k + tq + 4) * Cfg::kKp + 2 * (8 * j + g));
        mma_tf32(S[j], v[k], b0.x, b1.x);
        mma_tf32(S[j], v[k], b0.y, b1.y);
      }
    }
  }
  float* dst = MODE == kLocal ? segs : (it.last ? own : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h)
        if (vr + 8 * h < p.V)
          *reinterpret_cast<float2*>(dst + static_cast<size_t>(vr + 8 * h) * DP + 8 * j + 2 * tq) = make_float2(S[j][2 * h], S[j][2 * h + 1]);
  }
  if (MODE == kLocal && blockIdx.x == 0 && static_cast<int>(threadIdx.x) < DP)
    p.seg_gate[(static_cast<size_t>(it.seg) * p.heads + head) * DP + threadIdx.x] = seg_gate;
}

// Turns every segment's local end state into the true state at its end: S_i <- gates_i * S_(i-1) + local_i, starting from the
// sequence's state.  One thread per four state values of a (head, chunk).
__global__ void __launch_bounds__(256) hgrn2_chain_kernel(RecParams p, int DP) {
  const int head = blockIdx.y, s = blockIdx.z;
  const StepRows& sr = p.sr;
  const int len = sr.cu_q[s + 1] - sr.cu_q[s], segs = (len + p.seg_len - 1) / p.seg_len;
  const int entry = sr.num_decode + s, slot = sr.state_slot[entry], ctx = sr.ctx_len[entry];
  if (segs < 2 || slot < 0 || slot >= sr.num_slots || ctx <= 0) return;
  int seg0 = 0;
  for (int i = 0; i < s; ++i) seg0 += (sr.cu_q[i + 1] - sr.cu_q[i] + p.seg_len - 1) / p.seg_len;
  const int quads = p.V * DP / 4, i = blockIdx.x * 256 + threadIdx.x;
  if (i >= quads) return;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  if (ctx > len) a = reinterpret_cast<const float4*>(p.state + (static_cast<size_t>(slot) * p.heads + head) * p.V * DP)[i];
  reinterpret_cast<float4*>(p.seg_state + (static_cast<size_t>(seg0 + segs - 1) * p.heads + head) * p.V * DP)[i] = a;   // where segment 0 starts
  for (int j = 0; j < segs - 1; ++j) {
    const size_t at = static_cast<size_t>(seg0 + j) * p.heads + head;
    float4* u = reinterpret_cast<float4*>(p.seg_state + at * p.V * DP) + i;
    const float4 g = reinterpret_cast<const float4*>(p.seg_gate + at * DP)[i % (DP / 4)];
    const float4 l = *u;
    a = make_float4(fmaf(g.x, a.x, l.x), fmaf(g.y, a.y, l.y), fmaf(g.z, a.z, l.z), fmaf(g.w, a.w, l.w));
    *u = a;
  }
}

template <int DP, int CPT>
static int launch_fma(RecParams p, int items, cudaStream_t stream) {
  if (items <= p.z0) return 0;
  int warps = (p.V + 2 * CPT - 1) / (2 * CPT);
  if (warps > 8) warps = 8;
  const int need = (DP + 31) / 32;               // the gate products of a segment take one thread per state row
  if (p.seg_len > 0 && warps < need) warps = need;
  const dim3 grid((p.V + warps * 2 * CPT - 1) / (warps * 2 * CPT), p.heads, items - p.z0);
  constexpr int smem = RecCfg<DP, CPT>::kSmemBytes;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(hgrn2_kernel<DP, CPT, kLocal>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(hgrn2_kernel<DP, CPT, kFull>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr_set = true;
  }
  if (p.seg_len > 0) {
    hgrn2_kernel<DP, CPT, kLocal><<<grid, warps * 32, smem, stream>>>(p);
    hgrn2_chain_kernel<<<dim3((p.V * DP / 4 + 255) / 256, p.heads, p.num_prefill), 256, 0, stream>>>(p, DP);
  }
  hgrn2_kernel<DP, CPT, kFull><<<grid, warps * 32, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int DP>
static int launch_mma(const RecParams& p, int items, cudaStream_t stream) {
  if (items <= p.z0) return 0;
  int warps = (p.V + 15) / 16;
  if (warps > 8) warps = 8;
  if (p.seg_len > 0 && warps < DP / 32) warps = DP / 32;
  const dim3 grid((p.V + warps * 16 - 1) / (warps * 16), p.heads, items - p.z0);
  constexpr int smem = MbCfg<DP>::kSmemBytes;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(hgrn2_mma_kernel<DP, kLocal>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(hgrn2_mma_kernel<DP, kFull>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr_set = true;
  }
  if (p.seg_len > 0) {
    hgrn2_mma_kernel<DP, kLocal><<<grid, warps * 32, smem, stream>>>(p);
    hgrn2_chain_kernel<<<dim3((p.V * DP / 4 + 255) / 256, p.heads, p.num_prefill), 256, 0, stream>>>(p, DP);
  }
  hgrn2_mma_kernel<DP, kFull><<<grid, warps * 32, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

// decode rows step by step on the fp32 units; prompts there too, or (split) in blocks on the tensor cores
template <int DP, int CPT>
static int launch_hgrn2(RecParams p, int items, bool split, cudaStream_t stream) {
  if constexpr (DP <= 128) {
    if (split) {
      RecParams d = p;
      d.seg_len = 0;
      d.num_prefill = 0;
      const int rc = launch_fma<DP, CPT>(d, p.sr.num_decode, stream);
      if (rc != 0) return rc;
      p.z0 = p.sr.num_decode;
      return launch_mma<DP>(p, items, stream);
    }
  }
  return launch_fma<DP, CPT>(p, items, stream);
}

}  // namespace ogb

using namespace ogb;

// Row width of the stored state for D key channels (0: not supported).
extern "C" int ogb_hgrn2_state_rows(int D) { return D <= 0 ? 0 : D <= 64 ? 64 : D <= 128 ? 128 : D <= 256 ? 256 : 0; }

// seg_len > 0: prefill chunks run as segments of that many tokens; num_segments counts them over all chunks, and seg_state
// [num_segments, heads, V, rows] / seg_gate [num_segments, heads, rows] are scratch.  split: prompts may run on the tensor cores with
// split fp32 factors (states of up to 128 rows).
extern "C" int ogb_hgrn2(const float* qfv, const float* bias, const float* low, float* state, float* out, int ld, int ldo, int heads, int D,
                         int V, const int* ctx_len, const int* state_slot, const int* cu_q, int num_decode, int num_prefill, int num_slots,
                         int seg_len, int num_segments, float* seg_state, float* seg_gate, int split, int* status, void* stream) {
  if (num_decode + num_prefill <= 0 || heads <= 0 || V <= 0) return 0;
  const int dp = ogb_hgrn2_state_rows(D);
  if (dp == 0) return -2;
  if (seg_len > 0 && (seg_state == nullptr || seg_gate == nullptr || num_segments < num_prefill)) return -3;
  RecParams p{qfv, bias, low, state, out, seg_state, seg_gate, ld, ldo, heads, D, V, num_prefill, seg_len > 0 ? seg_len : 0, 0,
              StepRows{ctx_len, state_slot, cu_q, nullptr, nullptr, num_decode, 0, num_slots}, status};
  const int items = num_decode + (seg_len > 0 ? num_segments : num_prefill);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dp == 64) return launch_hgrn2<64, 8>(p, items, split != 0, s);
  if (dp == 128) return launch_hgrn2<128, 8>(p, items, split != 0, s);
  return launch_hgrn2<256, 4>(p, items, split != 0, s);
}
