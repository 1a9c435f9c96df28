// Matrix memories with one decay per head over per-sequence state.  Per head, with key k, value v, query q and numbers a, b of the token:
//
//   S <- a S + b k v^T      o = S^T q
//
// Retention: a is a fixed decay of the head, b = 1; q and k are rotated here.  mLSTM (logits given): with log gates i and f of the token
// and a running maximum m,  m' = max(f + m, i),  a = exp(f + m - m'),  b = exp(i - m');  a normalizer n <- a n + b k is the state's last
// column, and o is divided by max(|n . q|, exp(-m')) + 1e-6.  The state is stored [slot][head][column][row], m as [slot][head]; fp32 like all
// arithmetic here.  The norm of the heads and the output gate follow in head_rmsnorm_kernel.
//
// memory_step_kernel walks the rows of one (head, sequence) with the state in registers, laid out as in delta_step_kernel: a warp owns 16
// value columns (8 for states of 256 rows), its 16 lane pairs own every sixteenth quad of state rows.
//
// Prompts of the bf16 engine run in blocks of 64 tokens (memory_write_kernel, memory_chain_kernel, memory_read_kernel below).
#include <algorithm>

#include "hybrid.cuh"
#include "ogb_kernels.h"

namespace ogb {

struct MemoryParams {
  const void* row;         // [rows, ld]: q | k | v
  const float2* turns;     // [rows, half]: cosine, sine; half 0: no rotation
  const float* logits;     // [rows, ldl]: input | forget gates; null: fixed decays
  const float* bias;       // [2 heads]
  const float* decay;      // [2 heads]: decays, their logarithms
  float* state;            // [slots, heads, VS, DP], VS = V + (logits != null)
  float* peak;             // [slots, heads]
  float* out;              // [rows, heads * V]
  int ld, half, ldl, heads, D, V, DP, z0;
  float cap, q_scale, k_scale;
  StepRows sr;
  int* status;
  OGB_DEVICE int columns() const { return V + (logits != nullptr); }
};

// rows of work item z: a decode row or a whole prefill chunk
struct MemoryItem {
  int base, n, slot;
  bool fresh;
  OGB_DEVICE bool set(const MemoryParams& p, int z) {
    const StepRows& sr = p.sr;
    base = z; n = 1;
    if (z >= sr.num_decode) {
      const int s = z - sr.num_decode;
      base = sr.num_decode + sr.cu_q[s];
      n = sr.cu_q[s + 1] - sr.cu_q[s];
    }
    const int ctx = sr.ctx_len[z];
    slot = sr.state_slot[z];
    if (ctx <= 0 || slot < 0 || n <= 0) return false;
    if (slot >= sr.num_slots) {
      if (threadIdx.x == 0) atomicOr(p.status, kStatusIndexOutOfRange);
      return false;
    }
    fresh = ctx <= n;
    return true;
  }
};

// channel d of a head's projected query or key `src` (rotated: d turns with its partner half a rotation away)
template <typename T>
OGB_DEVICE float memory_channel(const MemoryParams& p, const T* src, int row, int d) {
  const float x = to_f32<T>(src[d]);
  if (d >= 2 * p.half) return x;
  const bool low = d < p.half;
  const float2 cs = p.turns[static_cast<size_t>(row) * p.half + (low ? d : d - p.half)];
  const float y = to_f32<T>(src[low ? d + p.half : d - p.half]);
  return low ? x * cs.x - y * cs.y : x * cs.x + y * cs.y;
}

// log input and forget gates of a row's head
OGB_DEVICE float2 memory_log_gates(const MemoryParams& p, int row, int head) {
  const float* z = p.logits + static_cast<size_t>(row) * p.ldl + head;
  const float i = p.cap * tanhf((z[0] + p.bias[head]) / p.cap), f = p.cap * tanhf((z[p.heads] + p.bias[p.heads + head]) / p.cap);
  return make_float2(i, f > 0.f ? -log1pf(expf(-f)) : f - log1pf(expf(f)));
}

constexpr int kMemTok = 8;

template <typename T, int DP, int CPT, bool GATED>
__global__ void __launch_bounds__(256, DP == 256 ? 1 : 2) memory_step_kernel(MemoryParams p) {
  constexpr int QPT = DP / 64, kMaxCols = 16 * CPT;
  __shared__ __align__(16) float sq[kMemTok][DP], sk[kMemTok][DP], sv[kMemTok][kMaxCols];
  __shared__ float sa[kMemTok], sb[kMemTok], sm[kMemTok + 1], si[kMemTok];
  const int threads = blockDim.x, ncols = threads / 32 * 2 * CPT, head = blockIdx.y, col0 = blockIdx.x * ncols;
  MemoryItem it;
  if (!it.set(p, blockIdx.z + p.z0)) return;             // the same for all blocks of a cluster
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane & 15;
  const int lc = (warp * 2 + (lane >> 4)) * CPT;
  float* own = p.state + (static_cast<size_t>(it.slot) * p.heads + head) * p.columns() * DP;
  f32x2 s[CPT][QPT][2], n[QPT][2];
  auto load = [&](int col, f32x2 (&x)[QPT][2]) {
#pragma unroll
    for (int i = 0; i < QPT; ++i) {
      ulonglong2 y = make_ulonglong2(0ull, 0ull);
      if (!it.fresh && col < p.columns()) y = *reinterpret_cast<const ulonglong2*>(own + static_cast<size_t>(col) * DP + (i * 16 + g) * 4);
      x[i][0] = y.x;
      x[i][1] = y.y;
    }
  };
#pragma unroll
  for (int c = 0; c < CPT; ++c) load(col0 + lc + c < p.V ? col0 + lc + c : p.columns(), s[c]);
  if (GATED) {                                           // every block keeps the normalizer and the maximum; the first one stores them
    load(p.V, n);
    if (threadIdx.x == 0) sm[kMemTok] = it.fresh ? 0.f : p.peak[static_cast<size_t>(it.slot) * p.heads + head];
    __syncwarp();
    if (gridDim.x > 1) asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  }
  for (int t0 = 0; t0 < it.n; t0 += kMemTok) {
    const int nt = min(kMemTok, it.n - t0);
    __syncthreads();
    const size_t row0 = static_cast<size_t>(it.base) + t0;
    for (int i = threadIdx.x; i < nt * DP; i += threads) {
      const int t = i / DP, d = i % DP;
      const T* src = static_cast<const T*>(p.row) + (row0 + t) * p.ld + static_cast<size_t>(head) * p.D;
      sq[t][d] = d < p.D ? memory_channel<T>(p, src, static_cast<int>(row0) + t, d) * p.q_scale : 0.f;
      sk[t][d] = d < p.D ? memory_channel<T>(p, src + p.heads * p.D, static_cast<int>(row0) + t, d) * p.k_scale : 0.f;
    }
    for (int i = threadIdx.x; i < nt * ncols; i += threads) {
      const int t = i / ncols, c = i - t * ncols;
      sv[t][c] = col0 + c < p.V ? to_f32<T>(static_cast<const T*>(p.row)[(row0 + t) * p.ld + 2 * p.heads * p.D + static_cast<size_t>(head) * p.V + col0 + c]) : 0.f;
    }
    if (static_cast<int>(threadIdx.x) < nt) {
      if (GATED) {
        const float2 x = memory_log_gates(p, static_cast<int>(row0) + threadIdx.x, head);
        si[threadIdx.x] = x.x;
        sa[threadIdx.x] = x.y;
      } else {
        sa[threadIdx.x] = p.decay[head];
        sb[threadIdx.x] = 1.f;
      }
    }
    if (GATED) {
      __syncthreads();
      if (threadIdx.x < 32) {                            // the maxima one after the other, their exponentials side by side
        float m = sm[kMemTok], before = m, at = m;
        for (int t = 0; t < nt; ++t) {
          if (static_cast<int>(threadIdx.x) == t) before = m;
          m = fmaxf(sa[t] + m, si[t]);
          if (static_cast<int>(threadIdx.x) == t) at = m;
        }
        float a = 0.f, b = 0.f;
        if (static_cast<int>(threadIdx.x) < nt) {
          a = expf(sa[threadIdx.x] + before - at);
          b = expf(si[threadIdx.x] - at);
        }
        __syncwarp();
        if (static_cast<int>(threadIdx.x) < nt) { sa[threadIdx.x] = a; sb[threadIdx.x] = b; sm[threadIdx.x] = expf(-at); }
        if (threadIdx.x == 0) sm[kMemTok] = m;
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      f32x2 k[QPT][2], q[QPT][2], dec;
      const float a = sa[t], b = sb[t];
      asm("mov.b64 %0, {%1, %1};" : "=l"(dec) : "f"(a));
#pragma unroll
      for (int i = 0; i < QPT; ++i) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(&sk[t][(i * 16 + g) * 4]);
        const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(&sq[t][(i * 16 + g) * 4]);
        k[i][0] = x.x; k[i][1] = x.y;
        q[i][0] = y.x; q[i][1] = y.y;
      }
      auto advance = [&](f32x2 (&x)[QPT][2], float v) {  // returns this lane's part of x . q after the write
        f32x2 vv, acc = 0ull;
        asm("mov.b64 %0, {%1, %1};" : "=l"(vv) : "f"(v));
#pragma unroll
        for (int i = 0; i < QPT; ++i)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            x[i][h] = f2_fma(k[i][h], vv, f2_mul(dec, x[i][h]));
            acc = f2_fma(q[i][h], x[i][h], acc);
          }
        return f2_sum(acc);
      };
      float r[CPT], den = 0.f;
#pragma unroll
      for (int c = 0; c < CPT; ++c) r[c] = advance(s[c], b * sv[t][lc + c]);
      if (GATED) den = advance(n, b);
      // lanes halve the values they carry: lane g ends with the sum of column `mine`
      int mine = 0;
#pragma unroll
      for (int w = CPT / 2, bit = 1; w >= 1; w >>= 1, bit <<= 1) {
        const bool up = (g & bit) != 0;
#pragma unroll
        for (int c = 0; c < w; ++c) {
          const float send = up ? r[c] : r[c + w], keep = up ? r[c + w] : r[c];
          r[c] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
        mine += up ? w : 0;
      }
#pragma unroll
      for (int bit = CPT; bit < 16; bit <<= 1) r[0] += __shfl_xor_sync(0xffffffffu, r[0], bit);
      if (GATED) {
#pragma unroll
        for (int bit = 1; bit < 16; bit <<= 1) den += __shfl_xor_sync(0xffffffffu, den, bit);
        r[0] /= fmaxf(fabsf(den), sm[t]) + 1e-6f;
      }
      if (g < CPT && col0 + lc + mine < p.V) p.out[(row0 + t) * (static_cast<size_t>(p.heads) * p.V) + static_cast<size_t>(head) * p.V + col0 + lc + mine] = r[0];
    }
  }
  auto store = [&](int col, const f32x2 (&x)[QPT][2]) {
#pragma unroll
    for (int i = 0; i < QPT; ++i)
      *reinterpret_cast<ulonglong2*>(own + static_cast<size_t>(col) * DP + (i * 16 + g) * 4) = make_ulonglong2(x[i][0], x[i][1]);
  };
#pragma unroll
  for (int c = 0; c < CPT; ++c)
    if (col0 + lc + c < p.V) store(col0 + lc + c, s[c]);
  if (GATED) {
    __syncwarp();
    if (gridDim.x > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");      // every block has read them
    if (blockIdx.x == 0 && threadIdx.x < 16) store(p.V, n);
    if (blockIdx.x == 0 && threadIdx.x == 0) p.peak[static_cast<size_t>(it.slot) * p.heads + head] = sm[kMemTok];
  }
}

template <typename T, int DP, int CPT>
static int launch_memory_step(MemoryParams p, int items, cudaStream_t stream) {
  const int warps = std::min(8, (p.V + 2 * CPT - 1) / (2 * CPT)), blocks = (p.V + warps * 2 * CPT - 1) / (warps * 2 * CPT);
  if (p.logits != nullptr && blocks > 8) return -3;
  for (int z0 = 0; z0 < items; z0 += 65535) {            // sequences lie along grid.z
    p.z0 = z0;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks, p.heads, std::min(65535, items - z0));
    cfg.blockDim = dim3(warps * 32);
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = blocks;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = p.logits != nullptr && blocks > 1 ? 1 : 0;
    if (p.logits != nullptr) OGB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, memory_step_kernel<T, DP, CPT, true>, p));
    else OGB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, memory_step_kernel<T, DP, CPT, false>, p));
  }
  return static_cast<int>(cudaGetLastError());
}
template <typename T>
static int dispatch_memory_step(const MemoryParams& p, int items, cudaStream_t stream) {
  if (items <= 0) return 0;
  if (p.DP == 64) return launch_memory_step<T, 64, 8>(p, items, stream);
  if (p.DP == 128) return launch_memory_step<T, 128, 8>(p, items, stream);
  if (p.DP == 256) return launch_memory_step<T, 256, 4>(p, items, stream);
  return -3;
}

// ------------------------------------------------------------------------------------------------------
// Blocks of 64 tokens.  With c_t the sum of the log decays (f, or the head's fixed one) of the block up to token t, g_s = i_s - c_s (i = 0
// without gates) and S, m the state and the maximum at the block's start, a read-out in the block is
//
//   G_t = max(m, max_{s <= t} g_s)  (without gates: -c_t)      m_t = c_t + G_t
//   o_t = exp(m - G_t) S^T q_t + sum_{s <= t} exp(g_s - G_t) (q_t . k_s) v_s      (m = 0 without gates)
//
// and the block's own writes, up to a factor that the chain brings in, are  U = sum_s exp(g_s - g*) k_s v_s^T  with g* = max_s g_s
// (without gates: -c_63).  A warp per block and head sums the gates up; all blocks write U side by side; a chain over the blocks of a
// sequence, elementwise in the state, turns every U into the state its block starts with; all blocks read out side by side.  Exponents are never positive; c and
// g are kept in double, so that differences of large sums stay good to fp32.  Products run on mma.sync tf32, fp32 factors split in
// two (values are bf16, which tf32 holds as they are).
// ------------------------------------------------------------------------------------------------------
constexpr int kMbThreads = 256;
constexpr int kMbTok = 64;                                        // tokens of a block
constexpr int kMbPP = kMbTok + 4;                                 // row pitch of the products of queries and keys

struct MemoryBlocks {
  const int* tile_seq;     // 64-row tiles of the prefill chunks
  const int* tile_q0;
  int num_tiles;
  float* u;                // [blocks, heads, VS, DP]: writes of the block, then the state it starts with
  float4* num;             // [blocks, heads]: sum of log decays, m* = c + g*, m at the block's start
  double* sums;            // [blocks, heads, 3, 64], with gates: c, g, the largest g up to the token
};

OGB_DEVICE int mb_first_block(const StepRows& sr, int s) {        // blocks of the entries before prefill entry s
  int n = 0;
  for (int i = 0; i < s; ++i) n += (sr.cu_q[i + 1] - sr.cu_q[i] + kMbTok - 1) / kMbTok;
  return n;
}

// the block of a CTA
struct MbTile {
  int seq, q0, len, nt;
  size_t row0, block;
  OGB_DEVICE bool set(const MemoryParams& p, const MemoryBlocks& bl, int tile) {
    const StepRows& sr = p.sr;
    seq = bl.tile_seq[tile];
    q0 = bl.tile_q0[tile];
    len = sr.cu_q[seq + 1] - sr.cu_q[seq];
    nt = min(kMbTok, len - q0);
    if (nt <= 0) return false;
    row0 = static_cast<size_t>(sr.num_decode) + sr.cu_q[seq] + q0;
    block = static_cast<size_t>(mb_first_block(sr, seq)) + q0 / kMbTok;
    return true;
  }
};

// Rotated, scaled channels of the block's rows to dst [64][pitch] -- of keys, or of queries and keys together (N = 2), which share their
// rotations; zeros behind the head's channels and the last token.  A thread has the same four channels in all its rows, whose loads are
// under way together.
template <typename T, int DP, int N>
OGB_DEVICE void mb_channels(const MemoryParams& p, const MbTile& b, const T* const (&src)[N], const float (&scale)[N], float* const (&dst)[N], int pitch) {
  bool vec = ((p.D | p.half) & 3) == 0 && (p.ld & 3) == 0;
#pragma unroll
  for (int a = 0; a < N; ++a) vec = vec && (reinterpret_cast<uintptr_t>(src[a]) & (4 * sizeof(T) - 1)) == 0;
  if (!vec) {
#pragma unroll
    for (int a = 0; a < N; ++a)
      for (int i = threadIdx.x; i < kMbTok * DP; i += kMbThreads) {
        const int t = i / DP, d = i % DP;
        dst[a][t * pitch + d] = t < b.nt && d < p.D ? memory_channel<T>(p, src[a] + (b.row0 + t) * p.ld, static_cast<int>(b.row0) + t, d) * scale[a] : 0.f;
      }
    return;
  }
  static_assert(sizeof(T) == 2, "four channels are two registers");
  constexpr int kStep = kMbThreads / (DP / 4), kBatch = 4;         // rows between a thread's, rows at a time
  const int d = threadIdx.x % (DP / 4) * 4, t0 = threadIdx.x / (DP / 4);
  const bool live = d < p.D, turn = d < 2 * p.half, low = d < p.half;
  const int dx = live ? d : 0, dy = turn ? (low ? d + p.half : d - p.half) : dx;
  const float2* cs = p.turns + (turn ? (low ? d : d - p.half) : 0);
  const float sign = low ? -1.f : 1.f;
#pragma unroll
  for (int j0 = 0; j0 < kMbTok / kStep; j0 += kBatch) {
    uint2 x[kBatch][N], y[kBatch][N];
    float4 c[kBatch][2];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const size_t row = b.row0 + min(t0 + (j0 + j) * kStep, b.nt - 1);
#pragma unroll
      for (int a = 0; a < N; ++a) {
        x[j][a] = *reinterpret_cast<const uint2*>(src[a] + row * p.ld + dx);
        if (turn) y[j][a] = *reinterpret_cast<const uint2*>(src[a] + row * p.ld + dy);
      }
      if (turn) {
        c[j][0] = *reinterpret_cast<const float4*>(cs + row * p.half);
        c[j][1] = *reinterpret_cast<const float4*>(cs + row * p.half + 2);
      }
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const int t = t0 + (j0 + j) * kStep;
#pragma unroll
      for (int a = 0; a < N; ++a) {
        float2 x0 = unpack_bf16(x[j][a].x), x1 = unpack_bf16(x[j][a].y);
        if (turn) {
          const float2 y0 = unpack_bf16(y[j][a].x), y1 = unpack_bf16(y[j][a].y);
          x0 = make_float2(x0.x * c[j][0].x + sign * (y0.x * c[j][0].y), x0.y * c[j][0].z + sign * (y0.y * c[j][0].w));
          x1 = make_float2(x1.x * c[j][1].x + sign * (y1.x * c[j][1].y), x1.y * c[j][1].z + sign * (y1.y * c[j][1].w));
        }
        const float f = live && t < b.nt ? scale[a] : 0.f;
        *reinterpret_cast<float4*>(dst[a] + t * pitch + d) = make_float4(x0.x * f, x0.y * f, x1.x * f, x1.y * f);
      }
    }
  }
}

// NC value columns v0 .. of the block's rows: fetched to registers, stored to dst [64][PITCH]
template <typename T, int NC, int PITCH>
struct MbValues {
  static constexpr int kRows = kMbTok * NC / 4 / kMbThreads, kStep = kMbThreads / (NC / 4);
  float x[kRows][4];
  OGB_DEVICE void fetch(const MemoryParams& p, const MbTile& b, int head, int v0) {
    const T* src = static_cast<const T*>(p.row) + 2 * p.heads * p.D + static_cast<size_t>(head) * p.V + v0;
    const bool vec = ((p.V | p.ld) & 3) == 0 && (reinterpret_cast<uintptr_t>(src) & (4 * sizeof(T) - 1)) == 0;
    const int c = threadIdx.x % (NC / 4) * 4, t0 = threadIdx.x / (NC / 4);
#pragma unroll
    for (int k = 0; k < kRows; ++k) {
      const int t = t0 + k * kStep;
#pragma unroll
      for (int j = 0; j < 4; ++j) x[k][j] = 0.f;
      if (t >= b.nt || v0 + c >= p.V) continue;
      const T* s = src + (b.row0 + t) * p.ld + c;
      if (vec) load_vec<4>(s, x[k]);
      else
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (v0 + c + j < p.V) x[k][j] = to_f32<T>(s[j]);
    }
  }
  OGB_DEVICE void store(float* dst) const {
    const int c = threadIdx.x % (NC / 4) * 4, t0 = threadIdx.x / (NC / 4);
#pragma unroll
    for (int k = 0; k < kRows; ++k) *reinterpret_cast<float4*>(dst + (t0 + k * kStep) * PITCH + c) = make_float4(x[k][0], x[k][1], x[k][2], x[k][3]);
  }
};

// The sums of a block's gates: one warp, whose lane l has tokens l and l + 32 (tokens behind the last have no weight: g = -inf).
__global__ void __launch_bounds__(256) memory_sums_kernel(MemoryParams p, MemoryBlocks bl) {
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, tile = item / p.heads, head = item % p.heads;
  MbTile b;
  if (tile >= bl.num_tiles || !b.set(p, bl, tile)) return;
  double c[2], g[2], top[2];
  float in[2] = {0.f, 0.f};
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int t = lane + 32 * h;
    c[h] = 0.0;
    if (t >= b.nt) continue;
    const float2 x = memory_log_gates(p, static_cast<int>(b.row0) + t, head);
    in[h] = x.x;
    c[h] = static_cast<double>(x.y);
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const double x = __shfl_up_sync(0xffffffffu, c[h], o);
      if (lane >= o) c[h] += x;
    }
  c[1] += __shfl_sync(0xffffffffu, c[0], 31);
#pragma unroll
  for (int h = 0; h < 2; ++h) top[h] = g[h] = lane + 32 * h < b.nt ? static_cast<double>(in[h]) - c[h] : -INFINITY;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const double x = __shfl_up_sync(0xffffffffu, top[h], o);
      if (lane >= o) top[h] = fmax(top[h], x);
    }
  top[1] = fmax(top[1], __shfl_sync(0xffffffffu, top[0], 31));
  double* out = bl.sums + (b.block * p.heads + head) * (3 * kMbTok);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    out[lane + 32 * h] = c[h];
    out[kMbTok + lane + 32 * h] = g[h];
    out[2 * kMbTok + lane + 32 * h] = top[h];
  }
}

struct MbSums {            // c, g, the largest g up to the token (without gates: -c) of token t of a block
  double c, g, top;
  OGB_DEVICE MbSums(const MemoryParams& p, const MemoryBlocks& bl, const MbTile& b, int head, int t) {
    if (p.logits != nullptr) {
      const double* in = bl.sums + (b.block * p.heads + head) * (3 * kMbTok) + t;
      c = in[0];
      g = in[kMbTok];
      top = in[2 * kMbTok];
    } else {
      c = static_cast<double>(p.decay[p.heads + head]) * (min(t, b.nt - 1) + 1);
      top = -c;
      g = t < b.nt ? -c : -INFINITY;
    }
  }
};

// 128 value columns of a block's writes: a warp has 16 of them and all channels of the keys, 64 at a time
constexpr int kMwCols = 128, kMwVP = kMwCols + 8;
template <int DP>
struct MwCfg {
  static constexpr int kPitch = DP + 8;
  static constexpr int kSmemBytes = 4 * (kMbTok + kMbTok * kMwVP + kMbTok * kPitch);
};

template <typename T, int DP>
__global__ void __launch_bounds__(kMbThreads, DP <= 128 ? 3 : 1) memory_write_kernel(MemoryParams p, MemoryBlocks bl) {
  constexpr int kPitch = MwCfg<DP>::kPitch, DC = 64, NT = DC / 8;
  extern __shared__ __align__(16) uint8_t mb_smem[];
  float* sw = reinterpret_cast<float*>(mb_smem);                  // [64] weights
  float* sv = sw + kMbTok;                                        // [64][kMwVP]
  float* sk = sv + kMbTok * kMwVP;                                // [64][kPitch]
  MbTile b;
  if (!b.set(p, bl, blockIdx.y)) return;
  const int head = blockIdx.x, v0 = blockIdx.z * kMwCols, VS = p.columns();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, tq = lane & 3;
  if (tid < kMbTok) {
    const MbSums x(p, bl, b, head, tid), last(p, bl, b, head, kMbTok - 1);
    sw[tid] = expf(static_cast<float>(x.g - last.top));
    if (tid == 0 && blockIdx.z == 0)
      bl.num[b.block * p.heads + head] = make_float4(static_cast<float>(last.c), static_cast<float>(last.c + last.top), 0.f, 0.f);
  }
  {
    const T* const keys[1] = {static_cast<const T*>(p.row) + static_cast<size_t>(p.heads + head) * p.D};
    const float scale[1] = {p.k_scale};
    float* const to[1] = {sk};
    mb_channels<T, DP, 1>(p, b, keys, scale, to, kPitch);
  }
  MbValues<T, kMwCols, kMwVP> val;
  val.fetch(p, b, head, v0);
  val.store(sv);
  __syncthreads();
  float* u = bl.u + (b.block * p.heads + head) * static_cast<size_t>(VS) * DP;
  if (v0 + 16 * warp < p.V) {
#pragma unroll 1
    for (int d0 = 0; d0 < DP; d0 += DC) {
      float acc[NT][4] = {};
#pragma unroll 2
      for (int k = 0; k < kMbTok / 8; ++k) {
        const int s0 = 8 * k + tq, s1 = s0 + 4, v = 16 * warp + gr;
        const float w0 = sw[s0], w1 = sw[s1];
        const float a[4] = {sv[s0 * kMwVP + v], sv[s0 * kMwVP + v + 8], sv[s1 * kMwVP + v], sv[s1 * kMwVP + v + 8]};
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int d = d0 + 8 * n + gr;
          const float2 b0 = tf32_cut(w0 * sk[s0 * kPitch + d]), b1 = tf32_cut(w1 * sk[s1 * kPitch + d]);
          mma_tf32(acc[n], a, b0.x, b1.x);
          mma_tf32(acc[n], a, b0.y, b1.y);
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int v = v0 + 16 * warp + gr + 8 * h;
          if (v < p.V) *reinterpret_cast<float2*>(u + static_cast<size_t>(v) * DP + d0 + 8 * n + 2 * tq) = make_float2(acc[n][2 * h], acc[n][2 * h + 1]);
        }
    }
  }
  if (p.logits != nullptr && blockIdx.z == 0)
    for (int d = tid; d < DP; d += kMbThreads) {
      float a = 0.f;
#pragma unroll 8
      for (int s = 0; s < kMbTok; ++s) a = fmaf(sw[s], sk[s * kPitch + d], a);
      u[static_cast<size_t>(p.V) * DP + d] = a;
    }
}

constexpr int kMcThreads = 128;
__global__ void __launch_bounds__(kMcThreads) memory_chain_kernel(MemoryParams p, MemoryBlocks bl) {
  constexpr int kAhead = 8;                                       // blocks whose writes are under way
  MemoryItem it;
  const int seq = blockIdx.z, head = blockIdx.y, quads = p.columns() * p.DP / 4, e = blockIdx.x * kMcThreads + threadIdx.x;
  if (!it.set(p, p.sr.num_decode + seq) || e >= quads) return;
  const size_t b0 = mb_first_block(p.sr, seq), at = (b0 * p.heads + head), step = p.heads;
  const int blocks = (it.n + kMbTok - 1) / kMbTok;
  float4* own = reinterpret_cast<float4*>(p.state + (static_cast<size_t>(it.slot) * p.heads + head) * p.columns() * p.DP) + e;
  float4 s = it.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *own;
  const bool gated = p.logits != nullptr;
  float m = gated && !it.fresh ? p.peak[static_cast<size_t>(it.slot) * p.heads + head] : 0.f;
  float4* u = reinterpret_cast<float4*>(bl.u) + at * quads + e;
  float4 w[kAhead];
  float2 num[kAhead];
  auto fetch = [&](int i, int j) {
    w[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    num[j] = make_float2(0.f, 0.f);
    if (i < blocks) {
      w[j] = __ldcg(u + i * step * quads);
      num[j] = __ldcg(reinterpret_cast<const float2*>(bl.num + at + i * step));
    }
  };
#pragma unroll
  for (int j = 0; j < kAhead; ++j) fetch(j, j);
  for (int i0 = 0; i0 < blocks; i0 += kAhead)
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (i0 + j >= blocks) break;
      const float4 x = w[j];
      const float2 y = num[j];
      fetch(i0 + kAhead + j, j);
      __stcg(u + (i0 + j) * step * quads, s);
      if (e == 0) bl.num[at + (i0 + j) * step].z = m;
      float a, f = 1.f;
      if (gated) {
        const float next = fmaxf(y.x + m, y.y);
        a = expf(y.x + m - next);
        f = expf(y.y - next);
        m = next;
      } else {
        a = expf(y.x);
      }
      s = make_float4(fmaf(f, x.x, a * s.x), fmaf(f, x.y, a * s.y), fmaf(f, x.z, a * s.z), fmaf(f, x.w, a * s.w));
    }
  *own = s;                                                       // the maximum is left by memory_read_kernel: others may yet read it here
}

OGB_DEVICE float2 two_terms(double x) {
  const float hi = static_cast<float>(x);
  return make_float2(hi, hi == -INFINITY ? 0.f : static_cast<float>(x - static_cast<double>(hi)));
}

// A read-out: products of queries and keys, then 32 value columns at a time, whose states and values come in while the columns before
// them are worked on.  Each of the eight warps has 16 tokens and half of the keys or columns.
constexpr int kMrCols = 32, kMrVP = kMrCols + 8;
template <int DP>
struct MrCfg {
  static constexpr int kPitch = DP + 4;
  static constexpr int kSmemBytes = 8 * (2 * kMbTok) + 4 * (2 * kMbTok * kPitch + 2 * kMbTok * kMrVP + kMbTok * kMbPP + 5 * kMbTok);
};

template <typename T, int DP>
__global__ void __launch_bounds__(kMbThreads, DP <= 128 ? 2 : 1) memory_read_kernel(MemoryParams p, MemoryBlocks bl) {
  using Cfg = MrCfg<DP>;
  constexpr int kPitch = Cfg::kPitch;
  extern __shared__ __align__(16) uint8_t mb_smem[];
  float2* sg = reinterpret_cast<float2*>(mb_smem);                // [64] g, [64] G, as sums of two terms
  float2* sG = sg + kMbTok;
  float* se = reinterpret_cast<float*>(sG + kMbTok);              // [64] exp(m - G)
  float* sinv = se + kMbTok;                                      // [64] exp(-m_t), then what read-outs are multiplied by
  float* sdot = sinv + kMbTok;                                    // [64] n . q
  float* srow = sdot + kMbTok;                                    // [2][64] sums of the rows of sP
  float* sq = srow + 2 * kMbTok;                                  // [64][kPitch]
  float* sk = sq + kMbTok * kPitch;                               // [64][kPitch] keys, then twice 32 columns of the state
  float* sv = sk + kMbTok * kPitch;                               // [2][64][kMrVP]
  float* sP = sv + 2 * kMbTok * kMrVP;                            // [64][kMbPP]
  MbTile b;
  if (!b.set(p, bl, blockIdx.y)) return;
  const int head = blockIdx.x, VS = p.columns();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, tq = lane & 3;
  const bool gated = p.logits != nullptr;
  const float* u = bl.u + (b.block * p.heads + head) * static_cast<size_t>(VS) * DP;
  const T* src = static_cast<const T*>(p.row) + static_cast<size_t>(head) * p.D;
  if (tid < kMbTok) {
    const float m_in = gated ? bl.num[b.block * p.heads + head].z : 0.f;
    const MbSums x(p, bl, b, head, tid);
    const double top = gated ? fmax(static_cast<double>(m_in), x.top) : x.top;
    const float peak = gated ? static_cast<float>(x.c + top) : 0.f;      // m_t
    sg[tid] = two_terms(x.g);
    sG[tid] = two_terms(top);
    se[tid] = expf(static_cast<float>(static_cast<double>(m_in) - top));
    sinv[tid] = expf(-peak);
    // the last block of a chunk leaves the maximum for the next step
    if (gated && tid == b.nt - 1 && b.q0 + b.nt == b.len) {
      const int slot = p.sr.state_slot[p.sr.num_decode + b.seq];
      if (slot >= 0 && slot < p.sr.num_slots) p.peak[static_cast<size_t>(slot) * p.heads + head] = peak;
    }
  }
  {
    const T* const both[2] = {src, src + p.heads * p.D};
    const float scale[2] = {p.q_scale, p.k_scale};
    float* const to[2] = {sq, sk};
    mb_channels<T, DP, 2>(p, b, both, scale, to, kPitch);
  }
  MbValues<T, kMrCols, kMrVP> val;
  val.fetch(p, b, head, 0);
  val.store(sv);
  __syncthreads();
  const int m = warp & 3, half = warp >> 2;
  float acc[4][4] = {};
  {
    const int tiles = min(4, max(0, 2 * m + 2 - 4 * half));       // key tiles up to the diagonal
    if (tiles > 0) split_product<DP / 8, 4>(acc, sq + 16 * m * kPitch, kPitch, sk + 32 * half * kPitch, kPitch, tiles, gr, tq);
  }
  __syncthreads();                                                // the keys have been read
  auto fetch_state = [&](int v0, int buf) {                       // columns behind the last are read as the last and dropped
    if (v0 < p.V) {
#pragma unroll
      for (int j = 0; j < kMrCols * DP / 4 / kMbThreads; ++j) {
        const int i = j * kMbThreads + tid, v = min(v0 + i / (DP / 4), VS - 1), d = i % (DP / 4) * 4;
        cp_async<16>(sk + (buf * kMrCols + i / (DP / 4)) * kPitch + d, u + static_cast<size_t>(v) * DP + d);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch_state(0, 0);
  {
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int t = 16 * m + gr + (x >> 1) * 8, s = 32 * half + 8 * n + 2 * tq + (x & 1);
        const float f = s <= t ? acc[n][x] * expf((sg[s].x - sG[t].x) + (sg[s].y - sG[t].y)) : 0.f;
        sP[t * kMbPP + s] = f;
        sum[x >> 1] += f;
      }
    if (gated) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
        sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
        if (tq == 0) srow[half * kMbTok + 16 * m + gr + 8 * h] = sum[h];
      }
      float n[DP / 32];
#pragma unroll
      for (int d = 0; d < DP / 32; ++d) n[d] = u[static_cast<size_t>(p.V) * DP + 32 * d + lane];
#pragma unroll 2
      for (int t = warp; t < kMbTok; t += 8) {
        float a = 0.f;
#pragma unroll
        for (int d = 0; d < DP / 32; ++d) a = fmaf(sq[t * kPitch + 32 * d + lane], n[d], a);
        a = warp_sum(a);
        if (lane == 0) sdot[t] = a;
      }
    }
  }
  for (int v0 = 0, buf = 0; v0 < p.V; v0 += kMrCols, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                              // these columns have arrived, the ones before are done
    if (v0 == 0 && tid < kMbTok)
      sinv[tid] = gated ? 1.f / (fmaxf(fabsf(se[tid] * sdot[tid] + srow[tid] + srow[kMbTok + tid]), sinv[tid]) + 1e-6f) : 1.f;
    fetch_state(v0 + kMrCols, buf ^ 1);
    val.fetch(p, b, head, v0 + kMrCols);
    const float* s_state = sk + buf * kMrCols * kPitch;
    const float* s_val = sv + buf * kMbTok * kMrVP;
    float o[2][4] = {};
    split_product<DP / 8, 2>(o, sq + 16 * m * kPitch, kPitch, s_state + 16 * half * kPitch, kPitch, 2, gr, tq);
    const float e0 = se[16 * m + gr], e1 = se[16 * m + gr + 8];
#pragma unroll
    for (int n = 0; n < 2; ++n) { o[n][0] *= e0; o[n][1] *= e0; o[n][2] *= e1; o[n][3] *= e1; }
#pragma unroll 2
    for (int k = 0; k < 2 * m + 2; ++k) {
      float hi[4], lo[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 h = tf32_cut(sP[(16 * m + gr + (x & 1) * 8) * kMbPP + 8 * k + tq + (x >> 1) * 4]);
        hi[x] = h.x; lo[x] = h.y;
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const float w0 = s_val[(8 * k + tq) * kMrVP + 16 * half + 8 * n + gr], w1 = s_val[(8 * k + tq + 4) * kMrVP + 16 * half + 8 * n + gr];
        mma_tf32(o[n], hi, w0, w1);
        mma_tf32(o[n], lo, w0, w1);
      }
    }
    val.store(sv + (buf ^ 1) * kMbTok * kMrVP);                   // last read a step ago
    if (v0 == 0) __syncthreads();                                 // sinv
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = 16 * m + gr + 8 * h;
      if (t >= b.nt) continue;
      const float f = sinv[t];
      float* dst = p.out + (b.row0 + t) * (static_cast<size_t>(p.heads) * p.V) + static_cast<size_t>(head) * p.V;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int v = v0 + 16 * half + 8 * n + 2 * tq;
        if ((p.V & 1) == 0 && v < p.V) *reinterpret_cast<float2*>(dst + v) = make_float2(o[n][2 * h] * f, o[n][2 * h + 1] * f);
        else {
          if (v < p.V) dst[v] = o[n][2 * h] * f;
          if (v + 1 < p.V) dst[v + 1] = o[n][2 * h + 1] * f;
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

template <typename T, int DP>
static int launch_memory_blocks(const MemoryParams& p, const MemoryBlocks& bl, int num_prefill, cudaStream_t stream) {
  static_assert(sizeof(T) == 2, "values are taken for exact tf32 terms");
  constexpr int write_bytes = MwCfg<DP>::kSmemBytes;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(memory_write_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, write_bytes));
    OGB_CUDA_CHECK(cudaFuncSetAttribute(memory_read_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, MrCfg<DP>::kSmemBytes));
    attr_set = true;
  }
  const int VS = p.V + (p.logits != nullptr), quads = VS * DP / 4;
  if (p.logits != nullptr) memory_sums_kernel<<<(bl.num_tiles * p.heads + 7) / 8, 256, 0, stream>>>(p, bl);
  memory_write_kernel<T, DP><<<dim3(p.heads, bl.num_tiles, (p.V + kMwCols - 1) / kMwCols), kMbThreads, write_bytes, stream>>>(p, bl);
  memory_chain_kernel<<<dim3((quads + kMcThreads - 1) / kMcThreads, p.heads, num_prefill), kMcThreads, 0, stream>>>(p, bl);
  memory_read_kernel<T, DP><<<dim3(p.heads, bl.num_tiles), kMbThreads, MrCfg<DP>::kSmemBytes, stream>>>(p, bl);
  return static_cast<int>(cudaGetLastError());
}

// ------------------------------------------------------------------------------------------------------
// rotations of a step's rows; the angle is reduced in double, so that it is good to fp32 at every position
// ------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) turn_table_kernel(const int* __restrict__ positions, const double* __restrict__ freq, float2* __restrict__ out,
                                                         int tokens, int half) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= static_cast<long long>(tokens) * half) return;
  const int t = static_cast<int>(i / half), k = static_cast<int>(i % half);
  const double a = static_cast<double>(positions[t]) * freq[k] * 0.15915494309189535;
  float s, c;
  sincospif(static_cast<float>(2.0 * (a - rint(a))), &s, &c);
  out[i] = make_float2(c, s);
}

}  // namespace ogb

using namespace ogb;

extern "C" int ogb_turn_table(const int* positions, const double* freq, float* out, int tokens, int half, void* stream) {
  const long long n = static_cast<long long>(tokens) * half;
  if (n <= 0) return 0;
  turn_table_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, static_cast<cudaStream_t>(stream)>>>(positions, freq, reinterpret_cast<float2*>(out),
                                                                                                          tokens, half);
  return static_cast<int>(cudaGetLastError());
}

// fp32 scratch per 64-row tile of a step's prompts
extern "C" int ogb_decay_block_floats(int heads, int D, int V, int gated) {
  const int dp = D <= 64 ? 64 : D <= 128 ? 128 : 256;
  return heads * ((V + (gated != 0)) * dp + 4 + (gated != 0 ? 6 * kMbTok : 0));
}

// row: q | k | v of `heads` heads; logits (or null) and decay (or null): one of them.  work (16-byte aligned, ogb_decay_block_floats of
// each of num_tiles tiles): prefill chunks run in blocks.
extern "C" int ogb_decay_memory(const void* row, int ld, const float* turns, int half, const float* logits, int ldl, const float* bias, float cap,
                                const float* decay, float* state, float* peak, float* out, int heads, int D, int V, int DP, float q_scale,
                                float k_scale, const int* ctx_len, const int* state_slot, const int* cu_q, const int* tile_seq, const int* tile_q0,
                                int num_decode, int num_prefill, int num_tiles, int num_slots, float* work, int elem, int* status, void* stream) {
  if (num_decode + num_prefill <= 0 || heads <= 0 || V <= 0) return 0;
  if (D < 1 || D > DP || 2 * half > D || (half > 0 && turns == nullptr) || (DP != 64 && DP != 128 && DP != 256)) return -3;
  if (logits != nullptr ? bias == nullptr || peak == nullptr || !(cap > 0.f) : decay == nullptr) return -3;
  MemoryParams p{row, reinterpret_cast<const float2*>(turns), logits, bias, decay, state, peak, out, ld, half, ldl, heads, D, V, DP, 0, cap, q_scale,
                 k_scale, StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, num_slots}, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool in_blocks = work != nullptr && elem == kElemBF16 && num_prefill > 0 && num_tiles > 0 && num_tiles <= 65535 && (reinterpret_cast<uintptr_t>(work) & 15) == 0 &&
                         (reinterpret_cast<uintptr_t>(out) & 7) == 0;
  const int items = num_decode + (in_blocks ? 0 : num_prefill);
  int rc = -3;
  if (elem == kElemBF16) rc = dispatch_memory_step<__nv_bfloat16>(p, items, s);
  else if (elem == kElemF32) rc = dispatch_memory_step<float>(p, items, s);
  if (rc != 0 || !in_blocks) return rc;
  MemoryBlocks bl;
  const size_t n = static_cast<size_t>(num_tiles) * heads;
  bl.tile_seq = tile_seq; bl.tile_q0 = tile_q0; bl.num_tiles = num_tiles;
  bl.num = reinterpret_cast<float4*>(work);
  bl.sums = reinterpret_cast<double*>(work + 4 * n);
  bl.u = work + 4 * n + (logits != nullptr ? 6 * kMbTok * n : 0);
  if (DP == 64) return launch_memory_blocks<__nv_bfloat16, 64>(p, bl, num_prefill, s);
  if (DP == 128) return launch_memory_blocks<__nv_bfloat16, 128>(p, bl, num_prefill, s);
  return launch_memory_blocks<__nv_bfloat16, 256>(p, bl, num_prefill, s);
}
