// Gated delta rule over per-sequence state.  Per head, with decay g, step size beta, unit key k and query q:
//
//   S <- g S      u = beta (v - S^T k)      S <- S + k u^T      o = S^T q
//
// delta_step_kernel walks the rows of one (head, sequence) with the state in registers, laid out as in hgrn2_kernel: a warp owns
// 16 value columns (8 for states of 256 rows), its 16 lane pairs own every sixteenth quad of state rows.  S^T k and S^T q are
// taken from the state before the write in one exchange between the lanes -- the read-out after it is g S^T q + (k . q) u -- so a
// token costs one halving exchange and one broadcast of u.  The state is stored [slot][head][column][row], fp32 like all
// arithmetic here.  The gated norm of the read-out follows in head_rmsnorm_kernel.
//
// Prompts of the bf16 engine run in blocks of 64 tokens on the tensor cores (delta_prepare_kernel, delta_blocks_kernel below).
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

// ------------------------------------------------------------------------------------------------------
// Blocks of 64 tokens.  With c_t the sum of the log decays of the block up to token t, S the state at its start and
//
//   A[t][s] = beta_t exp(c_t - c_s) (k_t . k_s)   (s < t)          P[t][s] = exp(c_t - c_s) (q_t . k_s)   (s <= t)
//
// the writes of the block solve (I + A) U = diag(beta) (V - diag(exp c) K S).  delta_prepare_kernel inverts I + A once per
// (block, head) -- all blocks side by side -- and leaves  W = (I + A)^-1 diag(beta exp c) K,  X = (I + A)^-1 diag(beta) V  and P;
// delta_blocks_kernel then walks the blocks of a sequence:
//
//   U = X - W S        o_t = exp(c_t) S^T q_t + sum_s P[t][s] u_s        S <- exp(c_63) S + sum_s exp(c_63 - c_s) k_s u_s^T
//
// Exponents are differences within a block and never positive, so nothing overflows and nothing is divided by a decay; c is kept
// in double, so that differences of large sums stay good to fp32.  Products run on mma.sync tf32 with every fp32 factor split in
// two (about 20 bits).
// ------------------------------------------------------------------------------------------------------
constexpr int kDbTok = 64;

// Scratch between the two kernels, per block (entry by entry, in order), every array padded with zeros to whole blocks.
struct DeltaBlocks {
  const int* tile_seq;     // 64-row tiles of the prefill chunks
  const int* tile_q0;
  int num_tiles;
  float* w;                // [blocks, heads, 64, DP]
  float* x;                // [blocks, heads, 64, VP]
  float* pm;               // [blocks, heads, 64, 64]
  float* q;                // [blocks, groups, 64, DP] queries
  float* kt;               // [blocks, groups, DP, 64] keys, transposed
  float2* dec;             // [blocks, heads, 64]: exp(c_t), exp(c_63 - c_t)
  int VP;
};

// blocks of the entries before prefill entry s
OGB_DEVICE int db_first_block(const StepRows& sr, int s) {
  int n = 0;
  for (int i = 0; i < s; ++i) n += (sr.cu_q[i + 1] - sr.cu_q[i] + kDbTok - 1) / kDbTok;
  return n;
}

template <int DP>
struct DbCfg {
  static constexpr int kPitch = DP + 4, kTP = kDbTok + 4;
  static constexpr int kSmemBytes = 4 * (2 * kDbTok * kPitch + 2 * kDbTok * kTP + 32 * 33 + 3 * kDbTok) + 8 * kDbTok;
};

template <typename T, int DP>
__global__ void __launch_bounds__(256, 2) delta_prepare_kernel(DeltaParams p, DeltaBlocks bl) {
  using Cfg = DbCfg<DP>;
  extern __shared__ __align__(16) uint8_t db_smem[];
  double* sc = reinterpret_cast<double*>(db_smem);                // [64] sums of log decays
  float* sk = reinterpret_cast<float*>(sc + kDbTok);              // [64][pitch] keys, queries
  float* sq = sk + kDbTok * Cfg::kPitch;
  float* sA = sq + kDbTok * Cfg::kPitch;                          // [64][kTP] A, its inverse
  float* sT = sA + kDbTok * Cfg::kTP;
  float* sM = sT + kDbTok * Cfg::kTP;                             // [32][33]
  float* sl = sM + 32 * 33;                                       // [64] log decay, step size, exp(c)
  float* sb = sl + kDbTok;
  float* se = sb + kDbTok;
  const StepRows& sr = p.sr;
  const int head = blockIdx.y, per = p.heads / p.groups, group = head / per, seq = bl.tile_seq[blockIdx.x], q0 = bl.tile_q0[blockIdx.x];
  const int len = sr.cu_q[seq + 1] - sr.cu_q[seq], nt = min(kDbTok, len - q0);
  if (nt <= 0) return;
  const size_t row0 = static_cast<size_t>(sr.num_decode) + sr.cu_q[seq] + q0;
  const size_t block = static_cast<size_t>(db_first_block(sr, seq)) + q0 / kDbTok, bh = block * p.heads + head, bg = block * p.groups + group;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  if (p.D == DP && nt == kDbTok) {
    for (int i = tid; i < kDbTok * DP / 4; i += 256) {
      const int t = i / (DP / 4), d = i % (DP / 4) * 4;
      const float* src = p.qk + (row0 + t) * (2 * p.groups * DP) + group * DP + d;
      cp_async<16>(sq + t * Cfg::kPitch + d, src);
      cp_async<16>(sk + t * Cfg::kPitch + d, src + p.groups * DP);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  } else {
    for (int i = tid; i < kDbTok * DP; i += 256) {
      const int t = i / DP, d = i % DP;
      const float* src = p.qk + (row0 + t) * (2 * p.groups * p.D) + group * p.D + d;
      const bool live = t < nt && d < p.D;
      sq[t * Cfg::kPitch + d] = live ? src[0] : 0.f;
      sk[t * Cfg::kPitch + d] = live ? src[p.groups * p.D] : 0.f;
    }
  }
  if (tid < kDbTok) {
    const float2 x = tid < nt ? p.gates[(row0 + tid) * p.heads + head] : make_float2(0.f, 0.f);
    sl[tid] = x.x;
    sb[tid] = x.y;
  }
  for (int i = tid; i < kDbTok * Cfg::kTP; i += 256) sT[i] = 0.f;
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (tid < kDbTok) {
    double c = 0.0;
    for (int j = 0; j <= tid; ++j) c += static_cast<double>(sl[j]);
    sc[tid] = c;
    se[tid] = expf(static_cast<float>(c));
  }
  if (head % per == 0) {                                          // the group's first head leaves queries and transposed keys behind
    for (int i = tid; i < kDbTok * DP / 4; i += 256) {
      const int t = i / (DP / 4), d = i % (DP / 4) * 4;
      reinterpret_cast<float4*>(bl.q + bg * kDbTok * DP)[i] = *reinterpret_cast<const float4*>(sq + t * Cfg::kPitch + d);
    }
    for (int i = tid; i < kDbTok * DP / 4; i += 256) {
      const int d = i / (kDbTok / 4), t = i % (kDbTok / 4) * 4;
      reinterpret_cast<float4*>(bl.kt + bg * kDbTok * DP)[i] =
          make_float4(sk[t * Cfg::kPitch + d], sk[(t + 1) * Cfg::kPitch + d], sk[(t + 2) * Cfg::kPitch + d], sk[(t + 3) * Cfg::kPitch + d]);
    }
  }
  __syncthreads();
  if (tid < kDbTok) bl.dec[bh * kDbTok + tid] = make_float2(se[tid], expf(static_cast<float>(sc[kDbTok - 1] - sc[tid])));
  // ---- A (warps 0 - 3) and P (warps 4 - 7): the m-tiles are paired so that the warps of a scheduler share the triangle ----
  {
    const bool isq = warp >= 4;
    const int m = isq ? 7 - warp : warp;
#pragma unroll 1
    for (int n0 = 0; n0 < 8; n0 += 4) {
      const int n_tiles = min(4, 2 * m + 2 - n0);
      float c[4][4] = {};
      if (n_tiles > 0)
        split_product<DP / 8, 4>(c, (isq ? sq : sk) + 16 * m * Cfg::kPitch, Cfg::kPitch, sk + 8 * n0 * Cfg::kPitch, Cfg::kPitch, n_tiles, g, tq);
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = 16 * m + g + h * 8, s = 8 * (n0 + n) + 2 * tq;
          const float f0 = s <= t ? c[n][2 * h] * expf(static_cast<float>(sc[t] - sc[s])) : 0.f;
          const float f1 = s + 1 <= t ? c[n][2 * h + 1] * expf(static_cast<float>(sc[t] - sc[s + 1])) : 0.f;
          if (isq) *reinterpret_cast<float2*>(bl.pm + (bh * kDbTok + t) * kDbTok + s) = make_float2(f0, f1);
          else *reinterpret_cast<float2*>(sA + t * Cfg::kTP + s) = make_float2(s < t ? f0 * sb[t] : 0.f, s + 1 < t ? f1 * sb[t] : 0.f);
        }
    }
  }
  __syncthreads();
  // the values take the place of the queries (T is at most four bytes wide, a value row at most as long as the pitch allows at a time)
  constexpr int kVP = Cfg::kPitch * 4 / static_cast<int>(sizeof(T));   // pitch in elements
  T* sv = reinterpret_cast<T*>(sq);
  auto fetch_v = [&](int v0) {                                    // columns v0 .. v0 + DP of the values
    constexpr int kVec = 16 / static_cast<int>(sizeof(T));
    const T* src = static_cast<const T*>(p.v) + row0 * (p.heads * p.V) + static_cast<size_t>(head) * p.V + v0;
    const int cols = min(DP, p.V - v0);
    if (nt == kDbTok && cols % kVec == 0 && p.V % kVec == 0) {
      for (int i = tid; i < kDbTok * (cols / kVec); i += 256) {
        const int t = i / (cols / kVec), c = i % (cols / kVec) * kVec;
        cp_async<16>(sv + t * kVP + c, src + static_cast<size_t>(t) * (p.heads * p.V) + c);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    } else {
      for (int i = tid; i < kDbTok * DP; i += 256) {
        const int t = i / DP, c = i % DP;
        sv[t * kVP + c] = t < nt && c < cols ? src[static_cast<size_t>(t) * (p.heads * p.V) + c] : from_f32<T>(0.f);
      }
    }
  };
  fetch_v(0);
  // ---- T = (I + A)^-1: 16 x 16 diagonal blocks column by column, then two levels of T21 = -T22 (A21 T11) ----
  if (tid < kDbTok) {
    const int b = tid & ~15, col = tid & 15;
#pragma unroll 1
    for (int r = col; r < 16; ++r) {
      float a = r == col ? 1.f : 0.f;
#pragma unroll 4
      for (int j = col; j < r; ++j) a = fmaf(-sA[(b + r) * Cfg::kTP + b + j], sT[(b + j) * Cfg::kTP + b + col], a);
      sT[(b + r) * Cfg::kTP + b + col] = a;
    }
  }
  __syncthreads();
#pragma unroll
  for (int n = 16; n <= 32; n *= 2) {
    const int pairs = kDbTok / (2 * n);
    for (int i = tid; i < pairs * n * n; i += 256) {
      const int o = i / (n * n) * 2 * n, r = i / n % n, c = i % n;
      float a = 0.f;
#pragma unroll 8
      for (int j = 0; j < n; ++j) a = fmaf(sA[(o + n + r) * Cfg::kTP + o + j], sT[(o + j) * Cfg::kTP + o + c], a);
      sM[(o / (2 * n) * n + r) * 33 + c] = a;
    }
    __syncthreads();
    for (int i = tid; i < pairs * n * n; i += 256) {
      const int o = i / (n * n) * 2 * n, r = i / n % n, c = i % n;
      float a = 0.f;
#pragma unroll 8
      for (int j = 0; j < n; ++j) a = fmaf(-sT[(o + n + r) * Cfg::kTP + o + n + j], sM[(o / (2 * n) * n + j) * 33 + c], a);
      sT[(o + n + r) * Cfg::kTP + o + c] = a;
    }
    __syncthreads();
  }
  // ---- T [diag(beta exp c) K | diag(beta) V]: a warp takes 16 columns at a time, their 64 rows in registers ----
  auto columns = [&](auto value, float* dst, int ld, int n_cols) {
    for (int n = warp; n < (n_cols + 15) / 16; n += 8) {
      float2 b[2][8][2];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int k = 0; k < 8; ++k)
#pragma unroll
          for (int h = 0; h < 2; ++h) b[i][k][h] = tf32_cut(value(8 * k + tq + 4 * h, 16 * n + 8 * i + g));
#pragma unroll 1
      for (int m = 0; m < 4; ++m) {
        float c[2][4] = {}, e[2][4] = {};
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (k >= 2 * m + 2) break;
          float hi[4], lo[4];
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const float2 h = tf32_cut(sT[(16 * m + g + (x & 1) * 8) * Cfg::kTP + 8 * k + tq + (x >> 1) * 4]);
            hi[x] = h.x; lo[x] = h.y;
          }
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_tf32(c[i], hi, b[i][k][0].x, b[i][k][1].x);
            mma_tf32(e[i], lo, b[i][k][0].x, b[i][k][1].x);
            mma_tf32(e[i], hi, b[i][k][0].y, b[i][k][1].y);
          }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
          if (16 * n + 8 * i < n_cols)
#pragma unroll
            for (int h = 0; h < 2; ++h)
              *reinterpret_cast<float2*>(dst + static_cast<size_t>(16 * m + g + 8 * h) * ld + 16 * n + 8 * i + 2 * tq) =
                  make_float2(c[i][2 * h] + e[i][2 * h], c[i][2 * h + 1] + e[i][2 * h + 1]);
      }
    }
  };
  columns([&](int s, int c) { return sk[s * Cfg::kPitch + c] * sb[s] * se[s]; }, bl.w + bh * kDbTok * DP, DP, DP);
  for (int v0 = 0; v0 < p.V; v0 += DP) {
    if (v0 > 0) {
      __syncthreads();
      fetch_v(v0);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    columns([&](int s, int c) { return v0 + c < p.V ? to_f32<T>(sv[s * kVP + c]) * sb[s] : 0.f; }, bl.x + bh * kDbTok * bl.VP + v0, bl.VP,
            min(DP, bl.VP - v0));
  }
}

// One CTA = (sequence, head, NV value columns), the blocks one after the other.  Warps 0 - 3 form U (16 tokens each), warps 4 - 7 the
// read-out; the state lies in the accumulators of the first DP / 16 warps (16 rows each) and, split, in shared memory as the next
// block's operand.  The other operands go straight from the scratch to registers, a block ahead: within 16 columns a thread holds
// four neighbouring ones, which are the columns (tq, tq + 4) of two steps of eight -- the shared operands are read to match.
template <int DP, int NV>
struct DwCfg {
  static constexpr int kPS = DP + 2, kPU = kDbTok + 2;            // row pitches in (hi, lo) pairs
  static constexpr int kSmemBytes = 8 * NV * (kPS + 2 * kPU);
};

template <int DP, int NV>
__global__ void __launch_bounds__(256, 1) delta_blocks_kernel(DeltaParams p, DeltaBlocks bl) {
  using Cfg = DwCfg<DP, NV>;
  constexpr int NT = NV / 8;
  extern __shared__ __align__(16) uint8_t db_smem[];
  float2* sS = reinterpret_cast<float2*>(db_smem);                // [NV][kPS]
  float2* sU = sS + NV * Cfg::kPS;                                // [NV][kPU] writes, decayed to the block's end below
  float2* sD = sU + NV * Cfg::kPU;
  DeltaItem it;
  if (!it.set(p, blockIdx.z + p.z0)) return;
  const int head = blockIdx.y, group = head / (p.heads / p.groups), col0 = blockIdx.x * NV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int m = warp & 3;
  const bool reads = warp >= 4, holds = warp < DP / 16;
  float* own = p.state + (static_cast<size_t>(it.slot) * p.heads + head) * p.V * DP;

  float s[NT][4];                                                 // rows 16 warp + g (+ 8), columns 8 n + 2 tq (+ 1)
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int v = col0 + 8 * n + 2 * tq + (x & 1), d = 16 * warp + g + (x >> 1) * 8;
      s[n][x] = holds && !it.fresh && v < p.V ? own[static_cast<size_t>(v) * DP + d] : 0.f;
    }
  auto put_state = [&]() {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) sS[(8 * n + 2 * tq + (x & 1)) * Cfg::kPS + 16 * warp + g + (x >> 1) * 8] = tf32_cut(s[n][x]);
  };
  if (holds) put_state();

  // this thread's places in the scratch of block b0 + b
  const size_t b0 = db_first_block(p.sr, it.entry - p.sr.num_decode), bh = b0 * p.heads + head, bg = b0 * p.groups + group;
  const size_t step_h = static_cast<size_t>(p.heads) * kDbTok, step_g = static_cast<size_t>(p.groups) * kDbTok * DP;
  const int t0 = 16 * m + g;
  const float* pa = reads ? bl.q + bg * kDbTok * DP + t0 * DP + 4 * tq : bl.w + (bh * kDbTok + t0) * DP + 4 * tq;
  const size_t step_a = reads ? step_g : step_h * DP;
  const float* px = bl.x + (bh * kDbTok + t0) * bl.VP + col0 + 2 * tq;
  const float* pp = bl.pm + (bh * kDbTok + t0) * kDbTok + 4 * tq;
  const float* pk = bl.kt + bg * kDbTok * DP + (16 * warp + g) * kDbTok + 4 * tq;
  const float2* pd = bl.dec + bh * kDbTok;

  float4 a[DP / 16][2], k4[4][2], p4[4][2];
  float2 xr[NT][2], de[2];
  float last = 1.f;
  auto fetch_a = [&]() {                                          // rows of W and X, or of the queries
#pragma unroll
    for (int j = 0; j < DP / 16; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) a[j][h] = *reinterpret_cast<const float4*>(pa + h * 8 * DP + 16 * j);
    pa += step_a;
#pragma unroll
    for (int h = 0; h < 2; ++h) de[h] = pd[t0 + 8 * h];
    if (!reads) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          xr[n][h] = col0 + 8 * n < bl.VP ? *reinterpret_cast<const float2*>(px + h * 8 * bl.VP + 8 * n) : make_float2(0.f, 0.f);
      px += step_h * bl.VP;
    }
  };
  auto fetch_k = [&]() {                                          // rows of the transposed keys and of P; the block's whole decay
    last = pd[kDbTok - 1].x;
    pd += step_h;
    if (holds) {
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h) k4[j][h] = *reinterpret_cast<const float4*>(pk + h * 8 * kDbTok + 16 * j);
      pk += step_g;
    }
    if (reads) {
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          if (j <= m) p4[j][h] = *reinterpret_cast<const float4*>(pp + h * 8 * kDbTok + 16 * j);
      pp += step_h * kDbTok;
    }
  };
  // c += (rows in registers) x (pairs in shared memory): 16 columns of the contraction per call
  auto mma16 = [&](float (&c)[NT][4], float (&e)[NT][4], const float4& r0, const float4& r1, const float2* b, int pitch) {
    const float av[2][2][2] = {{{r0.x, r0.y}, {r1.x, r1.y}}, {{r0.z, r0.w}, {r1.z, r1.w}}};
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const float2 h0 = tf32_cut(av[u][0][0]), h1 = tf32_cut(av[u][1][0]), h2 = tf32_cut(av[u][0][1]), h3 = tf32_cut(av[u][1][1]);
      const float hi[4] = {h0.x, h1.x, h2.x, h3.x}, lo[4] = {h0.y, h1.y, h2.y, h3.y};
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float4 bb = *reinterpret_cast<const float4*>(b + (8 * n + g) * pitch + 4 * tq + 2 * u);
        mma_tf32(c[n], hi, bb.x, bb.z);
        mma_tf32(e[n], lo, bb.x, bb.z);
        mma_tf32(e[n], hi, bb.y, bb.w);
      }
    }
  };

  const int blocks = (it.n + kDbTok - 1) / kDbTok;
  fetch_a();
  fetch_k();
  __syncthreads();
  for (int b = 0; b < blocks; ++b) {
    float c[NT][4] = {}, e[NT][4] = {};
#pragma unroll
    for (int j = 0; j < DP / 16; ++j) mma16(c, e, a[j][0], a[j][1], sS + 16 * j, Cfg::kPS);
    if (!reads) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int h = x >> 1, at = (8 * n + 2 * tq + (x & 1)) * Cfg::kPU + t0 + 8 * h;
          const float u = ((x & 1) ? xr[n][h].y : xr[n][h].x) - (c[n][x] + e[n][x]);
          sU[at] = tf32_cut(u);
          sD[at] = tf32_cut(u * de[h].y);
        }
    }
    const float d0 = de[0].x, d1 = de[1].x;
    if (b + 1 < blocks) fetch_a();
    __syncthreads();
    if (holds) {
      float f[NT][4] = {};
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) s[n][x] *= last;
#pragma unroll
      for (int j = 0; j < 4; ++j) mma16(s, f, k4[j][0], k4[j][1], sD + 16 * j, Cfg::kPU);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) s[n][x] += f[n][x];
      put_state();
    }
    if (reads) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          c[n][x] = (c[n][x] + e[n][x]) * (x < 2 ? d0 : d1);
          e[n][x] = 0.f;
        }
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (j <= m) mma16(c, e, p4[j][0], p4[j][1], sU + 16 * j, Cfg::kPU);
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = b * kDbTok + t0 + 8 * h;
        if (t < it.n) {
          float* dst = p.out + (static_cast<size_t>(it.base) + t) * (p.heads * p.V) + head * p.V;
#pragma unroll
          for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int x = 0; x < 2; ++x) {
              const int v = col0 + 8 * n + 2 * tq + x;
              if (v < p.V) dst[v] = c[n][2 * h + x] + e[n][2 * h + x];
            }
        }
      }
    }
    if (b + 1 < blocks) fetch_k();
    __syncthreads();
  }
  if (holds) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int v = col0 + 8 * n + 2 * tq + (x & 1), d = 16 * warp + g + (x >> 1) * 8;
        if (v < p.V) own[static_cast<size_t>(v) * DP + d] = s[n][x];
      }
  }
}

template <int DP, int NV>
static int launch_delta_walk(const DeltaParams& p, const DeltaBlocks& bl, int entries, cudaStream_t stream) {
  constexpr int smem = DwCfg<DP, NV>::kSmemBytes;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(delta_blocks_kernel<DP, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr_set = true;
  }
  delta_blocks_kernel<DP, NV><<<dim3((p.V + NV - 1) / NV, p.heads, entries), 256, smem, stream>>>(p, bl);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int DP>
static int launch_delta_blocks(DeltaParams p, const DeltaBlocks& bl, int entries, cudaStream_t stream) {
  constexpr int smem = DbCfg<DP>::kSmemBytes;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(delta_prepare_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr_set = true;
  }
  delta_prepare_kernel<T, DP><<<dim3(bl.num_tiles, p.heads), 256, smem, stream>>>(p, bl);
  const int rc = static_cast<int>(cudaGetLastError());
  if (rc != 0) return rc;
  p.z0 = p.sr.num_decode;
  // narrow slices put more SMs to work on few heads; wide ones read the shared operands less often
  if (static_cast<long long>((p.V + 15) / 16) * p.heads * entries <= ogb_num_sms()) return launch_delta_walk<DP, 16>(p, bl, entries, stream);
  return launch_delta_walk<DP, 32>(p, bl, entries, stream);
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

// Floats of scratch that the block form needs per block of 64 tokens (0: the size has none).
extern "C" int ogb_delta_block_floats(int heads, int groups, int D, int V) {
  const int dp = D <= 64 ? 64 : D <= 128 ? 128 : 0;
  return dp == 0 ? 0 : heads * kDbTok * (dp + (V + 7) / 8 * 8 + kDbTok + 2) + groups * 2 * kDbTok * dp;
}

// scratch (16-byte aligned, ogb_delta_block_floats of each of num_tiles blocks): prefill chunks run in blocks on the tensor cores.
extern "C" int ogb_delta_rule(const float* qk, const void* v, const void* gates, float* state, float* out, int heads, int groups, int D, int V,
                              const int* ctx_len, const int* state_slot, const int* cu_q, const int* tile_seq, const int* tile_q0, int num_decode,
                              int num_prefill, int num_tiles, int num_slots, float* scratch, int elem, int* status, void* stream) {
  if (num_decode + num_prefill <= 0 || heads <= 0 || V <= 0) return 0;
  if (D < 1 || D > 256 || groups < 1 || heads % groups != 0) return -3;
  DeltaParams p{qk, v, static_cast<const float2*>(gates), state, out, heads, groups, D, V, 0,
                StepRows{ctx_len, state_slot, cu_q, tile_seq, tile_q0, num_decode, num_tiles, num_slots}, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool in_blocks = scratch != nullptr && D <= 128 && num_prefill > 0 && num_tiles > 0 &&
                         ((reinterpret_cast<uintptr_t>(qk) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(scratch)) & 15) == 0;
  const int items = num_decode + (in_blocks ? 0 : num_prefill);
  int rc = -3;
  if (elem == kElemBF16) rc = dispatch_delta_step<__nv_bfloat16>(p, items, s);
  else if (elem == kElemF32) rc = dispatch_delta_step<float>(p, items, s);
  if (rc != 0 || !in_blocks) return rc;
  DeltaBlocks bl;
  const int dp = D <= 64 ? 64 : 128;
  const size_t n = static_cast<size_t>(num_tiles) * heads * kDbTok, ng = static_cast<size_t>(num_tiles) * groups * kDbTok * dp;
  bl.tile_seq = tile_seq; bl.tile_q0 = tile_q0; bl.num_tiles = num_tiles;
  bl.VP = (V + 7) / 8 * 8;
  bl.w = scratch;
  bl.x = bl.w + n * dp;
  bl.pm = bl.x + n * bl.VP;
  bl.q = bl.pm + n * kDbTok;
  bl.kt = bl.q + ng;
  bl.dec = reinterpret_cast<float2*>(bl.kt + ng);
  if (elem == kElemBF16) return dp == 64 ? launch_delta_blocks<__nv_bfloat16, 64>(p, bl, num_prefill, s) : launch_delta_blocks<__nv_bfloat16, 128>(p, bl, num_prefill, s);
  return dp == 64 ? launch_delta_blocks<float, 64>(p, bl, num_prefill, s) : launch_delta_blocks<float, 128>(p, bl, num_prefill, s);
}
