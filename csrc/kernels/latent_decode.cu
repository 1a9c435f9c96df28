// Decode attention over paged latents: one token per sequence, up to 32 heads per CTA against one stream of latents.
//
// A decode row has few query rows (the heads), so the 128-row tensor-memory tiles of the prefill kernel would spend most of
// their shared-memory traffic on rows that do not exist.  Here the products run on mma.sync m16n8k16 with 16 or 32 rows and
// the kernel is laid out around the byte stream instead:
//
//   last warp    : TMA producer, 64 tokens (4 pages) x R values per stage, 128-byte swizzled column chunks
//   8 or 16 warps: (R key columns, of which the first V are values) S = Q' C^T split four ways over the latent's columns and two or four ways over the tokens (a warp keeps its
//                  slice of Q' in registers where they suffice), partial scores summed through shared memory, softmax with all
//                  threads, then O += P C with every warp owning its share of the output columns
//
// Keys split `num_splits` ways leave fp32 partials for latent_combine_kernel.  Waits are bounded; page ids are checked.
#include "attention_common.cuh"
#include "attention_tc.cuh"
#include "latent_attention.cuh"
#include "ogb_kernels.h"

namespace ogb {

constexpr int kLdKeys = 64;
constexpr int kLdPitch = 72;             // floats per row of partial scores: conflict-free 8-byte stores

template <int R, int V, int MT, int ST, int NW>
struct LdCfg {
  static constexpr int kRows = 16 * MT;
  static constexpr int kChunks = R / 64;
  static constexpr int kStage = kLdKeys * R * 2;
  static constexpr int kQBytes = kRows * R * 2;
  static constexpr int kPBytes = kRows * 128;
  static constexpr int kSBytes = 4 * kRows * kLdPitch * 4;
  static constexpr int kSmemBytes = ST * kStage + kQBytes + kPBytes + kSBytes + 1024 /*alignment*/ + 512 /*barriers, row factors*/ + 256;
  static_assert(R % 64 == 0 && V % (8 * NW) == 0 && V <= R, "tile shape");
  static_assert(kSmemBytes <= 227 * 1024, "shared memory");
};

// byte offset of (row, column) in a tile of [64-column chunk][rows][128 bytes], 128-byte swizzle
OGB_DEVICE uint32_t ld_off(int rows, int row, int col) {
  return static_cast<uint32_t>(((col >> 6) * rows + row) * 128 + ((((col & 63) >> 3) ^ (row & 7)) << 4));
}

// Called by the consumer threads of every split of a row once its partials are written: the last one to arrive merges them.
template <int NW>
OGB_DEVICE void ld_merge(const LatParams& p, int* counter, size_t row0, int heads, volatile int* flag) {
  __threadfence();
  asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
  if (threadIdx.x == 0) {
    const int last = atomicAdd(counter, 1) == p.num_splits - 1;
    if (last) *counter = 0;              // every split has arrived: ready for the next launch
    *flag = last;
  }
  asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
  if (*flag == 0) return;
  __threadfence();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int row = warp; row < heads; row += NW) {
    const float* ml = p.part_ml + 2 * (row0 + row) * p.num_splits;
    float m = -INFINITY, l = 0.f;
    for (int s = 0; s < p.num_splits; ++s) m = fmaxf(m, __ldcg(ml + 2 * s));
    for (int s = 0; s < p.num_splits; ++s) {
      const float ms = __ldcg(ml + 2 * s);
      if (ms != -INFINITY) l += __ldcg(ml + 2 * s + 1) * expf(ms - m);
    }
    const float inv = (l > 0.f ? 1.f / l : 0.f) * latent_gate<__nv_bfloat16>(p, row0 + row);
    for (int c = lane * 4; c < p.vrank; c += 128) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s = 0; s < p.num_splits; ++s) {
        const float ms = __ldcg(ml + 2 * s);
        if (ms == -INFINITY) continue;
        const float w = expf(ms - m) * inv;
        const float4 o = __ldcg(reinterpret_cast<const float4*>(p.part_o + ((row0 + row) * p.num_splits + s) * p.vrank + c));
        a.x = fmaf(w, o.x, a.x); a.y = fmaf(w, o.y, a.y); a.z = fmaf(w, o.z, a.z); a.w = fmaf(w, o.w, a.w);
      }
      *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p.out) + (row0 + row) * p.ldo + c) = make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
    }
  }
}

template <int R, int V, int MT, int ST, int NW>
__global__ void __launch_bounds__((NW + 1) * 32, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap c_map, const LatParams p) {
  using Cfg = LdCfg<R, V, MT, ST, NW>;
  constexpr int KS = R / 64;             // k-steps of a warp's column slice (R / 4 columns)
  constexpr int NT = V / (8 * NW);       // 8-column output tiles of a warp
  constexpr int KN = 4 / (NW / 4);       // 16-token score tiles of a warp: NW / 4 warps share a column slice
  constexpr int TPR = NW * 32 / (16 * MT), KPT = kLdKeys / TPR;   // softmax: threads a row, tokens a thread
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sK = smem;
  uint8_t* sQ = sK + ST * Cfg::kStage;
  uint8_t* sP = sQ + Cfg::kQBytes;
  float* sS = reinterpret_cast<float*>(sP + Cfg::kPBytes);
  uint64_t* full = reinterpret_cast<uint64_t*>(sS + 4 * Cfg::kRows * kLdPitch);
  uint64_t* empty = full + ST;
  uint64_t* q_full = empty + ST;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(q_full + 1);
  float* sA = reinterpret_cast<float*>(q_full + 2);      // [rows] rescale factors, at the end 1 / l or the split's (m, l)

  const int entry = blockIdx.x, head0 = blockIdx.y * Cfg::kRows;
  const int ctx = p.ctx_len[entry];
  if (ctx <= 0) return;                                  // padding row
  const int heads = min(Cfg::kRows, p.heads - head0);
  const int lo = p.window > 0 ? max(0, ctx - p.window) : 0;
  int b0 = lo / kLdKeys, b1 = (ctx + kLdKeys - 1) / kLdKeys;
  if (p.num_splits > 1) {
    const int per = (b1 - b0 + p.num_splits - 1) / p.num_splits;
    b0 += static_cast<int>(blockIdx.z) * per;
    b1 = min(b1, b0 + per);
  }
  const size_t row0 = static_cast<size_t>(entry) * p.heads + head0;
  const int nblk = b1 - b0;
  if (nblk <= 0) {
    if (static_cast<int>(threadIdx.x) < heads) {
      const size_t pr = (row0 + threadIdx.x) * p.num_splits + blockIdx.z;
      p.part_ml[2 * pr] = -INFINITY;
      p.part_ml[2 * pr + 1] = 0.f;
    }
    if (p.counters != nullptr && threadIdx.x < NW * 32)
      ld_merge<NW>(p, p.counters + entry * gridDim.y + blockIdx.y, row0, heads, abort_flag);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < ST; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], NW); }
    mbar_init(q_full, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();

  if (warp == NW) {
    if (lane == 0) {
      mbar_expect_tx(q_full, Cfg::kQBytes);
      for (int h = 0; h < Cfg::kChunks; ++h) tma_load_2d(sQ + h * Cfg::kRows * 128, &q_map, q_full, h * 64, static_cast<int>(row0));
      const int n_pages = (ctx + kLatPage - 1) / kLatPage;
      const int* table = p.page_table + static_cast<size_t>(entry) * p.max_pages;
      for (int it = 0; it < nblk; ++it) {
        const int st = it % ST;
        int row_of_page[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int pi = min(max((b0 + it) * 4 + i, lo / kLatPage), min(n_pages, p.max_pages) - 1);   // the rest is masked
          int64_t page = table[pi];
          if (page < 0 || page >= p.num_pages) {
            atomicOr(p.status, kStatusIndexOutOfRange);
            page = 0;
          }
          row_of_page[i] = static_cast<int>(page) * kLatPage;
        }
        if (!fa_wait(&empty[st], ((it / ST) & 1) ^ 1, abort_flag)) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; break; }
        mbar_expect_tx(&full[st], Cfg::kStage);
        uint8_t* dst = sK + st * Cfg::kStage;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int h = 0; h < Cfg::kChunks; ++h) tma_load_2d(dst + h * kLdKeys * 128 + i * 2048, &c_map, &full[st], h * 64, row_of_page[i]);
      }
    }
    // the copies in flight are waited for by the consumers (bounded), which leave after the last one
    return;
  }

  // ------------------------------ consumers ------------------------------
  const int g = lane >> 2, t = lane & 3;
  const int ks = warp & 3, kh = warp >> 2;               // column slice and token group of the score product
  const uint32_t aK = smem_u32(sK), aQ = smem_u32(sQ), aP = smem_u32(sP);
  bool ok = fa_wait(q_full, 0, abort_flag);
  constexpr bool kQRegs = MT * KS <= (NW == 16 ? 4 : 8);                  // else the registers are worth more as loads in flight
  uint32_t qf[MT][kQRegs ? KS : 1][4];
  auto load_q = [&](int m, int k, uint32_t (&f)[4]) {
    ldsm_x4(aQ + ld_off(Cfg::kRows, m * 16 + (lane & 15), ks * (R / 4) + k * 16 + (lane >> 4) * 8), f[0], f[1], f[2], f[3]);
  };
  if constexpr (kQRegs) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int k = 0; k < KS; ++k) load_q(m, k, qf[m][k]);
  }
  float o[MT][NT][4] = {};
  const int srow = threadIdx.x / TPR, sub = threadIdx.x % TPR;
  float m_run = -INFINITY, l_run = 0.f;
  const float scale = p.scale * 1.4426950408889634f;
  for (int it = 0; it < nblk; ++it) {
    const int st = it % ST;
    ok = __all_sync(0xffffffffu, ok && fa_wait(&full[st], (it / ST) & 1, abort_flag));
    if (!ok && lane == 0) { atomicOr(p.status, kStatusWaitTimeout); *abort_flag = 1; }
    const uint32_t kb = aK + st * Cfg::kStage;
    // ---- partial scores ----
    float s[MT][2 * KN][4] = {};
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if constexpr (!kQRegs) {
#pragma unroll
        for (int m = 0; m < MT; ++m) load_q(m, k, qf[m][0]);
      }
#pragma unroll
      for (int n2 = 0; n2 < KN; ++n2) {
        uint32_t b[4];
        ldsm_x4(kb + ld_off(kLdKeys, (kh * KN + n2) * 16 + (lane >> 4) * 8 + (lane & 7), ks * (R / 4) + k * 16 + ((lane >> 3) & 1) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16_16816(s[m][2 * n2], qf[m][kQRegs ? k : 0], b[0], b[1]);
          mma_bf16_16816(s[m][2 * n2 + 1], qf[m][kQRegs ? k : 0], b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 2 * KN; ++n) {
        float* d = sS + (ks * Cfg::kRows + m * 16 + g) * kLdPitch + kh * KN * 16 + n * 8 + 2 * t;
        *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
        *reinterpret_cast<float2*>(d + 8 * kLdPitch) = make_float2(s[m][n][2], s[m][n][3]);
      }
    asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
    // ---- softmax ----
    {
      float v[KPT];
#pragma unroll
      for (int j = 0; j < KPT; ++j) v[j] = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float* src = sS + (x * Cfg::kRows + srow) * kLdPitch + sub * KPT;
#pragma unroll
        for (int j = 0; j < KPT; j += 2) {
          const float2 b = *reinterpret_cast<const float2*>(src + j);
          v[j] += b.x; v[j + 1] += b.y;
        }
      }
      const int key0 = (b0 + it) * kLdKeys + sub * KPT;
      float mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < KPT; ++j) {
        v[j] = key0 + j >= lo && key0 + j < ctx ? v[j] * scale : -INFINITY;
        mx = fmaxf(mx, v[j]);
      }
#pragma unroll
      for (int x = 1; x < TPR; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
      const float m_new = fmaxf(m_run, mx);
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_new);
      const float neg = m_new == -INFINITY ? 0.f : -m_new;
      float sum = 0.f;
      uint32_t pk[KPT / 2];
#pragma unroll
      for (int j = 0; j < KPT; j += 2) {
        const float e0 = exp2f(v[j] + neg), e1 = exp2f(v[j + 1] + neg);
        sum += e0 + e1;
        pk[j / 2] = pack_bf16(e0, e1);
      }
      l_run = l_run * alpha + sum;                       // this thread's keys; the row's sum is formed at the end
      m_run = m_new;
      uint8_t* pd = sP + ld_off(Cfg::kRows, srow, sub * KPT) + (sub * KPT & 7) * 2;
      if constexpr (KPT == 8) *reinterpret_cast<uint4*>(pd) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
      else if constexpr (KPT == 4) *reinterpret_cast<uint2*>(pd) = make_uint2(pk[0], pk[1]);
      else *reinterpret_cast<uint32_t*>(pd) = pk[0];
      if (sub == 0) sA[srow] = alpha;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
    // ---- O += P C ----
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = sA[m * 16 + g], a1 = sA[m * 16 + g + 8];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
      }
    }
#pragma unroll
    for (int kk = 0; kk < 2; ++kk) {
      uint32_t pf[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int k = 0; k < 2; ++k)
          ldsm_x4(aP + ld_off(Cfg::kRows, m * 16 + (lane & 15), kk * 32 + k * 16 + (lane >> 4) * 8), pf[m][k][0], pf[m][k][1], pf[m][k][2], pf[m][k][3]);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        uint32_t b[4];
        ldsm_x4_t(kb + ld_off(kLdKeys, kk * 32 + lane, warp * (V / NW) + n * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16_16816(o[m][n], pf[m][0], b[0], b[1]);
          mma_bf16_16816(o[m][n], pf[m][1], b[2], b[3]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
  }
  // ---- row sums, output ----
  asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
  const bool split = p.num_splits > 1;
  {
#pragma unroll
    for (int x = 1; x < TPR; x <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, x);
    if (sub == 0) {
      sA[srow] = split ? 1.f : (l_run > 0.f && srow < heads ? latent_gate<__nv_bfloat16>(p, row0 + srow) / l_run : 0.f);
      if (split && srow < heads) {
        const size_t pr = (row0 + srow) * p.num_splits + blockIdx.z;
        p.part_ml[2 * pr] = m_run * 0.6931471805599453f;
        p.part_ml[2 * pr + 1] = l_run;
      }
    }
  }
  asm volatile("bar.sync 1, %0;" ::"n"(NW * 32) : "memory");
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int hrow = 0; hrow < 2; ++hrow) {
      const int row = m * 16 + hrow * 8 + g;
      if (row >= heads) continue;
      const float f = sA[row];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = warp * (V / NW) + n * 8 + 2 * t;
        if (col >= p.vrank) continue;
        const float x = o[m][n][2 * hrow] * f, y = o[m][n][2 * hrow + 1] * f;
        if (split)
          *reinterpret_cast<float2*>(p.part_o + ((row0 + row) * p.num_splits + blockIdx.z) * p.vrank + col) = make_float2(x, y);
        else
          *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(p.out) + (row0 + row) * p.ldo + col) = pack_bf16(x, y);
      }
    }
  const bool aborted = *abort_flag != 0;
  if (split && p.counters != nullptr) ld_merge<NW>(p, p.counters + entry * gridDim.y + blockIdx.y, row0, heads, reinterpret_cast<volatile int*>(sS));
  if (aborted) {
    // a wait ran out: give copies that may still be in flight a bounded time to land
    const uint64_t t0 = global_timer_ns();
    while (global_timer_ns() - t0 < 200000ull) { __nanosleep(1000); }
  }
}

template <int R, int V, int MT, int ST, int NW>
static int launch_ld(const LatParams& p, cudaStream_t stream) {
  using Cfg = LdCfg<R, V, MT, ST, NW>;
  CUtensorMap q_map, c_map;
  int rc = make_tmap_bf16_2d(&q_map, p.q, static_cast<uint64_t>(p.rows) * p.heads, p.rank, p.ldq, Cfg::kRows, 64);
  if (rc != 0) return rc;
  rc = make_tmap_bf16_2d(&c_map, p.pool, static_cast<uint64_t>(p.num_pages) * kLatPage, p.rank, p.ldp, kLatPage, 64);
  if (rc != 0) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    OGB_CUDA_CHECK(cudaFuncSetAttribute(latent_decode_kernel<R, V, MT, ST, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes));
    attr_set = true;
  }
  const dim3 grid(p.rows, (p.heads + Cfg::kRows - 1) / Cfg::kRows, p.num_splits);
  latent_decode_kernel<R, V, MT, ST, NW><<<grid, (NW + 1) * 32, Cfg::kSmemBytes, stream>>>(q_map, c_map, p);
  return static_cast<int>(cudaGetLastError());
}

template <int MT>
static int dispatch_ld(const LatParams& p, cudaStream_t stream) {
  if (p.rank <= 64) return launch_ld<64, 64, MT, 4, 8>(p, stream);
  if (p.rank <= 128) return launch_ld<128, 128, MT, 4, 8>(p, stream);
  if (p.rank <= 192 && p.vrank <= 128) return launch_ld<192, 128, MT, 4, 8>(p, stream);
  if (p.rank <= 256) return launch_ld<256, 256, MT, 4, 16>(p, stream);
  if (p.rank <= 320 && p.vrank <= 256) return launch_ld<320, 256, MT, 3, 16>(p, stream);
  if (p.rank <= 512) return launch_ld<512, 512, MT, 2, 16>(p, stream);
  if (p.vrank <= 512) return launch_ld<576, 512, MT, 2, 16>(p, stream);
  return -2;
}

int launch_latent_decode(const LatParams& p, cudaStream_t stream) {
  return p.heads <= 16 ? dispatch_ld<1>(p, stream) : dispatch_ld<2>(p, stream);
}

}  // namespace ogb
