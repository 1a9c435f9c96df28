// Shared pieces of the kernels behind models with a per-layer mixer choice (hybrid.cu, recurrent.cu,
// latent_attention.cu): the row structure of a step, loads / stores of the two activation types, packed fp32
// arithmetic and the split tf32 products of the recurrences.
// These files are compiled without fast math: tanh, exponentials, divisions and roots keep their full precision.
#pragma once
#include "common.cuh"

namespace ogb {

enum ElemType : int { kElemF32 = 0, kElemBF16 = 1 };

template <typename T> OGB_DEVICE float to_f32(T v);
template <> OGB_DEVICE float to_f32<float>(float v) { return v; }
template <> OGB_DEVICE float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> OGB_DEVICE T from_f32(float v);
template <> OGB_DEVICE float from_f32<float>(float v) { return v; }
template <> OGB_DEVICE __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// V consecutive elements as fp32 (one vector access where V is 2 or 4; the pointer is then aligned to it)
template <int V, typename T>
OGB_DEVICE void load_vec(const T* p, float (&r)[V]) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r[0] = f.x; r[1] = f.y; r[2] = f.z; r[3] = f.w;
  } else if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
    r[0] = a.x; r[1] = a.y; r[2] = b.x; r[3] = b.y;
  } else if constexpr (V == 2 && sizeof(T) == 4) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    r[0] = f.x; r[1] = f.y;
  } else if constexpr (V == 2) {
    const float2 f = unpack_bf16(*reinterpret_cast<const uint32_t*>(p));
    r[0] = f.x; r[1] = f.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) r[i] = to_f32<T>(p[i]);
  }
}
template <int V, typename T>
OGB_DEVICE void store_vec(T* p, const float (&r)[V]) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]);
  } else if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r[0], r[1]), pack_bf16(r[2], r[3]));
  } else if constexpr (V == 2 && sizeof(T) == 4) {
    *reinterpret_cast<float2*>(p) = make_float2(r[0], r[1]);
  } else if constexpr (V == 2) {
    *reinterpret_cast<uint32_t*>(p) = pack_bf16(r[0], r[1]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = from_f32<T>(r[i]);
  }
}

// Rows of a step: `num_decode` single-token rows (row r belongs to sequence entry r), then the packed prefill chunks
// (sequence entry num_decode + s holds rows num_decode + cu_q[s] .. num_decode + cu_q[s + 1]).  ctx_len counts an entry's
// tokens after the step, so its first row sits at position ctx_len - rows.
struct StepRows {
  const int* ctx_len;
  const int* state_slot;
  const int* cu_q;
  const int* tile_seq;
  const int* tile_q0;
  int num_decode, num_tiles, num_slots;
};

// The rows of block `b`: a decode row, or up to R (a divisor of 64) rows of one prefill chunk; a grid has span_blocks of them.
template <int R>
struct RowSpan {
  int base, n, j0, j1, start, slot;            // first row of the entry, its rows, this block's rows within them, tokens before, slot (-1: none)
  OGB_DEVICE bool set(const StepRows& sr, int b, int* status) {
    int entry;
    if (b < sr.num_decode) {
      entry = b; base = b; n = 1; j0 = 0;
    } else {
      const int g = b - sr.num_decode, tile = g / (64 / R), s = sr.tile_seq[tile];
      entry = sr.num_decode + s;
      base = sr.num_decode + sr.cu_q[s];
      n = sr.cu_q[s + 1] - sr.cu_q[s];
      j0 = sr.tile_q0[tile] + (g % (64 / R)) * R;
    }
    j1 = min(j0 + R, n);
    start = sr.ctx_len[entry] - n;
    if (j0 >= n || start < 0) return false;    // a padding row has no tokens
    slot = sr.state_slot[entry];
    if (slot >= sr.num_slots) {
      if (threadIdx.x == 0) atomicOr(status, kStatusIndexOutOfRange);
      slot = -1;
    }
    return true;
  }
};
template <int R>
inline int span_blocks(const StepRows& sr) { return sr.num_decode + sr.num_tiles * (64 / R); }

// two fp32 values in one 64-bit register
typedef unsigned long long f32x2;
OGB_DEVICE f32x2 f2_fma(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
OGB_DEVICE f32x2 f2_mul(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
OGB_DEVICE float f2_sum(f32x2 a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}

template <int BYTES>
OGB_DEVICE void cp_async(void* dst, const void* src) {
  if constexpr (BYTES == 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

OGB_DEVICE float tf32_round(float x) {
  uint32_t r;
  asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x));
  return __uint_as_float(r);
}
OGB_DEVICE float2 tf32_split(float x) {
  const float hi = tf32_round(x);
  return make_float2(hi, tf32_round(x - hi));
}
// The cheaper split: the leading 11 bits as they are, and the rest (of which a tf32 operand keeps the leading 11 again).
OGB_DEVICE float2 tf32_cut(float x) {
  const float hi = __uint_as_float(__float_as_uint(x) & 0xffffe000u);
  return make_float2(hi, x - hi);
}
OGB_DEVICE void mma_tf32(float (&c)[4], const float (&a)[4], float b0, float b1) {
  asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])), "r"(__float_as_uint(b0)),
        "r"(__float_as_uint(b1)));
}

// C += A B^T over K in steps of 8, fp32 factors split in two tf32 terms (about 20 bits): A rows a + g, B rows b + g (K-major, row pitches
// pa, pb); the first nt tiles of eight B rows
template <int KS, int NT>
OGB_DEVICE void split_product(float (&c)[NT][4], const float* a, int pa, const float* b, int pb, int nt, int g, int tq) {
  float e[NT][4] = {};
#pragma unroll 2
  for (int k = 0; k < KS; ++k) {
    float hi[4], lo[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float2 h = tf32_cut(a[(g + (x & 1) * 8) * pa + 8 * k + tq + (x >> 1) * 4]);
      hi[x] = h.x; lo[x] = h.y;
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
      if (n < nt) {
        const float2 b0 = tf32_cut(b[(8 * n + g) * pb + 8 * k + tq]), b1 = tf32_cut(b[(8 * n + g) * pb + 8 * k + tq + 4]);
        mma_tf32(c[n], hi, b0.x, b1.x);
        mma_tf32(e[n], lo, b0.x, b1.x);
        mma_tf32(e[n], hi, b0.y, b1.y);
      }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) c[n][x] += e[n][x];
}

}  // namespace ogb
