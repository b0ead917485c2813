// Products of a few token rows with a streamed weight, shared by the decode kernels of the mixture of experts and of latent attention.
//
// One warp owns 16 weight rows (K contiguous) and up to 8 * NT tokens held in shared memory: mma.sync m16n8k16 with the weight rows as the M side
// and the tokens as the N side. The K order inside a 32-element step is permuted the same way on both sides, so that a thread's share of a row is
// 16 contiguous bytes: weights go from global memory straight to registers with 16-byte loads (four steps of a row pair in flight per thread), and
// no staging of the weight stream through shared memory is needed. The shape (<= 16 tokens) is bound by that stream, not by the tensor pipe.
#pragma once
#include "common.cuh"

FT_DEVICE uint4 ldg_stream(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
FT_DEVICE void mma_bf16_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// bytes between token rows in shared memory: a multiple of 64 that is 64 mod 128, so the 16-byte reads of a warp are conflict free. kp: padded K
__host__ __device__ inline int skinny_pitch(int kp) { return (kp * 2) % 128 == 0 ? kp * 2 + 64 : kp * 2; }

// acc[nt] += W[row g | row g + 8][0..kp) . X[token][0..kp): c0, c1 = row g of tokens 2t, 2t+1 and c2, c3 = row g + 8 (g = lane / 4, t = lane % 4).
// w: first of the 16 rows; ldw: elements between rows (16-byte aligned rows); kp: multiple of 32, both operands zero (or finite against zero) past K.
template <int NT>
FT_DEVICE void skinny_rows16(const __nv_bfloat16* __restrict__ w, int64_t ldw, int kp, const uint8_t* xs, int pitch, float (&acc)[NT][4]) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const __nv_bfloat16* lo = w + (size_t)g * ldw + t * 8;
  const __nv_bfloat16* hi = w + (size_t)(g + 8) * ldw + t * 8;
  const uint8_t* xr = xs + g * pitch + t * 16;
  auto step = [&](const uint4& a, const uint4& b, int k) {
#pragma unroll
    for (int n = 0; n < NT; n++) {
      const uint4 x = *reinterpret_cast<const uint4*>(xr + n * 8 * pitch + k * 2);
      mma_bf16_16816(acc[n], a.x, b.x, a.y, b.y, x.x, x.y);
      mma_bf16_16816(acc[n], a.z, b.z, a.w, b.w, x.z, x.w);
    }
  };
  constexpr int U = 4;
  int k = 0;
  for (; k + 32 * U <= kp; k += 32 * U) {
    uint4 a[U], b[U];
#pragma unroll
    for (int i = 0; i < U; i++) { a[i] = ldg_stream(lo + k + 32 * i); b[i] = ldg_stream(hi + k + 32 * i); }
#pragma unroll
    for (int i = 0; i < U; i++) step(a[i], b[i], k + 32 * i);
  }
  for (; k < kp; k += 32) {
    const uint4 a = ldg_stream(lo + k), b = ldg_stream(hi + k);
    step(a, b, k);
  }
}

// token row `n` of shared memory <- src[0..K), zeros up to kp; src is 16-byte aligned and readable up to the next multiple of 8 elements
FT_DEVICE void skinny_fill_row(uint8_t* xs, int pitch, int n, const __nv_bfloat16* src, int K, int kp, int tid, int nthreads) {
  for (int i = tid; i < kp / 8; i += nthreads) {
    uint4 v = make_uint4(0, 0, 0, 0);
    if (src != nullptr && i * 8 < K) {
      v = *reinterpret_cast<const uint4*>(src + i * 8);
      if (i * 8 + 8 > K) {
        __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&v);
        for (int j = K - i * 8; j < 8; j++) e[j] = __float2bfloat16(0.f);
      }
    }
    *reinterpret_cast<uint4*>(xs + (size_t)n * pitch + i * 16) = v;
  }
}
