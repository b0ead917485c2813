// Products of a few token rows with a streamed weight, shared by the decode kernels of the mixture of experts and of latent attention.
//
// A work item is 16 weight rows (K contiguous) of one group (an expert, a head) against up to 8 * NT tokens held in shared memory: mma.sync m16n8k16
// with the weight rows as the M side and the tokens as the N side. The K order inside a 32-element step is permuted the same way on both sides, so
// that a thread's share of a row is 16 contiguous bytes: weights go from global memory straight to registers with 16-byte loads. The eight warps of a
// CTA take an eighth of K each (the partial tiles meet in shared memory), so that an item is one or two memory round trips long, and the next item's
// first loads are issued before the current one is reduced. CTAs walk contiguous ranges of items of equal cost. The shape (<= 16 tokens) is bound by
// the weight stream, not by the tensor pipe.
#pragma once
#include "common.cuh"
#include "host_common.h"

FT_DEVICE uint4 ldg_stream(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
FT_DEVICE void mma_bf16_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
constexpr int SKINNY_SMEM_MAX = 208 * 1024;
// bytes between token rows in shared memory: a multiple of 64 that is 64 mod 128, so the 16-byte reads of a warp are conflict free. kp: padded K
__host__ __device__ inline int skinny_pitch(int kp) { return (kp * 2) % 128 == 0 ? kp * 2 + 64 : kp * 2; }

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

// P describes the groups: struct with
//   int count[2], per[2], cost[2]   two classes of groups: number of groups, items per group, cost of an item   (device function shape())
//   K(g), w(g, blk), ldw(g)         inner size, first row of 16-row block blk, row pitch; blocks are readable whole, rows up to K rounded up to 32
//   x_id(g), x_row(g, n)            groups with equal x_id share their tokens; row of token column n (null: empty)
//   finish(g, blk, nt, c, lane)     c.x, c.y: row lane / 4 of columns nt * 8 + 2 (lane % 4) + {0, 1}; c.z, c.w: row lane / 4 + 8
struct SkinnyShape {
  int count[2], per[2], cost[2];
};
constexpr int SKINNY_U = 4;        // 32-element steps per batch of loads

template <class P, int NT>
__global__ void __launch_bounds__(256, 2) skinny_stream_kernel(const P p) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t xs[];
  __shared__ float4 red[2][8][NT][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t8 = (lane & 3) * 8;
  const SkinnyShape S = p.shape();
  const int n0 = S.count[0] * S.per[0], n1 = S.count[1] * S.per[1];
  const long long total0 = (long long)n0 * S.cost[0], total = total0 + (long long)n1 * S.cost[1];
  auto bound = [&](int c) -> int {
    const long long b = total * c / gridDim.x;
    return b <= total0 ? (int)((b + S.cost[0] - 1) / S.cost[0]) : n0 + (int)((b - total0 + S.cost[1] - 1) / S.cost[1]);
  };
  const int lo = bound(blockIdx.x), hi = bound(blockIdx.x + 1);
  if (lo >= hi) return;
  auto group_of = [&](int it) { return it < n0 ? it / S.per[0] : S.count[0] + (it - n0) / S.per[1]; };
  auto block_of = [&](int it) { return it < n0 ? it % S.per[0] : (it - n0) % S.per[1]; };
  uint4 ca[SKINNY_U], cb[SKINNY_U];
  // this warp's steps of an item: [s0, s1)
  auto span = [&](int K, int& s0, int& s1, int& batches) {
    const int steps = (K + 31) >> 5, each = (steps + 7) >> 3;
    s0 = warp * each;
    s1 = min(steps, s0 + each);
    batches = (each + SKINNY_U - 1) / SKINNY_U;
  };
  auto load = [&](const __nv_bfloat16* base, int64_t ldw, int first, int s1, uint4 (&a)[SKINNY_U], uint4 (&b)[SKINNY_U]) {
    const __nv_bfloat16* r = base + (size_t)g8 * ldw + t8;
#pragma unroll
    for (int i = 0; i < SKINNY_U; i++)
      if (first + i < s1) {
        a[i] = ldg_stream(r + (size_t)(first + i) * 32);
        b[i] = ldg_stream(r + 8 * ldw + (size_t)(first + i) * 32);
      }
  };
  int g = group_of(lo), s0, s1, batches;
  span(p.K(g), s0, s1, batches);
  const __nv_bfloat16* base = p.w(g, block_of(lo));
  load(base, p.ldw(g), s0, s1, ca, cb);
  int xid = -1, pitch = 0;
  for (int it = lo; it < hi; it++) {
    const int blk = block_of(it);
    // the next item's rows (its first batch is requested while this item's last one is multiplied)
    const bool more = it + 1 < hi;
    const int gn = more ? group_of(it + 1) : g;
    const __nv_bfloat16* base_n = more ? p.w(gn, block_of(it + 1)) : base;
    int s0n = s0, s1n = s1, batches_n = batches;
    if (gn != g) span(p.K(gn), s0n, s1n, batches_n);
    if (p.x_id(g) != xid) {          // every warp has left the previous tokens behind at the last item's barrier
      const int K = p.K(g), kp = (K + 31) & ~31;
      pitch = skinny_pitch(kp);
      for (int n = 0; n < 8 * NT; n++) skinny_fill_row(xs, pitch, n, p.x_row(g, n), K, kp, threadIdx.x, 256);
      xid = p.x_id(g);
      __syncthreads();
    }
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; n++) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    const int64_t ldw = p.ldw(g);
    for (int bt = 0; bt < batches; bt++) {
      uint4 na[SKINNY_U], nb[SKINNY_U];
      if (bt + 1 < batches) load(base, ldw, s0 + (bt + 1) * SKINNY_U, s1, na, nb);
      else if (more) load(base_n, p.ldw(gn), s0n, s1n, na, nb);
#pragma unroll
      for (int i = 0; i < SKINNY_U; i++) {
        const int st = s0 + bt * SKINNY_U + i;
        if (st < s1) {
#pragma unroll
          for (int n = 0; n < NT; n++) {
            const uint4 x = *reinterpret_cast<const uint4*>(xs + (size_t)(n * 8 + g8) * pitch + st * 64 + t8 * 2);
            mma_bf16_16816(acc[n], ca[i].x, cb[i].x, ca[i].y, cb[i].y, x.x, x.y);
            mma_bf16_16816(acc[n], ca[i].z, cb[i].z, ca[i].w, cb[i].w, x.z, x.w);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < SKINNY_U; i++) { ca[i] = na[i]; cb[i] = nb[i]; }
    }
    const int buf = it & 1;
#pragma unroll
    for (int n = 0; n < NT; n++) red[buf][warp][n][lane] = make_float4(acc[n][0], acc[n][1], acc[n][2], acc[n][3]);
    __syncthreads();
#pragma unroll
    for (int n = 0; n < NT; n++)
      if (warp == ((it + n) & 7)) {
        float4 c = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int w = 0; w < 8; w++) {
          const float4 v = red[buf][w][n][lane];
          c.x += v.x; c.y += v.y; c.z += v.z; c.w += v.w;
        }
        p.finish(g, blk, n, c, lane);
      }
    g = gn; base = base_n; s0 = s0n; s1 = s1n; batches = batches_n;
  }
}

// launch with 8 * NT token rows of kmax elements in shared memory; grid: two CTAs per SM where their tokens fit
template <class P, int NT>
inline int skinny_launch(const P& p, int kmax, int max_items, cudaStream_t st) {
  const int smem = 8 * NT * skinny_pitch((kmax + 31) & ~31) + 64;
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    FT_CUDA_TRY(cudaFuncSetAttribute(skinny_stream_kernel<P, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, SKINNY_SMEM_MAX));
    done[dev] = true;
  }
  int grid = smem > 96 * 1024 ? 148 : 296;
  if (grid > max_items) grid = max_items;
  return (int)ft_launch_pdl(skinny_stream_kernel<P, NT>, dim3(grid), dim3(256), (size_t)smem, st, p);
}
