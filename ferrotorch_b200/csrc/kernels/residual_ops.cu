// One f32 residual per token, with the norm on the sublayer's output or ahead of two sublayers that run side by side, averages over the layers' results, the token shift ahead of a
// mixer, and the activations of feed-forwards.
//
//   ft_residual_embed    x = scale * table[id];  h = x in the operand type
//   ft_residual_update   y = sum of the sublayer's f32 planes;  x += y / rms(y) * w;  h = x, or x / rms(x) * w_last ahead of the output projection
//   ft_parallel_embed    x = table[id];  h1 = x / rms(x) * w1, h2 = x / rms(x) * w2: the operands of two sublayers
//   ft_parallel_update   x += mult * (what both sublayers returned: f32 planes, expert rows through an index, a bias);  h1 and h2 from the new x
//   ft_depth_update      X = x + y / rms(y) * w, kept beside the results of the earlier layers;  x = a weighted sum of all of them;  its norm, shifted by one token or not
//   ft_token_shift       h = n + (n of the token before - n) * s with n = x / rms(x) * w:  the shifted operand of a prompt's rows
//   ft_gated_act         act(gate) * up of interleaved gate / up columns, from a 16-bit or f32 matrix or from split-K planes
//   ft_poly_norm         a N(z) + b N(z^2) + c N(z^3) + e with N dividing a row by its root mean square, from a 16-bit or f32 matrix or from split-K planes
//
// The updates take one row per cluster of CTAs: one CTA where there are rows enough to fill the GPU, up to eight (sums of squares meet in
// distributed shared memory) for the few rows of a decode step, whose planes are then read by eight SMs instead of one. Everything a row needs stays in
// registers between its two norms. Compiled without fast-math.
#include <cooperative_groups.h>

#include <utility>

#include "common.cuh"
#include "host_common.h"

namespace {

template <typename H> FT_DEVICE void put4(H* dst, float4 v);
template <> FT_DEVICE void put4<float>(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
template <> FT_DEVICE void put4<__nv_bfloat16>(__nv_bfloat16* dst, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&a);
  pk.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(dst) = pk;
}
template <typename H> FT_DEVICE float4 get4(const H* src);
template <> FT_DEVICE float4 get4<float>(const float* src) { return *reinterpret_cast<const float4*>(src); }
template <> FT_DEVICE float4 get4<__nv_bfloat16>(const __nv_bfloat16* src) {
  const uint2 r = *reinterpret_cast<const uint2*>(src);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
FT_DEVICE float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
// elements past the row's width: padding of the buffers, of unknown content
FT_DEVICE float4 keep4(float4 v, int c, int W) {
  if (c + 1 > W) v.x = 0.f;
  if (c + 2 > W) v.y = 0.f;
  if (c + 3 > W) v.z = 0.f;
  if (c + 4 > W) v.w = 0.f;
  return v;
}

template <typename H>
__global__ void __launch_bounds__(256) residual_embed_kernel(const int64_t* __restrict__ ids, const H* __restrict__ table, int64_t ld_table, int64_t vocab, float scale,
                                                             float* __restrict__ x, int64_t ldx, H* __restrict__ h, int64_t ldh, int rows, int W) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (c >= W) return;
  for (int r = blockIdx.y; r < rows; r += gridDim.y) {
    const int64_t id = ids[r];
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (id >= 0 && id < vocab) v = keep4(get4(table + (size_t)id * ld_table + c), c, W);
    v = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
    *reinterpret_cast<float4*>(x + (size_t)r * ldx + c) = v;
    put4(h + (size_t)r * ldh + c, v);
  }
}

constexpr int UPD_THREADS = 256;
// NV: float4 columns per thread, of TH threads
template <int NV, int TH, typename H>
__global__ void __launch_bounds__(TH) residual_update_kernel(float* __restrict__ x, int64_t ldx, const float* __restrict__ y, int planes, size_t pstride, int64_t ldy,
                                                                      const float* __restrict__ w, const float* __restrict__ w_last, float eps, H* __restrict__ h,
                                                                      int64_t ldh, int ncta, int W, int cols, int store_x) {
  namespace cg = cooperative_groups;
  __shared__ float red[32];
  __shared__ float cta_ss[2];
  cg::cluster_group cluster = cg::this_cluster();
  const int row = blockIdx.x / ncta, c0 = blockIdx.x % ncta * cols, cend = min(W, c0 + cols);
  float4 wv[NV];                                    // weights do not depend on the predecessor
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * TH + threadIdx.x) * 4;
    wv[i] = c < cend ? *reinterpret_cast<const float4*>(w + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  pdl_launch_dependents();
  auto row_sum = [&](float ss, int slot) -> float {
    ss = block_sum(ss, red);
    if (ncta == 1) return ss;
    if (threadIdx.x == 0) cta_ss[slot] = ss;
    cluster.sync();
    float t = 0.f;
    for (int r = 0; r < ncta; r++) t += *cluster.map_shared_rank(&cta_ss[slot], r);
    return t;
  };
  const float* yr = y + (size_t)row * ldy;
  float* xr = x + (size_t)row * ldx;
  float4 v[NV], xv[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * TH + threadIdx.x) * 4;
    v[i] = xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < cend) {
      xv[i] = *reinterpret_cast<const float4*>(xr + c);
      int p = 0;
      for (; p + 4 <= planes; p += 4) {
        float4 t[4];
#pragma unroll
        for (int j = 0; j < 4; j++) t[j] = __ldcg(reinterpret_cast<const float4*>(yr + (p + j) * pstride + c));
        v[i].x += (t[0].x + t[1].x) + (t[2].x + t[3].x);
        v[i].y += (t[0].y + t[1].y) + (t[2].y + t[3].y);
        v[i].z += (t[0].z + t[1].z) + (t[2].z + t[3].z);
        v[i].w += (t[0].w + t[1].w) + (t[2].w + t[3].w);
      }
      for (; p < planes; p++) {
        const float4 t = __ldcg(reinterpret_cast<const float4*>(yr + p * pstride + c));
        v[i].x += t.x; v[i].y += t.y; v[i].z += t.z; v[i].w += t.w;
      }
      v[i] = keep4(v[i], c, W);
      ss += sq4(v[i]);
    }
  }
  const float rstd = 1.f / sqrtf(row_sum(ss, 0) / (float)W + eps);
  float s2 = 0.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * TH + threadIdx.x) * 4;
    xv[i] = make_float4(xv[i].x + v[i].x * rstd * wv[i].x, xv[i].y + v[i].y * rstd * wv[i].y, xv[i].z + v[i].z * rstd * wv[i].z, xv[i].w + v[i].w * rstd * wv[i].w);
    if (c < cend) {
      xv[i] = keep4(xv[i], c, W);
      if (store_x) *reinterpret_cast<float4*>(xr + c) = xv[i];
      if (w_last == nullptr) put4(h + (size_t)row * ldh + c, xv[i]);
      s2 += sq4(xv[i]);
    }
  }
  if (w_last != nullptr) {
    const float r2 = 1.f / sqrtf(row_sum(s2, 1) / (float)W + eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = c0 + (i * TH + threadIdx.x) * 4;
      if (c < cend) {
        const float4 l = *reinterpret_cast<const float4*>(w_last + c);
        put4(h + (size_t)row * ldh + c, make_float4(xv[i].x * r2 * l.x, xv[i].y * r2 * l.y, xv[i].z * r2 * l.z, xv[i].w * r2 * l.w));
      }
    }
  }
  if (ncta > 1) cluster.sync();                     // nobody leaves while a partner may still read its shared memory
}

// Two sublayers of the same x: f32 planes of either (a: the mixer, b: the feed-forward), rows of experts through row_of, and a bias
template <typename H> struct PairOutput {
  const float *a, *b;
  int na, nb;
  size_t stride_a, stride_b;
  int64_t lda, ldb;
  const H* rows;
  const int* row_of;
  int top;
  int64_t ldr;
  const float* bias;
};
FT_DEVICE void add_planes(float4& v, const float* p, int planes, size_t stride) {
  int k = 0;
  for (; k + 4 <= planes; k += 4) {
    float4 t[4];
#pragma unroll
    for (int j = 0; j < 4; j++) t[j] = __ldcg(reinterpret_cast<const float4*>(p + (k + j) * stride));
    v.x += (t[0].x + t[1].x) + (t[2].x + t[3].x);
    v.y += (t[0].y + t[1].y) + (t[2].y + t[3].y);
    v.z += (t[0].z + t[1].z) + (t[2].z + t[3].z);
    v.w += (t[0].w + t[1].w) + (t[2].w + t[3].w);
  }
  for (; k < planes; k++) {
    const float4 t = __ldcg(reinterpret_cast<const float4*>(p + k * stride));
    v.x += t.x; v.y += t.y; v.z += t.z; v.w += t.w;
  }
}
// EMBED: x starts as the embedding row of ids[row]. w2 null: one operand
template <int NV, bool EMBED, typename H>
__global__ void __launch_bounds__(UPD_THREADS) parallel_update_kernel(float* __restrict__ x, int64_t ldx, const int64_t* __restrict__ ids, const H* __restrict__ table,
                                                                      int64_t ld_table, int64_t vocab, PairOutput<H> Y, float mult, const float* __restrict__ w1,
                                                                      const float* __restrict__ w2, float eps, H* __restrict__ h1, H* __restrict__ h2, int64_t ldh, int ncta,
                                                                      int W, int cols, int store_x) {
  namespace cg = cooperative_groups;
  __shared__ float red[32];
  __shared__ float cta_ss;
  cg::cluster_group cluster = cg::this_cluster();
  const int row = blockIdx.x / ncta, c0 = blockIdx.x % ncta * cols, cend = min(W, c0 + cols);
  pdl_wait();
  pdl_launch_dependents();
  float* xr = x + (size_t)row * ldx;
  int64_t id = -1;
  if constexpr (EMBED) id = ids[row];
  float4 xv[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * UPD_THREADS + threadIdx.x) * 4;
    xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < cend) {
      if constexpr (EMBED) {
        if (id >= 0 && id < vocab) xv[i] = get4(table + (size_t)id * ld_table + c);
      } else {
        const float4 old = *reinterpret_cast<const float4*>(xr + c);
        float4 v = Y.bias ? *reinterpret_cast<const float4*>(Y.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (Y.na) add_planes(v, Y.a + (size_t)row * Y.lda + c, Y.na, Y.stride_a);
        if (Y.nb) add_planes(v, Y.b + (size_t)row * Y.ldb + c, Y.nb, Y.stride_b);
#pragma unroll 4
        for (int k = 0; k < Y.top; k++) {
          const float4 t = get4(Y.rows + (size_t)Y.row_of[(size_t)row * Y.top + k] * Y.ldr + c);
          v.x += t.x; v.y += t.y; v.z += t.z; v.w += t.w;
        }
        xv[i] = make_float4(old.x + mult * v.x, old.y + mult * v.y, old.z + mult * v.z, old.w + mult * v.w);
      }
      xv[i] = keep4(xv[i], c, W);
      if (store_x) *reinterpret_cast<float4*>(xr + c) = xv[i];
      ss += sq4(xv[i]);
    }
  }
  ss = block_sum(ss, red);
  if (ncta > 1) {
    if (threadIdx.x == 0) cta_ss = ss;
    cluster.sync();
    ss = 0.f;
    for (int r = 0; r < ncta; r++) ss += *cluster.map_shared_rank(&cta_ss, r);
  }
  const float rstd = 1.f / sqrtf(ss / (float)W + eps);
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * UPD_THREADS + threadIdx.x) * 4;
    if (c < cend) {
      const float4 n = make_float4(xv[i].x * rstd, xv[i].y * rstd, xv[i].z * rstd, xv[i].w * rstd), a = *reinterpret_cast<const float4*>(w1 + c);
      put4(h1 + (size_t)row * ldh + c, make_float4(n.x * a.x, n.y * a.y, n.z * a.z, n.w * a.w));
      if (w2 != nullptr) {
        const float4 b = *reinterpret_cast<const float4*>(w2 + c);
        put4(h2 + (size_t)row * ldh + c, make_float4(n.x * b.x, n.y * b.y, n.z * b.z, n.w * b.w));
      }
    }
  }
  if (ncta > 1) cluster.sync();                     // nobody leaves while a partner may still read its shared memory
}

// ------------------------------------------------------------------------------------------------------------
// averages over depth, token shift
// ------------------------------------------------------------------------------------------------------------
// results[j]: what layer j - 1 returned (0: the embedding output). The update stores results[count] and hands on x = sum over j <= count of avg[j] results[j]. What becomes of
// the norm of x: `rstd` set: only its factor is stored, per row (ft_token_shift does the rest); `shift` set (a decode step): h = n + (n of the token before - n) shift, with
// the state of this row's slot; else h = n.
template <typename H> struct DepthArgs {
  const float* y;                    // f32 planes of the sublayer, or
  int planes;
  size_t pstride;
  int64_t ldy;
  const H* rows;                     // rows of experts through row_of
  const int* row_of;
  int top;
  int64_t ldr;
  const float* w_out;
  float* x;
  float* results;
  size_t rstride;
  int64_t ldx;
  int count;
  const float* avg;
  const float* w_next;
  float eps;
  H* h;
  int64_t ldh;
  float* rstd;
  const float* shift;
  float* state;
  int64_t ld_state;
  const int *slots, *positions;
  int store;                         // 0: neither x nor the result is needed any more
};
FT_DEVICE void fma4(float4& a, float k, float4 v) { a.x += k * v.x; a.y += k * v.y; a.z += k * v.z; a.w += k * v.w; }
FT_DEVICE float4 mul4(float4 a, float k, float4 w) { return make_float4(a.x * k * w.x, a.y * k * w.y, a.z * k * w.z, a.w * k * w.w); }
// shifted operand from this token's and the previous token's normed values
FT_DEVICE float4 shift4(float4 n, float4 before, float4 s) {
  return make_float4(n.x + (before.x - n.x) * s.x, n.y + (before.y - n.y) * s.y, n.z + (before.z - n.z) * s.z, n.w + (before.w - n.w) * s.w);
}

// TH threads per CTA: at most two float4 columns a thread, of which it holds three sets
template <int NV, int TH, bool EMBED, typename H>
__global__ void __launch_bounds__(TH) depth_update_kernel(DepthArgs<H> A, const int64_t* __restrict__ ids, const H* __restrict__ table, int64_t ld_table, int64_t vocab,
                                                                   int ncta, int W, int cols) {
  namespace cg = cooperative_groups;
  __shared__ float red[32];
  __shared__ float cta_ss[2];
  cg::cluster_group cluster = cg::this_cluster();
  const int row = blockIdx.x / ncta, c0 = blockIdx.x % ncta * cols, cend = min(W, c0 + cols);
  pdl_wait();
  pdl_launch_dependents();
  auto row_sum = [&](float ss, int slot) -> float {
    ss = block_sum(ss, red);
    if (ncta == 1) return ss;
    if (threadIdx.x == 0) cta_ss[slot] = ss;
    cluster.sync();
    float t = 0.f;
    for (int r = 0; r < ncta; r++) t += *cluster.map_shared_rank(&cta_ss[slot], r);
    return t;
  };
  float* xr = A.x + (size_t)row * A.ldx;
  float* res = A.results + (size_t)row * A.ldx;
  float4 xv[NV];
  float s2 = 0.f;
  if constexpr (EMBED) {
    const int64_t id = ids[row];
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = c0 + (i * TH + threadIdx.x) * 4;
      xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < cend) {
        if (id >= 0 && id < vocab) xv[i] = keep4(get4(table + (size_t)id * ld_table + c), c, W);
        *reinterpret_cast<float4*>(xr + c) = xv[i];
        *reinterpret_cast<float4*>(res + c) = xv[i];
        s2 += sq4(xv[i]);
      }
    }
  } else {
    float4 v[NV], old[NV];
    float ss = 0.f;
    const float last = A.avg[A.count];
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = c0 + (i * TH + threadIdx.x) * 4;
      v[i] = xv[i] = old[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < cend) {
        old[i] = *reinterpret_cast<const float4*>(xr + c);
        if (A.planes) add_planes(v[i], A.y + (size_t)row * A.ldy + c, A.planes, A.pstride);
#pragma unroll 4
        for (int k = 0; k < A.top; k++) {
          const float4 t = get4(A.rows + (size_t)A.row_of[(size_t)row * A.top + k] * A.ldr + c);
          v[i].x += t.x; v[i].y += t.y; v[i].z += t.z; v[i].w += t.w;
        }
        v[i] = keep4(v[i], c, W);
        ss += sq4(v[i]);
#pragma unroll 4
        for (int j = 0; j < A.count; j++) fma4(xv[i], A.avg[j], *reinterpret_cast<const float4*>(res + j * A.rstride + c));
      }
    }
    const float rstd = 1.f / sqrtf(row_sum(ss, 0) / (float)W + A.eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = c0 + (i * TH + threadIdx.x) * 4;
      if (c < cend) {
        const float4 w = *reinterpret_cast<const float4*>(A.w_out + c), o = old[i];
        const float4 r = keep4(make_float4(o.x + v[i].x * rstd * w.x, o.y + v[i].y * rstd * w.y, o.z + v[i].z * rstd * w.z, o.w + v[i].w * rstd * w.w), c, W);
        fma4(xv[i], last, r);
        if (A.store) {
          *reinterpret_cast<float4*>(res + A.count * A.rstride + c) = r;
          *reinterpret_cast<float4*>(xr + c) = xv[i];
        }
        s2 += sq4(xv[i]);
      }
    }
  }
  const float r2 = 1.f / sqrtf(row_sum(s2, 1) / (float)W + A.eps);
  if (A.rstd != nullptr) {
    if (blockIdx.x % ncta == 0 && threadIdx.x == 0) A.rstd[row] = r2;
  } else {
    float* state = A.shift ? A.state + (size_t)A.slots[row] * A.ld_state : nullptr;
    const bool first = A.shift && A.positions[row] == 0;
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = c0 + (i * TH + threadIdx.x) * 4;
      if (c < cend) {
        float4 n = mul4(xv[i], r2, *reinterpret_cast<const float4*>(A.w_next + c));
        if (A.shift) {
          const float4 before = first ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(state + c);
          *reinterpret_cast<float4*>(state + c) = n;
          n = shift4(n, before, *reinterpret_cast<const float4*>(A.shift + c));
        }
        put4(A.h + (size_t)row * A.ldh + c, n);
      }
    }
  }
  if (ncta > 1) cluster.sync();                     // nobody leaves while a partner may still read its shared memory
}

// A thread takes four columns of SHIFT_ROWS neighbouring rows, and the row ahead of them where that belongs to the same sequence. The thread that meets a sequence's first
// row of this batch replaces its state, after it has read it: spans[sequence] = {first row, rows, state slot, whether the sequence starts here}.
constexpr int SHIFT_ROWS = 8;
template <typename H>
__global__ void __launch_bounds__(256) token_shift_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ rstd, const float* __restrict__ w,
                                                          const float* __restrict__ shift, const int4* __restrict__ spans, const int* __restrict__ seq_of,
                                                          float* __restrict__ state, int64_t ld_state, H* __restrict__ h, int64_t ldh, int rows, int W) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= W) return;
  const float4 wv = *reinterpret_cast<const float4*>(w + c), sv = *reinterpret_cast<const float4*>(shift + c);
  const int r0 = blockIdx.y * SHIFT_ROWS;
  float4 v[SHIFT_ROWS + 1];
#pragma unroll
  for (int i = 0; i <= SHIFT_ROWS; i++) {
    const int r = min(max(r0 + i - 1, 0), rows - 1);
    v[i] = mul4(*reinterpret_cast<const float4*>(x + (size_t)r * ldx + c), rstd[r], wv);
  }
#pragma unroll
  for (int i = 0; i < SHIFT_ROWS; i++) {
    const int r = r0 + i;
    if (r >= rows) break;
    float4 before = v[i];
    const int4 sp = spans[seq_of[r]];
    if (r == sp.x) {
      float* st = state + (size_t)sp.z * ld_state + c;
      before = sp.w ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
      const int e = sp.x + sp.y - 1;
      *reinterpret_cast<float4*>(st) = mul4(*reinterpret_cast<const float4*>(x + (size_t)e * ldx + c), rstd[e], wv);
    }
    put4(h + (size_t)r * ldh + c, shift4(v[i + 1], before, sv));
  }
}

// ------------------------------------------------------------------------------------------------------------
// polynomial of normed powers
// ------------------------------------------------------------------------------------------------------------
FT_DEVICE void add_powers(float (&s)[3], float z) {
  const float q = z * z, f = q * q;
  s[0] += q; s[1] += f; s[2] += f * q;
}
// sums of z^2, z^4 and z^6 over a CTA
FT_DEVICE void block_powers(float (&s)[3], float (*red)[32]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
#pragma unroll
  for (int k = 0; k < 3; k++) {
    s[k] = warp_sum(s[k]);
    if (lane == 0) red[k][warp] = s[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 3; k++) {
    s[k] = 0.f;
    for (int i = 0; i < warps; i++) s[k] += red[k][i];
  }
}
struct PolyNorm {
  float a, b, d, e;
  FT_DEVICE PolyNorm(const float (&s)[3], const float* coef, float eps, int W) {
    const float inv = 1.f / (float)W;
    a = coef[0] / sqrtf(s[0] * inv + eps);
    b = coef[1] / sqrtf(s[1] * inv + eps);
    d = coef[2] / sqrtf(s[2] * inv + eps);
    e = coef[3];
  }
  FT_DEVICE float operator()(float t) const { return ((d * t + b) * t + a) * t + e; }
};

// one row per cluster as in the updates above
template <int NV, typename I, typename O>
__global__ void __launch_bounds__(UPD_THREADS) poly_norm_kernel(const I* __restrict__ z, int planes, size_t pstride, int64_t ldz, const float* __restrict__ coef, float eps,
                                                                O* __restrict__ out, int64_t ldo, int ncta, int W, int cols) {
  namespace cg = cooperative_groups;
  __shared__ float red[3][32];
  __shared__ float cta_ss[3];
  cg::cluster_group cluster = cg::this_cluster();
  const int row = blockIdx.x / ncta, c0 = blockIdx.x % ncta * cols, cend = min(W, c0 + cols);
  pdl_wait();
  pdl_launch_dependents();
  float4 v[NV];
  float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * UPD_THREADS + threadIdx.x) * 4;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < cend) {
      if constexpr (sizeof(I) == 4) add_planes(v[i], z + (size_t)row * ldz + c, planes, pstride);
      else v[i] = get4(z + (size_t)row * ldz + c);
      v[i] = keep4(v[i], c, W);
      add_powers(s, v[i].x); add_powers(s, v[i].y); add_powers(s, v[i].z); add_powers(s, v[i].w);
    }
  }
  block_powers(s, red);
  if (ncta > 1) {
    if (threadIdx.x < 3) cta_ss[threadIdx.x] = threadIdx.x == 0 ? s[0] : threadIdx.x == 1 ? s[1] : s[2];
    cluster.sync();
#pragma unroll
    for (int k = 0; k < 3; k++) {
      s[k] = 0.f;
      for (int r = 0; r < ncta; r++) s[k] += *cluster.map_shared_rank(&cta_ss[k], r);
    }
  }
  const PolyNorm f(s, coef, eps, W);
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = c0 + (i * UPD_THREADS + threadIdx.x) * 4;
    if (c < cend) put4(out + (size_t)row * ldo + c, keep4(make_float4(f(v[i].x), f(v[i].y), f(v[i].z), f(v[i].w)), c, W));
  }
  if (ncta > 1) cluster.sync();                     // nobody leaves while a partner may still read its shared memory
}

// many bf16 rows: one CTA each, which keeps the row in registers as it was loaded (16 bytes at a time; pitches are multiples of eight)
template <int NV>
__global__ void __launch_bounds__(UPD_THREADS) poly_norm_rows_kernel(const __nv_bfloat16* __restrict__ z, int64_t ldz, const float* __restrict__ coef, float eps,
                                                                     __nv_bfloat16* __restrict__ out, int64_t ldo, int W) {
  __shared__ float red[3][32];
  const __nv_bfloat16* zr = z + (size_t)blockIdx.x * ldz;
  bf16x8 v[NV];
  float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = (i * UPD_THREADS + threadIdx.x) * 8;
    if (c < W) v[i] = *reinterpret_cast<const bf16x8*>(zr + c);
  }
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = (i * UPD_THREADS + threadIdx.x) * 8;
    if (c < W) {
      float x[8];
      bf16x8_to_float(v[i], x);
#pragma unroll
      for (int e = 0; e < 8; e++)
        if (c + e < W) add_powers(s, x[e]);
    }
  }
  block_powers(s, red);
  const PolyNorm f(s, coef, eps, W);
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = (i * UPD_THREADS + threadIdx.x) * 8;
    if (c < W) {
      float x[8];
      bf16x8_to_float(v[i], x);
#pragma unroll
      for (int e = 0; e < 8; e++) x[e] = c + e < W ? f(x[e]) : 0.f;
      *reinterpret_cast<bf16x8*>(out + (size_t)blockIdx.x * ldo + c) = float_to_bf16x8(x);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// gated activation
// ------------------------------------------------------------------------------------------------------------
enum { ACT_GELU_TANH = 0, ACT_SILU = 1 };
FT_DEVICE float gate_act(float z, int kind) {
  if (kind == ACT_SILU) return z / (1.f + __expf(-z));
  // 0.5 (1 + tanh(u)) = 1 / (1 + exp(-2u))
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return z / (1.f + __expf(-2.f * u));
}
FT_DEVICE float gate_act_exact(float z, int kind) {
  if (kind == ACT_SILU) return z / (1.f + expf(-z));
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
template <bool EXACT> FT_DEVICE float4 gated4(float4 g, float4 u, int kind) {
  if constexpr (EXACT) return make_float4(gate_act_exact(g.x, kind) * u.x, gate_act_exact(g.y, kind) * u.y, gate_act_exact(g.z, kind) * u.z, gate_act_exact(g.w, kind) * u.w);
  else return make_float4(gate_act(g.x, kind) * u.x, gate_act(g.y, kind) * u.y, gate_act(g.z, kind) * u.z, gate_act(g.w, kind) * u.w);
}
FT_DEVICE float4 unpack4(uint2 r) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

FT_DEVICE float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }

// columns come in blocks of eight gates and the eight ups of the same neurons; a thread takes one block (bf16: two 16-byte loads, one 16-byte store). bias: f32 in the
// order of the columns, or null
template <typename T>
__global__ void __launch_bounds__(256) gated_act_kernel(const T* __restrict__ gu, int64_t ld, const float* __restrict__ bias, int rows, int blocks, int kind,
                                                        T* __restrict__ out, int64_t ldo) {
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= blocks) return;
  float4 bv[4];
#pragma unroll
  for (int i = 0; i < 4; i++) bv[i] = bias ? *reinterpret_cast<const float4*>(bias + b * 16 + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  constexpr int RU = sizeof(T) == 2 ? 4 : 1;
  for (int r0 = blockIdx.y * RU; r0 < rows; r0 += gridDim.y * RU) {
    if constexpr (sizeof(T) == 2) {
      uint4 g[RU], u[RU];
#pragma unroll
      for (int i = 0; i < RU; i++) {
        const uint4* s = reinterpret_cast<const uint4*>(gu + (size_t)min(r0 + i, rows - 1) * ld + b * 16);
        g[i] = s[0];
        u[i] = s[1];
      }
#pragma unroll
      for (int i = 0; i < RU; i++) {
        const float4 a = gated4<false>(add4(unpack4(make_uint2(g[i].x, g[i].y)), bv[0]), add4(unpack4(make_uint2(u[i].x, u[i].y)), bv[2]), kind);
        const float4 c = gated4<false>(add4(unpack4(make_uint2(g[i].z, g[i].w)), bv[1]), add4(unpack4(make_uint2(u[i].z, u[i].w)), bv[3]), kind);
        const float e[8] = {a.x, a.y, a.z, a.w, c.x, c.y, c.z, c.w};
        if (r0 + i < rows) *reinterpret_cast<bf16x8*>(out + (size_t)(r0 + i) * ldo + b * 8) = float_to_bf16x8(e);
      }
    } else {
      const float* s = gu + (size_t)r0 * ld + b * 16;
#pragma unroll
      for (int i = 0; i < 8; i += 4)
        *reinterpret_cast<float4*>(out + (size_t)r0 * ldo + b * 8 + i) =
            gated4<true>(add4(*reinterpret_cast<const float4*>(s + i), bv[i / 4]), add4(*reinterpret_cast<const float4*>(s + 8 + i), bv[2 + i / 4]), kind);
    }
  }
}

__global__ void __launch_bounds__(128) gated_act_planes_kernel(const float* __restrict__ p, int splits, int64_t ldp, size_t pstride, const float* __restrict__ bias, int rows,
                                                               int quads, int kind, __nv_bfloat16* __restrict__ out, int64_t ldo) {
  pdl_wait();
  pdl_launch_dependents();
  const int i = blockIdx.x * 128 + threadIdx.x;
  if (i >= rows * quads) return;
  const int r = i / quads, q = i % quads;                       // four neurons
  const float* s = p + (size_t)r * ldp + (q >> 1) * 16 + (q & 1) * 4;
  float4 g = make_float4(0.f, 0.f, 0.f, 0.f), u = g;
  if (bias) {
    g = *reinterpret_cast<const float4*>(bias + (q >> 1) * 16 + (q & 1) * 4);
    u = *reinterpret_cast<const float4*>(bias + (q >> 1) * 16 + (q & 1) * 4 + 8);
  }
#pragma unroll 4
  for (int k = 0; k < splits; k++) {
    const float4 a = __ldcg(reinterpret_cast<const float4*>(s + k * pstride)), b = __ldcg(reinterpret_cast<const float4*>(s + k * pstride + 8));
    g.x += a.x; g.y += a.y; g.z += a.z; g.w += a.w;
    u.x += b.x; u.y += b.y; u.z += b.z; u.w += b.w;
  }
  put4(out + (size_t)r * ldo + q * 4, gated4<false>(g, u, kind));
}

// how a row of W columns is spread: CTAs of its cluster, columns of a CTA, float4 columns of a thread
struct RowSpread { int ncta, cols, nv; };
RowSpread row_spread(int rows, int W) {
  // rows alone fill the GPU, or a row is spread over up to eight SMs (at least 256 columns each)
  int ncta = 1;
  while (ncta < 8 && (rows * ncta < 148 && W > 256 * ncta * 2)) ncta *= 2;
  while (ncta < 8 && (W + ncta - 1) / ncta > UPD_THREADS * 4 * 8) ncta *= 2;
  const int cols = ((W + ncta - 1) / ncta + 3) & ~3;
  return RowSpread{ncta, cols, (cols + UPD_THREADS * 4 - 1) / (UPD_THREADS * 4)};
}

// one row per cluster of sp.ncta CTAs
template <typename... K, typename... A>
int launch_rows(const RowSpread& sp, int rows, int threads, cudaStream_t st, void (*kernel)(K...), A&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(sp.ncta * rows);
  cfg.blockDim = dim3(threads);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = sp.ncta;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ft_pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, kernel, std::forward<A>(args)...);
}

template <bool EMBED, typename H>
int dispatch_depth(const DepthArgs<H>& A, const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, int rows, int W, cudaStream_t st) {
  const RowSpread sp = row_spread(rows, W);
  if (sp.nv > 8) return FT_ERR_TOO_LARGE;
#define FT_DU(N, TH) return launch_rows(sp, rows, TH, st, depth_update_kernel<N, TH, EMBED, H>, A, ids, (const H*)table, ld_table, vocab, sp.ncta, W, sp.cols)
  if (sp.nv <= 1) FT_DU(1, 256);
  if (sp.nv <= 2) FT_DU(2, 256);
  if (sp.nv <= 4) FT_DU(2, 512);
  FT_DU(2, 1024);
#undef FT_DU
}

template <typename I, typename O>
int dispatch_poly(const void* z, int planes, int64_t pstride, int64_t ldz, const float* coef, float eps, void* out, int64_t ldo, int rows, int W, cudaStream_t st) {
  const RowSpread sp = row_spread(rows, W);
  if (sp.nv > 8) return FT_ERR_TOO_LARGE;
#define FT_PN(N) return launch_rows(sp, rows, UPD_THREADS, st, poly_norm_kernel<N, I, O>, (const I*)z, planes, (size_t)pstride, ldz, coef, eps, (O*)out, ldo, sp.ncta, W, sp.cols)
  if (sp.nv <= 1) FT_PN(1);
  if (sp.nv <= 2) FT_PN(2);
  if (sp.nv <= 4) FT_PN(4);
  FT_PN(8);
#undef FT_PN
}

template <bool EMBED, typename H>
int dispatch_parallel(float* x, int64_t ldx, const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, const PairOutput<H>& Y, float mult, const float* w1,
                      const float* w2, float eps, void* h1, void* h2, int64_t ldh, int rows, int W, int store, cudaStream_t st) {
  const RowSpread sp = row_spread(rows, W);
  if (sp.nv > 8) return FT_ERR_TOO_LARGE;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(sp.ncta * rows);
  cfg.blockDim = dim3(UPD_THREADS);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = sp.ncta;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ft_pdl_enabled() ? 2 : 1;
#define FT_PU(N) return (int)cudaLaunchKernelEx(&cfg, parallel_update_kernel<N, EMBED, H>, x, ldx, ids, (const H*)table, ld_table, vocab, Y, mult, w1, w2, eps, (H*)h1, (H*)h2, ldh,                                                 sp.ncta, W, sp.cols, store)
  if (sp.nv <= 1) FT_PU(1);
  if (sp.nv <= 2) FT_PU(2);
  if (sp.nv <= 4) FT_PU(4);
  FT_PU(8);
#undef FT_PU
}

template <typename H>
int dispatch_update(float* x, int64_t ldx, const float* y, int planes, int64_t pstride, int64_t ldy, const float* w, const float* w_last, float eps, void* h, int64_t ldh,
                    int rows, int W, int store, cudaStream_t st) {
  const RowSpread sp = row_spread(rows, W);
  if (sp.nv > 8) return FT_ERR_TOO_LARGE;
#define FT_RU(N, TH) return launch_rows(sp, rows, TH, st, residual_update_kernel<N, TH, H>, x, ldx, y, planes, (size_t)pstride, ldy, w, w_last, eps, (H*)h, ldh, sp.ncta, W, sp.cols, store)
  if (sp.nv <= 1) FT_RU(1, 256);
  if (sp.nv <= 2) FT_RU(2, 256);
  if (sp.nv <= 4) FT_RU(4, 256);
  FT_RU(8, 256);
#undef FT_RU
}

}  // namespace

// x [rows][ldx] f32 = scale * table[ids[r]] (zeros for ids outside [0, vocab)), h [rows][ldh] the same in the table's type (bf16, or f32 with is_f32).
// Leading dimensions are multiples of four.
FT_EXPORT int ft_residual_embed(const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, float scale, float* x, int64_t ldx, void* h, int64_t ldh,
                                int is_f32, int rows, int W, cudaStream_t st) {
  if (rows < 1 || W < 1 || (ld_table & 3) || (ldx & 3) || (ldh & 3)) return FT_ERR_ARG;
  const dim3 grid((W + 1023) / 1024, rows < 2048 ? rows : 2048);
  if (is_f32) return (int)ft_launch_pdl(residual_embed_kernel<float>, grid, dim3(256), 0, st, ids, (const float*)table, ld_table, vocab, scale, x, ldx, (float*)h, ldh, rows, W);
  return (int)ft_launch_pdl(residual_embed_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, ids, (const __nv_bfloat16*)table, ld_table, vocab, scale, x, ldx, (__nv_bfloat16*)h,
                            ldh, rows, W);
}

// y = sum of `planes` f32 planes [row][ldy]; x += y / sqrt(mean(y^2) + eps) * w; h = x, or with w_last x / sqrt(mean(x^2) + eps) * w_last, bf16 (f32 with
// is_f32). w, w_last: f32, readable up to W rounded up to a multiple of four. x is left alone when store_x is 0. Widths up to 65536.
FT_EXPORT int ft_residual_update(float* x, int64_t ldx, const float* y, int planes, int64_t plane_stride, int64_t ldy, const float* w, const float* w_last, float eps,
                                 void* h, int64_t ldh, int is_f32, int rows, int W, int store_x, cudaStream_t st) {
  if (rows < 1 || W < 1 || planes < 1 || (ldx & 3) || (ldy & 3) || (ldh & 3) || (plane_stride & 3)) return FT_ERR_ARG;
  if (is_f32) return dispatch_update<float>(x, ldx, y, planes, plane_stride, ldy, w, w_last, eps, h, ldh, rows, W, store_x, st);
  return dispatch_update<__nv_bfloat16>(x, ldx, y, planes, plane_stride, ldy, w, w_last, eps, h, ldh, rows, W, store_x, st);
}

// Start of a pass whose layers norm ahead of two sublayers: x [rows][ldx] f32 = table[ids[r]] (zeros for ids outside [0, vocab)), h1 = x / sqrt(mean(x^2) + eps) * w1 and, unless
// w2 is null, h2 the same with w2; both [rows][ldh] in the table's type. Widths up to 65536.
FT_EXPORT int ft_parallel_embed(const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, const float* w1, const float* w2, float eps, float* x, int64_t ldx,
                                void* h1, void* h2, int64_t ldh, int is_f32, int rows, int W, cudaStream_t st) {
  if (rows < 1 || W < 1 || !w1 || (w2 && !h2) || (ld_table & 3) || (ldx & 3) || (ldh & 3)) return FT_ERR_ARG;
  if (is_f32) return dispatch_parallel<true, float>(x, ldx, ids, table, ld_table, vocab, PairOutput<float>{}, 0.f, w1, w2, eps, h1, h2, ldh, rows, W, 1, st);
  return dispatch_parallel<true, __nv_bfloat16>(x, ldx, ids, table, ld_table, vocab, PairOutput<__nv_bfloat16>{}, 0.f, w1, w2, eps, h1, h2, ldh, rows, W, 1, st);
}

// x += mult * (planes of a [na][row][lda] + planes of b [nb][row][ldb] + expert rows row_of[row][0..top) (type of h) + bias); h1, h2 as in ft_parallel_embed. a, b: f32, either
// may be absent (0 planes); bias f32 or null; all vectors readable up to W rounded up to a multiple of four. x is left alone when store_x is 0.
FT_EXPORT int ft_parallel_update(float* x, int64_t ldx, float mult, const float* a, int na, int64_t stride_a, int64_t lda, const float* b, int nb, int64_t stride_b, int64_t ldb,
                                 const void* expert_rows, const int* row_of, int top, int64_t ldr, const float* bias, const float* w1, const float* w2, float eps, void* h1,
                                 void* h2, int64_t ldh, int is_f32, int rows, int W, int store_x, cudaStream_t st) {
  if (rows < 1 || W < 1 || na < 0 || nb < 0 || top < 0 || !w1 || (w2 && !h2) || (ldx & 3) || (lda & 3) || (ldb & 3) || (ldr & 3) || (ldh & 3) || (stride_a & 3) || (stride_b & 3) ||
      (top && (!expert_rows || !row_of)))
    return FT_ERR_ARG;
  if (is_f32) {
    const PairOutput<float> Y{a, b, na, nb, (size_t)stride_a, (size_t)stride_b, lda, ldb, (const float*)expert_rows, row_of, top, ldr, bias};
    return dispatch_parallel<false, float>(x, ldx, nullptr, nullptr, 0, 0, Y, mult, w1, w2, eps, h1, h2, ldh, rows, W, store_x, st);
  }
  const PairOutput<__nv_bfloat16> Y{a, b, na, nb, (size_t)stride_a, (size_t)stride_b, lda, ldb, (const __nv_bfloat16*)expert_rows, row_of, top, ldr, bias};
  return dispatch_parallel<false, __nv_bfloat16>(x, ldx, nullptr, nullptr, 0, 0, Y, mult, w1, w2, eps, h1, h2, ldh, rows, W, store_x, st);
}

// Start of a pass with averages over depth: x and results, both [rows][ldx] f32, = table[ids[r]] (zeros for ids outside [0, vocab)). What becomes of the norm n = x / sqrt(mean(x^2)
// + eps) * w_next: rstd (f32 [rows]) not null: only 1 / sqrt(mean(x^2) + eps) is stored; else h [rows][ldh] in the table's type, shifted with the state of row slots[r] (f32 rows of
// ld_state; not read at position 0, replaced by n) unless shift is null. Widths up to 65536.
FT_EXPORT int ft_depth_embed(const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, float* x, float* results, int64_t ldx, const float* w_next, float eps,
                             void* h, int64_t ldh, float* rstd, const float* shift, float* state, int64_t ld_state, const int* slots, const int* positions, int is_f32, int rows,
                             int W, cudaStream_t st) {
  if (rows < 1 || W < 1 || (!rstd && (!w_next || !h)) || (shift && (!state || !slots || !positions)) || (ld_table & 3) || (ldx & 3) || (ldh & 3) || (ld_state & 3)) return FT_ERR_ARG;
#define FT_DE(T)                                                                                                                                                       \
  {                                                                                                                                                                    \
    DepthArgs<T> A{};                                                                                                                                                  \
    A.x = x; A.results = results; A.ldx = ldx; A.w_next = w_next; A.eps = eps; A.h = (T*)h; A.ldh = ldh; A.rstd = rstd; A.shift = shift; A.state = state;               \
    A.ld_state = ld_state; A.slots = slots; A.positions = positions; A.store = 1;                                                                                      \
    return dispatch_depth<true, T>(A, ids, table, ld_table, vocab, rows, W, st);                                                                                       \
  }
  if (is_f32) FT_DE(float);
  FT_DE(__nv_bfloat16);
#undef FT_DE
}

// X = x + y / sqrt(mean(y^2) + eps) * w_out with y = sum of f32 planes [planes][row][ldy] + expert rows row_of[row][0..top) (type of h); results[count] = X; x = sum over j <= count
// of avg[j] results[j] (f32, results_stride elements apart, rows of ldx); then as in ft_depth_embed. x and results[count] are left alone when store is 0. All vectors readable up to W
// rounded up to a multiple of four.
FT_EXPORT int ft_depth_update(float* x, float* results, int64_t results_stride, int64_t ldx, int count, const float* avg, const float* y, int planes, int64_t plane_stride,
                              int64_t ldy, const void* expert_rows, const int* row_of, int top, int64_t ldr, const float* w_out, const float* w_next, float eps, void* h,
                              int64_t ldh, float* rstd, const float* shift, float* state, int64_t ld_state, const int* slots, const int* positions, int is_f32, int rows, int W,
                              int store, cudaStream_t st) {
  if (rows < 1 || W < 1 || count < 1 || planes < 0 || top < 0 || !w_out || !avg || (!rstd && (!w_next || !h)) || (shift && (!state || !slots || !positions)) || (ldx & 3) ||
      (ldy & 3) || (ldr & 3) || (ldh & 3) || (ld_state & 3) || (results_stride & 3) || (plane_stride & 3) || (top && (!expert_rows || !row_of)))
    return FT_ERR_ARG;
#define FT_DU(T)                                                                                                                                                        \
  {                                                                                                                                                                     \
    const DepthArgs<T> A{y, planes, (size_t)plane_stride, ldy, (const T*)expert_rows, row_of, top, ldr, w_out, x, results, (size_t)results_stride, ldx, count, avg, w_next, \
                         eps, (T*)h, ldh, rstd, shift, state, ld_state, slots, positions, store};                                                                       \
    return dispatch_depth<false, T>(A, nullptr, nullptr, 0, 0, rows, W, st);                                                                                            \
  }
  if (is_f32) FT_DU(float);
  FT_DU(__nv_bfloat16);
#undef FT_DU
}

// h[r] = n[r] + (n before r - n[r]) * shift with n[r] = x[r] * rstd[r] * w, for a batch of sequences whose rows lie one after another: spans int4 per sequence {first row, rows, slot,
// whether it starts here}, seq_of[r] the sequence of a row. Before a sequence's first row comes its state (f32 row `slot` of ld_state) or, where it starts, zeros; the state
// becomes n of its last row. h in bf16, or f32 with is_f32.
FT_EXPORT int ft_token_shift(const float* x, int64_t ldx, const float* rstd, const float* w, const float* shift, const int* spans, const int* seq_of, float* state, int64_t ld_state,
                             void* h, int64_t ldh, int is_f32, int rows, int W, cudaStream_t st) {
  if (rows < 1 || W < 1 || !rstd || !w || !shift || !spans || !seq_of || !state || (ldx & 3) || (ldh & 3) || (ld_state & 3) || (reinterpret_cast<uintptr_t>(spans) & 15)) return FT_ERR_ARG;
  const int quads = (W + 3) / 4, threads = quads >= 256 ? 256 : (quads + 31) & ~31, groups = (rows + SHIFT_ROWS - 1) / SHIFT_ROWS;
  if (groups > 65535) return FT_ERR_TOO_LARGE;
  const dim3 grid((quads + threads - 1) / threads, groups);
  if (is_f32) token_shift_kernel<float><<<grid, threads, 0, st>>>(x, ldx, rstd, w, shift, (const int4*)spans, seq_of, state, ld_state, (float*)h, ldh, rows, W);
  else token_shift_kernel<__nv_bfloat16><<<grid, threads, 0, st>>>(x, ldx, rstd, w, shift, (const int4*)spans, seq_of, state, ld_state, (__nv_bfloat16*)h, ldh, rows, W);
  return (int)cudaGetLastError();
}

// out[r] = a N(z) + b N(z^2) + c N(z^3) + e for rows z of n columns, powers element by element, N(v) = v / sqrt(mean(v^2) + eps); coef: f32 {a, b, c, e}. z and out bf16, or f32 with is_f32;
// rows end with a whole group of four columns (of eight where a pitch is a multiple of eight). Up to 65536 columns.
FT_EXPORT int ft_poly_norm(const void* z, int64_t ldz, const float* coef, float eps, int rows, int n, void* out, int64_t ldo, int is_f32, cudaStream_t st) {
  if (rows < 1 || n < 1 || !coef || (ldz & 3) || (ldo & 3)) return FT_ERR_ARG;
  if (is_f32) return dispatch_poly<float, float>(z, 1, 0, ldz, coef, eps, out, ldo, rows, n, st);
  const int nv = (n + UPD_THREADS * 8 - 1) / (UPD_THREADS * 8);
  if (rows >= 148 && nv <= 8 && !(ldz & 7) && !(ldo & 7) && !((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15)) {
#define FT_PR(N) poly_norm_rows_kernel<N><<<rows, UPD_THREADS, 0, st>>>((const __nv_bfloat16*)z, ldz, coef, eps, (__nv_bfloat16*)out, ldo, n)
    if (nv <= 1) FT_PR(1);
    else if (nv <= 2) FT_PR(2);
    else if (nv <= 4) FT_PR(4);
    else if (nv <= 6) FT_PR(6);
    else FT_PR(8);
#undef FT_PR
    return (int)cudaGetLastError();
  }
  return dispatch_poly<__nv_bfloat16, __nv_bfloat16>(z, 1, 0, ldz, coef, eps, out, ldo, rows, n, st);
}

// The same from split-K planes [split][row][ldp] (f32) to bf16 rows.
FT_EXPORT int ft_poly_norm_planes(const float* planes, int splits, int64_t ldp, int64_t plane_stride, const float* coef, float eps, int rows, int n, void* out, int64_t ldo,
                                  cudaStream_t st) {
  if (rows < 1 || splits < 1 || n < 1 || !coef || (ldp & 3) || (plane_stride & 3) || (ldo & 3)) return FT_ERR_ARG;
  return dispatch_poly<float, __nv_bfloat16>(planes, splits, plane_stride, ldp, coef, eps, out, ldo, rows, n, st);
}

// out[r][f] = act(gate + bias) * (up + bias) for f < fp (a multiple of 8) from columns in blocks of eight gates and eight ups; kind 0: gelu (tanh form), 1: silu; bias: f32 in
// the order of the columns, or null.
FT_EXPORT int ft_gated_act(const void* gu, int64_t ld, const float* bias, int rows, int fp, int kind, void* out, int64_t ldo, int is_f32, cudaStream_t st) {
  if (rows < 1 || fp < 8 || (fp & 7) || (ld & 7) || (ldo & 7) || kind < 0 || kind > 1) return FT_ERR_ARG;
  const int blocks = fp / 8, threads = blocks >= 256 ? 256 : (blocks + 31) & ~31, ru = is_f32 ? 1 : 4;
  const int gx = (blocks + threads - 1) / threads, want = (rows + ru - 1) / ru, cap = 148 * 16 / gx + 1;
  const dim3 grid(gx, want < cap ? want : cap);
  if (is_f32) gated_act_kernel<float><<<grid, threads, 0, st>>>((const float*)gu, ld, bias, rows, blocks, kind, (float*)out, ldo);
  else gated_act_kernel<__nv_bfloat16><<<grid, threads, 0, st>>>((const __nv_bfloat16*)gu, ld, bias, rows, blocks, kind, (__nv_bfloat16*)out, ldo);
  return (int)cudaGetLastError();
}

// The same from split-K planes [split][row][ldp] (f32) to bf16 rows.
FT_EXPORT int ft_gated_act_planes(const float* planes, int splits, int64_t ldp, int64_t plane_stride, const float* bias, int rows, int fp, int kind, void* out, int64_t ldo, cudaStream_t st) {
  if (rows < 1 || splits < 1 || fp < 8 || (fp & 7) || (ldp & 3) || (plane_stride & 3) || (ldo & 3) || kind < 0 || kind > 1) return FT_ERR_ARG;
  const int quads = fp / 4;
  return (int)ft_launch_pdl(gated_act_planes_kernel, dim3((rows * quads + 127) / 128), dim3(128), 0, st, planes, splits, ldp, (size_t)plane_stride, bias, rows, quads,
                            kind, (__nv_bfloat16*)out, ldo);
}
