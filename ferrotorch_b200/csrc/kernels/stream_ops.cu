// Residual streams: several f32 copies of the residual ("hyper-connections"), mixed after every sublayer, together with the element-wise norm
// (Dynamic Tanh) that feeds the next sublayer. Both act on every column by itself, so one kernel does the whole step between two sublayers:
//
//   y      = sum of the sublayer's partial results (split-K planes, one plane per expert slot, or expert rows picked up through an index)
//   x_t   <- sum_s mix[s][t] x_s + out[t] y                      (all streams at once from the old ones, f32)
//   u      = sum_s in[s] x_s    (or the plain sum of the streams ahead of the model's last norm)
//   h      = tanh(alpha u) w + b                                 (bf16 or f32, the next projection's operand)
//
// so the streams are read once and written once per sublayer and nothing between two projections touches memory twice. A thread keeps its four
// columns (norm weights in registers) and walks the rows. Compiled without fast-math: tanhf is the accurate one.
#include "common.cuh"
#include "host_common.h"

namespace {

constexpr int MAX_STREAMS = 16;

struct TanhNorm {
  const float* alpha;            // one value
  const float* w;
  const float* b;
};

// Partial results of the sublayer: `planes` f32 planes [plane][row][ld], then (optional) `top` picked rows per token of a 16-bit or f32 matrix.
struct SubOut {
  const float* p;
  int planes;
  int64_t plane_stride, ld;
  const void* rows;              // expert output rows, dtype of h
  const int* row_of;             // [tokens][top]
  int top;
  int64_t ld_rows;
};

template <typename H> FT_DEVICE void store4(H* dst, float4 v);
template <> FT_DEVICE void store4<float>(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
template <> FT_DEVICE void store4<__nv_bfloat16>(__nv_bfloat16* dst, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&a);
  pk.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(dst) = pk;
}
template <typename H> FT_DEVICE float4 load4(const H* src);
template <> FT_DEVICE float4 load4<float>(const float* src) { return *reinterpret_cast<const float4*>(src); }
template <> FT_DEVICE float4 load4<__nv_bfloat16>(const __nv_bfloat16* src) {
  const uint2 r = *reinterpret_cast<const uint2*>(src);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
FT_DEVICE float4 fma4(float s, float4 a, float4 c) { return make_float4(fmaf(s, a.x, c.x), fmaf(s, a.y, c.y), fmaf(s, a.z, c.z), fmaf(s, a.w, c.w)); }
FT_DEVICE float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
FT_DEVICE float4 tanh_norm4(float alpha, float4 u, float4 w, float4 b) {
  return make_float4(fmaf(tanhf(alpha * u.x), w.x, b.x), fmaf(tanhf(alpha * u.y), w.y, b.y), fmaf(tanhf(alpha * u.z), w.z, b.z), fmaf(tanhf(alpha * u.w), w.w, b.w));
}

// SM: compile-time bound on the number of streams (S <= SM)
template <int SM, typename H>
__global__ void __launch_bounds__(128) hyper_update_kernel(float* __restrict__ x, int S, int64_t ldx, const float* __restrict__ mix, const float* __restrict__ out,
                                                           SubOut y, const float* __restrict__ in_next, TanhNorm norm, H* __restrict__ h, int64_t ldh, int rows,
                                                           int W, int store_x) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= W) return;
  float cm[SM][SM], co[SM], ci[SM];
#pragma unroll
  for (int s = 0; s < SM; s++) {
    co[s] = s < S ? out[s] : 0.f;
    ci[s] = s < S ? (in_next ? in_next[s] : 1.f) : 0.f;
#pragma unroll
    for (int t = 0; t < SM; t++) cm[s][t] = (s < S && t < S) ? mix[s * S + t] : 0.f;
  }
  const float alpha = *norm.alpha;
  const float4 w = *reinterpret_cast<const float4*>(norm.w + c), b = *reinterpret_cast<const float4*>(norm.b + c);
  for (int r = blockIdx.y; r < rows; r += gridDim.y) {
    float* xr = x + (size_t)r * S * ldx + c;
    float4 old[SM];
#pragma unroll
    for (int s = 0; s < SM; s++) old[s] = s < S ? *reinterpret_cast<const float4*>(xr + s * ldx) : make_float4(0.f, 0.f, 0.f, 0.f);
    float4 yv = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int p = 0; p < y.planes; p++) yv = add4(yv, *reinterpret_cast<const float4*>(y.p + p * y.plane_stride + r * y.ld + c));
    for (int j = 0; j < y.top; j++) yv = add4(yv, load4(reinterpret_cast<const H*>(y.rows) + (size_t)y.row_of[(size_t)r * y.top + j] * y.ld_rows + c));
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int t = 0; t < SM; t++) {
      if (t < S) {
        float4 v = make_float4(co[t] * yv.x, co[t] * yv.y, co[t] * yv.z, co[t] * yv.w);
#pragma unroll
        for (int s = 0; s < SM; s++) v = fma4(cm[s][t], old[s], v);
        if (store_x) *reinterpret_cast<float4*>(xr + t * ldx) = v;
        u = fma4(ci[t], v, u);
      }
    }
    store4(h + (size_t)r * ldh + c, tanh_norm4(alpha, u, w, b));
  }
}

// the same for any number of streams up to MAX_STREAMS, coefficients read from memory
template <typename H>
__global__ void __launch_bounds__(128) hyper_update_many_kernel(float* __restrict__ x, int S, int64_t ldx, const float* __restrict__ mix, const float* __restrict__ out,
                                                                SubOut y, const float* __restrict__ in_next, TanhNorm norm, H* __restrict__ h, int64_t ldh, int rows,
                                                                int W, int store_x) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= W) return;
  const float alpha = *norm.alpha;
  const float4 w = *reinterpret_cast<const float4*>(norm.w + c), b = *reinterpret_cast<const float4*>(norm.b + c);
  for (int r = blockIdx.y; r < rows; r += gridDim.y) {
    float* xr = x + (size_t)r * S * ldx + c;
    float4 old[MAX_STREAMS];
    for (int s = 0; s < S; s++) old[s] = *reinterpret_cast<const float4*>(xr + s * ldx);
    float4 yv = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int p = 0; p < y.planes; p++) yv = add4(yv, *reinterpret_cast<const float4*>(y.p + p * y.plane_stride + r * y.ld + c));
    for (int j = 0; j < y.top; j++) yv = add4(yv, load4(reinterpret_cast<const H*>(y.rows) + (size_t)y.row_of[(size_t)r * y.top + j] * y.ld_rows + c));
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int t = 0; t < S; t++) {
      float4 v = make_float4(out[t] * yv.x, out[t] * yv.y, out[t] * yv.z, out[t] * yv.w);
      for (int s = 0; s < S; s++) v = fma4(mix[s * S + t], old[s], v);
      if (store_x) *reinterpret_cast<float4*>(xr + t * ldx) = v;
      u = fma4(in_next ? in_next[t] : 1.f, v, u);
    }
    store4(h + (size_t)r * ldh + c, tanh_norm4(alpha, u, w, b));
  }
}

// x_s = norm(table[id]) for every stream s; h = next norm of sum_s in[s] x_s
template <typename H>
__global__ void __launch_bounds__(128) hyper_embed_kernel(const int64_t* __restrict__ ids, const H* __restrict__ table, int64_t ld_table, int64_t vocab,
                                                          TanhNorm first, float* __restrict__ x, int S, int64_t ldx, const float* __restrict__ in_next, TanhNorm norm,
                                                          H* __restrict__ h, int64_t ldh, int rows, int W) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= W) return;
  float ci = 0.f;
  for (int s = 0; s < S; s++) ci += in_next ? in_next[s] : 1.f;
  const float a0 = *first.alpha, a1 = *norm.alpha;
  const float4 w0 = *reinterpret_cast<const float4*>(first.w + c), b0 = *reinterpret_cast<const float4*>(first.b + c);
  const float4 w1 = *reinterpret_cast<const float4*>(norm.w + c), b1 = *reinterpret_cast<const float4*>(norm.b + c);
  for (int r = blockIdx.y; r < rows; r += gridDim.y) {
    const int64_t id = ids[r];
    const float4 e = (id >= 0 && id < vocab) ? load4(table + (size_t)id * ld_table + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 v = tanh_norm4(a0, e, w0, b0);
    for (int s = 0; s < S; s++) *reinterpret_cast<float4*>(x + ((size_t)r * S + s) * ldx + c) = v;
    store4(h + (size_t)r * ldh + c, tanh_norm4(a1, make_float4(ci * v.x, ci * v.y, ci * v.z, ci * v.w), w1, b1));
  }
}

template <typename H>
__global__ void __launch_bounds__(128) dynamic_tanh_kernel(const H* __restrict__ x, int64_t ldx, TanhNorm norm, H* __restrict__ y, int64_t ldy, int rows, int W) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= W) return;
  const float alpha = *norm.alpha;
  const float4 w = *reinterpret_cast<const float4*>(norm.w + c), b = *reinterpret_cast<const float4*>(norm.b + c);
  for (int r = blockIdx.y; r < rows; r += gridDim.y) store4(y + (size_t)r * ldy + c, tanh_norm4(alpha, load4(x + (size_t)r * ldx + c), w, b));
}

dim3 row_grid(int rows, int W, int per_sm) {
  const int gx = (W + 511) / 512;
  int gy = (148 * per_sm + gx - 1) / gx;
  if (gy > rows) gy = rows;
  if (gy > 65535) gy = 65535;
  return dim3(gx, gy < 1 ? 1 : gy);
}
bool quad(int64_t v) { return (v & 3) == 0; }

}  // namespace

// One step between two sublayers. x: f32 [rows][streams][ldx], updated in place (store_x = 0: only h is wanted, as ahead of the last norm).
// mix: f32 [streams][streams] indexed [from][to]; out, in_next: f32 [streams] (in_next null: plain sum). The sublayer's result is the sum of
// `planes` f32 planes (plane_stride, ld_plane in elements) and, when top > 0, of the rows row_of[token][0..top) of `expert_rows` (dtype of h).
// norm: alpha f32[1], w and b f32 padded to a multiple of four. h: bf16 or (h_f32) f32 [rows][ldh]. All leading dimensions are multiples of four.
FT_EXPORT int ft_hyper_update(float* x, int streams, int64_t ldx, const float* mix, const float* out, const float* planes_ptr, int planes, int64_t plane_stride,
                              int64_t ld_plane, const void* expert_rows, const int* row_of, int top, int64_t ld_rows, const float* in_next, const float* alpha,
                              const float* w, const float* b, void* h, int64_t ldh, int h_f32, int rows, int W, int store_x, cudaStream_t st) {
  if (streams < 1 || streams > MAX_STREAMS || rows < 1 || W < 1 || planes < 0 || top < 0 || !quad(ldx) || !quad(ldh) || ldx < W || ldh < W) return FT_ERR_ARG;
  if (planes > 0 && (!planes_ptr || !quad(plane_stride) || !quad(ld_plane))) return FT_ERR_ARG;
  if (top > 0 && (!expert_rows || !row_of || !quad(ld_rows))) return FT_ERR_ARG;
  const SubOut y{planes_ptr, planes, plane_stride, ld_plane, expert_rows, row_of, top, ld_rows};
  const TanhNorm nn{alpha, w, b};
  const dim3 grid = row_grid(rows, W, 12);
#define FT_HYPER(K, T) return (int)ft_launch_pdl(K, grid, dim3(128), 0, st, x, streams, ldx, mix, out, y, in_next, nn, (T*)h, ldh, rows, W, store_x)
#define FT_HYPER_T(T)                                                     \
  switch (streams) {                                                      \
    case 1: FT_HYPER((hyper_update_kernel<1, T>), T);                     \
    case 2: FT_HYPER((hyper_update_kernel<2, T>), T);                     \
    case 3: FT_HYPER((hyper_update_kernel<3, T>), T);                     \
    case 4: FT_HYPER((hyper_update_kernel<4, T>), T);                     \
    default: FT_HYPER((hyper_update_many_kernel<T>), T);                  \
  }
  if (h_f32) { FT_HYPER_T(float) }
  FT_HYPER_T(__nv_bfloat16)
#undef FT_HYPER_T
#undef FT_HYPER
}

// Start of a forward pass: every stream of x becomes the normalised embedding row of the token (first norm), h the next sublayer's operand.
// table: dtype of h, [vocab][ld_table]; ids outside the table read as zero rows.
FT_EXPORT int ft_hyper_embed(const void* ids, const void* table, int64_t ld_table, int64_t vocab, const float* alpha0, const float* w0, const float* b0, float* x,
                             int streams, int64_t ldx, const float* in_next, const float* alpha, const float* w, const float* b, void* h, int64_t ldh, int h_f32,
                             int rows, int W, cudaStream_t st) {
  if (streams < 1 || streams > MAX_STREAMS || rows < 1 || W < 1 || !quad(ldx) || !quad(ldh) || !quad(ld_table) || ldx < W || ldh < W || ld_table < W) return FT_ERR_ARG;
  const TanhNorm n0{alpha0, w0, b0}, n1{alpha, w, b};
  const dim3 grid = row_grid(rows, W, 12);
  if (h_f32)
    return (int)ft_launch_pdl(hyper_embed_kernel<float>, grid, dim3(128), 0, st, (const int64_t*)ids, (const float*)table, ld_table, vocab, n0, x, streams, ldx, in_next,
                              n1, (float*)h, ldh, rows, W);
  return (int)ft_launch_pdl(hyper_embed_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, (const int64_t*)ids, (const __nv_bfloat16*)table, ld_table, vocab, n0, x, streams,
                            ldx, in_next, n1, (__nv_bfloat16*)h, ldh, rows, W);
}

// y = tanh(alpha x) w + b by rows; x and y bf16 or (is_f32) f32, alpha f32[1], w and b f32 padded to a multiple of four columns.
FT_EXPORT int ft_dynamic_tanh(const void* x, int64_t ldx, const float* alpha, const float* w, const float* b, void* y, int64_t ldy, int is_f32, int rows, int W,
                              cudaStream_t st) {
  if (rows < 1 || W < 1 || !quad(ldx) || !quad(ldy) || ldx < W || ldy < W) return FT_ERR_ARG;
  const TanhNorm n{alpha, w, b};
  const dim3 grid = row_grid(rows, W, 12);
  if (is_f32) dynamic_tanh_kernel<float><<<grid, 128, 0, st>>>((const float*)x, ldx, n, (float*)y, ldy, rows, W);
  else dynamic_tanh_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>((const __nv_bfloat16*)x, ldx, n, (__nv_bfloat16*)y, ldy, rows, W);
  return (int)cudaGetLastError();
}
