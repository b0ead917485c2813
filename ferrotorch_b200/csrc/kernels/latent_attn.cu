// Latent attention: keys and values are linear images of one small vector per token (the latent c, RMS-normalised) plus one rotated key part shared by
// all heads, so a token's cache row is [c | k_rot] whatever the number of heads. Rows are padded: c to a multiple of 16 elements (`r16`), k_rot to a
// multiple of 16 (`row` = r16 + padded rot), zeros in the padding. Pages hold 16 rows. The rotated part may be absent (rot = 0), queries may come through a
// normalised latent of their own, a layer may read the latent that an earlier layer cached, and the heads' outputs may be gated (per element or per head).
//
//   score(q, j) = scale (q_plain . W_uk c_j + q_rot . k_rot_j) = scale (W_uk^T q_plain | q_rot) . (c_j | k_rot_j)
//   out         = W_uv sum_j p_j c_j
//
//   ft_latent_prep          projection rows of a prompt -> rotated queries (in place), normalised latent and rotated key -> cache page (+ dense row)
//   ft_latent_ctx_gather    cached rows of earlier portions -> dense rows
//   ft_latent_flash         prompts: per-head keys / values expanded from the latent by a GEMM; tcgen05 flash attention over ragged sequences
//   ft_latent_decode_norms  split-K planes of a query latent and a latent -> both normalised, one for the query expansion, one into the cache page
//   ft_latent_decode_prep   split-K planes of one token per sequence -> absorbed queries W_uk^T q_plain, rotations, norm, cache write (one launch)
//   ft_latent_decode        one query token per sequence over the cached rows, all heads of a tile share every loaded row (mma.sync), split over the
//                           sequence; ft_latent_combine merges the splits
//   ft_latent_rows          plain f32-arithmetic kernel for f32 or bf16 data and any sizes (the 32-bit path)
//   ft_latent_gate          the output gate as a pass of its own, behind ft_latent_rows
// Compiled without fast-math.
#include "common.cuh"
#include "host_common.h"

namespace {

constexpr int KV_BLOCK = 16;

template <typename T> FT_DEVICE float to_f(T v);
template <> FT_DEVICE float to_f<float>(float v) { return v; }
template <> FT_DEVICE float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> FT_DEVICE T from_f(float v);
template <> FT_DEVICE float from_f<float>(float v) { return v; }
template <> FT_DEVICE __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
FT_DEVICE float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

FT_DEVICE float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
FT_DEVICE float sigmoid_fast(float x) { return 1.f / (1.f + __expf(-x)); }

// Output gate: pre-activations [rows][ldg] in the data type, a column per element (heads padded to 8) or per head
enum { GATE_NONE = 0, GATE_ELEMENT = 1, GATE_HEAD = 2 };
struct OutputGate {
  const void* p;
  int64_t ldg;
  int kind;
};

// Column layout of a projection row: heads of [plain padded to d8 | rot padded to dr8] (or, with q_rank, the query latent padded to a multiple of 8), then the latent
// (rank padded to rank8), then the shared rot part.
struct LatentDims {
  int H, d, dr, rank;
  int q_rank, q_cols;
  int d8, dr8, rank8, r16, row;      // padded sizes; row = cache row length
};

// ------------------------------------------------------------------------------------------------------------
// prompt rows: grid rows, 128 threads; a warp takes whole heads, a lane neighbouring pairs (two elements at a time everywhere: all offsets are even)
// ------------------------------------------------------------------------------------------------------------
template <typename T> FT_DEVICE float2 load2(const T* p);
template <> FT_DEVICE float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> FT_DEVICE float2 load2<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
template <typename T> FT_DEVICE void store2(T* p, float a, float b);
template <> FT_DEVICE void store2<float>(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
template <> FT_DEVICE void store2<__nv_bfloat16>(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(T* __restrict__ qkv, int64_t ld, LatentDims D, const float* __restrict__ w, float eps,
                                                          const int* __restrict__ positions, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                                          const int* __restrict__ slots, const int* __restrict__ ctx_rows, T* __restrict__ cache, T* __restrict__ ctx,
                                                          const float* __restrict__ wq) {
  __shared__ float red[32];
  const int r = blockIdx.x, half = D.dr / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = positions[r];
  T* row = qkv + (size_t)r * ld;
  const float* ct = cos_t + (size_t)pos * half;
  const float* st = sin_t + (size_t)pos * half;
  const T* lat = row + D.q_cols;
  float ss = 0.f;
  if (D.q_rank) {                                    // the query latent, in place
    for (int i = threadIdx.x * 2; i < D.q_rank; i += 256) {
      const float2 v = load2(row + i);
      ss += v.x * v.x + (i + 1 < D.q_rank ? v.y * v.y : 0.f);
    }
    const float rq = 1.f / sqrtf(block_sum(ss, red) / (float)D.q_rank + eps);
    for (int i = threadIdx.x * 2; i < D.q_rank; i += 256) {
      const float2 v = load2(row + i);
      store2(row + i, v.x * rq * wq[i], i + 1 < D.q_rank ? v.y * rq * wq[i + 1] : 0.f);
    }
    if (cache == nullptr) return;                    // keys and values from an earlier layer's latent
    ss = 0.f;
  }
  for (int i = threadIdx.x * 2; i < D.rank; i += 256) {
    const float2 v = load2(lat + i);
    ss += v.x * v.x + (i + 1 < D.rank ? v.y * v.y : 0.f);
  }
  for (int p = lane; p < half && !D.q_rank; p += 32) {
    const float c = ct[p], s = st[p];
#pragma unroll 4
    for (int hd = warp; hd < D.H; hd += 4) {
      T* q = row + hd * (D.d8 + D.dr8) + D.d8 + 2 * p;
      const float2 v = load2(q);
      store2(q, v.x * c - v.y * s, v.y * c + v.x * s);
    }
  }
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)D.rank + eps);
  T* dst = cache + (size_t)slots[r] * D.row;
  T* dense = ctx ? ctx + (size_t)ctx_rows[r] * D.row : nullptr;
  for (int i = threadIdx.x * 2; i < D.r16; i += 256) {
    float a = 0.f, b = 0.f;
    if (i < D.rank) {
      const float2 v = load2(lat + i);
      a = v.x * rstd * w[i];
      if (i + 1 < D.rank) b = v.y * rstd * w[i + 1];
    }
    store2(dst + i, a, b);
    if (dense) store2(dense + i, a, b);
  }
  const T* kr = lat + D.rank8;
  for (int i = threadIdx.x; i < (D.row - D.r16) / 2; i += 128) {
    float a = 0.f, b = 0.f;
    if (i < half) {
      const float2 v = load2(kr + 2 * i);
      const float c = ct[i], s = st[i];
      a = v.x * c - v.y * s;
      b = v.y * c + v.x * s;
    }
    store2(dst + D.r16 + 2 * i, a, b);
    if (dense) store2(dense + D.r16 + 2 * i, a, b);
  }
}

// Rows that have nothing but a latent to norm (no rotated part, no query latent): a warp each, eight columns a lane
template <typename T> FT_DEVICE void load8(const T* p, float (&v)[8]);
template <> FT_DEVICE void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> FT_DEVICE void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) { bf16x8_to_float(*reinterpret_cast<const bf16x8*>(p), v); }
template <typename T> FT_DEVICE void store8(T* p, const float (&v)[8]);
template <> FT_DEVICE void store8<float>(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
template <> FT_DEVICE void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) { *reinterpret_cast<bf16x8*>(p) = float_to_bf16x8(v); }
template <typename T>
__global__ void __launch_bounds__(128) latent_norm_kernel(const T* __restrict__ lat, int64_t ld, int rows, LatentDims D, const float* __restrict__ w, float eps,
                                                          const int* __restrict__ slots, const int* __restrict__ ctx_rows, T* __restrict__ cache, T* __restrict__ ctx) {
  const int r = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const T* src = lat + (size_t)r * ld;
  float ss = 0.f, v[8];
  for (int i = lane * 8; i < D.rank8; i += 256) {
    load8(src + i, v);
#pragma unroll
    for (int e = 0; e < 8; e++) ss += i + e < D.rank ? v[e] * v[e] : 0.f;
  }
  const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D.rank + eps);
  T* dst = cache + (size_t)slots[r] * D.row;
  T* dense = ctx ? ctx + (size_t)ctx_rows[r] * D.row : nullptr;
  for (int i = lane * 8; i < D.r16; i += 256) {
    if (i < D.rank8) load8(src + i, v);
#pragma unroll
    for (int e = 0; e < 8; e++) v[e] = i + e < D.rank ? v[e] * rstd * w[i + e] : 0.f;
    store8(dst + i, v);
    if (dense) store8(dense + i, v);
  }
}

__global__ void __launch_bounds__(128) latent_ctx_gather_kernel(const uint4* __restrict__ cache, uint4* __restrict__ ctx, int vecs, const int* __restrict__ slots,
                                                                const int* __restrict__ rows) {
  const uint4* src = cache + (size_t)slots[blockIdx.x] * vecs;
  uint4* dst = ctx + (size_t)rows[blockIdx.x] * vecs;
  for (int i = threadIdx.x; i < vecs; i += 128) dst[i] = src[i];
}

// ------------------------------------------------------------------------------------------------------------
// plain kernel: q [rows][H][D.row] (absorbed | rotated), grid (H, rows), 128 threads
// ------------------------------------------------------------------------------------------------------------
constexpr int ROWS_CHUNK = 64, ROWS_MAX_COLS = 16;     // latent columns per thread: r16 <= 128 * 16
template <typename T>
__global__ void __launch_bounds__(128) latent_rows_kernel(const T* __restrict__ q, const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                                                          const int* __restrict__ seq_of, const int* __restrict__ positions, LatentDims D, float scale,
                                                          T* __restrict__ out) {
  extern __shared__ float sm[];
  float* sq = sm;                  // D.row
  __shared__ float sp[ROWS_CHUNK];
  const int hd = blockIdx.x, r = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int len = positions[r] + 1;
  const int* bt = block_table + (size_t)(seq_of ? seq_of[r] : r) * max_blocks;
  const T* qr = q + ((size_t)r * D.H + hd) * D.row;
  for (int i = threadIdx.x; i < D.row; i += 128) sq[i] = to_f(qr[i]);
  float o[ROWS_MAX_COLS];
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++) o[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int t0 = 0; t0 < len; t0 += ROWS_CHUNK) {
    const int cnt = min(ROWS_CHUNK, len - t0);
    for (int k = warp; k < cnt; k += 4) {
      const int t = t0 + k;
      const T* kr = cache + ((size_t)bt[t / KV_BLOCK] * KV_BLOCK + t % KV_BLOCK) * D.row;
      float a = 0.f;
      for (int i = lane; i < D.row; i += 32) a += sq[i] * to_f(kr[i]);
      a = warp_sum(a);
      if (lane == 0) sp[k] = a * scale;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < cnt; k++) mx = fmaxf(mx, sp[k]);
    const float alpha = expf(m - mx);
    l *= alpha;
#pragma unroll
    for (int i = 0; i < ROWS_MAX_COLS; i++) o[i] *= alpha;
    for (int k = 0; k < cnt; k++) {
      const int t = t0 + k;
      const T* kr = cache + ((size_t)bt[t / KV_BLOCK] * KV_BLOCK + t % KV_BLOCK) * D.row;
      const float p = expf(sp[k] - mx);
      l += p;
#pragma unroll
      for (int i = 0; i < ROWS_MAX_COLS; i++)
        if (threadIdx.x + 128 * i < D.r16) o[i] += p * to_f(kr[threadIdx.x + 128 * i]);
    }
    m = mx;
    __syncthreads();
  }
  T* dst = out + ((size_t)r * D.H + hd) * D.r16;
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++)
    if (threadIdx.x + 128 * i < D.r16) dst[threadIdx.x + 128 * i] = from_f<T>(o[i] / l);
}

// a [rows][lda], heads of v8 columns, gated in place; four columns a thread
template <typename T>
__global__ void __launch_bounds__(256) latent_gate_kernel(T* __restrict__ a, int64_t lda, OutputGate gate, int quads, int v8) {
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= quads) return;
  T* x = a + (size_t)blockIdx.y * lda + i * 4;
  const T* g = reinterpret_cast<const T*>(gate.p) + (size_t)blockIdx.y * gate.ldg;
  const int hd = i * 4 / v8;
#pragma unroll
  for (int e = 0; e < 4; e++) x[e] = from_f<T>(to_f(x[e]) * sigmoid_exact(to_f(g[gate.kind == GATE_HEAD ? hd : i * 4 + e])));
}

// ------------------------------------------------------------------------------------------------------------
// decode preparation on split-K planes: CTAs [0, H * slices) absorb 64 latent columns of one head for every token, then one CTA per token handles its cache row, and with a
// gate the rest take 256 of its columns each
// ------------------------------------------------------------------------------------------------------------
constexpr int DEC_TOK = 16, ABS_COLS = 64, PREP_THREADS = 256;
FT_DEVICE float plane_sum(const float* __restrict__ p, int splits, size_t stride, size_t idx) {
  float a = 0.f;
  int s = 0;
  for (; s + 4 <= splits; s += 4) {
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; j++) v[j] = __ldcg(p + (s + j) * stride + idx);
    a += (v[0] + v[1]) + (v[2] + v[3]);
  }
  for (; s < splits; s++) a += __ldcg(p + s * stride + idx);
  return a;
}
__global__ void __launch_bounds__(PREP_THREADS) latent_decode_prep_kernel(const float* __restrict__ planes, int splits, int64_t ldp, size_t pstride, LatentDims D, int B,
                                                                          const __nv_bfloat16* __restrict__ wuk, int64_t ldw, const float* __restrict__ w, float eps,
                                                                          const int* __restrict__ positions, const float* __restrict__ cos_t,
                                                                          const float* __restrict__ sin_t, const int* __restrict__ block_table, int max_blocks,
                                                                          __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ cache, int gate_cols,
                                                                          float* __restrict__ gate) {
  extern __shared__ __align__(16) uint8_t prep_smem[];
  __shared__ float red[32];
  const int slices = (D.r16 + ABS_COLS - 1) / ABS_COLS, half = D.dr / 2;
  const bool absorb = (int)blockIdx.x < D.H * slices;
  const int hd = blockIdx.x / slices, sl = blockIdx.x % slices;
  __nv_bfloat16* sw = reinterpret_cast<__nv_bfloat16*>(prep_smem);             // [d][ABS_COLS]
  float* sq = reinterpret_cast<float*>(prep_smem + (size_t)D.d * ABS_COLS * 2);   // [d][DEC_TOK]
  if (absorb) {
    // the weight slice does not depend on the predecessor: it is on its way before the wait
    const __nv_bfloat16* wp = wuk + (size_t)hd * D.d8 * ldw + sl * ABS_COLS;
    const int vecs = min(ABS_COLS, (int)(ldw - sl * ABS_COLS)) / 8;
    for (int i = threadIdx.x; i < D.d * vecs; i += PREP_THREADS) {
      const int k = i / vecs, v = i % vecs;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(sw + k * ABS_COLS + v * 8)), "l"(wp + (size_t)k * ldw + v * 8) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  pdl_wait();
  pdl_launch_dependents();
  if (absorb) {
    const size_t qcol = (size_t)hd * (D.d8 + D.dr8);
    for (int i = threadIdx.x; i < B * D.d; i += PREP_THREADS) {
      const int b = i / D.d, k = i % D.d;
      // the query as the bf16 operand that the prompt kernels see
      sq[k * DEC_TOK + b] = __bfloat162float(__float2bfloat16(plane_sum(planes, splits, pstride, (size_t)b * ldp + qcol + k)));
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int cp = threadIdx.x & 31, tg = (threadIdx.x >> 5) * 2, c0 = sl * ABS_COLS + cp * 2;   // two columns of two tokens
    if (c0 < D.r16 && tg < B) {
      float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
#pragma unroll 8
      for (int k = 0; k < D.d; k++) {
        const float2 wv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sw + k * ABS_COLS + cp * 2));
        const float2 x = *reinterpret_cast<const float2*>(sq + k * DEC_TOK + tg);
        a00 += x.x * wv.x; a01 += x.x * wv.y;
        a10 += x.y * wv.x; a11 += x.y * wv.y;
      }
      *reinterpret_cast<__nv_bfloat162*>(q + ((size_t)tg * D.H + hd) * D.row + c0) = __floats2bfloat162_rn(a00, a01);
      if (tg + 1 < B) *reinterpret_cast<__nv_bfloat162*>(q + ((size_t)(tg + 1) * D.H + hd) * D.row + c0) = __floats2bfloat162_rn(a10, a11);
    }
    if (sl == 0) {
      const int pairs = (D.row - D.r16) / 2;
      for (int i = threadIdx.x; i < B * pairs; i += PREP_THREADS) {
        const int b = i / pairs, p = i % pairs;
        float a = 0.f, bb = 0.f;
        if (p < half) {
          const size_t idx = (size_t)b * ldp + qcol + D.d8 + 2 * p;
          const float u = plane_sum(planes, splits, pstride, idx), v = plane_sum(planes, splits, pstride, idx + 1);
          const float c = cos_t[(size_t)positions[b] * half + p], s = sin_t[(size_t)positions[b] * half + p];
          a = u * c - v * s;
          bb = v * c + u * s;
        }
        *reinterpret_cast<__nv_bfloat162*>(q + ((size_t)b * D.H + hd) * D.row + D.r16 + 2 * p) = __floats2bfloat162_rn(a, bb);
      }
    }
    return;
  }
  const int extra = blockIdx.x - D.H * slices, rows = cache ? B : 0;
  if (extra >= rows) {                                // sigmoid of the gate's columns, behind the shared rotated part
    const int per = (gate_cols + PREP_THREADS - 1) / PREP_THREADS, tk = (extra - rows) / per, c = (extra - rows) % per * PREP_THREADS + threadIdx.x;
    if (c < gate_cols)
      gate[(size_t)tk * gate_cols + c] = sigmoid_exact(plane_sum(planes, splits, pstride, (size_t)tk * ldp + (size_t)D.H * (D.d8 + D.dr8) + (cache ? D.rank8 + D.dr8 : 0) + c));
    return;
  }
  const int b = extra, pos = positions[b];
  const size_t base = (size_t)b * ldp + (size_t)D.H * (D.d8 + D.dr8);
  float* lat = reinterpret_cast<float*>(prep_smem);     // rank floats (the launcher sizes the buffer for both uses)
  float ss = 0.f;
  for (int i = threadIdx.x; i < D.rank; i += PREP_THREADS) {
    const float v = plane_sum(planes, splits, pstride, base + i);
    lat[i] = v;
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / (float)D.rank + eps);
  const int blk = block_table[(size_t)b * max_blocks + pos / KV_BLOCK];
  if (blk < 0) return;
  __nv_bfloat16* dst = cache + ((size_t)blk * KV_BLOCK + pos % KV_BLOCK) * D.row;
  for (int i = threadIdx.x; i < D.r16; i += PREP_THREADS) dst[i] = __float2bfloat16(i < D.rank ? lat[i] * rstd * w[i] : 0.f);
  for (int p = threadIdx.x; p < (D.row - D.r16) / 2; p += PREP_THREADS) {
    float a = 0.f, bb = 0.f;
    if (p < half) {
      const float u = plane_sum(planes, splits, pstride, base + D.rank8 + 2 * p), v = plane_sum(planes, splits, pstride, base + D.rank8 + 2 * p + 1);
      const float c = cos_t[(size_t)pos * half + p], s = sin_t[(size_t)pos * half + p];
      a = u * c - v * s;
      bb = v * c + u * s;
    }
    *reinterpret_cast<__nv_bfloat162*>(dst + D.r16 + 2 * p) = __floats2bfloat162_rn(a, bb);
  }
}

// grid (B, 1 or 2): y = 0 the query latent of a token, y = 1 its cached latent
__global__ void __launch_bounds__(PREP_THREADS) latent_decode_norms_kernel(const float* __restrict__ planes, int splits, int64_t ldp, size_t pstride, LatentDims D,
                                                                           const float* __restrict__ wq, const float* __restrict__ w, float eps,
                                                                           const int* __restrict__ positions, const int* __restrict__ block_table, int max_blocks,
                                                                           __nv_bfloat16* __restrict__ cq, int64_t ldq, __nv_bfloat16* __restrict__ cache) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t prep_smem[];
  __shared__ float red[32];
  float* v = reinterpret_cast<float*>(prep_smem);
  const int b = blockIdx.x;
  const bool is_q = blockIdx.y == 0;
  const int n = is_q ? D.q_rank : D.rank;
  const size_t base = (size_t)b * ldp + (is_q ? 0 : D.q_cols);
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += PREP_THREADS) {
    const float x = plane_sum(planes, splits, pstride, base + i);
    v[i] = x;
    ss += x * x;
  }
  const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
  if (is_q) {
    for (int i = threadIdx.x; i < n; i += PREP_THREADS) cq[(size_t)b * ldq + i] = __float2bfloat16(v[i] * rstd * wq[i]);
    return;
  }
  const int pos = positions[b], blk = block_table[(size_t)b * max_blocks + pos / KV_BLOCK];
  if (blk < 0) return;
  __nv_bfloat16* dst = cache + ((size_t)blk * KV_BLOCK + pos % KV_BLOCK) * D.row;
  for (int i = threadIdx.x; i < D.r16; i += PREP_THREADS) dst[i] = __float2bfloat16(i < n ? v[i] * rstd * w[i] : 0.f);
}

// ------------------------------------------------------------------------------------------------------------
// decode attention: grid (nsplit, ceil(H / (16 MT)), B), 256 threads.
// Chunks of 64 cached rows go through a two-stage shared-memory ring (16-byte cp.async; rows an odd number of 16-byte units apart, so the ldmatrix
// reads are conflict free). Scores: warp w takes eight rows of the chunk against the MT * 16 heads over the whole row length; softmax statistics meet
// in shared memory; output: warp w takes NP * 16 latent columns over all 64 rows. ws: [B][head tile][split][MT * 16][r16 + 4] f32 (accumulators, running
// maximum in the log2 domain, running sum).
// ------------------------------------------------------------------------------------------------------------
constexpr int LD_CHUNK = 64, LD_STAGES = 2, LD_P_PITCH = 144;

FT_DEVICE void cp_async16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
FT_DEVICE void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
FT_DEVICE void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
FT_DEVICE void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
FT_DEVICE void ldmatrix_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
FT_DEVICE void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
FT_DEVICE void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__host__ __device__ inline int latent_smem_pitch(int row) { return row * 2 + 16; }

template <int MT, int NP>
__global__ void __launch_bounds__(256, 1) latent_decode_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache,
                                                               const int* __restrict__ block_table, int max_blocks, const int* __restrict__ seq_lens, LatentDims D,
                                                               float scale, float* __restrict__ ws) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float sm_mx[8][MT * 16], sm_l[8][MT * 16];
  constexpr int HT = MT * 16;
  const int split = blockIdx.x, nsplit = gridDim.x, tile = blockIdx.y, b = blockIdx.z, h0 = tile * HT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int len = seq_lens[b];
  const int per = ((len + nsplit - 1) / nsplit + KV_BLOCK - 1) / KV_BLOCK * KV_BLOCK;
  const int t0 = split * per, t1 = min(len, t0 + per);
  float* my_ws = ws + (((size_t)b * gridDim.y + tile) * nsplit + split) * HT * (D.r16 + 4);
  if (t1 <= t0) {                                                   // nothing for this split
    for (int i = threadIdx.x; i < HT; i += 256) { my_ws[(size_t)i * (D.r16 + 4) + D.r16] = -INFINITY; my_ws[(size_t)i * (D.r16 + 4) + D.r16 + 1] = 0.f; }
    return;
  }
  const int nchunks = (t1 - t0 + LD_CHUNK - 1) / LD_CHUNK;
  const int pitch = latent_smem_pitch(D.row), vecs = D.row / 8;
  const uint32_t sQ = smem_u32(smem), sK = sQ + HT * pitch, sP = sK + LD_STAGES * LD_CHUNK * pitch;
  const int* bt = block_table + (size_t)b * max_blocks;

  auto load_chunk = [&](int c, int stage) {
    const int c0 = t0 + c * LD_CHUNK, cnt = min(LD_CHUNK, t1 - c0);
    const uint32_t dst = sK + stage * LD_CHUNK * pitch;
    for (int r = warp; r < cnt; r += 8) {
      const int t = c0 + r;
      const __nv_bfloat16* src = cache + ((size_t)__ldg(bt + t / KV_BLOCK) * KV_BLOCK + t % KV_BLOCK) * D.row;
      for (int i = lane; i < vecs; i += 32) cp_async16(dst + r * pitch + i * 16, src + i * 8);
    }
    // rows up to the next multiple of 16 meet weight zero: they must be finite
    for (int r = cnt + warp; r < ((cnt + 15) & ~15); r += 8)
      for (int i = lane; i < vecs; i += 32) *reinterpret_cast<uint4*>(smem + (dst - sQ) + r * pitch + i * 16) = make_uint4(0, 0, 0, 0);
  };
  for (int r = warp; r < HT; r += 8)
    for (int i = lane; i < vecs; i += 32) {
      if (h0 + r < D.H) cp_async16(sQ + r * pitch + i * 16, q + ((size_t)b * D.H + h0 + r) * D.row + i * 8);
      else *reinterpret_cast<uint4*>(smem + r * pitch + i * 16) = make_uint4(0, 0, 0, 0);
    }
#pragma unroll
  for (int s = 0; s < LD_STAGES; s++) {
    if (s < nchunks) load_chunk(s, s);
    cp_async_commit();
  }
  const float sl2 = scale * 1.4426950408889634f;
  float o[MT][NP][2][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int p = 0; p < NP; p++)
#pragma unroll
      for (int e = 0; e < 4; e++) o[m][p][0][e] = o[m][p][1][e] = 0.f;
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int m = 0; m < MT; m++) { m_run[m][0] = m_run[m][1] = -INFINITY; l_run[m][0] = l_run[m][1] = 0.f; }
  const int npairs = D.r16 / 16, ksteps = D.row / 16;

  for (int c = 0; c < nchunks; c++) {
    cp_async_wait<LD_STAGES - 1>();
    __syncthreads();
    const int stage = c % LD_STAGES, cnt = min(LD_CHUNK, t1 - (t0 + c * LD_CHUNK));
    const uint32_t kb = sK + stage * LD_CHUNK * pitch;
    float s[MT][4];
#pragma unroll
    for (int m = 0; m < MT; m++) s[m][0] = s[m][1] = s[m][2] = s[m][3] = 0.f;
    if (warp * 8 < cnt) {
      const uint32_t krow = kb + (warp * 8 + (lane & 7)) * pitch;
      const uint32_t qrow = sQ + (lane & 15) * pitch + (lane >> 4) * 16;
      int ks = 0;
      for (; ks + 2 <= ksteps; ks += 2) {
        uint32_t kf[4];
        ldmatrix_x4(kf, krow + ks * 32 + (lane >> 3) * 16);
#pragma unroll
        for (int m = 0; m < MT; m++) {
          uint32_t qa[4], qb[4];
          ldmatrix_x4(qa, qrow + m * 16 * pitch + ks * 32);
          ldmatrix_x4(qb, qrow + m * 16 * pitch + ks * 32 + 32);
          mma_16816(s[m], qa[0], qa[1], qa[2], qa[3], kf[0], kf[1]);
          mma_16816(s[m], qb[0], qb[1], qb[2], qb[3], kf[2], kf[3]);
        }
      }
      if (ks < ksteps) {
        uint32_t k0, k1;
        ldmatrix_x2(k0, k1, krow + ks * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
        for (int m = 0; m < MT; m++) {
          uint32_t qa[4];
          ldmatrix_x4(qa, qrow + m * 16 * pitch + ks * 32);
          mma_16816(s[m], qa[0], qa[1], qa[2], qa[3], k0, k1);
        }
      }
    }
    const bool v0 = warp * 8 + t2 < cnt, v1 = warp * 8 + t2 + 1 < cnt;
#pragma unroll
    for (int m = 0; m < MT; m++) {
      float a = fmaxf(v0 ? s[m][0] : -INFINITY, v1 ? s[m][1] : -INFINITY), bq = fmaxf(v0 ? s[m][2] : -INFINITY, v1 ? s[m][3] : -INFINITY);
      a = fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 1));
      a = fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 2));
      bq = fmaxf(bq, __shfl_xor_sync(0xffffffffu, bq, 1));
      bq = fmaxf(bq, __shfl_xor_sync(0xffffffffu, bq, 2));
      if ((lane & 3) == 0) { sm_mx[warp][m * 16 + g] = a; sm_mx[warp][m * 16 + g + 8] = bq; }
    }
    __syncthreads();
    float alpha[MT][2];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        float mx = m_run[m][e];
#pragma unroll
        for (int w = 0; w < 8; w++) mx = fmaxf(mx, sm_mx[w][m * 16 + g + 8 * e]);
        alpha[m][e] = ex2((m_run[m][e] - mx) * sl2);                // 0 on the first chunk
        m_run[m][e] = mx;
        const float p0 = v0 ? ex2((s[m][2 * e] - mx) * sl2) : 0.f, p1 = v1 ? ex2((s[m][2 * e + 1] - mx) * sl2) : 0.f;
        l_run[m][e] = l_run[m][e] * alpha[m][e] + p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(smem + (sP - sQ) + (m * 16 + g + 8 * e) * LD_P_PITCH + (warp * 8 + t2) * 2) = __floats2bfloat162_rn(p0, p1);
      }
    __syncthreads();
    const int psteps = (cnt + 15) / 16;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int p = 0; p < NP; p++)
#pragma unroll
        for (int n = 0; n < 2; n++) {
          o[m][p][n][0] *= alpha[m][0]; o[m][p][n][1] *= alpha[m][0];
          o[m][p][n][2] *= alpha[m][1]; o[m][p][n][3] *= alpha[m][1];
        }
    for (int ps = 0; ps < psteps; ps++) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; m++) ldmatrix_x4(pf[m], sP + (m * 16 + (lane & 15)) * LD_P_PITCH + ps * 32 + (lane >> 4) * 16);
      const uint32_t vrow = kb + (ps * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * pitch + (lane >> 4) * 16;
#pragma unroll
      for (int p = 0; p < NP; p++) {
        const int pr = warp * NP + p;
        if (pr < npairs) {
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, vrow + pr * 32);
#pragma unroll
          for (int m = 0; m < MT; m++) {
            mma_16816(o[m][p][0], pf[m][0], pf[m][1], pf[m][2], pf[m][3], vb[0], vb[1]);
            mma_16816(o[m][p][1], pf[m][0], pf[m][1], pf[m][2], pf[m][3], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();
    if (c + LD_STAGES < nchunks) load_chunk(c + LD_STAGES, stage);
    cp_async_commit();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float l = l_run[m][e];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if ((lane & 3) == 0) sm_l[warp][m * 16 + g + 8 * e] = l;
      const int hrow = m * 16 + g + 8 * e;
      float* dst = my_ws + (size_t)hrow * (D.r16 + 4);
#pragma unroll
      for (int p = 0; p < NP; p++) {
        const int pr = warp * NP + p;
        if (pr < npairs && h0 + hrow < D.H) {
          *reinterpret_cast<float2*>(dst + pr * 16 + t2) = make_float2(o[m][p][0][2 * e], o[m][p][0][2 * e + 1]);
          *reinterpret_cast<float2*>(dst + pr * 16 + 8 + t2) = make_float2(o[m][p][1][2 * e], o[m][p][1][2 * e + 1]);
        }
      }
      if (warp == 0 && (lane & 3) == 0) dst[D.r16] = m_run[m][e] * sl2;
    }
  __syncthreads();
  for (int i = threadIdx.x; i < HT; i += 256) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) l += sm_l[w][i];
    my_ws[(size_t)i * (D.r16 + 4) + D.r16 + 1] = l;
  }
}

// merge the splits: grid (H, B), 128 threads; out [B][H][r16] bf16
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ ws, int H, int HT, int tiles, int nsplit, int r16, __nv_bfloat16* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float f[64];
  __shared__ float inv_sh;
  const int hd = blockIdx.x, b = blockIdx.y;
  const int ldw = r16 + 4;
  const size_t sstride = (size_t)HT * ldw;
  const float* base = ws + (((size_t)b * tiles + hd / HT) * nsplit) * sstride + (size_t)(hd % HT) * ldw;
  if (threadIdx.x < 32) {
    float m[2], l[2], mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int s = threadIdx.x + 32 * i;
      m[i] = s < nsplit ? __ldcg(base + s * sstride + r16) : -INFINITY;
      l[i] = s < nsplit ? __ldcg(base + s * sstride + r16 + 1) : 0.f;
      mx = fmaxf(mx, m[i]);
    }
    mx = warp_max(mx);
    float tot = 0.f;
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const float w = m[i] == -INFINITY ? 0.f : ex2(m[i] - mx);
      f[threadIdx.x + 32 * i] = w;
      tot += w * l[i];
    }
    tot = warp_sum(tot);
    if (threadIdx.x == 0) inv_sh = tot > 0.f ? 1.f / tot : 0.f;
  }
  __syncthreads();
  const float inv = inv_sh;
  for (int c = threadIdx.x * 4; c < r16; c += 512) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = 0; s0 < nsplit; s0 += 8) {
      float4 v[8];
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const bool live = s0 + j < nsplit && f[min(s0 + j, 63)] > 0.f;    // a split without rows left its accumulators unwritten
        v[j] = live ? __ldcg(reinterpret_cast<const float4*>(base + (s0 + j) * sstride + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const float w = s0 + j < nsplit ? f[s0 + j] : 0.f;
        a.x += w * v[j].x; a.y += w * v[j].y; a.z += w * v[j].z; a.w += w * v[j].w;
      }
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(a.x * inv, a.y * inv), hi = __floats2bfloat162_rn(a.z * inv, a.w * inv);
    uint2 pk;
    pk.x = *reinterpret_cast<uint32_t*>(&lo);
    pk.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(out + ((size_t)b * H + hd) * r16 + c) = pk;
  }
}

// ------------------------------------------------------------------------------------------------------------
// prompt attention (tcgen05): one CTA per (tile of NT * 128 queries of one sequence, head).
//   warp 0       TMA: the queries' column blocks once, then keys (plain blocks of this head + the shared rotated block) and values, 64 rows at a time,
//                two-stage rings. Heads are a tensor-map dimension of their own, so columns past a head's size arrive as zeros.
//   warp 1       TMEM owner; one lane issues S_t = Q_t K^T for the NT query tiles (double buffered) and O_t += P_t V
//   warps 2..    one thread per query row and tile: causal mask, online softmax in the log2 domain, P (bf16) through swizzled shared memory
// With NT = 2 one tile's softmax runs under the other tile's tensor work and both share every loaded key and value block.
// ------------------------------------------------------------------------------------------------------------
constexpr int LF_BM = 128, LF_BN = 64;
constexpr int LF_QB = LF_BM * 128;         // one 64-column block of 128 queries
constexpr int LF_KB = LF_BN * 128;         // one 64-column block of 64 keys
constexpr int LF_PB = LF_BM * 128;
constexpr uint32_t FT_K_LATENT = 9;

FT_DEVICE bool lf_wait(uint64_t* bar, uint32_t parity) {
  if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = globaltimer_ns();
  for (uint32_t i = 1;; i++) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 0xff) == 0 && globaltimer_ns() - t0 > 2000000000ull) return false;
  }
}

struct FlashDims {
  int d, dr, dv;                   // per-head sizes
  int nn, nr, nv;                  // 64-column blocks of plain, rotated and value dimensions
  int dv8;
};

// NQ, NV: 64-column blocks of the query / key and value dimensions at compile time (the issuing thread's descriptors then are constants added to a base;
// built at run time they cost more than the MMAs themselves), or 0 to read them from F.
template <int NT, int NQ, int NV>
__global__ void __launch_bounds__(64 + 128 * NT, (NT == 1 && NV == 1) ? 2 : 1)
latent_flash_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmKr, const __grid_constant__ CUtensorMap tmV, const int4* __restrict__ tiles, FlashDims F, float scale_log2,
                    OutputGate gate, __nv_bfloat16* __restrict__ out, int64_t ldo, uint32_t* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nq = NQ > 0 ? NQ : F.nn + F.nr, nv = NV > 0 ? NV : F.nv;
  const int k_bytes = nq * LF_KB, v_bytes = nv * LF_KB;
  uint8_t* sQ = smem;                               // [NT][nq]
  uint8_t* sK = sQ + NT * nq * LF_QB;               // [2][nq]
  uint8_t* sV = sK + 2 * k_bytes;                   // [2][nv]
  uint8_t* sP = sV + 2 * v_bytes;                   // [NT]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + NT * LF_PB);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;                      // [2]
  uint64_t* k_empty = bars + 3;
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 7;
  uint64_t* s_full = bars + 9;                      // [NT][2]
  uint64_t* p_ready = bars + 9 + 2 * NT;            // [NT]
  uint64_t* pv_done = bars + 9 + 3 * NT;            // [NT]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 9 + 4 * NT);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 tl = tiles[blockIdx.x];                // first query row, rows, position of the first row, first context row of the sequence
  const int hd = blockIdx.y;
  int nblk[NT], nmax = 0;
#pragma unroll
  for (int t = 0; t < NT; t++) {
    const int rows = min(LF_BM, tl.y - t * LF_BM);
    nblk[t] = rows > 0 ? (tl.z + t * LF_BM + rows + LF_BN - 1) / LF_BN : 0;
    nmax = max(nmax, nblk[t]);
  }
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; i++) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    for (int t = 0; t < NT; t++) { mbar_init(&s_full[2 * t], 1); mbar_init(&s_full[2 * t + 1], 1); mbar_init(&p_ready[t], 128); mbar_init(&pv_done[t], 1); }
    mbar_fence_init();
  }
  if (warp == 0 && lane == 0) { tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmQr); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmKr); tma_prefetch_desc(&tmV); }
  constexpr uint32_t TMEM = (NT == 1 && NV == 1) ? 256 : 512;       // small heads leave room for a second CTA
  if (warp == 1) { tmem_alloc(tmem_slot, TMEM); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tS = *tmem_slot, tO = tS + NT * 2 * LF_BN;

  if (warp == 0) {
    if (lane == 0) {
      int live = 0;
      for (int t = 0; t < NT; t++) live += nblk[t] > 0;
      mbar_expect_tx(q_full, live * nq * LF_QB);
      for (int t = 0; t < NT; t++) {
        if (nblk[t] == 0) continue;
        for (int c = 0; c < F.nn; c++) tma_load_3d(sQ + (t * nq + c) * LF_QB, &tmQ, q_full, c * 64, hd, tl.x + t * LF_BM);
        for (int c = 0; c < F.nr; c++) tma_load_3d(sQ + (t * nq + F.nn + c) * LF_QB, &tmQr, q_full, c * 64, hd, tl.x + t * LF_BM);
      }
      auto load_k = [&](int j) -> bool {
        const int s = j & 1;
        if (!lf_wait(&k_empty[s], ((j >> 1) & 1) ^ 1)) { ft_set_status(status, FT_K_LATENT, 1, j); return false; }
        mbar_expect_tx(&k_full[s], k_bytes);
        for (int c = 0; c < F.nn; c++) tma_load_3d(sK + s * k_bytes + c * LF_KB, &tmK, &k_full[s], c * 64, hd, tl.w + j * LF_BN);
        for (int c = 0; c < F.nr; c++) tma_load_2d(sK + s * k_bytes + (F.nn + c) * LF_KB, &tmKr, &k_full[s], c * 64, tl.w + j * LF_BN);
        return true;
      };
      bool ok = load_k(0);
      for (int j = 0; j < nmax && ok; j++) {
        if (j + 1 < nmax) ok = load_k(j + 1);
        if (!ok) break;
        const int s = j & 1;
        if (!lf_wait(&v_empty[s], ((j >> 1) & 1) ^ 1)) { ft_set_status(status, FT_K_LATENT, 2, j); ok = false; break; }
        mbar_expect_tx(&v_full[s], v_bytes);
        for (int c = 0; c < nv; c++) tma_load_3d(sV + s * v_bytes + c * LF_KB, &tmV, &v_full[s], c * 64, hd, tl.w + j * LF_BN);
      }
      if (!ok)
        for (int i = 0; i < 64; i++) __nanosleep(1000);      // copies in flight land before the shared memory goes away
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_f16(LF_BM, LF_BN, 1, 0, 0);
      const uint32_t idesc_o = make_idesc_f16(LF_BM, nv * 64, 1, 0, 1);
      // a descriptor's start address counts 16-byte units in its low bits: moving inside the operand is an addition
      const uint64_t q_desc = make_smem_desc(smem_u32(sQ), 16, 1024, FT_SWZ_128B), k_desc = make_smem_desc(smem_u32(sK), 16, 1024, FT_SWZ_128B);
      const uint64_t p_desc = make_smem_desc(smem_u32(sP), 16, 1024, FT_SWZ_128B), v_desc = make_smem_desc(smem_u32(sV), LF_KB, 1024, FT_SWZ_128B);
      auto issue_s = [&](int t, int j) {
        const uint64_t qd = q_desc + (uint32_t)(t * nq) * (LF_QB / 16), kd = k_desc + (uint32_t)(j & 1) * (k_bytes / 16);
        const uint32_t d = tS + t * 2 * LF_BN + (j & 1) * LF_BN;
#pragma unroll
        for (int c = 0; c < nq; c++) {
#pragma unroll
          for (int k = 0; k < 4; k++) umma_f16_ss(d, qd + c * (LF_QB / 16) + k * 2, kd + c * (LF_KB / 16) + k * 2, idesc_s, (c | k) != 0);
        }
        umma_commit(&s_full[2 * t + (j & 1)]);
      };
      bool ok = lf_wait(q_full, 0) && lf_wait(&k_full[0], 0);
      if (!ok) ft_set_status(status, FT_K_LATENT, 3, 0);
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < NT; t++)
          if (nblk[t] > 0) issue_s(t, 0);
        umma_commit(&k_empty[0]);
        for (int j = 0; j < nmax && ok; j++) {
          if (j + 1 < nmax) {
            if (!lf_wait(&k_full[(j + 1) & 1], ((j + 1) >> 1) & 1)) { ft_set_status(status, FT_K_LATENT, 4, j); break; }
            tc_fence_after();
#pragma unroll
            for (int t = 0; t < NT; t++)
              if (j + 1 < nblk[t]) issue_s(t, j + 1);
            umma_commit(&k_empty[(j + 1) & 1]);
          }
          if (!lf_wait(&v_full[j & 1], (j >> 1) & 1)) { ft_set_status(status, FT_K_LATENT, 5, j); break; }
          const uint64_t vd = v_desc + (uint32_t)(j & 1) * (v_bytes / 16);
#pragma unroll
          for (int t = 0; t < NT; t++) {
            if (j >= nblk[t] || !ok) continue;
            if (!lf_wait(&p_ready[t], j & 1)) { ft_set_status(status, FT_K_LATENT, 6, j); ok = false; continue; }
            tc_fence_after();
#pragma unroll
            for (int k = 0; k < LF_BN / 16; k++)
              umma_f16_ss(tO + t * nv * 64, p_desc + t * (LF_PB / 16) + k * 2, vd + k * 128, idesc_o, (j | k) != 0);
            umma_commit(&pv_done[t]);
          }
          umma_commit(&v_empty[j & 1]);
        }
      }
    }
  } else {
    const int t = (warp - 2) >> 2, q = warp & 3, r = q * 32 + lane;
    const int nb = t == 0 ? nblk[0] : nblk[NT - 1];
    const int qpos = tl.z + t * LF_BM + r;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    uint8_t* prow = sP + t * LF_PB + r * 128;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nb && ok; j++) {
      if (!lf_wait(&s_full[2 * t + (j & 1)], (j >> 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_LATENT, 7, j); ok = false; break; }
      tc_fence_after();
      __syncwarp();                                            // the TMEM loads are warp-wide: every lane is here
      uint32_t sv[64];
      tmem_ld_32x32b_x32(tS + lane_off + t * 2 * LF_BN + (j & 1) * LF_BN, sv);
      tmem_ld_32x32b_x32(tS + lane_off + t * 2 * LF_BN + (j & 1) * LF_BN + 32, sv + 32);
      tmem_ld_wait();
      const int kv0 = j * LF_BN;
      if (kv0 + LF_BN - 1 > tl.z + t * LF_BM) {                // the diagonal can cross this block
#pragma unroll
        for (int c = 0; c < 64; c++)
          if (kv0 + c > qpos) sv[c] = __float_as_uint(-INFINITY);
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 64; c++) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(sv[c]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      float m_new = fmaxf(m_used, mx);
      if (m_new == -INFINITY) m_new = 0.f;
      const bool grow = (m_new - m_used) * scale_log2 > 8.f;
      const bool rescale = __any_sync(0xffffffffu, grow);
      float alpha = 1.f;
      if (rescale) {
        alpha = ex2((m_used - m_new) * scale_log2);
        m_used = m_new;
      }
      const float moff = m_used * scale_log2;
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pk[32];
#pragma unroll
      for (int c = 0; c < 32; c++) {
        const float p0 = ex2(fmaf(__uint_as_float(sv[2 * c]), scale_log2, -moff));
        const float p1 = ex2(fmaf(__uint_as_float(sv[2 * c + 1]), scale_log2, -moff));
        rs4[c & 3] += p0 + p1;
        __nv_bfloat162 hh = __floats2bfloat162_rn(p0, p1);
        pk[c] = *reinterpret_cast<uint32_t*>(&hh);
      }
      l = l * alpha + ((rs4[0] + rs4[1]) + (rs4[2] + rs4[3]));
      if (j > 0) {
        if (!lf_wait(&pv_done[t], (j - 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_LATENT, 8, j); ok = false; break; }
        tc_fence_after();
        __syncwarp();
        if (rescale) {
#pragma unroll 1
          for (int c = 0; c < nv * 2; c++) {
            uint32_t ov[32];
            const uint32_t addr = tO + lane_off + t * nv * 64 + c * 32;
            tmem_ld_32x32b_x32(addr, ov);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; e++) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * alpha);
            tmem_st_32x32b_x32(addr, ov);
          }
          tmem_st_wait();
        }
      }
#pragma unroll
      for (int c8 = 0; c8 < 8; c8++)
        *reinterpret_cast<uint4*>(prow + ((c8 ^ (r & 7)) << 4)) = make_uint4(pk[4 * c8], pk[4 * c8 + 1], pk[4 * c8 + 2], pk[4 * c8 + 3]);
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&p_ready[t]);
    }
    if (ok && nb > 0) {
      if (!lf_wait(&pv_done[t], (nb - 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_LATENT, 9, 0); ok = false; }
    }
    if (ok && nb > 0) {
      tc_fence_after();
      float inv_l = 1.f / l;
      const bool live = t * LF_BM + r < tl.y;
      const size_t row = (size_t)(tl.x + t * LF_BM + r);
      const __nv_bfloat16* gp = reinterpret_cast<const __nv_bfloat16*>(gate.p) + row * gate.ldg;
      if (gate.kind == GATE_HEAD && live) inv_l *= sigmoid_fast(__bfloat162float(gp[hd]));
      const bool gated = gate.kind == GATE_ELEMENT;
      gp += (size_t)hd * F.dv8;
      __nv_bfloat16* dst = out + row * ldo + (size_t)hd * F.dv8;
      // rows past the end of the sequence only skip the stores: the warp-wide TMEM loads stay in code that all lanes run together
#pragma unroll 1
      for (int c = 0; c < nv * 2; c++) {
        uint32_t ov[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tO + lane_off + t * nv * 64 + c * 32, ov);
        tmem_ld_wait();
        uint4 w[4];
        if (gated) {
#pragma unroll
          for (int c8 = 0; c8 < 4; c8++) {
            if (live && c * 32 + c8 * 8 + 8 <= F.dv8) {
              float gv[8];
              bf16x8_to_float(*reinterpret_cast<const bf16x8*>(gp + c * 32 + c8 * 8), gv);
#pragma unroll
              for (int i = 0; i < 8; i++) ov[8 * c8 + i] = __float_as_uint(__uint_as_float(ov[8 * c8 + i]) * sigmoid_fast(gv[i]));
            }
          }
        }
#pragma unroll
        for (int c8 = 0; c8 < 4; c8++) {
          uint32_t e[4];
#pragma unroll
          for (int i = 0; i < 4; i++) {
            __nv_bfloat162 hh = __floats2bfloat162_rn(__uint_as_float(ov[8 * c8 + 2 * i]) * inv_l, __uint_as_float(ov[8 * c8 + 2 * i + 1]) * inv_l);
            e[i] = *reinterpret_cast<uint32_t*>(&hh);
          }
          w[c8] = make_uint4(e[0], e[1], e[2], e[3]);
        }
#pragma unroll
        for (int c8 = 0; c8 < 4; c8++)
          if (live && c * 32 + c8 * 8 + 8 <= F.dv8) *reinterpret_cast<uint4*>(dst + c * 32 + c8 * 8) = w[c8];
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tS, TMEM);
  }
}

LatentDims make_dims(int H, int d, int dr, int rank, int q_rank = 0) {
  LatentDims D;
  D.H = H; D.d = d; D.dr = dr; D.rank = rank;
  D.d8 = (d + 7) & ~7;
  D.dr8 = (dr + 7) & ~7;
  D.rank8 = (rank + 7) & ~7;
  D.r16 = (rank + 15) & ~15;
  D.row = D.r16 + ((dr + 15) & ~15);
  D.q_rank = q_rank;
  D.q_cols = q_rank ? (q_rank + 7) & ~7 : H * (D.d8 + D.dr8);
  return D;
}
bool dims_ok(int H, int d, int dr, int rank) { return H >= 1 && d >= 1 && dr >= 0 && (dr & 1) == 0 && rank >= 1; }
int flash_smem(int NT, int nq, int nv) { return NT * nq * LF_QB + 2 * (nq + nv) * LF_KB + NT * LF_PB + 256 + 1024; }
constexpr int SMEM_MAX = 232448;

template <int NT, int NQ, int NV>
int launch_flash(const CUtensorMap (&m)[5], const int* tiles, int ntiles, int H, const FlashDims& F, float scale, const OutputGate& gate, void* out, int64_t ldo, int smem,
                 cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    FT_CUDA_TRY(cudaFuncSetAttribute(latent_flash_kernel<NT, NQ, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    configured = true;
  }
  latent_flash_kernel<NT, NQ, NV><<<dim3(ntiles, H), 64 + 128 * NT, smem, st>>>(m[0], m[1], m[2], m[3], m[4], reinterpret_cast<const int4*>(tiles), F,
                                                                       scale * 1.4426950408889634f, gate, (__nv_bfloat16*)out, ldo, ft_status_ptr());
  return (int)cudaGetLastError();
}

template <int MT, int NP>
int launch_decode(dim3 grid, int smem, cudaStream_t st, const void* q, const void* cache, const int* bt, int mb, const int* lens, const LatentDims& D, float scale,
                  float* ws) {
  static bool configured = false;
  if (!configured) {
    FT_CUDA_TRY(cudaFuncSetAttribute(latent_decode_kernel<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX - 8192));
    configured = true;
  }
  return (int)ft_launch_pdl(latent_decode_kernel<MT, NP>, grid, dim3(256), (size_t)smem, st, (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, bt, mb, lens, D, scale,
                            ws);
}

}  // namespace

// Projection rows qkv [rows][ld] (bf16, or f32 with is_f32): heads of [plain | rot] (each padded to 8 columns), latent (padded to 8), shared rot part.
// Rotates the queries' rot parts in place (pairs of neighbouring columns, tables cos/sin f32 [position][dr / 2]), normalises the latent (w f32[rank])
// and rotates the shared key part into cache row slots[r] (= page * 16 + offset) and, when ctx is given, dense row ctx_rows[r]. Cache rows have
// 16-padded latent + 16-padded rot elements. q_rank > 0 (with dr = 0): the heads' columns hold the query latent instead (padded to 8), which is normalised in place
// with wq (f32[q_rank]); cache may then be null, for rows without a latent of their own.
FT_EXPORT int ft_latent_prep(void* qkv, int64_t ld, int rows, int H, int d, int dr, int rank, int q_rank, const float* wq, const float* w, float eps, const int* positions,
                             const float* cos_t, const float* sin_t, const int* slots, const int* ctx_rows, void* cache, void* ctx, int is_f32, cudaStream_t st) {
  if (rows < 1 || !dims_ok(H, d, dr, rank) || q_rank < 0 || (ctx && !ctx_rows) || (q_rank ? dr != 0 || !wq : !cache)) return FT_ERR_ARG;
  const LatentDims D = make_dims(H, d, dr, rank, q_rank);
  if (ld < (int64_t)D.q_cols + (cache ? D.rank8 + dr : 0) || (ld & 7)) return FT_ERR_ARG;
  if (dr == 0 && q_rank == 0) {
    const int ctas = (rows + 3) / 4;
    if (is_f32) latent_norm_kernel<float><<<ctas, 128, 0, st>>>((const float*)qkv + D.q_cols, ld, rows, D, w, eps, slots, ctx_rows, (float*)cache, (float*)ctx);
    else latent_norm_kernel<__nv_bfloat16><<<ctas, 128, 0, st>>>((const __nv_bfloat16*)qkv + D.q_cols, ld, rows, D, w, eps, slots, ctx_rows, (__nv_bfloat16*)cache, (__nv_bfloat16*)ctx);
    return (int)cudaGetLastError();
  }
  if (is_f32) latent_prep_kernel<float><<<rows, 128, 0, st>>>((float*)qkv, ld, D, w, eps, positions, cos_t, sin_t, slots, ctx_rows, (float*)cache, (float*)ctx, wq);
  else latent_prep_kernel<__nv_bfloat16><<<rows, 128, 0, st>>>((__nv_bfloat16*)qkv, ld, D, w, eps, positions, cos_t, sin_t, slots, ctx_rows, (__nv_bfloat16*)cache,
                                                               (__nv_bfloat16*)ctx, wq);
  return (int)cudaGetLastError();
}

// ctx row rows[i] <- cache row slots[i] for n rows of row_bytes (a multiple of 16)
FT_EXPORT int ft_latent_ctx_gather(const void* cache, void* ctx, int row_bytes, const int* slots, const int* rows, int n, cudaStream_t st) {
  if (n < 1 || row_bytes < 16 || (row_bytes & 15)) return FT_ERR_ARG;
  latent_ctx_gather_kernel<<<n, 128, 0, st>>>((const uint4*)cache, (uint4*)ctx, row_bytes / 16, slots, rows);
  return (int)cudaGetLastError();
}

// Plain attention over cached rows: q [rows][H][row] (absorbed | rotated), row r of sequence seq_of[r] (null: r) sees positions 0..positions[r];
// out [rows][H][r16], both f32 (is_f32) or bf16. Latent sizes up to 2048.
FT_EXPORT int ft_latent_rows(const void* q, const void* cache, const int* block_table, int max_blocks, const int* seq_of, const int* positions, int rows, int H, int dr,
                             int rank, float scale, void* out, int is_f32, cudaStream_t st) {
  if (rows < 1 || rows > 65535 || !dims_ok(H, 1, dr, rank)) return FT_ERR_ARG;
  const LatentDims D = make_dims(H, 1, dr, rank);
  if (D.r16 > 128 * ROWS_MAX_COLS) return FT_ERR_TOO_LARGE;
  const dim3 grid(H, rows);
  if (is_f32) latent_rows_kernel<float><<<grid, 128, D.row * 4, st>>>((const float*)q, (const float*)cache, block_table, max_blocks, seq_of, positions, D, scale, (float*)out);
  else latent_rows_kernel<__nv_bfloat16><<<grid, 128, D.row * 4, st>>>((const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_table, max_blocks, seq_of, positions, D,
                                                                       scale, (__nv_bfloat16*)out);
  return (int)cudaGetLastError();
}

// a [rows][lda] (heads of v8 columns, v8 a multiple of 8) times the sigmoid of gate [rows][ldg], kinds as in ft_latent_flash; both f32 (is_f32) or bf16.
FT_EXPORT int ft_latent_gate(void* a, int64_t lda, const void* gate, int64_t ldg, int gate_kind, int rows, int H, int v8, int is_f32, cudaStream_t st) {
  if (rows < 1 || H < 1 || v8 < 8 || (v8 & 7) || (gate_kind != GATE_ELEMENT && gate_kind != GATE_HEAD) || !gate) return FT_ERR_ARG;
  const int quads = H * v8 / 4, es = is_f32 ? 4 : 2;
  for (int r0 = 0; r0 < rows; r0 += 65535) {
    const int n = rows - r0 < 65535 ? rows - r0 : 65535;
    char* x = (char*)a + (size_t)r0 * lda * es;
    const OutputGate G{(const char*)gate + (size_t)r0 * ldg * es, ldg, gate_kind};
    const dim3 grid((quads + 255) / 256, n);
    if (is_f32) latent_gate_kernel<float><<<grid, 256, 0, st>>>((float*)x, lda, G, quads, v8);
    else latent_gate_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((__nv_bfloat16*)x, lda, G, quads, v8);
  }
  return (int)cudaGetLastError();
}

// Decode step of B <= 16 sequences whose queries come through a latent, from split-K planes [query latent padded to 8 | latent padded to 8]: the normalised query
// latent (bf16 [B][ldq]) and, unless cache is null, the cache row of every sequence's current position. Latents of up to 12288.
FT_EXPORT int ft_latent_decode_norms(const float* planes, int splits, int64_t ldp, int64_t plane_stride, int B, int q_rank, int rank, const float* wq, const float* w, float eps,
                                     const int* positions, const int* block_table, int max_blocks, void* cq, int64_t ldq, void* cache, cudaStream_t st) {
  if (B < 1 || B > DEC_TOK || splits < 1 || q_rank < 1 || rank < 1 || ldq < q_rank) return FT_ERR_ARG;
  const size_t smem = sizeof(float) * (size_t)(q_rank > rank ? q_rank : rank);
  if (smem > 48 * 1024) return FT_ERR_TOO_LARGE;
  return (int)ft_launch_pdl(latent_decode_norms_kernel, dim3(B, cache ? 2 : 1), dim3(PREP_THREADS), smem, st, planes, splits, ldp, (size_t)plane_stride,
                            make_dims(1, 1, 0, rank, q_rank), wq, w, eps, positions, block_table, max_blocks, (__nv_bfloat16*)cq, ldq, (__nv_bfloat16*)cache);
}

// Decode step of B <= 16 sequences, from the split-K planes of the fused query / latent projection (column layout as in ft_latent_prep): absorbed and
// rotated queries q [B][H][row] bf16, cache row of every sequence's current position (cache null: the planes hold queries alone). wuk: bf16 [H * d8][ldw], ldw >= rank padded to 16, zeros past rank.
// gate_cols > 0: gate (f32 [B][gate_cols]) gets the sigmoid of the columns behind those.
FT_EXPORT int ft_latent_decode_prep(const float* planes, int splits, int64_t ldp, int64_t plane_stride, int B, int H, int d, int dr, int rank, const void* wuk,
                                    int64_t ldw, const float* w, float eps, const int* positions, const float* cos_t, const float* sin_t, const int* block_table,
                                    int max_blocks, void* q, void* cache, int gate_cols, float* gate, cudaStream_t st) {
  if (B < 1 || B > DEC_TOK || splits < 1 || !dims_ok(H, d, dr, rank) || gate_cols < 0 || (gate_cols && !gate)) return FT_ERR_ARG;
  const LatentDims D = make_dims(H, d, dr, rank);
  if ((ldw & 7) || ldw < D.r16) return FT_ERR_ARG;
  const int slices = (D.r16 + ABS_COLS - 1) / ABS_COLS;
  const size_t absorb = (size_t)d * (ABS_COLS * 2 + DEC_TOK * 4), norm = sizeof(float) * (size_t)rank;
  const size_t smem = absorb > norm ? absorb : norm;
  if (smem > 48 * 1024) return FT_ERR_TOO_LARGE;
  return (int)ft_launch_pdl(latent_decode_prep_kernel, dim3(H * slices + (cache ? B : 0) + B * ((gate_cols + PREP_THREADS - 1) / PREP_THREADS)), dim3(PREP_THREADS), smem, st, planes, splits, ldp, (size_t)plane_stride, D, B,
                            (const __nv_bfloat16*)wuk, ldw, w, eps, positions, cos_t, sin_t, block_table, max_blocks, (__nv_bfloat16*)q, (__nv_bfloat16*)cache, gate_cols,
                            gate);
}

// Attention of one token per sequence over its cached rows (seq_lens[b] rows, the newest included); q as written by ft_latent_decode_prep. Partial
// results go to ws: f32 [B][ceil(H / (16 mt))][nsplit][16 mt][r16 + 4]; mt = 1 or 2 tiles of 16 heads per CTA; nsplit <= 64; latent sizes up to 1024
// (512 with mt = 2).
FT_EXPORT int ft_latent_decode(const void* q, const void* cache, const int* block_table, int max_blocks, const int* seq_lens, int B, int H, int dr, int rank, float scale,
                               int nsplit, int mt, float* ws, cudaStream_t st) {
  if (B < 1 || nsplit < 1 || nsplit > 64 || !dims_ok(H, 1, dr, rank) || (mt != 1 && mt != 2) || (reinterpret_cast<uintptr_t>(ws) & 15)) return FT_ERR_ARG;
  const LatentDims D = make_dims(H, 1, dr, rank);
  const int smem = (mt * 16 + LD_STAGES * LD_CHUNK) * latent_smem_pitch(D.row) + mt * 16 * LD_P_PITCH;
  const int np = (D.r16 / 16 + 7) / 8;
  if (smem > SMEM_MAX - 8192 || np > 8 || (mt == 2 && np > 4)) return FT_ERR_TOO_LARGE;
  const dim3 grid(nsplit, (H + mt * 16 - 1) / (mt * 16), B);
#define FT_LD(M, N) return launch_decode<M, N>(grid, smem, st, q, cache, block_table, max_blocks, seq_lens, D, scale, ws)
  if (mt == 1) {
    if (np <= 1) FT_LD(1, 1);
    if (np <= 2) FT_LD(1, 2);
    if (np <= 4) FT_LD(1, 4);
    FT_LD(1, 8);
  }
  if (np <= 1) FT_LD(2, 1);
  if (np <= 2) FT_LD(2, 2);
  FT_LD(2, 4);
#undef FT_LD
}

// Merges the splits of ft_latent_decode: out [B][H][r16] bf16, normalised.
FT_EXPORT int ft_latent_combine(const float* ws, int B, int H, int rank, int nsplit, int mt, void* out, cudaStream_t st) {
  if (B < 1 || H < 1 || rank < 1 || nsplit < 1 || nsplit > 64 || (mt != 1 && mt != 2)) return FT_ERR_ARG;
  const int HT = mt * 16;
  return (int)ft_launch_pdl(latent_combine_kernel, dim3(H, B), dim3(128), 0, st, ws, H, HT, (H + HT - 1) / HT, nsplit, (rank + 15) & ~15, (__nv_bfloat16*)out);
}

// Query rows of one tile of ft_latent_flash for these head sizes: 256 or 128; 0 when the sizes do not fit the kernel (use ft_latent_rows).
FT_EXPORT int ft_latent_flash_tile(int d, int dr, int dv) {
  const int nq = (d + 63) / 64 + (dr + 63) / 64, nv = (dv + 63) / 64;
  if (nq <= 2 && nv == 1) return 128;                  // two CTAs of one tile per SM
  if (nv <= 2 && flash_smem(2, nq, nv) <= SMEM_MAX) return 256;
  if (nv <= 4 && flash_smem(1, nq, nv) <= SMEM_MAX) return 128;
  return 0;
}

// Causal attention over ragged sequences. q: [q_rows][ldq] with heads of [d padded to 8 | dr padded to 8]; kv: [ctx_rows][ldkv] with H heads of keys (d
// padded to 8), then H heads of values (dv padded to 8); kr: rotated key part, [ctx_rows][ldkr]; out: [q_rows][ldo], heads of dv padded to 8. tiles: int4
// per tile {first query row, rows (<= the tile size), position of the first row, first context row of its sequence}: the row at position p sees context
// rows 0..p of its sequence. dr may be 0 (kr is not read then). gate_kind 1: gate rows (pitch ldg) of H * (dv padded to 8) pre-activations, 2: of H; 0: none. All bf16, leading
// dimensions multiples of 8.
FT_EXPORT int ft_latent_flash(const void* q, int64_t ldq, int q_rows, const void* kv, int64_t ldkv, const void* kr, int64_t ldkr, int ctx_rows, const int* tiles, int ntiles,
                              int H, int d, int dr, int dv, float scale, const void* gate, int64_t ldg, int gate_kind, void* out, int64_t ldo, cudaStream_t st) {
  const OutputGate G{gate, ldg, gate_kind};
  if (gate_kind < 0 || gate_kind > 2 || (gate_kind && !gate) || (gate_kind == GATE_ELEMENT && ((ldg & 7) || (reinterpret_cast<uintptr_t>(gate) & 15)))) return FT_ERR_ARG;
  if (q_rows < 1 || ctx_rows < 1 || ntiles < 1 || H < 1 || H > 65535 || d < 1 || dr < 0 || dv < 1 || (ldq & 7) || (ldkv & 7) || (ldkr & 7) || (ldo & 7)) return FT_ERR_ARG;
  const int tile = ft_latent_flash_tile(d, dr, dv);
  if (tile == 0) return FT_ERR_TOO_LARGE;
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  FT_CUDA_TRY(ft_bind_context(dev));
  const int d8 = (d + 7) & ~7, dr8 = (dr + 7) & ~7, dv8 = (dv + 7) & ~7;
  const uint64_t hq = (uint64_t)(d8 + dr8) * 2;
  CUtensorMap m[5];
  const __nv_bfloat16 *qp = (const __nv_bfloat16*)q, *kp = (const __nv_bfloat16*)kv;
  int r = ft_make_tmap_3d(&m[0], qp, 2, true, d, H, q_rows, hq, (uint64_t)ldq * 2, 64, 1, LF_BM, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r && dr) r = ft_make_tmap_3d(&m[1], qp + d8, 2, true, dr, H, q_rows, hq, (uint64_t)ldq * 2, 64, 1, LF_BM, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[2], kp, 2, true, d, H, ctx_rows, (uint64_t)d8 * 2, (uint64_t)ldkv * 2, 64, 1, LF_BN, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r && dr) r = ft_make_tmap_2d(&m[3], kr, 2, true, dr, ctx_rows, (uint64_t)ldkr * 2, 64, LF_BN, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[4], kp + (size_t)H * d8, 2, true, dv, H, ctx_rows, (uint64_t)dv8 * 2, (uint64_t)ldkv * 2, 64, 1, LF_BN, CU_TENSOR_MAP_SWIZZLE_128B);
  if (r) return r;
  if (!dr) { m[1] = m[0]; m[3] = m[2]; }               // named by the kernel, never read
  const FlashDims F{d, dr, dv, (d + 63) / 64, (dr + 63) / 64, (dv + 63) / 64, dv8};
  const int nq = F.nn + F.nr;
  const int smem = flash_smem(tile / 128, nq, F.nv);
#define FT_LF(T, Q, V) return launch_flash<T, Q, V>(m, tiles, ntiles, H, F, scale, G, out, ldo, smem, st)
  if (tile == 256) {
    if (nq == 2 && F.nv == 2) FT_LF(2, 2, 2);
    if (nq == 3 && F.nv == 1) FT_LF(2, 3, 1);
    if (nq == 3 && F.nv == 2) FT_LF(2, 3, 2);
    FT_LF(2, 0, 0);
  }
  if (nq == 1 && F.nv == 1) FT_LF(1, 1, 1);
  if (nq == 2 && F.nv == 1) FT_LF(1, 2, 1);
  FT_LF(1, 0, 0);
#undef FT_LF
}
