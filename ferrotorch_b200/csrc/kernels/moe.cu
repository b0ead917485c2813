// Mixture of experts: sigmoid router with the top experts per token, experts of the clamped gated form
//   g = min(W_gate x, limit),  u = clamp(W_up x, -limit, limit),  expert(x) = W_down (g sigmoid(slope g) (u + 1)),
// every chosen expert applied to score * x. The projections are linear, so W (score x) = score (W x): the score multiplies the f32 accumulators and
// no scaled copy of the tokens is made (or rounded).
//
// Weights: gate and up rows are interleaved in blocks of eight (eight gate rows, then the eight up rows of the same neurons), so that a warp's 16
// weight rows -- and a thread's accumulators -- hold a neuron's gate and up together, and the tiles of the grouped GEMM hold both as well.
//
// Prefill: router GEMM -> ft_moe_topk (choice, scores, position inside the expert) -> ft_moe_layout (128-row aligned segment per expert, tile
// table) -> ft_moe_gather -> grouped tcgen05 GEMM (gemm_tcgen05.cu) -> ft_moe_act -> grouped GEMM -> picked up by ft_hyper_update.
// Decode (up to 16 tokens): ft_moe_route_small (logits, choice and the list of active experts in one launch), ft_moe_gate_up_small (weight stream ->
// activation), ft_moe_down_small (one f32 plane per expert slot, summed by the kernel that updates the streams); the shared expert rides in the
// same launches.
#include "common.cuh"
#include "host_common.h"
#include "skinny.cuh"

namespace {

constexpr int SMALL_TOK = 16;      // tokens of the decode kernels
constexpr int MAX_TOP = 32;
constexpr int SEG = 128;           // rows per tile of the grouped GEMM

FT_DEVICE float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
FT_DEVICE float gated_clamped(float g, float u, float limit, float slope) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(slope * g) * (u + 1.f);
}

// whole warp: (value, index) of the largest logit that comes after (pv, pi) in the order "value descending, index ascending"
FT_DEVICE void next_best(const float* z, int E, float pv, int pi, float& bv, int& bi) {
  bv = -INFINITY;
  bi = 0x7fffffff;
  for (int e = threadIdx.x & 31; e < E; e += 32) {
    const float v = z[e];
    const bool after = v < pv || (v == pv && e > pi);
    if (after && (v > bv || (v == bv && e < bi))) { bv = v; bi = e; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
  }
}

// one warp per token
__global__ void __launch_bounds__(256) moe_topk_kernel(const float* __restrict__ logits, int64_t ld, int T, int E, int top, int* __restrict__ expert,
                                                       float* __restrict__ score, int* __restrict__ pos, int* __restrict__ count) {
  const int tok = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (tok >= T) return;
  const float* z = logits + (size_t)tok * ld;
  float pv = INFINITY;
  int pi = -1;
  for (int j = 0; j < top; j++) {
    float v;
    int e;
    next_best(z, E, pv, pi, v, e);
    if (e >= E) e = j;                               // only with NaN logits
    if ((threadIdx.x & 31) == 0) {
      expert[(size_t)tok * top + j] = e;
      score[(size_t)tok * top + j] = sigmoid_f(v);
      pos[(size_t)tok * top + j] = atomicAdd(&count[e], 1);
    }
    pv = v;
    pi = e;
  }
}

// one CTA: segment starts (multiples of SEG), group of every SEG-row tile (-1: unused), number of rows in use; count is zeroed for the next launch
__global__ void __launch_bounds__(1024) moe_layout_kernel(int* __restrict__ count, int E, int max_tiles, int* __restrict__ start, int* __restrict__ tile_group,
                                                          int* __restrict__ rows_used) {
  __shared__ int warp_tot[32];
  __shared__ int base_sh;
  if (threadIdx.x == 0) base_sh = 0;
  __syncthreads();
  for (int e0 = 0; e0 < E; e0 += 1024) {
    const int e = e0 + threadIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int tiles = e < E ? (count[e] + SEG - 1) / SEG : 0;
    int inc = tiles;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    if (lane == 31) warp_tot[warp] = inc;
    __syncthreads();
    int before = base_sh;
    for (int w = 0; w < warp; w++) before += warp_tot[w];
    const int first = before + inc - tiles;
    if (e < E) {
      start[e] = first * SEG;
      count[e] = 0;
      for (int i = 0; i < tiles && first + i < max_tiles; i++) tile_group[first + i] = e;
    }
    __syncthreads();
    if (threadIdx.x == 1023) base_sh = before + inc;
    __syncthreads();
  }
  for (int i = base_sh + threadIdx.x; i < max_tiles; i += 1024) tile_group[i] = -1;
  if (threadIdx.x == 0) *rows_used = min(base_sh, max_tiles) * SEG;
}

// one CTA per (token, slot): its row, and a copy of the token there
__global__ void __launch_bounds__(128) moe_gather_kernel(const uint4* __restrict__ h, int64_t ldh16, const int* __restrict__ expert, const float* __restrict__ score,
                                                         const int* __restrict__ pos, const int* __restrict__ start, int top, int vecs, uint4* __restrict__ xs,
                                                         int64_t ldx16, int* __restrict__ row_of, float* __restrict__ row_score) {
  const int pair = blockIdx.x;
  const int row = start[expert[pair]] + pos[pair];
  if (threadIdx.x == 0) { row_of[pair] = row; row_score[row] = score[pair]; }
  const uint4* src = h + (size_t)(pair / top) * ldh16;
  uint4* dst = xs + (size_t)row * ldx16;
  for (int i = threadIdx.x; i < vecs; i += 128) dst[i] = src[i];
}

// gu: [rows][2 * fp] in blocks of eight gate | eight up columns -> act [rows][ld_act]
template <typename T>
__global__ void __launch_bounds__(256) moe_act_kernel(const T* __restrict__ gu, int64_t ld_gu, const float* __restrict__ row_score, const int* __restrict__ rows_used,
                                                      int rows, int fp, float limit, float slope, T* __restrict__ act, int64_t ld_act) {
  const int n = rows_used ? min(rows, *rows_used) : rows;
  const int per_row = fp / 8;
  const size_t total = (size_t)n * per_row;
  for (size_t i = blockIdx.x * (size_t)256 + threadIdx.x; i < total; i += (size_t)gridDim.x * 256) {
    const int r = (int)(i / per_row), blk = (int)(i % per_row);
    const float s = row_score ? row_score[r] : 1.f;
    const T* src = gu + (size_t)r * ld_gu + blk * 16;
    T* dst = act + (size_t)r * ld_act + blk * 8;
    float o[8];
    if constexpr (sizeof(T) == 2) {
      float g[8], u[8];
      bf16x8_to_float(*reinterpret_cast<const bf16x8*>(src), g);
      bf16x8_to_float(*reinterpret_cast<const bf16x8*>(src + 8), u);
#pragma unroll
      for (int e = 0; e < 8; e++) o[e] = gated_clamped(s * g[e], s * u[e], limit, slope);
      *reinterpret_cast<bf16x8*>(dst) = float_to_bf16x8(o);
    } else {
#pragma unroll
      for (int e = 0; e < 8; e++) dst[e] = gated_clamped(s * src[e], s * src[8 + e], limit, slope);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
// Routing of a decode step in device memory: n[0] active experts; id[a], cnt[a] and pair[a][i] = token * top + slot of active expert a;
// score[token * top + slot].
struct SmallRoute {
  int* n;
  int* id;
  int* cnt;
  int* pair;                       // [experts][SMALL_TOK]
  float* score;
};

// grid ceil(E / 8): one warp per expert computes its logit for every token; the last CTA chooses and builds the lists
__global__ void __launch_bounds__(256) moe_route_small_kernel(const __nv_bfloat16* __restrict__ h, int64_t ldh, const __nv_bfloat16* __restrict__ router, int64_t ldr,
                                                              int B, int W, int E, int top, float* __restrict__ logits, int* __restrict__ counter, SmallRoute R) {
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, e = blockIdx.x * 8 + warp;
  if (e < E) {
    const __nv_bfloat16* w = router + (size_t)e * ldr;
    for (int b0 = 0; b0 < B; b0 += 8) {
      float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      for (int k = lane * 8; k < W; k += 256) {
        float wv[8];
        bf16x8_to_float(*reinterpret_cast<const bf16x8*>(w + k), wv);
        const int lim = W - k;
#pragma unroll
        for (int b = 0; b < 8; b++) {
          if (b0 + b < B) {
            float hv[8];
            bf16x8_to_float(*reinterpret_cast<const bf16x8*>(h + (size_t)(b0 + b) * ldh + k), hv);
#pragma unroll
            for (int j = 0; j < 8; j++) acc[b] += j < lim ? wv[j] * hv[j] : 0.f;
          }
        }
      }
#pragma unroll
      for (int b = 0; b < 8; b++) {
        acc[b] = warp_sum(acc[b]);
        if (lane == 0 && b0 + b < B) logits[(size_t)(b0 + b) * E + e] = acc[b];
      }
    }
  }
  __shared__ int is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    is_last = atomicAdd(counter, 1) == (int)gridDim.x - 1;
    if (is_last) *counter = 0;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  __shared__ int chosen[SMALL_TOK * MAX_TOP];
  for (int b = warp; b < B; b += 8) {
    float pv = INFINITY;
    int pi = -1;
    for (int j = 0; j < top; j++) {
      float v;
      int c;
      next_best(logits + (size_t)b * E, E, pv, pi, v, c);
      if (c >= E) c = j;
      if (lane == 0) { chosen[b * top + j] = c; R.score[b * top + j] = sigmoid_f(v); }
      pv = v;
      pi = c;
    }
  }
  __syncthreads();
  if (warp == 0) {                                   // active experts in ascending order
    int n = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int x = e0 + lane;
      int cnt = 0;
      if (x < E)
        for (int p = 0; p < B * top; p++) cnt += chosen[p] == x;
      const unsigned m = __ballot_sync(0xffffffffu, cnt > 0);
      if (cnt > 0) {
        const int a = n + __popc(m & ((1u << lane) - 1));
        R.id[a] = x;
        R.cnt[a] = cnt;
        int i = 0;
        for (int p = 0; p < B * top; p++)
          if (chosen[p] == x && i < SMALL_TOK) R.pair[a * SMALL_TOK + i++] = p;
      }
      n += __popc(m);
    }
    if (lane == 0) *R.n = n;
  }
}

// One side of a decode launch: a stack of experts (or the one shared expert) in the packed layout
struct ExpertSet {
  const __nv_bfloat16* gu;         // [experts][2 * fp][ld_in]
  const __nv_bfloat16* down;       // [experts][rows_out][ld_mid]
  int f, fp;                       // neurons, padded to a multiple of 8
  int64_t ld_in, ld_mid;           // padded to multiples of 32
  float limit;
};

// grid (blocks of 64 neurons, groups + shared), 256 threads: warp w computes 8 neurons (16 interleaved rows) for all tokens; tokens that did not
// choose the expert are computed along (the tensor tile has room for eight) and dropped.
template <int NT>
__global__ void __launch_bounds__(256) moe_gate_up_small_kernel(const __nv_bfloat16* __restrict__ h, int64_t ldh, int B, int W, int top, SmallRoute R, int groups,
                                                                ExpertSet ex, ExpertSet sh, float slope, __nv_bfloat16* __restrict__ act, int64_t ld_act,
                                                                __nv_bfloat16* __restrict__ act_sh, int64_t ld_act_sh, int tok0) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t xs[];
  __shared__ int pair_of[8 * NT];
  __shared__ float sc[8 * NT];
  const int a = blockIdx.y;
  const bool shared_ex = a == groups;
  if (!shared_ex && a >= *R.n) return;
  const ExpertSet& S = shared_ex ? sh : ex;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((int)blockIdx.x * 64 >= S.fp) return;
  const int nb = min(8 * NT, B - tok0), kp = (W + 31) & ~31, pitch = skinny_pitch(kp);
  if (threadIdx.x < 8 * NT) {
    pair_of[threadIdx.x] = shared_ex && (int)threadIdx.x < nb ? tok0 + threadIdx.x : -1;
    sc[threadIdx.x] = 1.f;
  }
  __syncthreads();
  if (!shared_ex && threadIdx.x < R.cnt[a]) {
    const int p = R.pair[a * SMALL_TOK + threadIdx.x], tk = p / top - tok0;
    if (tk >= 0 && tk < 8 * NT) { pair_of[tk] = p; sc[tk] = R.score[p]; }
  }
  for (int n = 0; n < 8 * NT; n++) skinny_fill_row(xs, pitch, n, n < nb ? h + (size_t)(tok0 + n) * ldh : nullptr, W, kp, threadIdx.x, 256);
  __syncthreads();
  const int blk = blockIdx.x * 8 + warp;
  if (blk * 8 >= S.fp) return;
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; n++) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  const __nv_bfloat16* w = S.gu + ((size_t)(shared_ex ? 0 : R.id[a]) * 2 * S.fp + (size_t)blk * 16) * S.ld_in;
  skinny_rows16<NT>(w, S.ld_in, kp, xs, pitch, acc);
  const int f = blk * 8 + (lane >> 2);
  if (f >= S.f) return;
  __nv_bfloat16* dst = shared_ex ? act_sh : act;
  const int64_t ld = shared_ex ? ld_act_sh : ld_act;
#pragma unroll
  for (int n = 0; n < NT; n++)
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int tk = n * 8 + (lane & 3) * 2 + j, p = pair_of[tk];
      if (p >= 0) dst[(size_t)p * ld + f] = __float2bfloat16(gated_clamped(sc[tk] * acc[n][j], sc[tk] * acc[n][2 + j], S.limit, slope));
    }
}

// grid (blocks of 128 output columns, groups + shared), 256 threads: plane `slot` of out gets the expert's contribution to its tokens, plane `top`
// the shared expert's. out: [top + 1][tok_stride][ldo] f32.
template <int NT>
__global__ void __launch_bounds__(256) moe_down_small_kernel(const __nv_bfloat16* __restrict__ act, int64_t ld_act, const __nv_bfloat16* __restrict__ act_sh,
                                                             int64_t ld_act_sh, int B, int W, int top, SmallRoute R, int groups, ExpertSet ex, ExpertSet sh,
                                                             int rows_out, float* __restrict__ out, int64_t plane_stride, int64_t ldo) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t xs[];
  __shared__ int pair_sh[SMALL_TOK];
  const int a = blockIdx.y;
  const bool shared_ex = a == groups;
  if (!shared_ex && a >= *R.n) return;
  const ExpertSet& S = shared_ex ? sh : ex;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cnt = shared_ex ? B : min(R.cnt[a], SMALL_TOK), kp = (S.f + 31) & ~31, pitch = skinny_pitch(kp);
  if (threadIdx.x < SMALL_TOK) pair_sh[threadIdx.x] = (int)threadIdx.x < cnt ? (shared_ex ? (int)threadIdx.x : R.pair[a * SMALL_TOK + threadIdx.x]) : -1;
  __syncthreads();
  const int row0 = blockIdx.x * 128 + warp * 16;
  const __nv_bfloat16* w = S.down + ((size_t)(shared_ex ? 0 : R.id[a]) * rows_out + row0) * S.ld_mid;
  for (int i0 = 0; i0 < cnt; i0 += 8 * NT) {
    if (i0) __syncthreads();
    for (int n = 0; n < 8 * NT; n++) {
      const int p = i0 + n < SMALL_TOK ? pair_sh[i0 + n] : -1;
      const __nv_bfloat16* src = p < 0 ? nullptr : (shared_ex ? act_sh + (size_t)p * ld_act_sh : act + (size_t)p * ld_act);
      skinny_fill_row(xs, pitch, n, src, S.f, kp, threadIdx.x, 256);
    }
    __syncthreads();
    if (row0 >= rows_out) continue;
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; n++) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    skinny_rows16<NT>(w, S.ld_mid, kp, xs, pitch, acc);
#pragma unroll
    for (int n = 0; n < NT; n++)
#pragma unroll
      for (int j = 0; j < 2; j++) {
        const int i = i0 + n * 8 + (lane & 3) * 2 + j;
        const int p = i < SMALL_TOK ? pair_sh[i] : -1;
        if (p < 0) continue;
        float* o = out + (shared_ex ? (size_t)top * plane_stride + (size_t)p * ldo : (size_t)(p % top) * plane_stride + (size_t)(p / top) * ldo);
        const int r = row0 + (lane >> 2);
        if (r < W) o[r] = acc[n][j];
        if (r + 8 < W) o[r + 8] = acc[n][2 + j];
      }
  }
}

// one product of a few tokens per group (group = attention head: latent output -> value): grid (rows / 128, groups)
template <int NT>
__global__ void __launch_bounds__(256) skinny_heads_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx, int64_t head_x, const __nv_bfloat16* __restrict__ w,
                                                           int64_t ldw, int64_t head_w, int B, int N, int K, __nv_bfloat16* __restrict__ out, int64_t ldo,
                                                           int64_t head_o) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t xs[];
  const int hd = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kp = (K + 31) & ~31, pitch = skinny_pitch(kp);
  for (int n = 0; n < 8 * NT; n++) skinny_fill_row(xs, pitch, n, n < B ? x + (size_t)n * ldx + hd * head_x : nullptr, K, kp, threadIdx.x, 256);
  __syncthreads();
  const int row0 = blockIdx.x * 128 + warp * 16;
  if (row0 >= N) return;
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; n++) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  skinny_rows16<NT>(w + (size_t)hd * head_w + (size_t)row0 * ldw, ldw, kp, xs, pitch, acc);
#pragma unroll
  for (int n = 0; n < NT; n++)
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int tk = n * 8 + (lane & 3) * 2 + j;
      if (tk >= B) continue;
      __nv_bfloat16* o = out + (size_t)tk * ldo + hd * head_o;
      const int r = row0 + (lane >> 2);
      if (r < N) o[r] = __float2bfloat16(acc[n][j]);
      if (r + 8 < N) o[r + 8] = __float2bfloat16(acc[n][2 + j]);
    }
}

constexpr int SMALL_SMEM_MAX = 220 * 1024;
template <typename K>
cudaError_t allow_smem(K kernel, bool (&done)[64]) {
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 64 && done[dev]) return cudaSuccess;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMALL_SMEM_MAX);
  if (e == cudaSuccess && dev < 64) done[dev] = true;
  return e;
}

}  // namespace

// Choice of the `top` largest logits per token (ties: lower index first), their sigmoids, and the running position of every (token, slot) inside its
// expert. count: int[E], zero before the launch (ft_moe_layout zeroes it again). expert, score, pos: [T * top].
FT_EXPORT int ft_moe_topk(const float* logits, int64_t ld, int T, int E, int top, int* expert, float* score, int* pos, int* count, cudaStream_t st) {
  if (T < 1 || E < 1 || top < 1 || top > E) return FT_ERR_ARG;
  moe_topk_kernel<<<(T + 7) / 8, 256, 0, st>>>(logits, ld, T, E, top, expert, score, pos, count);
  return (int)cudaGetLastError();
}

// Segment start of every expert (multiples of 128 rows), expert of every 128-row tile (-1 unused), rows in use. max_tiles >= the number of tiles
// that any choice can need (T * top / 128 + min(E, T * top), rounded up).
FT_EXPORT int ft_moe_layout(int* count, int E, int max_tiles, int* start, int* tile_group, int* rows_used, cudaStream_t st) {
  if (E < 1 || max_tiles < 1) return FT_ERR_ARG;
  moe_layout_kernel<<<1, 1024, 0, st>>>(count, E, max_tiles, start, tile_group, rows_used);
  return (int)cudaGetLastError();
}

// Copies token rows into the expert segments: xs[row_of[pair]] = h[pair / top] (row_bytes, both pitches multiples of 16 bytes); row_of [T * top] and
// row_score [rows of xs] are written along.
FT_EXPORT int ft_moe_gather(const void* h, int64_t ldh_bytes, const int* expert, const float* score, const int* pos, const int* start, int T, int top, int row_bytes,
                            void* xs, int64_t ldx_bytes, int* row_of, float* row_score, cudaStream_t st) {
  if (T < 1 || top < 1 || (ldh_bytes & 15) || (ldx_bytes & 15) || (row_bytes & 15) || row_bytes > ldh_bytes || row_bytes > ldx_bytes) return FT_ERR_ARG;
  moe_gather_kernel<<<T * top, 128, 0, st>>>((const uint4*)h, ldh_bytes / 16, expert, score, pos, start, top, row_bytes / 16, (uint4*)xs, ldx_bytes / 16, row_of,
                                             row_score);
  return (int)cudaGetLastError();
}

// act[r][f] = g sigmoid(slope g) (u + 1) with g = min(s gate, limit), u = clamp(s up, -limit, limit), s = row_score[r] (1 when null). gu: columns in
// blocks of eight gate, eight up (2 * fp columns); dtype bf16 or (is_f32) f32. rows_used: device int bounding the rows, or null.
FT_EXPORT int ft_moe_act(const void* gu, int64_t ld_gu, const float* row_score, const int* rows_used, int rows, int fp, float limit, float slope, void* act,
                         int64_t ld_act, int is_f32, cudaStream_t st) {
  if (rows < 1 || fp < 8 || (fp & 7) || (ld_gu & 7) || (ld_act & 7) || ld_gu < 2 * fp || ld_act < fp) return FT_ERR_ARG;
  const size_t work = ((size_t)rows * (fp / 8) + 255) / 256;
  const int grid = (int)(work > 148 * 16 ? 148 * 16 : work);
  if (is_f32) moe_act_kernel<float><<<grid, 256, 0, st>>>((const float*)gu, ld_gu, row_score, rows_used, rows, fp, limit, slope, (float*)act, ld_act);
  else moe_act_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((const __nv_bfloat16*)gu, ld_gu, row_score, rows_used, rows, fp, limit, slope, (__nv_bfloat16*)act, ld_act);
  return (int)cudaGetLastError();
}

// Decode routing (B <= 16 tokens, bf16 operands, f32 accumulation): logits [B][E] f32 scratch, counter int zero before the first launch. Outputs:
// n_active int[1], id int[E], cnt int[E], pair int[E][16], score f32 [B * top].
FT_EXPORT int ft_moe_route_small(const void* h, int64_t ldh, const void* router, int64_t ldr, int B, int W, int E, int top, float* logits, int* counter, int* n_active,
                                 int* id, int* cnt, int* pair, float* score, cudaStream_t st) {
  if (B < 1 || B > SMALL_TOK || E < 1 || top < 1 || top > E || top > MAX_TOP || (ldh & 7) || (ldr & 7)) return FT_ERR_ARG;
  return (int)ft_launch_pdl(moe_route_small_kernel, dim3((E + 7) / 8), dim3(256), 0, st, (const __nv_bfloat16*)h, ldh, (const __nv_bfloat16*)router, ldr, B, W, E, top,
                            logits, counter, SmallRoute{n_active, id, cnt, pair, score});
}

// Gate / up projections and activation of a decode step. gu: [E][2 * fp][ld_in] interleaved rows, ld_in >= W rounded up to 32; act: bf16 [B * top][ld_act],
// row = token * top + slot. Shared expert (shared_gu null: none): act_sh bf16 [B][ld_act_sh]. fp and fp_sh are the neuron counts rounded up to 8.
FT_EXPORT int ft_moe_gate_up_small(const void* h, int64_t ldh, int B, int W, int E, int top, int* n_active, int* id, int* cnt, int* pair, float* score, const void* gu,
                                   int f, int64_t ld_in, float limit, const void* shared_gu, int f_sh, int64_t ld_in_sh, float limit_sh, float slope, void* act,
                                   int64_t ld_act, void* act_sh, int64_t ld_act_sh, cudaStream_t st) {
  const int kp = (W + 31) & ~31;
  if (B < 1 || B > SMALL_TOK || f < 1 || (ldh & 7) || (ld_in & 7) || ld_in < kp || ld_act < f || (shared_gu && ((ld_in_sh & 7) || ld_in_sh < kp || ld_act_sh < f_sh)))
    return FT_ERR_ARG;
  const SmallRoute R{n_active, id, cnt, pair, score};
  const ExpertSet ex{(const __nv_bfloat16*)gu, nullptr, f, (f + 7) & ~7, ld_in, 0, limit};
  const ExpertSet sh{(const __nv_bfloat16*)shared_gu, nullptr, f_sh, (f_sh + 7) & ~7, ld_in_sh, 0, limit_sh};
  const int groups = E < B * top ? E : B * top, fmax = shared_gu && sh.fp > ex.fp ? sh.fp : ex.fp;
  const dim3 grid((fmax + 63) / 64, groups + (shared_gu ? 1 : 0));
  const int pitch = skinny_pitch(kp);
  static bool done1[64] = {}, done2[64] = {};
  if (B > 8 && 16 * pitch <= SMALL_SMEM_MAX) {
    FT_CUDA_TRY(allow_smem(moe_gate_up_small_kernel<2>, done2));
    return (int)ft_launch_pdl(moe_gate_up_small_kernel<2>, grid, dim3(256), (size_t)16 * pitch, st, (const __nv_bfloat16*)h, ldh, B, W, top, R, groups, ex, sh, slope,
                              (__nv_bfloat16*)act, ld_act, (__nv_bfloat16*)act_sh, ld_act_sh, 0);
  }
  if (8 * pitch > SMALL_SMEM_MAX) return FT_ERR_TOO_LARGE;
  FT_CUDA_TRY(allow_smem(moe_gate_up_small_kernel<1>, done1));
  for (int t0 = 0; t0 < B; t0 += 8) {
    const cudaError_t e = ft_launch_pdl(moe_gate_up_small_kernel<1>, grid, dim3(256), (size_t)8 * pitch, st, (const __nv_bfloat16*)h, ldh, B, W, top, R, groups, ex, sh,
                                        slope, (__nv_bfloat16*)act, ld_act, (__nv_bfloat16*)act_sh, ld_act_sh, t0);
    if (e != cudaSuccess) return (int)e;
  }
  return FT_OK;
}

// Down projections of a decode step: out[slot][token][W] f32 (plane_stride, ldo in elements), the shared expert in plane `top`. down: [E][rows_out][ld_mid]
// with rows_out >= W a multiple of 16 and ld_mid >= f rounded up to 32 (zeros past f).
FT_EXPORT int ft_moe_down_small(const void* act, int64_t ld_act, const void* act_sh, int64_t ld_act_sh, int B, int W, int E, int top, int* n_active, int* id, int* cnt,
                                int* pair, float* score, const void* down, int f, int64_t ld_mid, const void* shared_down, int f_sh, int64_t ld_mid_sh, int rows_out,
                                float* out, int64_t plane_stride, int64_t ldo, cudaStream_t st) {
  if (B < 1 || B > SMALL_TOK || f < 1 || (rows_out & 15) || rows_out < W || (ld_act & 7) || ld_mid < ((f + 31) & ~31) || (ld_mid & 7) ||
      (shared_down && ((ld_act_sh & 7) || (ld_mid_sh & 7) || ld_mid_sh < ((f_sh + 31) & ~31))))
    return FT_ERR_ARG;
  const SmallRoute R{n_active, id, cnt, pair, score};
  const ExpertSet ex{nullptr, (const __nv_bfloat16*)down, f, (f + 7) & ~7, 0, ld_mid, 0.f};
  const ExpertSet sh{nullptr, (const __nv_bfloat16*)shared_down, f_sh, (f_sh + 7) & ~7, 0, ld_mid_sh, 0.f};
  const int groups = E < B * top ? E : B * top;
  const int kmax = ((shared_down && f_sh > f ? f_sh : f) + 31) & ~31;
  int smem = 8 * skinny_pitch(kmax);
  if (smem > SMALL_SMEM_MAX) return FT_ERR_TOO_LARGE;
  const dim3 grid((W + 127) / 128, groups + (shared_down ? 1 : 0));
  static bool done1[64] = {}, done2[64] = {};
  if (B > 8 && 2 * smem + 128 <= SMALL_SMEM_MAX) {
    FT_CUDA_TRY(allow_smem(moe_down_small_kernel<2>, done2));
    return (int)ft_launch_pdl(moe_down_small_kernel<2>, grid, dim3(256), (size_t)2 * smem + 128, st, (const __nv_bfloat16*)act, ld_act, (const __nv_bfloat16*)act_sh,
                              ld_act_sh, B, W, top, R, groups, ex, sh, rows_out, out, plane_stride, ldo);
  }
  FT_CUDA_TRY(allow_smem(moe_down_small_kernel<1>, done1));
  return (int)ft_launch_pdl(moe_down_small_kernel<1>, grid, dim3(256), (size_t)smem + 64, st, (const __nv_bfloat16*)act, ld_act, (const __nv_bfloat16*)act_sh, ld_act_sh,
                            B, W, top, R, groups, ex, sh, rows_out, out, plane_stride, ldo);
}

// out[b][head][n] = sum_k w[head][n][k] x[b][head][k] for B <= 16 tokens: x bf16 (ldx between tokens, head_x between heads, 16-byte aligned), w bf16 rows of
// ldw >= K rounded up to 32 elements with head_w elements between heads (16-row blocks are read whole: the buffer extends past the last head's rows
// to the next multiple of 16), out bf16.
FT_EXPORT int ft_skinny_heads(const void* x, int64_t ldx, int64_t head_x, const void* w, int64_t ldw, int64_t head_w, int B, int heads, int N, int K, void* out,
                              int64_t ldo, int64_t head_o, cudaStream_t st) {
  const int kp = (K + 31) & ~31, pitch = skinny_pitch(kp);
  if (B < 1 || B > SMALL_TOK || heads < 1 || N < 1 || K < 1 || (ldx & 7) || (head_x & 7) || (ldw & 7) || ldw < kp || (head_w & 7)) return FT_ERR_ARG;
  static bool done1[64] = {}, done2[64] = {};
  const dim3 grid((N + 127) / 128, heads);
  if (B > 8) {
    if (16 * pitch > SMALL_SMEM_MAX) return FT_ERR_TOO_LARGE;
    FT_CUDA_TRY(allow_smem(skinny_heads_kernel<2>, done2));
    return (int)ft_launch_pdl(skinny_heads_kernel<2>, grid, dim3(256), (size_t)16 * pitch, st, (const __nv_bfloat16*)x, ldx, head_x, (const __nv_bfloat16*)w, ldw, head_w,
                              B, N, K, (__nv_bfloat16*)out, ldo, head_o);
  }
  if (8 * pitch > SMALL_SMEM_MAX) return FT_ERR_TOO_LARGE;
  FT_CUDA_TRY(allow_smem(skinny_heads_kernel<1>, done1));
  return (int)ft_launch_pdl(skinny_heads_kernel<1>, grid, dim3(256), (size_t)8 * pitch, st, (const __nv_bfloat16*)x, ldx, head_x, (const __nv_bfloat16*)w, ldw, head_w, B,
                            N, K, (__nv_bfloat16*)out, ldo, head_o);
}
