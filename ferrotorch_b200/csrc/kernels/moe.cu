// Mixture of experts: sigmoid router with the top experts per token, and experts of two forms.
//   clamped   g = min(W_gate x, limit),  u = clamp(W_up x, -limit, limit),  expert(x) = W_down (g sigmoid(slope g) (u + 1)), applied to score * x: the
//             projections are linear, so W (score x) = score (W x), and the score multiplies the f32 accumulators: no scaled copy of the tokens is made (or rounded)
//   silu      expert(x) = score W_down (g sigmoid(g) u): the score multiplies the activation, in f32, ahead of the down projection
// The router takes the largest logits, weighted with their sigmoids, or (RouteRule) the largest sums of sigmoid and a per-expert correction, or of logit and bias, among the
// experts of the best groups, with weights that are normed to a given sum.
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

// the same on the fast exponential and division, for results that are rounded to bf16
FT_DEVICE float gated_clamped_fast(float g, float u, float limit, float slope) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g * (u + 1.f), 1.f + __expf(-slope * g));
}
enum { EXPERT_CLAMPED = 0, EXPERT_SILU = 1 };
template <bool FAST> FT_DEVICE float expert_act(int kind, float k, float g, float u, float limit, float slope) {
  if (kind == EXPERT_SILU) return FAST ? k * u * (g / (1.f + __expf(-g))) : k * u * (g * sigmoid_f(g));
  return FAST ? gated_clamped_fast(k * g, k * u, limit, slope) : gated_clamped(k * g, k * u, limit, slope);
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

// How a router chooses: by logit, weights are the sigmoids (ROUTE_SIGMOID); or by a choice score within the `keep` groups (of neighbours) whose two best experts have the
// largest sum (groups 0: all experts), weights normed to the sum `scale`: sigmoid(logit) + vector, weights proportional to the chosen sigmoids (ROUTE_CORRECTED); logit +
// vector, weights proportional to the exponentials of the chosen scores (ROUTE_SOFTMAX).
enum { ROUTE_SIGMOID = 0, ROUTE_CORRECTED = 1, ROUTE_SOFTMAX = 2 };
struct RouteRule {
  int kind;
  const float* vector;
  int groups, keep;
  float scale;
};
constexpr float WEIGHT_SUM_EPS = 1e-20f;
constexpr int MAX_GROUPS = 256;

// whole warp: ch[e] = choice score of expert e, minus infinity outside the best groups. gs: [groups] scratch
FT_DEVICE void choice_scores(const float* z, float* ch, int E, const RouteRule& rule, float* gs) {
  const int lane = threadIdx.x & 31;
  for (int e = lane; e < E; e += 32) ch[e] = (rule.kind == ROUTE_SOFTMAX ? __ldcg(z + e) : sigmoid_f(__ldcg(z + e))) + rule.vector[e];
  __syncwarp();
  if (rule.groups == 0) return;
  const int size = E / rule.groups;
  for (int g = lane; g < rule.groups; g += 32) {
    float a = -INFINITY, b = -INFINITY;              // the two largest
    for (int i = 0; i < size; i++) {
      const float v = ch[g * size + i];
      b = fmaxf(b, fminf(a, v));
      a = fmaxf(a, v);
    }
    gs[g] = size > 1 ? a + b : a;
  }
  __syncwarp();
  float pv = INFINITY;
  int pi = -1;
  for (int k = 0; k < rule.keep; k++) {              // the last group that stays, in the order "score descending, index ascending"
    float v;
    int g;
    next_best(gs, rule.groups, pv, pi, v, g);
    pv = v;
    pi = g;
  }
  for (int e = lane; e < E; e += 32) {
    const int g = e / size;
    if (gs[g] < pv || (gs[g] == pv && g > pi)) ch[e] = -INFINITY;
  }
  __syncwarp();
}
// whole warp: the `top` best of ch in order, take(slot, expert, its weight before norming) on every lane; a ruled router's normed weights follow, lane j with
// take(-1 - j, 0, weight)
template <typename Take>
FT_DEVICE void choose(const float* z, const float* ch, int E, int top, const RouteRule& rule, Take take) {
  float pv = INFINITY, sum = 0.f, best = 0.f;
  int pi = -1;
  const bool ruled = rule.kind != ROUTE_SIGMOID;
  float mine = 0.f;                                  // lane j keeps the weight of slot j (of a ruled router: top <= 32)
  for (int j = 0; j < top; j++) {
    float v;
    int e;
    next_best(ch, E, pv, pi, v, e);
    if (e >= E) e = j;                               // only with NaN logits
    if (j == 0) best = v;
    const float s = rule.kind == ROUTE_SOFTMAX ? expf(v - best) : sigmoid_f(ruled ? __ldcg(z + e) : v);
    sum += s;
    if ((threadIdx.x & 31) == j) mine = s;
    take(j, e, s);
    pv = v;
    pi = e;
  }
  if (ruled) {
    const float k = rule.scale / (sum + WEIGHT_SUM_EPS);
    if ((int)(threadIdx.x & 31) < top) take(-1 - (int)(threadIdx.x & 31), 0, mine * k);
  }
}

// one warp per token; dynamic shared memory (ruled routers): [8][E + groups]
__global__ void __launch_bounds__(256) moe_topk_kernel(const float* __restrict__ logits, int64_t ld, int T, int E, int top, RouteRule rule, int* __restrict__ expert,
                                                       float* __restrict__ score, int* __restrict__ pos, int* __restrict__ count) {
  extern __shared__ float choice_sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tok = blockIdx.x * 8 + warp;
  if (tok >= T) return;
  const float* z = logits + (size_t)tok * ld;
  float* ch = choice_sh + (size_t)warp * (E + rule.groups);
  const bool ruled = rule.kind != ROUTE_SIGMOID;
  if (ruled) choice_scores(z, ch, E, rule, ch + E);
  const size_t at = (size_t)tok * top;
  choose(z, ruled ? ch : z, E, top, rule, [&](int j, int e, float s) {
    if (j < 0) {                                     // final weights, a lane each
      score[at - 1 - j] = s;
    } else if (lane == 0) {
      expert[at + j] = e;
      if (!ruled) score[at + j] = s;
      pos[at + j] = atomicAdd(&count[e], 1);
    }
  });
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

// gu: [rows][2 * fp] in blocks of eight gate | eight up columns -> act [rows][ld_act]. grid (column blocks, row groups). bf16: neighbouring lanes load the
// gate and the up half of a block (16 bytes each, a warp reads 512 contiguous bytes) and swap halves, so each ends up with four neurons.
template <typename T>
__global__ void __launch_bounds__(256) moe_act_kernel(const T* __restrict__ gu, int64_t ld_gu, const float* __restrict__ row_score, const int* __restrict__ rows_used,
                                                      int rows, int fp, int kind, float limit, float slope, T* __restrict__ act, int64_t ld_act) {
  const int n = rows_used ? min(rows, *rows_used) : rows;
  const int unit = blockIdx.x * blockDim.x + threadIdx.x, units = fp / 4;
  if constexpr (sizeof(T) == 2) {
    constexpr int RU = 4;                              // rows in flight
    const bool live = unit < units;
    const int u = live ? unit : units - 2 + (unit & 1);
    const bool odd = unit & 1;
    for (int r0 = blockIdx.y; r0 < n; r0 += gridDim.y * RU) {
      uint4 v[RU];
      float sc[RU];
#pragma unroll
      for (int i = 0; i < RU; i++) {
        const int r = min(r0 + i * (int)gridDim.y, n - 1);
        v[i] = *reinterpret_cast<const uint4*>(gu + (size_t)r * ld_gu + u * 8);
        sc[i] = row_score ? row_score[r] : 1.f;
      }
#pragma unroll
      for (int i = 0; i < RU; i++) {
        const int r = r0 + i * (int)gridDim.y;
        // even lane: gate 0..3 kept, up 0..3 received; odd lane: gate 4..7 received, up 4..7 kept
        const uint32_t m0 = __shfl_xor_sync(0xffffffffu, odd ? v[i].x : v[i].z, 1), m1 = __shfl_xor_sync(0xffffffffu, odd ? v[i].y : v[i].w, 1);
        const uint32_t g0 = odd ? m0 : v[i].x, g1 = odd ? m1 : v[i].y, u0 = odd ? v[i].z : m0, u1 = odd ? v[i].w : m1;
        const float2 ga = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g0)), gb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&g1));
        const float2 ua = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u0)), ub = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u1));
        const float k = sc[i];
        __nv_bfloat162 o0 = __floats2bfloat162_rn(expert_act<true>(kind, k, ga.x, ua.x, limit, slope), expert_act<true>(kind, k, ga.y, ua.y, limit, slope));
        __nv_bfloat162 o1 = __floats2bfloat162_rn(expert_act<true>(kind, k, gb.x, ub.x, limit, slope), expert_act<true>(kind, k, gb.y, ub.y, limit, slope));
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&o0);
        pk.y = *reinterpret_cast<uint32_t*>(&o1);
        if (live && r < n) *reinterpret_cast<uint2*>(act + (size_t)r * ld_act + unit * 4) = pk;
      }
    }
  } else {
    if (unit >= units) return;
    for (int r = blockIdx.y; r < n; r += gridDim.y) {
      const float s = row_score ? row_score[r] : 1.f;
      const T* src = gu + (size_t)r * ld_gu + (unit / 2) * 16 + (unit % 2) * 4;
#pragma unroll
      for (int e = 0; e < 4; e++) act[(size_t)r * ld_act + unit * 4 + e] = expert_act<false>(kind, s, src[e], src[8 + e], limit, slope);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
// Routing of a decode step in device memory: n[0] active experts; id[a], cnt[a], pair[a][i] = token * top + slot of active expert a in token order, and
// pair_of[a][token] (-1: the token did not choose it); score[token * top + slot].
struct SmallRoute {
  int* n;
  int* id;
  int* cnt;
  int* pair;                       // [experts][SMALL_TOK]
  int* pair_of;                    // [experts][SMALL_TOK]
  float* score;
};

constexpr int ROUTE_LOGITS = 8192;   // logits of the choosing CTA that fit its shared memory

// grid E: one CTA per expert computes its logit for every token; the last CTA chooses and builds the lists. logits: [16][E], and [16][E] more of scratch behind them
__global__ void __launch_bounds__(128) moe_route_small_kernel(const __nv_bfloat16* __restrict__ h, int64_t ldh, const __nv_bfloat16* __restrict__ router, int64_t ldr,
                                                              int B, int W, int E, int top, RouteRule rule, float* __restrict__ logits, int* __restrict__ counter,
                                                              SmallRoute R) {
  pdl_wait();
  pdl_launch_dependents();
  __shared__ float part[4][SMALL_TOK];
  __shared__ float zs[ROUTE_LOGITS];
  __shared__ float gs[4][MAX_GROUPS];
  __shared__ int chosen[SMALL_TOK * MAX_TOP];
  __shared__ int is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, e = blockIdx.x;
  const __nv_bfloat16* w = router + (size_t)e * ldr;
  for (int b0 = 0; b0 < B; b0 += 8) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int k = threadIdx.x * 8; k < W; k += 1024) {
      float wv[8];
      const bf16x8 wr = *reinterpret_cast<const bf16x8*>(w + k);
      bf16x8 hr[8];
#pragma unroll
      for (int b = 0; b < 8; b++) hr[b] = *reinterpret_cast<const bf16x8*>(h + (size_t)min(b0 + b, B - 1) * ldh + k);
      bf16x8_to_float(wr, wv);
      const int lim = W - k;
#pragma unroll
      for (int b = 0; b < 8; b++) {
        float hv[8];
        bf16x8_to_float(hr[b], hv);
#pragma unroll
        for (int j = 0; j < 8; j++) acc[b] += j < lim ? wv[j] * hv[j] : 0.f;
      }
    }
#pragma unroll
    for (int b = 0; b < 8; b++) {
      acc[b] = warp_sum(acc[b]);
      if (lane == 0) part[warp][b0 + b] = acc[b];
    }
  }
  __syncthreads();
  if (threadIdx.x < B) logits[(size_t)threadIdx.x * E + e] = (part[0][threadIdx.x] + part[1][threadIdx.x]) + (part[2][threadIdx.x] + part[3][threadIdx.x]);
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    is_last = atomicAdd(counter, 1) == (int)gridDim.x - 1;
    if (is_last) *counter = 0;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  const bool staged = B * E <= ROUTE_LOGITS, ruled = rule.kind != ROUTE_SIGMOID;
  if (staged && !ruled) {
    for (int i = threadIdx.x; i < B * E; i += 128) zs[i] = __ldcg(logits + i);
    __syncthreads();
  }
  for (int b = warp; b < B; b += 4) {
    const float* z = logits + (size_t)b * E;
    float* ch = staged ? zs + (size_t)b * E : logits + (size_t)SMALL_TOK * E + (size_t)b * E;
    if (ruled) choice_scores(z, ch, E, rule, gs[warp]);
    choose(z, ruled || staged ? ch : z, E, top, rule, [&](int j, int c, float s) {
      if (j < 0) {
        R.score[b * top - 1 - j] = s;
      } else if (lane == 0) {
        chosen[b * top + j] = c;
        if (!ruled) R.score[b * top + j] = s;
      }
    });
  }
  __syncthreads();
  // active experts in ascending order; thread t of a round looks at expert e0 + t
  __shared__ int warp_n[4];
  int base = 0;
  for (int e0 = 0; e0 < E; e0 += 128) {
    const int x = e0 + threadIdx.x;
    int cnt = 0;
    if (x < E)
      for (int q = 0; q < B * top; q++) cnt += chosen[q] == x;
    const unsigned m = __ballot_sync(0xffffffffu, cnt > 0);
    if (lane == 0) warp_n[warp] = __popc(m);
    __syncthreads();
    int a = base + __popc(m & ((1u << lane) - 1u));
    for (int i = 0; i < warp; i++) a += warp_n[i];
    if (cnt > 0) {
      R.id[a] = x;
      R.cnt[a] = min(cnt, SMALL_TOK);
      int i = 0;
      for (int b = 0; b < B; b++) {
        int mine = -1;
        for (int j = 0; j < top; j++)
          if (chosen[b * top + j] == x) mine = b * top + j;
        R.pair_of[a * SMALL_TOK + b] = mine;
        if (mine >= 0) R.pair[a * SMALL_TOK + i++] = mine;
      }
    }
    base += (warp_n[0] + warp_n[1]) + (warp_n[2] + warp_n[3]);
    __syncthreads();
  }
  if (threadIdx.x == 0) *R.n = base;
}

// One side of a decode launch: a stack of experts (or the one shared expert) in the packed layout
struct ExpertSet {
  const __nv_bfloat16* w;          // gate / up: [experts][2 * fp][ld] interleaved; down: [experts][rows][ld]
  int f, fp;                       // neurons, padded to a multiple of 8
  int64_t ld, stride;              // row pitch, elements between experts
  float limit;
};

// Gate and up rows of eight neurons per item; all tokens are multiplied (the tensor tile has room for eight), those that chose the expert kept. Groups:
// the active experts, then the shared one.
struct GateUpWork {
  const __nv_bfloat16* h;
  int64_t ldh;
  int B, W, tok0;
  SmallRoute R;
  ExpertSet ex, sh;
  int has_shared, kind;
  float slope;
  __nv_bfloat16 *act, *act_sh;
  int64_t ld_act, ld_act_sh;

  FT_DEVICE SkinnyShape shape() const { return SkinnyShape{{*R.n, has_shared}, {ex.fp / 8, has_shared ? sh.fp / 8 : 1}, {1, 1}}; }
  FT_DEVICE bool shared(int g) const { return has_shared && g == *R.n; }
  FT_DEVICE int K(int) const { return W; }
  FT_DEVICE int64_t ldw(int g) const { return shared(g) ? sh.ld : ex.ld; }
  FT_DEVICE const __nv_bfloat16* w(int g, int blk) const {
    return shared(g) ? sh.w + (size_t)blk * 16 * sh.ld : ex.w + (size_t)R.id[g] * ex.stride + (size_t)blk * 16 * ex.ld;
  }
  FT_DEVICE int x_id(int) const { return 0; }
  FT_DEVICE const __nv_bfloat16* x_row(int, int n) const { return tok0 + n < B ? h + (size_t)(tok0 + n) * ldh : nullptr; }
  FT_DEVICE void finish(int g, int blk, int nt, float4 c, int lane) const {
    const bool s = shared(g);
    const ExpertSet& S = s ? sh : ex;
    const int f = blk * 8 + (lane >> 2), tk = tok0 + nt * 8 + (lane & 3) * 2;
    if (f >= S.f) return;
#pragma unroll
    for (int j = 0; j < 2; j++) {
      if (tk + j >= B) break;
      const int pr = s ? tk + j : R.pair_of[g * SMALL_TOK + tk + j];
      if (pr < 0) continue;
      const float k = s ? 1.f : R.score[pr];
      (s ? act_sh + (size_t)pr * ld_act_sh : act + (size_t)pr * ld_act)[f] =
          __float2bfloat16(expert_act<true>(kind, k, j ? c.y : c.x, j ? c.w : c.z, S.limit, slope));
    }
  }
};

// Sixteen output columns per item, the expert's own tokens as columns: plane `slot` of out gets its contribution, plane `top` the shared expert's.
struct DownWork {
  const __nv_bfloat16 *act, *act_sh;
  int64_t ld_act, ld_act_sh;
  int B, W, top, col0;
  SmallRoute R;
  ExpertSet ex, sh;
  int has_shared, blocks;
  float* out;
  int64_t plane_stride, ldo;

  FT_DEVICE SkinnyShape shape() const { return SkinnyShape{{*R.n, has_shared}, {blocks, blocks}, {(ex.f + 31) >> 5, has_shared ? (sh.f + 31) >> 5 : 1}}; }
  FT_DEVICE bool shared(int g) const { return has_shared && g == *R.n; }
  FT_DEVICE int K(int g) const { return shared(g) ? sh.f : ex.f; }
  FT_DEVICE int64_t ldw(int g) const { return shared(g) ? sh.ld : ex.ld; }
  FT_DEVICE const __nv_bfloat16* w(int g, int blk) const {
    return shared(g) ? sh.w + (size_t)blk * 16 * sh.ld : ex.w + (size_t)R.id[g] * ex.stride + (size_t)blk * 16 * ex.ld;
  }
  FT_DEVICE int x_id(int g) const { return g; }
  FT_DEVICE int pair(int g, int n) const {
    if (shared(g)) return n < B ? n : -1;
    return n < SMALL_TOK && n < R.cnt[g] ? R.pair[g * SMALL_TOK + n] : -1;
  }
  FT_DEVICE const __nv_bfloat16* x_row(int g, int n) const {
    const int pr = pair(g, col0 + n);
    return pr < 0 ? nullptr : (shared(g) ? act_sh + (size_t)pr * ld_act_sh : act + (size_t)pr * ld_act);
  }
  FT_DEVICE void finish(int g, int blk, int nt, float4 c, int lane) const {
    const bool s = shared(g);
    const int r = blk * 16 + (lane >> 2), i = col0 + nt * 8 + (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int pr = pair(g, i + j);
      if (pr < 0) continue;
      float* o = out + (s ? (size_t)top * plane_stride + (size_t)pr * ldo : (size_t)(pr % top) * plane_stride + (size_t)(pr / top) * ldo);
      if (r < W) o[r] = j ? c.y : c.x;
      if (r + 8 < W) o[r + 8] = j ? c.w : c.z;
    }
  }
};

// One matrix per group with the same tokens in every group (attention heads: latent output -> value)
struct HeadsWork {
  const __nv_bfloat16 *x, *weights;
  int64_t ldx, head_x, ld, head_w;
  int B, heads, N, Kin;
  __nv_bfloat16* out;
  int64_t ldo, head_o;
  const float* gate;                 // factors [token][ldg] or null: head_g columns between heads, elem_g (0 or 1) between a head's outputs
  int64_t ldg;
  int head_g, elem_g;

  FT_DEVICE SkinnyShape shape() const { return SkinnyShape{{heads, 0}, {(N + 15) / 16, 1}, {1, 1}}; }
  FT_DEVICE int K(int) const { return Kin; }
  FT_DEVICE int64_t ldw(int) const { return ld; }
  FT_DEVICE const __nv_bfloat16* w(int g, int blk) const { return weights + (size_t)g * head_w + (size_t)blk * 16 * ld; }
  FT_DEVICE int x_id(int g) const { return g; }
  FT_DEVICE const __nv_bfloat16* x_row(int g, int n) const { return n < B ? x + (size_t)n * ldx + (size_t)g * head_x : nullptr; }
  FT_DEVICE void finish(int g, int blk, int nt, float4 c, int lane) const {
    const int r = blk * 16 + (lane >> 2), tk = nt * 8 + (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < 2; j++) {
      if (tk + j >= B) break;
      __nv_bfloat16* o = out + (size_t)(tk + j) * ldo + (size_t)g * head_o;
      const float* f = gate ? gate + (size_t)(tk + j) * ldg + (size_t)g * head_g : nullptr;
      if (r < N) o[r] = __float2bfloat16((j ? c.y : c.x) * (f ? f[r * elem_g] : 1.f));
      if (r + 8 < N) o[r + 8] = __float2bfloat16((j ? c.w : c.z) * (f ? f[(r + 8) * elem_g] : 1.f));
    }
  }
};

bool rule_ok(const RouteRule& r, int E, int top) {
  if (r.kind < ROUTE_SIGMOID || r.kind > ROUTE_SOFTMAX || (r.kind != ROUTE_SIGMOID) != (r.vector != nullptr)) return false;
  if (r.kind == ROUTE_SIGMOID) return r.groups == 0;
  if (r.groups < 0 || r.groups > MAX_GROUPS || top > 32) return false;
  return r.groups == 0 || (E % r.groups == 0 && r.keep >= 1 && r.keep <= r.groups && top <= r.keep * (E / r.groups));
}
bool skinny_fits(int nt, int kmax) { return 8 * nt * skinny_pitch((kmax + 31) & ~31) + 64 <= SKINNY_SMEM_MAX; }

}  // namespace

// Choice of the `top` largest logits per token (ties: lower index first), their sigmoids, and the running position of every (token, slot) inside its
// expert. count: int[E], zero before the launch (ft_moe_layout zeroes it again). expert, score, pos: [T * top]. rule 1 with a vector (f32[E]): the choice goes by sigmoid +
// vector, within the `keep` best of `groups` equal groups of neighbours (0: no groups; a group counts its two best), and the scores are the chosen sigmoids
// divided by their sum, times scale (top up to 32, groups up to 256); rule 2: by logit + vector, and the scores are the softmax over the chosen, times scale.
FT_EXPORT int ft_moe_topk(const float* logits, int64_t ld, int T, int E, int top, int rule_kind, const float* vector, int groups, int keep, float scale, int* expert, float* score,
                          int* pos, int* count, cudaStream_t st) {
  const RouteRule rule{rule_kind, vector, groups, keep, scale};
  if (T < 1 || E < 1 || top < 1 || top > E || !rule_ok(rule, E, top)) return FT_ERR_ARG;
  const size_t smem = rule_kind ? (size_t)8 * (E + groups) * 4 : 0;
  if (smem > 200 * 1024) return FT_ERR_TOO_LARGE;
  if (smem > 48 * 1024) FT_CUDA_TRY(cudaFuncSetAttribute(moe_topk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  moe_topk_kernel<<<(T + 7) / 8, 256, smem, st>>>(logits, ld, T, E, top, rule, expert, score, pos, count);
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

// kind 0: act[r][f] = g sigmoid(slope g) (u + 1) with g = min(s gate, limit), u = clamp(s up, -limit, limit), s = row_score[r] (1 when null); kind 1:
// s gate sigmoid(gate) up. gu: columns in blocks of eight gate, eight up (2 * fp columns); dtype bf16 or (is_f32) f32. rows_used: device int bounding the rows, or null.
FT_EXPORT int ft_moe_act(const void* gu, int64_t ld_gu, const float* row_score, const int* rows_used, int rows, int fp, int kind, float limit, float slope,
                         void* act, int64_t ld_act, int is_f32, cudaStream_t st) {
  if (rows < 1 || kind < 0 || kind > 1 || fp < 8 || (fp & 7) || (ld_gu & 7) || (ld_act & 7) || ld_gu < 2 * fp || ld_act < fp) return FT_ERR_ARG;
  const int units = fp / 4, gx = (units + 255) / 256, threads = ((units + gx - 1) / gx + 31) / 32 * 32;
  const int gy = (148 * 8 * (256 / threads) + gx - 1) / gx;
  const dim3 grid(gx, gy < rows ? gy : rows);
  if (is_f32) moe_act_kernel<float><<<grid, threads, 0, st>>>((const float*)gu, ld_gu, row_score, rows_used, rows, fp, kind, limit, slope, (float*)act, ld_act);
  else moe_act_kernel<__nv_bfloat16><<<grid, threads, 0, st>>>((const __nv_bfloat16*)gu, ld_gu, row_score, rows_used, rows, fp, kind, limit, slope, (__nv_bfloat16*)act, ld_act);
  return (int)cudaGetLastError();
}

// Decode routing (B <= 16 tokens, bf16 operands, f32 accumulation): logits f32 scratch of 32 E, counter int zero before the first launch. Outputs:
// n_active int[1], id int[E], cnt int[E], pair int[E][16], pair_of int[E][16], score f32 [B * top]. Choice and scores as in ft_moe_topk.
FT_EXPORT int ft_moe_route_small(const void* h, int64_t ldh, const void* router, int64_t ldr, int B, int W, int E, int top, int rule_kind, const float* vector, int groups, int keep,
                                 float scale, float* logits, int* counter, int* n_active, int* id, int* cnt, int* pair, int* pair_of, float* score, cudaStream_t st) {
  const RouteRule rule{rule_kind, vector, groups, keep, scale};
  if (B < 1 || B > SMALL_TOK || E < 1 || top < 1 || top > E || top > MAX_TOP || (ldh & 7) || (ldr & 7) || !rule_ok(rule, E, top)) return FT_ERR_ARG;
  return (int)ft_launch_pdl(moe_route_small_kernel, dim3(E), dim3(128), 0, st, (const __nv_bfloat16*)h, ldh, (const __nv_bfloat16*)router, ldr, B, W, E, top, rule,
                            logits, counter, SmallRoute{n_active, id, cnt, pair, pair_of, score});
}

// Gate / up projections and activation of a decode step. gu: [E][2 * fp][ld_in] interleaved rows, ld_in >= W rounded up to 32; act: bf16 [B * top][ld_act],
// row = token * top + slot; kind as in ft_moe_act. Shared expert (shared_gu null: none): act_sh bf16 [B][ld_act_sh]. fp is the neuron count rounded up to 8.
FT_EXPORT int ft_moe_gate_up_small(const void* h, int64_t ldh, int B, int W, int E, int top, int* n_active, int* id, int* cnt, int* pair, int* pair_of, float* score,
                                   const void* gu, int f, int64_t ld_in, float limit, const void* shared_gu, int f_sh, int64_t ld_in_sh, float limit_sh, int kind,
                                   float slope, void* act, int64_t ld_act, void* act_sh, int64_t ld_act_sh, cudaStream_t st) {
  const int kp = (W + 31) & ~31, fp = (f + 7) & ~7, fps = (f_sh + 7) & ~7;
  if (B < 1 || B > SMALL_TOK || f < 1 || (ldh & 7) || (ld_in & 7) || ld_in < kp || ld_act < f || (shared_gu && (f_sh < 1 || (ld_in_sh & 7) || ld_in_sh < kp || ld_act_sh < f_sh)))
    return FT_ERR_ARG;
  if (!skinny_fits(1, W)) return FT_ERR_TOO_LARGE;
  GateUpWork p{(const __nv_bfloat16*)h, ldh, B, W, 0, SmallRoute{n_active, id, cnt, pair, pair_of, score},
               ExpertSet{(const __nv_bfloat16*)gu, f, fp, ld_in, 2 * fp * ld_in, limit}, ExpertSet{(const __nv_bfloat16*)shared_gu, f_sh, fps, ld_in_sh, 0, limit_sh},
               shared_gu ? 1 : 0, kind, slope, (__nv_bfloat16*)act, (__nv_bfloat16*)act_sh, ld_act, ld_act_sh};
  const int items = (E < B * top ? E : B * top) * (fp / 8) + (shared_gu ? fps / 8 : 0);
  if (B > 8 && skinny_fits(2, W)) return skinny_launch<GateUpWork, 2>(p, W, items, st);
  for (p.tok0 = 0; p.tok0 < B; p.tok0 += 8) {
    const int r = skinny_launch<GateUpWork, 1>(p, W, items, st);
    if (r) return r;
  }
  return FT_OK;
}

// Down projections of a decode step: out[slot][token][W] f32 (plane_stride, ldo in elements), the shared expert in plane `top`. down: [E][rows_out][ld_mid]
// with rows_out >= W a multiple of 16 and ld_mid >= f rounded up to 32 (zeros past f).
FT_EXPORT int ft_moe_down_small(const void* act, int64_t ld_act, const void* act_sh, int64_t ld_act_sh, int B, int W, int E, int top, int* n_active, int* id, int* cnt,
                                int* pair, int* pair_of, float* score, const void* down, int f, int64_t ld_mid, const void* shared_down, int f_sh, int64_t ld_mid_sh,
                                int rows_out, float* out, int64_t plane_stride, int64_t ldo, cudaStream_t st) {
  if (B < 1 || B > SMALL_TOK || f < 1 || (rows_out & 15) || rows_out < W || (ld_act & 7) || ld_mid < ((f + 31) & ~31) || (ld_mid & 7) ||
      (shared_down && (f_sh < 1 || (ld_act_sh & 7) || (ld_mid_sh & 7) || ld_mid_sh < ((f_sh + 31) & ~31))))
    return FT_ERR_ARG;
  const int kmax = shared_down && f_sh > f ? f_sh : f, blocks = (W + 15) / 16;
  if (!skinny_fits(1, kmax)) return FT_ERR_TOO_LARGE;
  DownWork p{(const __nv_bfloat16*)act, (const __nv_bfloat16*)act_sh, ld_act, ld_act_sh, B, W, top, 0, SmallRoute{n_active, id, cnt, pair, pair_of, score},
             ExpertSet{(const __nv_bfloat16*)down, f, 0, ld_mid, rows_out * ld_mid, 0.f}, ExpertSet{(const __nv_bfloat16*)shared_down, f_sh, 0, ld_mid_sh, 0, 0.f},
             shared_down ? 1 : 0, blocks, out, plane_stride, ldo};
  const int items = ((E < B * top ? E : B * top) + (shared_down ? 1 : 0)) * blocks;
  if (B > 8 && skinny_fits(2, kmax)) return skinny_launch<DownWork, 2>(p, kmax, items, st);
  for (p.col0 = 0; p.col0 < B; p.col0 += 8) {
    const int r = skinny_launch<DownWork, 1>(p, kmax, items, st);
    if (r) return r;
  }
  return FT_OK;
}

// out[b][head][n] = sum_k w[head][n][k] x[b][head][k] for B <= 16 tokens: x bf16 (ldx between tokens, head_x between heads, 16-byte aligned), w bf16 rows of
// ldw >= K rounded up to 32 elements with head_w elements between heads (16-row blocks are read whole: the buffer extends past the last head's rows
// to the next multiple of 16), out bf16, times gate[b][head * head_g + n * elem_g] (f32 rows of ldg) unless gate is null.
FT_EXPORT int ft_skinny_heads(const void* x, int64_t ldx, int64_t head_x, const void* w, int64_t ldw, int64_t head_w, int B, int heads, int N, int K, void* out,
                              int64_t ldo, int64_t head_o, const float* gate, int64_t ldg, int head_g, int elem_g, cudaStream_t st) {
  if (B < 1 || B > SMALL_TOK || heads < 1 || N < 1 || K < 1 || (ldx & 7) || (head_x & 7) || (ldw & 7) || ldw < ((K + 31) & ~31) || (head_w & 7)) return FT_ERR_ARG;
  const HeadsWork p{(const __nv_bfloat16*)x, (const __nv_bfloat16*)w, ldx, head_x, ldw, head_w, B, heads, N, K, (__nv_bfloat16*)out, ldo, head_o, gate,
                    ldg, head_g, elem_g};
  const int items = heads * ((N + 15) / 16);
  if (!skinny_fits(B > 8 ? 2 : 1, K)) return FT_ERR_TOO_LARGE;
  return B > 8 ? skinny_launch<HeadsWork, 2>(p, K, items, st) : skinny_launch<HeadsWork, 1>(p, K, items, st);
}
