// Grouped-query attention with per-head key and value sizes, over a paged row cache: rotary positions on the first dimensions of a head (neighbouring pairs, or the
// two halves of the rotated part), RMS norms on queries and keys (per head, over the whole projection, or none), an optional sliding window beside which the first
// tokens of a sequence may stay visible, or chunks of the sequence that do not see one another, softmax with an optional sink per head, values optionally mixed with
// those of an earlier layer, and an output gate (per element or per head) with a scale. A layer may read the keys and values that an earlier layer cached.
//
// Differential heads have two query / key maps (maps = 2) over the same values: o = a_1 - lambda a_2, normed over the head's values (RMS, no weight), times a scale.
//
// Head sizes are padded to multiples of 16 (zeros): d16, v16. A token's cache row is [G keys of maps x d16 | G values of v16]; pages hold 16 rows. The maps of a head lie
// next to one another.
//
//   ft_gqa_prep          projection rows of a prompt -> normalised, rotated queries (in place), keys and values -> cache rows
//   ft_gqa_flash         prompts (tcgen05): ragged sequences, keys and values straight from the pages; the heads of a group share a tile, the maps of a head a CTA
//   ft_gqa_decode_prep   the same as ft_gqa_prep for one token per sequence, from split-K planes
//   ft_gqa_decode        one query token per sequence, the heads of a group share every loaded row (mma.sync), split over the visible range; the last CTA
//                        of a group merges the splits, adds the sink and applies the gate
//   ft_gqa_rows          plain f32-arithmetic kernel for f32 or bf16 data and any sizes (the 32-bit path)
//   ft_gqa_differential  what differential heads do with the outputs of their maps, where the attention kernel left them apart
// Compiled without fast-math.
#include <cooperative_groups.h>

#include "common.cuh"
#include "host_common.h"

namespace {

constexpr int KV_BLOCK = 16;
constexpr float LOG2E = 1.4426950408889634f;

FT_DEVICE float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
FT_DEVICE float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
FT_DEVICE float sigmoid_fast(float x) { return 1.f / (1.f + __expf(-x)); }

struct GqaDims {
  int H, G, d, dv, d16, v16, rot;    // query heads, key / value heads, sizes and padded sizes, rotated dimensions
  int row;                           // cache row: G * (maps * d16 + v16)
  int maps, HQ, GK;                  // maps of a head; H * maps queries, G * maps keys
};
// what a differential head does with its maps; on = 0: nothing
struct Differential {
  int on;
  float lambda, scale, eps;
};
enum { GATE_NONE = 0, GATE_ELEMENT = 1, GATE_HEAD = 2 };
enum { NORM_HEAD = 0, NORM_WHOLE = 1, NORM_NONE = 2 };

// eight consecutive elements
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
template <typename T> FT_DEVICE float one(T v);
template <> FT_DEVICE float one<float>(float v) { return v; }
template <> FT_DEVICE float one<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
FT_DEVICE void put1(float* p, float v) { *p = v; }
FT_DEVICE void put1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// ------------------------------------------------------------------------------------------------------------
// prompt rows: one CTA per row; a thread holds eight neighbouring columns (four rotation pairs) of a head. WHOLE: one norm over all heads.
// ------------------------------------------------------------------------------------------------------------
struct PrepArgs {
  GqaDims D;
  const float *wq, *wk;              // per head: [d16]; whole: [heads * d16]; null: no norm
  float eps;
  int halves;                        // dimension i turns with i + rot / 2, not 2 i with 2 i + 1
  const int* positions;
  const float *cos_t, *sin_t;
  const int* slots;
};
constexpr int PREP_T = 128;

template <typename T, bool WHOLE>
__global__ void __launch_bounds__(PREP_T) gqa_prep_kernel(T* __restrict__ qkv, int64_t ld, PrepArgs A, T* __restrict__ cache, const T* __restrict__ vfirst, int64_t ldf,
                                                          const float* __restrict__ lambda) {
  __shared__ float red[32];
  const GqaDims& D = A.D;
  const int r = blockIdx.x, pos = A.positions[r], half = D.rot / 2, hv = D.d16 / 8, nq = D.HQ * hv, nk = cache ? D.GK * hv : 0, heads = D.HQ + (cache ? D.GK : 0);
  T* row = qkv + (size_t)r * ld;
  T* dst = cache ? cache + (size_t)A.slots[r] * D.row : nullptr;       // null: queries alone
  const float* ct = A.cos_t + (size_t)pos * half;
  const float* st = A.sin_t + (size_t)pos * half;
  const bool normed = WHOLE || A.wq != nullptr;
  auto weights = [&](int head) -> const float* { return (head < D.HQ ? A.wq : A.wk) + (WHOLE ? (head < D.HQ ? head : head - D.HQ) * D.d16 : 0); };
  auto finish = [&](int head, int vi, bool is_q, const float (&x)[8], float rstd) {       // norm weight, rotation, store
    const float* w = normed ? weights(head) + vi * 8 : nullptr;
    float v[8];
#pragma unroll
    for (int e = 0; e < 8; e++) v[e] = normed ? x[e] * rstd * w[e] : x[e];
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int p = vi * 4 + e;
      if (p < half) {
        const float c = ct[p], s = st[p], a = v[2 * e], b = v[2 * e + 1];
        v[2 * e] = a * c - b * s;
        v[2 * e + 1] = b * c + a * s;
      }
    }
    store8(is_q ? row + head * D.d16 + vi * 8 : dst + (head - D.HQ) * D.d16 + vi * 8, v);
  };
  // the same for pairs (i, i + half): a lane takes both of a pair, so nothing is read after it was overwritten
  auto finish_halves = [&](int head, int l, int lanes, float rstd) {
    const bool is_q = head < D.HQ;
    const T* src = row + head * D.d16;
    T* to = is_q ? row + head * D.d16 : dst + (head - D.HQ) * D.d16;
    const float* w = normed ? weights(head) : nullptr;
    if ((half & 7) == 0) {
      for (int vi = l; vi < half / 8; vi += lanes) {
        float a[8], b[8];
        load8(src + vi * 8, a);
        load8(src + half + vi * 8, b);
#pragma unroll
        for (int e = 0; e < 8; e++) {
          const int p = vi * 8 + e;
          const float c = ct[p], s = st[p], u = normed ? a[e] * rstd * w[p] : a[e], v = normed ? b[e] * rstd * w[half + p] : b[e];
          a[e] = u * c - v * s;
          b[e] = v * c + u * s;
        }
        store8(to + vi * 8, a);
        store8(to + half + vi * 8, b);
      }
      if (is_q && !normed) return;                   // the rest stays as it is
      for (int vi = D.rot / 8 + l; vi < hv; vi += lanes) {
        float a[8];
        load8(src + vi * 8, a);
        if (normed)
#pragma unroll
          for (int e = 0; e < 8; e++) a[e] = a[e] * rstd * w[vi * 8 + e];
        store8(to + vi * 8, a);
      }
    } else {
      auto at = [&](int c) { return normed ? one(src[c]) * rstd * w[c] : one(src[c]); };
      for (int p = l; p < half; p += lanes) {
        const float c = ct[p], s = st[p], u = at(p), v = at(half + p);
        put1(to + p, u * c - v * s);
        put1(to + half + p, v * c + u * s);
      }
      for (int c = D.rot + l; c < D.d16; c += lanes) put1(to + c, at(c));
    }
  };
  if (!normed && half == 0) {                        // queries stay as they are
    for (int i = threadIdx.x; i < nk; i += PREP_T) {
      float a[8];
      load8(row + D.HQ * D.d16 + i * 8, a);
      store8(dst + i * 8, a);
    }
  } else if constexpr (WHOLE) {
    float sq = 0.f, sk = 0.f, x[8];
    for (int i = threadIdx.x; i < nq + nk; i += PREP_T) {
      load8(row + i * 8, x);
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < 8; e++) s += x[e] * x[e];
      if (i < nq) sq += s; else sk += s;
    }
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
    const float rq = 1.f / sqrtf(sq / (float)(D.HQ * D.d) + A.eps), rk = 1.f / sqrtf(sk / (float)(D.GK * D.d) + A.eps);
    if (A.halves) {
      for (int head = threadIdx.x >> 5; head < heads; head += PREP_T / 32) finish_halves(head, threadIdx.x & 31, 32, head < D.HQ ? rq : rk);
    } else {
      for (int i = threadIdx.x; i < nq + nk; i += PREP_T) {
        load8(row + i * 8, x);
        finish(i / hv, i % hv, i < nq, x, i < nq ? rq : rk);
      }
    }
  } else if (!normed && A.halves && (half & 7) == 0) {
    const int hw = half / 8, tail = hv - 2 * hw;     // nothing to reduce: pairs of vectors of all heads in a row, then the keys' columns behind the rotated ones
    for (int i = threadIdx.x; i < heads * hw; i += PREP_T) {
      const int head = i / hw, vi = i % hw;
      const T* src = row + head * D.d16 + vi * 8;
      T* to = head < D.HQ ? row + head * D.d16 + vi * 8 : dst + (head - D.HQ) * D.d16 + vi * 8;
      float a[8], b[8], c[8], s[8];
      load8(src, a);
      load8(src + half, b);
      load8(ct + vi * 8, c);
      load8(st + vi * 8, s);
#pragma unroll
      for (int e = 0; e < 8; e++) {
        const float u = a[e];
        a[e] = u * c[e] - b[e] * s[e];
        b[e] = b[e] * c[e] + u * s[e];
      }
      store8(to, a);
      store8(to + half, b);
    }
    for (int i = threadIdx.x; i < (cache ? D.GK : 0) * tail; i += PREP_T) {
      const int at = i / tail * D.d16 + (2 * hw + i % tail) * 8;
      float a[8];
      load8(row + D.HQ * D.d16 + at, a);
      store8(dst + at, a);
    }
  } else {
    int lanes = 1;                                   // lanes of a head: a power of two that covers its columns, at most a warp
    while (lanes < hv && lanes < 32) lanes *= 2;
    const int l = threadIdx.x % lanes, groups = PREP_T / lanes;
    for (int h0 = 0; h0 < heads; h0 += groups) {
      const int head = h0 + threadIdx.x / lanes;
      const bool live = head < heads;
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, s = 0.f;
      if (live && (normed || !A.halves))
        for (int vi = l; vi < hv; vi += lanes) {
          load8(row + head * D.d16 + vi * 8, x);
#pragma unroll
          for (int e = 0; e < 8; e++) s += x[e] * x[e];
        }
      for (int o = lanes / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      const float rstd = 1.f / sqrtf(s / (float)D.d + A.eps);
      if (live && A.halves) finish_halves(head, l, lanes, rstd);
      if (live && !A.halves)
        for (int vi = l; vi < hv; vi += lanes) {
          if (hv > lanes) load8(row + head * D.d16 + vi * 8, x);       // a single vector per lane is still in registers
          finish(head, vi, head < D.HQ, x, rstd);
        }
    }
  }
  if (cache == nullptr) return;
  const float lam = lambda ? *lambda : 0.f;
  for (int i = threadIdx.x; i < D.G * D.v16 / 8; i += PREP_T) {
    float v[8];
    load8(row + (D.HQ + D.GK) * D.d16 + i * 8, v);
    if (lambda) {
      float f[8];
      load8(vfirst + (size_t)r * ldf + i * 8, f);
#pragma unroll
      for (int e = 0; e < 8; e++) v[e] = (1.f - lam) * v[e] + lam * f[e];
    }
    store8(dst + D.GK * D.d16 + i * 8, v);
  }
}

// ------------------------------------------------------------------------------------------------------------
// plain kernel: grid (rows, H * maps), 128 threads
// ------------------------------------------------------------------------------------------------------------
struct MaskGate {
  float scale;
  int window;                        // keys a position sees, itself included (INT_MAX: all)
  int keep;                          // and the first keys of the sequence
  int chunk;                         // a position sees only its own chunk of the sequence (0: no chunks)
  const float* sink;                 // [H] or null
  const void* gate;                  // per element: rows of H * v16 in the data type; per head: f32 rows of H (pre-activation)
  int64_t ldg;
  int gate_kind;
  float out_scale;
};
// first key that a position sees, the kept ones aside
FT_DEVICE int first_visible(const MaskGate& M, int pos) {
  const int w = max(0, pos - M.window + 1);
  return M.chunk ? max(w, pos / M.chunk * M.chunk) : w;
}
constexpr int ROWS_CHUNK = 64, ROWS_MAX_COLS = 8;
template <typename T, typename O>
__global__ void __launch_bounds__(128) gqa_rows_kernel(const T* __restrict__ q, int64_t ldq, const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                                                       const int* __restrict__ seq_of, const int* __restrict__ positions, GqaDims D, MaskGate M, O* __restrict__ out,
                                                       int64_t ldo) {
  extern __shared__ float sq[];      // d16
  __shared__ float sp[ROWS_CHUNK];
  const int r = blockIdx.x, hd = blockIdx.y, g = hd / D.maps / (D.H / D.G), gk = g * D.maps + hd % D.maps, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int len = positions[r] + 1, first = first_visible(M, len - 1);
  const int kept = min(M.keep, first), gap = first - kept, total = len - gap;        // visible keys in order: 0..kept, first..len
  const int* bt = block_table + (size_t)seq_of[r] * max_blocks;
  for (int i = threadIdx.x; i < D.d16; i += 128) sq[i] = one(q[(size_t)r * ldq + hd * D.d16 + i]);
  float o[ROWS_MAX_COLS];
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++) o[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  if (M.sink) { m = M.sink[hd]; l = 1.f; }           // the sink is a score without a value
  __syncthreads();
  for (int t0 = 0; t0 < total; t0 += ROWS_CHUNK) {
    const int cnt = min(ROWS_CHUNK, total - t0);
    for (int k = warp; k < cnt; k += 4) {
      const int t = t0 + k < kept ? t0 + k : t0 + k + gap;
      const T* kr = cache + ((size_t)bt[t / KV_BLOCK] * KV_BLOCK + t % KV_BLOCK) * D.row + gk * D.d16;
      float a = 0.f;
      for (int i = lane; i < D.d16; i += 32) a += sq[i] * one(kr[i]);
      a = warp_sum(a);
      if (lane == 0) sp[k] = a * M.scale;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < cnt; k++) mx = fmaxf(mx, sp[k]);
    const float alpha = expf(m - mx);
    l *= alpha;
#pragma unroll
    for (int i = 0; i < ROWS_MAX_COLS; i++) o[i] *= alpha;
    for (int k = 0; k < cnt; k++) {
      const int t = t0 + k < kept ? t0 + k : t0 + k + gap;
      const T* vr = cache + ((size_t)bt[t / KV_BLOCK] * KV_BLOCK + t % KV_BLOCK) * D.row + D.GK * D.d16 + g * D.v16;
      const float p = expf(sp[k] - mx);
      l += p;
#pragma unroll
      for (int i = 0; i < ROWS_MAX_COLS; i++)
        if (threadIdx.x + 128 * i < D.v16) o[i] += p * one(vr[threadIdx.x + 128 * i]);
    }
    m = mx;
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++) {
    const int c = threadIdx.x + 128 * i;
    if (c < D.v16) {
      float v = o[i] / l * M.out_scale;
      if (M.gate_kind == GATE_ELEMENT) v *= sigmoid_exact(one(reinterpret_cast<const T*>(M.gate)[(size_t)r * M.ldg + hd * D.v16 + c]));
      if (M.gate_kind == GATE_HEAD) v *= sigmoid_exact(reinterpret_cast<const float*>(M.gate)[(size_t)r * M.ldg + hd]);
      put1(out + (size_t)r * ldo + hd * D.v16 + c, v);
    }
  }
}

// differential heads from the f32 outputs of their maps [rows][H][2][v16]: a warp per row and head
template <typename T>
__global__ void __launch_bounds__(256) gqa_differential_kernel(const float* __restrict__ a, int64_t lda, GqaDims D, Differential F, int units, T* __restrict__ out, int64_t ldo) {
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= units) return;
  const int r = unit / D.H, hd = unit % D.H;
  const float* src = a + (size_t)r * lda + (size_t)hd * 2 * D.v16;
  T* dst = out + (size_t)r * ldo + (size_t)hd * D.v16;
  float o[ROWS_MAX_COLS][4], ss = 0.f;
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++) {
    const int c = lane * 4 + i * 128;
    if (c < D.v16) {
      const float4 x = *reinterpret_cast<const float4*>(src + c), y = *reinterpret_cast<const float4*>(src + D.v16 + c);
      o[i][0] = x.x - F.lambda * y.x; o[i][1] = x.y - F.lambda * y.y; o[i][2] = x.z - F.lambda * y.z; o[i][3] = x.w - F.lambda * y.w;
      ss += o[i][0] * o[i][0] + o[i][1] * o[i][1] + o[i][2] * o[i][2] + o[i][3] * o[i][3];
    }
  }
  const float k = F.scale / sqrtf(warp_sum(ss) / (float)D.dv + F.eps);
#pragma unroll
  for (int i = 0; i < ROWS_MAX_COLS; i++) {
    const int c = lane * 4 + i * 128;
    if (c < D.v16)
#pragma unroll
      for (int e = 0; e < 4; e++) put1(dst + c + e, o[i][e] * k);
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode preparation from split-K planes: a warp takes one head (or 128 gate columns) of one token, four columns a lane. WHOLE: the CTAs of a token form a
// cluster, sums of squares meet in distributed shared memory, the plane sums wait in shared memory meanwhile.
// ------------------------------------------------------------------------------------------------------------
constexpr int DEC_TOK = 16, DP_WARPS = 8, DP_MAXC = 4;       // head sizes up to 128 * DP_MAXC
FT_DEVICE float4 plane_sum4(const float* __restrict__ p, int splits, size_t stride) {
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  int s = 0;
  for (; s + 4 <= splits; s += 4) {
    float4 t[4];
#pragma unroll
    for (int j = 0; j < 4; j++) t[j] = __ldcg(reinterpret_cast<const float4*>(p + (s + j) * stride));
    a.x += (t[0].x + t[1].x) + (t[2].x + t[3].x);
    a.y += (t[0].y + t[1].y) + (t[2].y + t[3].y);
    a.z += (t[0].z + t[1].z) + (t[2].z + t[3].z);
    a.w += (t[0].w + t[1].w) + (t[2].w + t[3].w);
  }
  for (; s < splits; s++) {
    const float4 t = __ldcg(reinterpret_cast<const float4*>(p + s * stride));
    a.x += t.x; a.y += t.y; a.z += t.z; a.w += t.w;
  }
  return a;
}
struct DecPrepArgs {
  PrepArgs P;
  const float* planes;
  int splits;
  int64_t ldp;
  size_t pstride;
  const int* block_table;
  int max_blocks;
  int gate_col, gate_kind;           // column of the gate's pre-activation in the planes
  float* gate;                       // [16][H * v16] or [16][H]: sigmoid of it
  float* vf_out;                     // [16][G * v16]: values kept for later layers, or
  const float* vf_in;                //   mixed in with weight *lambda
  const float* lambda;
};
FT_DEVICE void put_bf16x4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&a);
  pk.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = pk;
}

template <bool WHOLE>
__global__ void __launch_bounds__(DP_WARPS * 32) gqa_decode_prep_kernel(DecPrepArgs A, __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ cache) {
  namespace cg = cooperative_groups;
  extern __shared__ __align__(16) float held[];      // plane sums of query and key heads: WHOLE [local unit][d16], else (halves) [warp][d16]
  __shared__ float red[32];
  __shared__ float cta_ss[2];
  pdl_wait();
  pdl_launch_dependents();
  const GqaDims& D = A.P.D;
  const int b = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pos = A.P.positions[b], half = D.rot / 2, stride = gridDim.x * DP_WARPS;
  const int u0 = blockIdx.x * DP_WARPS + warp, heads = D.HQ + (cache ? D.GK : 0);
  const float* src = A.planes + (size_t)b * A.ldp;
  const int blk = A.block_table[(size_t)b * A.max_blocks + pos / KV_BLOCK];
  __nv_bfloat16* dst = blk < 0 || cache == nullptr ? nullptr : cache + ((size_t)blk * KV_BLOCK + pos % KV_BLOCK) * D.row;
  const float* ct = A.P.cos_t + (size_t)pos * half;
  const float* st = A.P.sin_t + (size_t)pos * half;
  const bool normed = WHOLE || A.P.wq != nullptr;
  auto finish = [&](int u, int c, float4 v, float rstd, const float* sums) {       // sums: this head's plane sums (read for pairs of halves only)
    const bool is_q = u < D.HQ;
    const float* wh = normed ? (is_q ? A.P.wq : A.P.wk) + (WHOLE ? (is_q ? u : u - D.HQ) * D.d16 : 0) : nullptr;
    if (normed) {
      const float4 w = *reinterpret_cast<const float4*>(wh + c);
      v = make_float4(v.x * rstd * w.x, v.y * rstd * w.y, v.z * rstd * w.z, v.w * rstd * w.w);
    }
    const int p = c / 2;
    if (A.P.halves) {
      float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const int d = c + i;
        if (d < D.rot) {
          const bool low = d < half;
          const int o = low ? d + half : d - half;
          const float other = normed ? sums[o] * rstd * wh[o] : sums[o], cc = ct[low ? d : o], ss = st[low ? d : o];
          e[i] = low ? e[i] * cc - other * ss : e[i] * cc + other * ss;
        }
      }
      v = make_float4(e[0], e[1], e[2], e[3]);
    } else {
      if (p < half) {
        const float cc = ct[p], ss = st[p], a = v.x;
        v.x = a * cc - v.y * ss;
        v.y = v.y * cc + a * ss;
      }
      if (p + 1 < half) {
        const float cc = ct[p + 1], ss = st[p + 1], a = v.z;
        v.z = a * cc - v.w * ss;
        v.w = v.w * cc + a * ss;
      }
    }
    if (is_q) put_bf16x4(q + (((size_t)b * D.HQ + u) * D.maps + u % D.maps) * D.d16 + c, v);
    else if (dst) put_bf16x4(dst + (u - D.HQ) * D.d16 + c, v);
  };
  float ssq = 0.f, ssk = 0.f;
  int local = warp;
  for (int u = u0; u < heads; u += stride, local += DP_WARPS) {
    float4 v[DP_MAXC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < DP_MAXC; i++) {
      const int c = lane * 4 + i * 128;
      if (c < D.d16) {
        v[i] = plane_sum4(src + (size_t)u * D.d16 + c, A.splits, A.pstride);
        ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        if constexpr (WHOLE) *reinterpret_cast<float4*>(held + local * D.d16 + c) = v[i];
        else if (A.P.halves) *reinterpret_cast<float4*>(held + warp * D.d16 + c) = v[i];
      }
    }
    if constexpr (WHOLE) {
      if (u < D.HQ) ssq += ss; else ssk += ss;
    } else {
      const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D.d + A.P.eps);
      __syncwarp();
#pragma unroll
      for (int i = 0; i < DP_MAXC; i++)
        if (lane * 4 + i * 128 < D.d16) finish(u, lane * 4 + i * 128, v[i], rstd, held + warp * D.d16);
      __syncwarp();
    }
  }
  if constexpr (WHOLE) {
    ssq = block_sum(ssq, red);
    ssk = block_sum(ssk, red);
    if (threadIdx.x == 0) { cta_ss[0] = ssq; cta_ss[1] = ssk; }
  }
  // values and gates: the first unit of this warp past the heads
  const int gate_cols = A.gate_kind == GATE_ELEMENT ? D.H * D.v16 : A.gate_kind == GATE_HEAD ? D.H : 0;
  const int values = cache ? D.G : 0, units = heads + values + (gate_cols + 127) / 128;
  const float lam = A.lambda ? *A.lambda : 0.f;
  int u = u0;
  if (u < heads) u += (heads - u + stride - 1) / stride * stride;
  for (; u < units; u += stride) {
    if (u < heads + values) {
      const int g = u - heads;
      for (int c = lane * 4; c < D.v16; c += 128) {
        float4 v = plane_sum4(src + (size_t)heads * D.d16 + g * D.v16 + c, A.splits, A.pstride);
        const size_t at = (size_t)b * D.G * D.v16 + g * D.v16 + c;
        if (A.lambda) {
          const float4 f = *reinterpret_cast<const float4*>(A.vf_in + at);
          v = make_float4((1.f - lam) * v.x + lam * f.x, (1.f - lam) * v.y + lam * f.y, (1.f - lam) * v.z + lam * f.z, (1.f - lam) * v.w + lam * f.w);
        } else if (A.vf_out) {
          *reinterpret_cast<float4*>(A.vf_out + at) = v;
        }
        if (dst) put_bf16x4(dst + D.GK * D.d16 + g * D.v16 + c, v);
      }
    } else {
      const int c = (u - heads - values) * 128 + lane * 4;
      if (c < gate_cols) {
        const float4 v = plane_sum4(src + A.gate_col + c, A.splits, A.pstride);      // columns past a head gate's end: readable, not stored
        const float e[4] = {sigmoid_exact(v.x), sigmoid_exact(v.y), sigmoid_exact(v.z), sigmoid_exact(v.w)};
        for (int j = 0; j < 4; j++)
          if (c + j < gate_cols) A.gate[(size_t)b * gate_cols + c + j] = e[j];
      }
    }
  }
  if constexpr (WHOLE) {
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    float tq = 0.f, tk = 0.f;
    for (unsigned r = 0; r < gridDim.x; r++) {
      const float* p = cluster.map_shared_rank(cta_ss, r);
      tq += p[0];
      tk += p[1];
    }
    const float rq = 1.f / sqrtf(tq / (float)(D.HQ * D.d) + A.P.eps), rk = 1.f / sqrtf(tk / (float)(D.GK * D.d) + A.P.eps);
    local = warp;
    for (int v = u0; v < heads; v += stride, local += DP_WARPS)
      for (int c = lane * 4; c < D.d16; c += 128) finish(v, c, *reinterpret_cast<const float4*>(held + local * D.d16 + c), v < D.HQ ? rq : rk, held + local * D.d16);
    cluster.sync();                                  // nobody leaves while a partner may still read its shared memory
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode attention: grid (nsplit, G * head tiles, B), 256 threads. Chunks of 64 visible rows go through a two-stage shared-memory ring (16-byte cp.async; rows an
// odd number of 16-byte units apart, so the ldmatrix reads are conflict free). Scores: warp w takes eight rows against the 16 heads of the tile; softmax
// statistics meet in shared memory; output: warp w takes NP * 16 value columns over all 64 rows. ws: [B][G * tiles][split][16][v16 + 4] f32 (accumulators,
// running maximum in the log2 domain, running sum); counters: [B][G * tiles], zero between launches. Differential heads come as 2 H heads of twice the size whose
// queries are zero outside their own map's half, so that one row of keys and values serves both maps; the merge combines them.
// ------------------------------------------------------------------------------------------------------------
constexpr int GD_CHUNK = 64, GD_STAGES = 2, GD_P_PITCH = 144, GD_MAX_SPLIT = 64, GD_HT = 16;
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
FT_DEVICE void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__host__ __device__ inline int gd_pitch(int d16, int v16) { return (d16 + v16) * 2 + 16; }
inline int gd_smem(int d16, int v16) {
  const int p = gd_pitch(d16, v16), ring = GD_HT * p + GD_STAGES * GD_CHUNK * p + GD_HT * GD_P_PITCH, merge = 2 * GD_MAX_SPLIT * GD_HT * 4 + GD_HT * 4;
  return ring > merge ? ring : merge;
}

template <int NP>
__global__ void __launch_bounds__(256) gqa_decode_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table,
                                                         int max_blocks, const int* __restrict__ seq_lens, GqaDims D, MaskGate M, int tiles, float* __restrict__ ws,
                                                         int* __restrict__ counters, Differential F, __nv_bfloat16* __restrict__ out, int64_t ldo) {
  pdl_wait();
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float sm_mx[8][GD_HT], sm_l[8][GD_HT];
  __shared__ int is_last;
  const int split = blockIdx.x, nsplit = gridDim.x, g = blockIdx.y / tiles, tile = blockIdx.y % tiles, b = blockIdx.z;
  const int R = D.H / D.G, h0 = g * R + tile * GD_HT, nh = min(GD_HT, R - tile * GD_HT);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  const int len = seq_lens[b], first = first_visible(M, len - 1);
  const int kept = min(M.keep, first), gap = first - kept, total = len - gap;        // visible rows in order: 0..kept, first..len
  const int per = ((total + nsplit - 1) / nsplit + 15) & ~15;
  const int t0 = split * per, t1 = min(total, t0 + per);
  const int nchunks = t1 > t0 ? (t1 - t0 + GD_CHUNK - 1) / GD_CHUNK : 0;
  const int wrow = D.v16 + 4;
  float* base = ws + ((size_t)b * gridDim.y + blockIdx.y) * nsplit * GD_HT * wrow;
  float* my_ws = base + (size_t)split * GD_HT * wrow;
  const int pitch = gd_pitch(D.d16, D.v16), kvecs = D.d16 / 8, vecs = kvecs + D.v16 / 8;
  const uint32_t sQ = smem_u32(smem), sK = sQ + GD_HT * pitch, sP = sK + GD_STAGES * GD_CHUNK * pitch;
  const int* bt = block_table + (size_t)b * max_blocks;
  const float sl2 = M.scale * LOG2E;

  auto load_chunk = [&](int c, int stage) {
    const int c0 = t0 + c * GD_CHUNK, cnt = min(GD_CHUNK, t1 - c0);
    const uint32_t dst = sK + stage * GD_CHUNK * pitch;
    for (int r = warp; r < cnt; r += 8) {
      const int t = c0 + r < kept ? c0 + r : c0 + r + gap;
      const __nv_bfloat16* src = cache + ((size_t)__ldg(bt + t / KV_BLOCK) * KV_BLOCK + t % KV_BLOCK) * D.row;
      for (int i = lane; i < vecs; i += 32)
        cp_async16(dst + r * pitch + i * 16, i < kvecs ? src + g * D.d16 + i * 8 : src + D.G * D.d16 + g * D.v16 + (i - kvecs) * 8);
    }
    // rows up to the next multiple of 16 meet weight zero: they must be finite
    for (int r = cnt + warp; r < ((cnt + 15) & ~15); r += 8)
      for (int i = lane; i < vecs; i += 32) *reinterpret_cast<uint4*>(smem + (dst - sQ) + r * pitch + i * 16) = make_uint4(0, 0, 0, 0);
  };
  if (nchunks > 0) {
    for (int r = warp; r < GD_HT; r += 8)
      for (int i = lane; i < kvecs; i += 32) {
        if (r < nh) cp_async16(sQ + r * pitch + i * 16, q + ((size_t)b * D.H + h0 + r) * D.d16 + i * 8);
        else *reinterpret_cast<uint4*>(smem + r * pitch + i * 16) = make_uint4(0, 0, 0, 0);
      }
#pragma unroll
    for (int s = 0; s < GD_STAGES; s++) {
      if (s < nchunks) load_chunk(s, s);
      cp_async_commit();
    }
  }
  float o[NP][2][4];
#pragma unroll
  for (int p = 0; p < NP; p++)
#pragma unroll
    for (int e = 0; e < 4; e++) o[p][0][e] = o[p][1][e] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const int npairs = D.v16 / 16, ksteps = D.d16 / 16;
  for (int c = 0; c < nchunks; c++) {
    cp_async_wait<GD_STAGES - 1>();
    __syncthreads();
    const int stage = c % GD_STAGES, cnt = min(GD_CHUNK, t1 - (t0 + c * GD_CHUNK));
    const uint32_t kb = sK + stage * GD_CHUNK * pitch;
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    if (warp * 8 < cnt) {
      const uint32_t krow = kb + (warp * 8 + (lane & 7)) * pitch, qrow = sQ + (lane & 15) * pitch + (lane >> 4) * 16;
      for (int ks = 0; ks < ksteps; ks++) {
        uint32_t k0, k1, qa[4];
        ldmatrix_x2(k0, k1, krow + ks * 32 + ((lane >> 3) & 1) * 16);
        ldmatrix_x4(qa, qrow + ks * 32);
        mma_16816(s, qa, k0, k1);
      }
    }
    const bool v0 = warp * 8 + t2 < cnt, v1 = warp * 8 + t2 + 1 < cnt;
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float a = fmaxf(v0 ? s[2 * e] : -INFINITY, v1 ? s[2 * e + 1] : -INFINITY);
      a = fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 1));
      a = fmaxf(a, __shfl_xor_sync(0xffffffffu, a, 2));
      if ((lane & 3) == 0) sm_mx[warp][gr + 8 * e] = a;
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float mx = m_run[e];
#pragma unroll
      for (int w = 0; w < 8; w++) mx = fmaxf(mx, sm_mx[w][gr + 8 * e]);
      alpha[e] = ex2((m_run[e] - mx) * sl2);                        // 0 on the first chunk
      m_run[e] = mx;
      const float p0 = v0 ? ex2((s[2 * e] - mx) * sl2) : 0.f, p1 = v1 ? ex2((s[2 * e + 1] - mx) * sl2) : 0.f;
      l_run[e] = l_run[e] * alpha[e] + p0 + p1;
      *reinterpret_cast<__nv_bfloat162*>(smem + (sP - sQ) + (gr + 8 * e) * GD_P_PITCH + (warp * 8 + t2) * 2) = __floats2bfloat162_rn(p0, p1);
    }
    __syncthreads();
    const int psteps = (cnt + 15) / 16;
#pragma unroll
    for (int p = 0; p < NP; p++)
#pragma unroll
      for (int n = 0; n < 2; n++) {
        o[p][n][0] *= alpha[0]; o[p][n][1] *= alpha[0];
        o[p][n][2] *= alpha[1]; o[p][n][3] *= alpha[1];
      }
    for (int ps = 0; ps < psteps; ps++) {
      uint32_t pf[4];
      ldmatrix_x4(pf, sP + (lane & 15) * GD_P_PITCH + ps * 32 + (lane >> 4) * 16);
      const uint32_t vrow = kb + (ps * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * pitch + D.d16 * 2 + (lane >> 4) * 16;
#pragma unroll
      for (int p = 0; p < NP; p++) {
        const int pr = warp * NP + p;
        if (pr < npairs) {
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, vrow + pr * 32);
          mma_16816(o[p][0], pf, vb[0], vb[1]);
          mma_16816(o[p][1], pf, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();
    if (c + GD_STAGES < nchunks) load_chunk(c + GD_STAGES, stage);
    cp_async_commit();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int e = 0; e < 2; e++) {
    float l = l_run[e];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const int hrow = gr + 8 * e;
    if ((lane & 3) == 0) sm_l[warp][hrow] = l;
    float* dst = my_ws + (size_t)hrow * wrow;
    if (nchunks > 0 && hrow < nh) {
#pragma unroll
      for (int p = 0; p < NP; p++) {
        const int pr = warp * NP + p;
        if (pr < npairs) {
          *reinterpret_cast<float2*>(dst + pr * 16 + t2) = make_float2(o[p][0][2 * e], o[p][0][2 * e + 1]);
          *reinterpret_cast<float2*>(dst + pr * 16 + 8 + t2) = make_float2(o[p][1][2 * e], o[p][1][2 * e + 1]);
        }
      }
    }
    if (warp == 0 && (lane & 3) == 0) dst[D.v16] = nchunks > 0 ? m_run[e] * sl2 : -INFINITY;
  }
  __syncthreads();
  if (threadIdx.x < GD_HT) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) l += sm_l[w][threadIdx.x];
    my_ws[(size_t)threadIdx.x * wrow + D.v16 + 1] = l;
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    int* ctr = counters + (size_t)b * gridDim.y + blockIdx.y;
    is_last = atomicAdd(ctr, 1) == nsplit - 1;
    if (is_last) *ctr = 0;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  // merge: weights of the splits and the row sums first, then one pass over the value columns
  float* fw = reinterpret_cast<float*>(smem);                       // [nsplit][16]
  float* fl = fw + GD_MAX_SPLIT * GD_HT;
  float* inv = fl + GD_MAX_SPLIT * GD_HT;                           // [16]
  for (int i = threadIdx.x; i < nsplit * nh; i += 256) {
    const int s = i / nh, r = i % nh;
    const float2 ml = __ldcg(reinterpret_cast<const float2*>(base + ((size_t)s * GD_HT + r) * wrow + D.v16));
    fw[s * GD_HT + r] = ml.x;
    fl[s * GD_HT + r] = ml.y;
  }
  __syncthreads();
  if (threadIdx.x < nh) {
    const int r = threadIdx.x;
    const float sink = M.sink ? M.sink[h0 + r] * LOG2E : -INFINITY;
    float mx = sink, l = 0.f;
    for (int s = 0; s < nsplit; s++) mx = fmaxf(mx, fw[s * GD_HT + r]);
    if (M.sink) l = ex2(sink - mx);
    for (int s = 0; s < nsplit; s++) {
      const float f = fw[s * GD_HT + r] == -INFINITY ? 0.f : ex2(fw[s * GD_HT + r] - mx);
      l += f * fl[s * GD_HT + r];
      fw[s * GD_HT + r] = f;
    }
    float k = M.out_scale / l;
    if (M.gate_kind == GATE_HEAD) k *= reinterpret_cast<const float*>(M.gate)[(size_t)b * D.H + h0 + r];
    inv[r] = k;
  }
  __syncthreads();
  auto merged = [&](int r, int c) -> float4 {        // four value columns of a row over all splits, not yet divided by the row sum
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = 0; s0 < nsplit; s0 += 8) {
      float4 v[8];
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const bool live = s0 + j < nsplit && fw[min(s0 + j, GD_MAX_SPLIT - 1) * GD_HT + r] > 0.f;    // a split without rows left its accumulators unwritten
        v[j] = live ? __ldcg(reinterpret_cast<const float4*>(base + ((size_t)(s0 + j) * GD_HT + r) * wrow + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int j = 0; j < 8; j++) {
        const float w = s0 + j < nsplit ? fw[(s0 + j) * GD_HT + r] : 0.f;
        a.x += w * v[j].x; a.y += w * v[j].y; a.z += w * v[j].z; a.w += w * v[j].w;
      }
    }
    return a;
  };
  if (F.on) {                                        // rows 2 i and 2 i + 1 are the maps of a head: one warp takes both
    for (int p = warp; p < nh / 2; p += 8) {
      const float k0 = inv[2 * p], k1 = inv[2 * p + 1] * F.lambda;
      float4 o4[4];                                  // value sizes up to 512
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const int c = lane * 4 + i * 128;
        o4[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < D.v16) {
          const float4 x = merged(2 * p, c), y = merged(2 * p + 1, c);
          o4[i] = make_float4(x.x * k0 - y.x * k1, x.y * k0 - y.y * k1, x.z * k0 - y.z * k1, x.w * k0 - y.w * k1);
          ss += o4[i].x * o4[i].x + o4[i].y * o4[i].y + o4[i].z * o4[i].z + o4[i].w * o4[i].w;
        }
      }
      const float k = F.scale / sqrtf(warp_sum(ss) / (float)D.dv + F.eps);
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const int c = lane * 4 + i * 128;
        if (c < D.v16) put_bf16x4(out + (size_t)b * ldo + (size_t)(h0 / 2 + p) * D.v16 + c, make_float4(o4[i].x * k, o4[i].y * k, o4[i].z * k, o4[i].w * k));
      }
    }
    return;
  }
  const int vq = D.v16 / 4;
  for (int i = threadIdx.x; i < nh * vq; i += 256) {
    const int r = i / vq, c = (i % vq) * 4;
    float4 a = merged(r, c);
    const float k = inv[r];
    a = make_float4(a.x * k, a.y * k, a.z * k, a.w * k);
    if (M.gate_kind == GATE_ELEMENT) {
      const float4 gt = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(M.gate) + ((size_t)b * D.H + h0 + r) * D.v16 + c);
      a = make_float4(a.x * gt.x, a.y * gt.y, a.z * gt.z, a.w * gt.w);
    }
    put_bf16x4(out + (size_t)b * ldo + (h0 + r) * D.v16 + c, a);
  }
}

// ------------------------------------------------------------------------------------------------------------
// prompt attention (tcgen05): one CTA per (tile of NT sub-tiles of one sequence, key / value head). A sub-tile's 128 rows are `tok` tokens times the R query heads
// of the group, so a window costs the keys of `tok` tokens more than its size, and a group's heads share every loaded key and value. DIFF: the two sub-tiles are the maps
// of the same heads and tokens, each with keys of its own and both with the same values; the rows of both maps lie in the same lanes of tensor memory, so that either half of the
// softmax threads combines half of the value columns. Sizes that do not fit it run every map as a head of its own, with f32 output.
//   warp 0       TMA: the queries' column blocks once, then keys and values, 64 rows at a time (four pages; a lane per page and column block), two-stage rings.
//                Heads are a tensor-map dimension of their own, so columns past a head's size arrive as zeros; pages past the end are out of bounds: zeros
//   warp 1       TMEM owner; one lane issues S_t = Q_t K^T for the NT sub-tiles (double buffered) and O_t += P_t V
//   warps 2..    one thread per row: causal, window and chunk mask, online softmax in the log2 domain, P (bf16) through swizzled shared memory
// ------------------------------------------------------------------------------------------------------------
constexpr int GF_BM = 128, GF_BN = 64;
constexpr int GF_QB = GF_BM * 128;         // one 64-column block of 128 query rows
constexpr int GF_KB = GF_BN * 128;         // one 64-column block of 64 keys
constexpr int GF_PB = GF_BM * 128;
constexpr int GF_PAGE = KV_BLOCK * 128;    // one page's share of a key block
constexpr uint32_t FT_K_GQA = 10;

FT_DEVICE bool gf_wait(uint64_t* bar, uint32_t parity) {
  if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = globaltimer_ns();
  for (uint32_t i = 1;; i++) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 0xff) == 0 && globaltimer_ns() - t0 > 2000000000ull) return false;
  }
}

struct FlashArgs {
  GqaDims D;
  MaskGate M;
  int R, tok;                      // query heads per key / value head, tokens per sub-tile
  int nq, nv;                      // 64-column blocks of key and value sizes
  int max_blocks;
  int slack;                       // bytes of shared memory left for alignment
  Differential F;
  int out_f32;                     // output rows are f32 (maps apart)
};

// two CTAs of one sub-tile per SM: their halves of tensor memory hold scores and up to two value blocks
constexpr bool gf_pair(int NT, int NV) { return NT == 1 && NV > 0 && NV <= 2; }

// NQ, NV: column blocks at compile time (the issuing thread's descriptors then are constants added to a base), or 0 to read them from A.
template <int NT, int NQ, int NV, bool DIFF>
__global__ void __launch_bounds__(64 + 128 * NT, gf_pair(NT, NV) ? 2 : 1)
gqa_flash_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQ2, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const int4* __restrict__ tiles,
                 const int* __restrict__ block_table, FlashArgs A, void* __restrict__ out, int64_t ldo, uint32_t* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  if ((int)(smem - smem_raw) > A.slack) { ft_set_status(status, FT_K_GQA, 10, 0); return; }      // dynamic shared memory starts at a multiple of 1024 here
  const int nq = NQ > 0 ? NQ : A.nq, nv = NV > 0 ? NV : A.nv;
  constexpr int KM = DIFF ? 2 : 1;                  // keys of a stage: one set per map
  const int k_bytes = KM * nq * GF_KB, v_bytes = nv * GF_KB;
  uint8_t* sQ = smem;                               // [NT][nq]
  uint8_t* sK = sQ + NT * nq * GF_QB;               // [2][KM][nq]
  uint8_t* sV = sK + 2 * k_bytes;                   // [2][nv]
  uint8_t* sP = sV + 2 * v_bytes;                   // [NT]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + NT * GF_PB);
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
  // the groups of a tile next to one another: tiles come longest first, so the CTAs do too
  const int heads = DIFF ? A.D.G : A.D.GK, maps = DIFF ? 1 : A.D.maps;
  const int4 tl = tiles[blockIdx.x / heads];        // first query row, tokens, position of the first token, sequence
  const int gk = blockIdx.x % heads, g = gk / maps, map = gk % maps;      // without DIFF a map is a key head of its own
  const int tok = A.tok, keep = A.M.keep;
  auto first_of = [&](int t) { return DIFF ? 0 : t * tok; };              // first token of a sub-tile
  // every sub-tile goes over the jk blocks of the kept first keys, then over those from j0 on, where the window of the tile's first token starts
  const int j0 = first_visible(A.M, tl.z) / GF_BN, jk = min((keep + GF_BN - 1) / GF_BN, j0);
  auto block_at = [&](int j) { return j < jk ? j : j - jk + j0; };
  int nblk[NT], nmax = 0;
#pragma unroll
  for (int t = 0; t < NT; t++) {
    const int n = min(tok, tl.y - first_of(t));
    nblk[t] = n > 0 ? (tl.z + first_of(t) + n + GF_BN - 1) / GF_BN - j0 + jk : 0;
    nmax = max(nmax, nblk[t]);
  }
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; i++) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    for (int t = 0; t < NT; t++) { mbar_init(&s_full[2 * t], 1); mbar_init(&s_full[2 * t + 1], 1); mbar_init(&p_ready[t], 128); mbar_init(&pv_done[t], 1); }
    mbar_fence_init();
  }
  if (warp == 0 && lane == 0) { tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmQ2); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV); }
  constexpr uint32_t TMEM = gf_pair(NT, NV) ? 256 : 512;
  if (warp == 1) { tmem_alloc(tmem_slot, TMEM); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tS = *tmem_slot, tO = tS + NT * 2 * GF_BN;

  if (warp == 0) {
    if (lane == 0) {
      int live = 0;
      for (int t = 0; t < NT; t++) live += nblk[t] > 0;
      mbar_expect_tx(q_full, live * nq * A.R * tok * 128);
      for (int t = 0; t < NT; t++)
        if (nblk[t] > 0)
          for (int c = 0; c < nq; c++) tma_load_3d(sQ + (t * nq + c) * GF_QB, (DIFF ? t : map) ? &tmQ2 : &tmQ, q_full, c * 64, g * A.R, tl.x + first_of(t));
    }
    __syncwarp();
    const int* bt = block_table + (size_t)tl.w * A.max_blocks;
    const int pg = lane & 3, cb = lane >> 2;        // this lane's page of a key block, and its first column block
    auto page_row = [&](int j) -> int {             // first row of that page in the cache, out of bounds past the sequence's pages
      const int p = block_at(j) * 4 + pg;
      const int blk = p < A.max_blocks ? __ldg(bt + p) : -1;
      return blk * KV_BLOCK;                        // -1: a negative coordinate, read as zeros
    };
    auto load_k = [&](int j, int y) -> bool {
      const int s = j & 1;
      const bool free_k = gf_wait(&k_empty[s], ((j >> 1) & 1) ^ 1);
      if (!__all_sync(0xffffffffu, free_k)) { if (lane == 0) ft_set_status(status, FT_K_GQA, 1, j); return false; }   // the whole warp at once
      if (lane == 0) mbar_expect_tx(&k_full[s], k_bytes);
      __syncwarp();
      for (int c = cb; c < KM * nq; c += 8)
        tma_load_3d(sK + s * k_bytes + c * GF_KB + pg * GF_PAGE, &tmK, &k_full[s], (DIFF ? c % nq : c) * 64, DIFF ? 2 * g + c / nq : gk, y);
      return true;
    };
    int y = nmax > 0 ? page_row(0) : 0;
    bool ok = nmax > 0 && load_k(0, y);
    for (int j = 0; j < nmax && ok; j++) {
      const int y_next = j + 1 < nmax ? page_row(j + 1) : 0;
      if (j + 1 < nmax) ok = load_k(j + 1, y_next);
      if (!ok) break;
      const int s = j & 1;
      const bool free_v = gf_wait(&v_empty[s], ((j >> 1) & 1) ^ 1);
      if (!__all_sync(0xffffffffu, free_v)) { if (lane == 0) ft_set_status(status, FT_K_GQA, 2, j); ok = false; break; }
      if (lane == 0) mbar_expect_tx(&v_full[s], v_bytes);
      __syncwarp();
      for (int c = cb; c < nv; c += 8) tma_load_3d(sV + s * v_bytes + c * GF_KB + pg * GF_PAGE, &tmV, &v_full[s], c * 64, g, y);
      y = y_next;
    }
    if (!ok)
      for (int i = 0; i < 64; i++) __nanosleep(1000);      // copies in flight land before the shared memory goes away
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = make_idesc_f16(GF_BM, GF_BN, 1, 0, 0);
      const uint32_t idesc_o = make_idesc_f16(GF_BM, nv * 64, 1, 0, 1);
      // a descriptor's start address counts 16-byte units in its low bits: moving inside the operand is an addition
      const uint64_t q_desc = make_smem_desc(smem_u32(sQ), 16, 1024, FT_SWZ_128B), k_desc = make_smem_desc(smem_u32(sK), 16, 1024, FT_SWZ_128B);
      const uint64_t p_desc = make_smem_desc(smem_u32(sP), 16, 1024, FT_SWZ_128B), v_desc = make_smem_desc(smem_u32(sV), GF_KB, 1024, FT_SWZ_128B);
      auto issue_s = [&](int t, int j) {
        const uint64_t qd = q_desc + (uint32_t)(t * nq) * (GF_QB / 16), kd = k_desc + (uint32_t)(j & 1) * (k_bytes / 16) + (DIFF ? (uint32_t)(t * nq) * (GF_KB / 16) : 0);
        const uint32_t d = tS + t * 2 * GF_BN + (j & 1) * GF_BN;
#pragma unroll
        for (int c = 0; c < nq; c++) {
#pragma unroll
          for (int k = 0; k < 4; k++) umma_f16_ss(d, qd + c * (GF_QB / 16) + k * 2, kd + c * (GF_KB / 16) + k * 2, idesc_s, (c | k) != 0);
        }
        umma_commit(&s_full[2 * t + (j & 1)]);
      };
      bool ok = gf_wait(q_full, 0) && gf_wait(&k_full[0], 0);
      if (!ok) ft_set_status(status, FT_K_GQA, 3, 0);
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < NT; t++)
          if (nblk[t] > 0) issue_s(t, 0);
        umma_commit(&k_empty[0]);
        for (int j = 0; j < nmax && ok; j++) {
          if (j + 1 < nmax) {
            if (!gf_wait(&k_full[(j + 1) & 1], ((j + 1) >> 1) & 1)) { ft_set_status(status, FT_K_GQA, 4, j); break; }
            tc_fence_after();
#pragma unroll
            for (int t = 0; t < NT; t++)
              if (j + 1 < nblk[t]) issue_s(t, j + 1);
            umma_commit(&k_empty[(j + 1) & 1]);
          }
          if (!gf_wait(&v_full[j & 1], (j >> 1) & 1)) { ft_set_status(status, FT_K_GQA, 5, j); break; }
          const uint64_t vd = v_desc + (uint32_t)(j & 1) * (v_bytes / 16);
#pragma unroll
          for (int t = 0; t < NT; t++) {
            if (j >= nblk[t] || !ok) continue;
            if (!gf_wait(&p_ready[t], j & 1)) { ft_set_status(status, FT_K_GQA, 6, j); ok = false; continue; }
            tc_fence_after();
#pragma unroll
            for (int k = 0; k < GF_BN / 16; k++)
              umma_f16_ss(tO + t * nv * 64, p_desc + t * (GF_PB / 16) + k * 2, vd + k * 128, idesc_o, (j | k) != 0);
            umma_commit(&pv_done[t]);
          }
          umma_commit(&v_empty[j & 1]);
        }
      }
    }
  } else {
    const int t = (warp - 2) >> 2, q = warp & 3, r = q * 32 + lane;
    const int nb = t == 0 ? nblk[0] : nblk[NT - 1];
    const int tk = r / A.R, head = (g * A.R + r % A.R) * maps + map;      // token inside the sub-tile, query head
    const bool live = tk < tok && first_of(t) + tk < tl.y;
    const int qpos = tl.z + first_of(t) + tk;
    const int lo_pos = tl.z + first_of(t), hi_pos = tl.z + min(tl.y, first_of(t) + tok) - 1;      // positions of the sub-tile
    const int wlow = first_visible(A.M, qpos) - 1, whigh = first_visible(A.M, hi_pos) - 1;   // the last positions that this row and the sub-tile's last one do not see any more
    const float scale_log2 = A.M.scale * LOG2E;
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    uint8_t* prow = sP + t * GF_PB + r * 128;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nb && ok; j++) {
      if (!gf_wait(&s_full[2 * t + (j & 1)], (j >> 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_GQA, 7, j); ok = false; break; }
      tc_fence_after();
      __syncwarp();                                            // the TMEM loads are warp-wide: every lane is here
      uint32_t sv[64];
      tmem_ld_32x32b_x32(tS + lane_off + t * 2 * GF_BN + (j & 1) * GF_BN, sv);
      tmem_ld_32x32b_x32(tS + lane_off + t * 2 * GF_BN + (j & 1) * GF_BN + 32, sv + 32);
      tmem_ld_wait();
      const int kv0 = block_at(j) * GF_BN;
      if (kv0 + GF_BN - 1 > lo_pos || (kv0 <= whigh && kv0 + GF_BN > keep)) {   // the diagonal or an edge of the visible keys can cross this block
#pragma unroll
        for (int c = 0; c < 64; c++)
          if (kv0 + c > qpos || (kv0 + c <= wlow && kv0 + c >= keep)) sv[c] = __float_as_uint(-INFINITY);
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 64; c++) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(sv[c]));
      const float m_new = fmaxf(m_used, fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])));
      // a row that has seen no key yet (all of them outside its window) stays at minus infinity with weights zero
      const bool grow = m_new != -INFINITY && (m_new - m_used) * scale_log2 > 8.f;
      const bool rescale = __any_sync(0xffffffffu, grow);
      float alpha = 1.f;
      if (rescale && m_new != -INFINITY) {
        alpha = ex2((m_used - m_new) * scale_log2);
        m_used = m_new;
      }
      const float moff = m_used == -INFINITY ? 0.f : m_used * scale_log2;
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
        if (!gf_wait(&pv_done[t], (j - 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_GQA, 8, j); ok = false; break; }
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
      if (!gf_wait(&pv_done[t], (nb - 1) & 1)) { if (lane == 0) ft_set_status(status, FT_K_GQA, 9, 0); ok = false; }
    }
    if constexpr (DIFF) {
      // row sums and sums of squares of both maps meet in shared memory; both warpgroups pass both barriers whatever happened
      float* sm_l = reinterpret_cast<float*>(tmem_slot + 4);           // [2][128], then [2][128]
      sm_l[t * 128 + r] = ok && l > 0.f ? l : 1.f;
      tc_fence_before();
      asm volatile("bar.sync 1, 256;" ::: "memory");
      tc_fence_after();
      const float k0 = 1.f / sm_l[r], k1 = A.F.lambda / sm_l[128 + r];
      const int half = nv * 32;                                        // this warpgroup's value columns
      float ss = 0.f;
#pragma unroll 1
      for (int c = 0; c < nv; c++) {
        uint32_t a[32], b[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tO + lane_off + t * half + c * 32, a);
        tmem_ld_32x32b_x32(tO + lane_off + nv * 64 + t * half + c * 32, b);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e++) {
          const float v = __uint_as_float(a[e]) * k0 - __uint_as_float(b[e]) * k1;
          ss += v * v;
        }
      }
      sm_l[256 + t * 128 + r] = ss;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      const float k = A.F.scale / sqrtf((sm_l[256 + r] + sm_l[384 + r]) / (float)A.D.dv + A.F.eps), f0 = k0 * k, f1 = k1 * k;
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(out) + (size_t)(tl.x + tk) * ldo + (size_t)head * A.D.v16;
#pragma unroll 1
      for (int c = 0; c < nv; c++) {
        uint32_t a[32], b[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tO + lane_off + t * half + c * 32, a);
        tmem_ld_32x32b_x32(tO + lane_off + nv * 64 + t * half + c * 32, b);
        tmem_ld_wait();
#pragma unroll
        for (int c8 = 0; c8 < 4; c8++) {
          const int col = t * half + c * 32 + c8 * 8;
          if (ok && live && col < A.D.v16) {
            float e[8];
#pragma unroll
            for (int i = 0; i < 8; i++) e[i] = __uint_as_float(a[8 * c8 + i]) * f0 - __uint_as_float(b[8 * c8 + i]) * f1;
            store8(dst + col, e);
          }
        }
        __syncwarp();
      }
    }
    if (!DIFF && ok && nb > 0) {
      tc_fence_after();
      const size_t row = (size_t)(tl.x + t * tok + tk);
      if (A.M.sink != nullptr && live) l += ex2(A.M.sink[head] * LOG2E - m_used * scale_log2);
      float k = A.M.out_scale / l;
      if (A.M.gate_kind == GATE_HEAD && live) k *= sigmoid_fast(reinterpret_cast<const float*>(A.M.gate)[row * A.M.ldg + head]);
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(out) + row * ldo + (size_t)head * A.D.v16;
      float* dst32 = reinterpret_cast<float*>(out) + row * ldo + (size_t)head * A.D.v16;
      const __nv_bfloat16* gate = reinterpret_cast<const __nv_bfloat16*>(A.M.gate) + row * A.M.ldg + (size_t)head * A.D.v16;
      const bool gated = A.M.gate_kind == GATE_ELEMENT;
      // rows outside the tile only skip the loads and stores: the warp-wide TMEM loads stay in code that all lanes run together
#pragma unroll 1
      for (int c = 0; c < nv * 2; c++) {
        uint32_t ov[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tO + lane_off + t * nv * 64 + c * 32, ov);
        tmem_ld_wait();
#pragma unroll
        for (int c8 = 0; c8 < 4; c8++) {
          if (live && c * 32 + c8 * 8 < A.D.v16) {
            float e[8];
#pragma unroll
            for (int i = 0; i < 8; i++) e[i] = __uint_as_float(ov[8 * c8 + i]) * k;
            if (gated) {
              float gv[8];
              load8(gate + c * 32 + c8 * 8, gv);
#pragma unroll
              for (int i = 0; i < 8; i++) e[i] *= sigmoid_fast(gv[i]);
            }
            if (A.out_f32) store8(dst32 + c * 32 + c8 * 8, e);
            else store8(dst + c * 32 + c8 * 8, e);
          }
        }
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

constexpr int SMEM_MAX = 232448;
int flash_slack(int NT, int nq, int nv) { return NT == 1 && nq == 2 && nv == 2 ? 640 : 1024; }      // two CTAs of the largest pair fit an SM to within this
int flash_smem(int NT, int nq, int nv) { return NT * nq * GF_QB + 2 * (nq + nv) * GF_KB + NT * GF_PB + 64 + 64 * NT + flash_slack(NT, nq, nv); }
int flash_diff_smem(int nq, int nv) { return flash_smem(2, nq, nv) + 2 * nq * GF_KB + 4 * 128 * 4 + 64; }      // the second map's keys, the meeting place of the maps

bool make_dims(GqaDims& D, int H, int G, int d, int dv, int rot, int maps = 1) {
  if (G < 1 || H < G || H % G || d < 1 || dv < 1 || rot < 0 || rot > d || (rot & 1) || maps < 1 || maps > 2 || H > 65535 / maps) return false;
  D = GqaDims{H, G, d, dv, (d + 15) & ~15, (dv + 15) & ~15, rot, 0, maps, H * maps, G * maps};
  D.row = G * (maps * D.d16 + D.v16);
  return true;
}
MaskGate make_mask(float scale, int window, int keep, int chunk, const float* sink, const void* gate, int64_t ldg, int kind, float out_scale) {
  return MaskGate{scale, window > 0 ? window : 0x3fffffff, keep, chunk > 0 ? chunk : 0, sink, gate, ldg, kind, out_scale};
}

template <int NT, int NQ, int NV, bool DIFF = false>
int launch_flash(const CUtensorMap (&m)[4], const int* tiles, int ntiles, const int* bt, const FlashArgs& A, void* out, int64_t ldo, int smem, cudaStream_t st) {
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    FT_CUDA_TRY(cudaFuncSetAttribute(gqa_flash_kernel<NT, NQ, NV, DIFF>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    done[dev] = true;
  }
  gqa_flash_kernel<NT, NQ, NV, DIFF><<<ntiles * (DIFF ? A.D.G : A.D.GK), 64 + 128 * NT, smem, st>>>(m[0], m[1], m[2], m[3], reinterpret_cast<const int4*>(tiles), bt, A, out,
                                                                                                    ldo, ft_status_ptr());
  return (int)cudaGetLastError();
}

template <int NP>
int launch_decode(dim3 grid, int smem, cudaStream_t st, const void* q, const void* cache, const int* bt, int mb, const int* lens, const GqaDims& D, const MaskGate& M,
                  int tiles, float* ws, int* counters, const Differential& F, void* out, int64_t ldo) {
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    FT_CUDA_TRY(cudaFuncSetAttribute(gqa_decode_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX - 8192));
    done[dev] = true;
  }
  return (int)ft_launch_pdl(gqa_decode_kernel<NP>, grid, dim3(256), (size_t)smem, st, (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, bt, mb, lens, D, M, tiles, ws,
                            counters, F, (__nv_bfloat16*)out, ldo);
}

}  // namespace

// Projection rows qkv [rows][ld] (bf16, or f32 with is_f32): H query heads, G key heads (d padded to d16 = a multiple of 16 columns each), G value heads (dv
// padded to v16). Norms queries and keys (norm 0: RMS over each head, 1: over all query and all key heads; wq, wk f32 in the same padding, one head long or
// all heads long; 2: no norm), turns the first `rot` dimensions of each (pairs of neighbouring columns, or with halves != 0 column i with i + rot / 2; tables cos / sin f32
// [position][rot / 2]), leaves the queries in place and writes keys and values to cache row slots[r] (= page * 16 + offset): [G x d16 | G x v16]. With lambda (one f32 on the device) the values become
// (1 - lambda) v + lambda vfirst (rows of G * v16, pitch ldf). maps = 2: two query and two key vectors per head, next to one another. cache null: queries alone.
FT_EXPORT int ft_gqa_prep(void* qkv, int64_t ld, int rows, int H, int G, int d, int dv, int maps, int rot, int norm, int halves, const float* wq, const float* wk, float eps,
                          const int* positions, const float* cos_t, const float* sin_t, const int* slots, void* cache, const void* vfirst, int64_t ldf, const float* lambda, int is_f32,
                          cudaStream_t st) {
  PrepArgs A{};
  if (rows < 1 || !make_dims(A.D, H, G, d, dv, rot, maps) || (ld & 7) || ld < (int64_t)A.D.HQ * A.D.d16 + (cache ? A.D.GK * A.D.d16 + G * A.D.v16 : 0) || (lambda && (!vfirst || (ldf & 7))) ||
      norm < NORM_HEAD || norm > NORM_NONE || (norm != NORM_NONE && !(wq && wk)))
    return FT_ERR_ARG;
  const bool whole = norm == NORM_WHOLE;
  A.halves = halves;
  A.wq = norm == NORM_NONE ? nullptr : wq; A.wk = wk; A.eps = eps; A.positions = positions; A.cos_t = cos_t; A.sin_t = sin_t; A.slots = slots;
#define FT_GP(T, W) gqa_prep_kernel<T, W><<<rows, PREP_T, 0, st>>>((T*)qkv, ld, A, (T*)cache, (const T*)vfirst, ldf, lambda)
  if (is_f32) { if (whole) FT_GP(float, true); else FT_GP(float, false); }
  else { if (whole) FT_GP(__nv_bfloat16, true); else FT_GP(__nv_bfloat16, false); }
#undef FT_GP
  return (int)cudaGetLastError();
}

// Plain attention over cached rows: q [rows][ldq] as left by ft_gqa_prep; row r of sequence seq_of[r] sees the last `window` (0: all) of the positions
// 0..positions[r] and the first `keep` of them; sink f32 [H] or null; gate_kind 0: none, 1: rows of H * v16 pre-activations in the data type (pitch ldg), 2: f32 rows of H; out [rows][ldo], heads of
// v16, times out_scale. chunk > 0: a position sees only those of its own chunk. maps = 2: rows of H * 2 heads, the maps apart. out is f32 with out_f32, else of the data
// type. Value sizes up to 1024.
FT_EXPORT int ft_gqa_rows(const void* q, int64_t ldq, const void* cache, const int* block_table, int max_blocks, const int* seq_of, const int* positions, int rows, int H, int G,
                          int d, int dv, int maps, float scale, int window, int keep, int chunk, const float* sink, const void* gate, int64_t ldg, int gate_kind,
                          float out_scale, void* out, int64_t ldo, int out_f32, int is_f32, cudaStream_t st) {
  GqaDims D;
  if (rows < 1 || keep < 0 || !make_dims(D, H, G, d, dv, 0, maps) || (gate_kind && !gate) || (maps > 1 && (gate_kind || sink))) return FT_ERR_ARG;
  if (D.v16 > 128 * ROWS_MAX_COLS || D.d16 > 8192) return FT_ERR_TOO_LARGE;
  const MaskGate M = make_mask(scale, window, keep, chunk, sink, gate, ldg, gate_kind, out_scale);
  const dim3 grid(rows, D.HQ);
#define FT_GR(T, O) gqa_rows_kernel<T, O><<<grid, 128, D.d16 * 4, st>>>((const T*)q, ldq, (const T*)cache, block_table, max_blocks, seq_of, positions, D, M, (O*)out, ldo)
  if (is_f32) FT_GR(float, float);
  else if (out_f32) FT_GR(__nv_bfloat16, float);
  else FT_GR(__nv_bfloat16, __nv_bfloat16);
#undef FT_GR
  return (int)cudaGetLastError();
}

// Differential heads: out[r][h] = o / sqrt(mean(o^2) + eps) * scale with o = a[r][h][0] - lambda a[r][h][1]; a: f32 rows of H * 2 heads of v16 (zeros past dv, pitch a
// multiple of 4), out: bf16, or f32 with is_f32. Value sizes up to 1024.
FT_EXPORT int ft_gqa_differential(const float* a, int64_t lda, int rows, int H, int dv, float lambda, float scale, float eps, void* out, int64_t ldo, int is_f32, cudaStream_t st) {
  GqaDims D;
  if (rows < 1 || !make_dims(D, H, 1, 1, dv, 0, 2) || (lda & 3)) return FT_ERR_ARG;
  if (D.v16 > 128 * ROWS_MAX_COLS || (int64_t)rows * H > 0x7ffffff0) return FT_ERR_TOO_LARGE;
  const Differential F{1, lambda, scale, eps};
  const int units = rows * H;
  if (is_f32) gqa_differential_kernel<float><<<(units + 7) / 8, 256, 0, st>>>(a, lda, D, F, units, (float*)out, ldo);
  else gqa_differential_kernel<__nv_bfloat16><<<(units + 7) / 8, 256, 0, st>>>(a, lda, D, F, units, (__nv_bfloat16*)out, ldo);
  return (int)cudaGetLastError();
}

// ft_gqa_prep for one token of B <= 16 sequences, from split-K planes of the projection (columns as there; gate pre-activations from column gate_col on, kind as in
// ft_gqa_rows): queries q bf16 [B][H][d16], cache row of each sequence's current position, sigmoid of the gate (f32 [B][H * v16] or [B][H]). vf_out (f32
// [B][G * v16]) keeps the values; vf_in and lambda mix such values in. cache null: queries alone. Head sizes up to 512. maps = 2: queries [B][H * 2][2 * d16], each in its own
// map's half (the other half, zero, is not written).
FT_EXPORT int ft_gqa_decode_prep(const float* planes, int splits, int64_t ldp, int64_t plane_stride, int B, int H, int G, int d, int dv, int maps, int rot, int norm, int halves,
                                 const float* wq, const float* wk, float eps, const int* positions, const float* cos_t, const float* sin_t, const int* block_table, int max_blocks,
                                 int gate_col, int gate_kind, float* gate, float* vf_out, const float* vf_in, const float* lambda, void* q, void* cache, cudaStream_t st) {
  DecPrepArgs A{};
  GqaDims& D = A.P.D;
  if (B < 1 || B > DEC_TOK || splits < 1 || !make_dims(D, H, G, d, dv, rot, maps) || (ldp & 3) || (plane_stride & 3) || (gate_col & 3) || (gate_kind && !gate) ||
      (lambda && !vf_in) || norm < NORM_HEAD || norm > NORM_NONE || (norm != NORM_NONE && !(wq && wk)))
    return FT_ERR_ARG;
  if (D.d16 > 128 * DP_MAXC) return FT_ERR_TOO_LARGE;
  A.P.halves = halves;
  A.P.wq = norm == NORM_NONE ? nullptr : wq; A.P.wk = wk; A.P.eps = eps; A.P.positions = positions; A.P.cos_t = cos_t; A.P.sin_t = sin_t;
  A.planes = planes; A.splits = splits; A.ldp = ldp; A.pstride = (size_t)plane_stride; A.block_table = block_table; A.max_blocks = max_blocks;
  A.gate_col = gate_col; A.gate_kind = gate_kind; A.gate = gate; A.vf_out = vf_out; A.vf_in = vf_in; A.lambda = lambda;
  const int gate_cols = gate_kind == GATE_ELEMENT ? H * D.v16 : gate_kind == GATE_HEAD ? H : 0;
  const int units = D.HQ + (cache ? D.GK + G : 0) + (gate_cols + 127) / 128;
  int ctas = (units + DP_WARPS - 1) / DP_WARPS;
  if (norm != NORM_WHOLE)
    return (int)ft_launch_pdl(gqa_decode_prep_kernel<false>, dim3(ctas, B), dim3(DP_WARPS * 32), halves ? (size_t)DP_WARPS * D.d16 * 4 : 0, st, A, (__nv_bfloat16*)q, (__nv_bfloat16*)cache);
  int cl = 1;
  while (cl < 8 && cl < ctas) cl *= 2;
  ctas = cl;
  const size_t smem = (size_t)((D.HQ + D.GK + ctas * DP_WARPS - 1) / (ctas * DP_WARPS)) * DP_WARPS * D.d16 * 4;
  if (smem > (size_t)SMEM_MAX - 1024) return FT_ERR_TOO_LARGE;
  if (smem > 48 * 1024) FT_CUDA_TRY(cudaFuncSetAttribute(gqa_decode_prep_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX - 1024));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(ctas, B);
  cfg.blockDim = dim3(DP_WARPS * 32);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = ctas;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ft_pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, gqa_decode_prep_kernel<true>, A, (__nv_bfloat16*)q, (__nv_bfloat16*)cache);
}

// Attention of one token per sequence over its visible cached rows (seq_lens[b] rows, the newest included, or the last `window` and the first `keep` of them); q and gate as written by
// ft_gqa_decode_prep. ws: f32 [B][G * ceil(H / G / 16)][nsplit][16][v16 + 4], 16-byte aligned; counters: int [B][G * ceil(H / G / 16)], zero before the first
// launch (the kernel leaves them zero). nsplit <= 64; value sizes up to 512. out: bf16 [B][ldo], heads of v16. chunk > 0: only rows of the newest position's chunk.
// maps = 2: q as ft_gqa_decode_prep leaves it, without sink and gate; groups count 2 H / G rows, the heads' outputs are those of ft_gqa_differential (lambda, dscale, eps).
FT_EXPORT int ft_gqa_decode(const void* q, const void* cache, const int* block_table, int max_blocks, const int* seq_lens, int B, int H, int G, int d, int dv, int maps,
                            float scale, int window, int keep, int chunk, const float* sink, const float* gate, int gate_kind, float out_scale, float lambda, float dscale,
                            float eps, int nsplit, float* ws, int* counters, void* out, int64_t ldo, cudaStream_t st) {
  GqaDims D;
  if (maps < 1 || maps > 2 || H < 1 || H > 32767 || d < 1 || d > 65536) return FT_ERR_ARG;
  if (maps == 2) { H *= 2; d = 2 * ((d + 15) & ~15); }
  if (B < 1 || keep < 0 || nsplit < 1 || nsplit > GD_MAX_SPLIT || !make_dims(D, H, G, d, dv, 0) || (reinterpret_cast<uintptr_t>(ws) & 15) || (ldo & 3) || (gate_kind && !gate) ||
      (maps == 2 && (gate_kind || sink)))
    return FT_ERR_ARG;
  const Differential F{maps == 2, lambda, dscale, eps};
  const MaskGate M = make_mask(scale, window, keep, chunk, sink, gate, 0, gate_kind, out_scale);
  const int smem = gd_smem(D.d16, D.v16), np = (D.v16 / 16 + 7) / 8, tiles = (H / G + GD_HT - 1) / GD_HT;
  if (smem > SMEM_MAX - 8192 || np > 4) return FT_ERR_TOO_LARGE;
  const dim3 grid(nsplit, G * tiles, B);
#define FT_GD(N) return launch_decode<N>(grid, smem, st, q, cache, block_table, max_blocks, seq_lens, D, M, tiles, ws, counters, F, out, ldo)
  if (np <= 1) FT_GD(1);
  if (np <= 2) FT_GD(2);
  FT_GD(4);
#undef FT_GD
}

// Whether ft_gqa_decode_prep and ft_gqa_decode take these sizes.
FT_EXPORT int ft_gqa_decode_fits(int H, int G, int d, int dv, int maps) {
  GqaDims D;
  return make_dims(D, H, G, d, dv, 0, maps) && D.d16 <= 128 * DP_MAXC && D.v16 <= 512 && gd_smem(maps * D.d16, D.v16) <= SMEM_MAX - 8192 &&
         (size_t)((D.HQ + D.GK + 63) / 64) * DP_WARPS * D.d16 * 4 <= (size_t)SMEM_MAX - 1024;
}

// How ft_gqa_flash combines the maps of differential heads of these sizes: 1 itself, 0 not at all (f32 rows of every map for ft_gqa_differential).
FT_EXPORT int ft_gqa_flash_joins_maps(int d, int dv) {
  const int nq = (d + 63) / 64, nv = (dv + 63) / 64;
  return nv <= 2 && flash_diff_smem(nq, nv) <= SMEM_MAX;
}

// Sub-tiles (of 128 / (H / G) tokens each) per tile of ft_gqa_flash: 1 or 2; 0 when these sizes do not fit the kernel (use ft_gqa_rows).
FT_EXPORT int ft_gqa_flash_subtiles(int H, int G, int d, int dv, int maps) {
  GqaDims D;
  if (!make_dims(D, H, G, d, dv, 0, maps) || H / G > GF_BM) return 0;
  const int nq = (d + 63) / 64, nv = (dv + 63) / 64;
  if (maps == 2 && ft_gqa_flash_joins_maps(d, dv)) return 1;
  if (nq <= 2 && nv <= 2) return 1;                    // two CTAs of one sub-tile per SM
  if (nv <= 2 && flash_smem(2, nq, nv) <= SMEM_MAX) return 2;
  if (nv <= 4 && flash_smem(1, nq, nv) <= SMEM_MAX) return 1;
  return 0;
}

// Attention of a ragged batch of prompts or portions: q bf16 [q_rows][ldq] as left by ft_gqa_prep; keys and values from the cache's pages [pages][16][row] (those
// of the new tokens included). tiles: int4 per tile {first query row, tokens (<= subtiles * (128 / (H / G))), position of the first token, row of block_table}.
// Mask, sink, gate and output as in ft_gqa_rows (out_f32: f32 rows). Leading dimensions are multiples of 8. maps = 2 (no sink, no gate): the combined heads, bf16, where
// ft_gqa_flash_joins_maps says so (lambda, dscale, eps as in ft_gqa_differential), else the maps apart.
FT_EXPORT int ft_gqa_flash(const void* q, int64_t ldq, int q_rows, const void* cache, int pages, const int* block_table, int max_blocks, const int* tiles, int ntiles, int H,
                           int G, int d, int dv, int maps, float scale, int window, int keep, int chunk, const float* sink, const void* gate, int64_t ldg, int gate_kind,
                           float out_scale, float lambda, float dscale, float eps, void* out, int64_t ldo, int out_f32, cudaStream_t st) {
  FlashArgs A{};
  GqaDims& D = A.D;
  if (q_rows < 1 || pages < 1 || ntiles < 1 || keep < 0 || !make_dims(D, H, G, d, dv, 0, maps) || (ldq & 7) || (ldo & 7) || (gate_kind && !gate) ||
      (gate_kind == GATE_ELEMENT && (ldg & 7)) || (maps == 2 && (gate_kind || sink)))
    return FT_ERR_ARG;
  const int nt = ft_gqa_flash_subtiles(H, G, d, dv, maps);
  if (nt == 0) return FT_ERR_TOO_LARGE;
  const bool join = maps == 2 && ft_gqa_flash_joins_maps(d, dv);
  if (join && out_f32) return FT_ERR_ARG;
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  FT_CUDA_TRY(ft_bind_context(dev));
  A.M = make_mask(scale, window, keep, chunk, sink, gate, ldg, gate_kind, out_scale);
  A.F = Differential{join, lambda, dscale, eps};
  A.out_f32 = out_f32;
  A.R = H / G;
  A.tok = GF_BM / A.R;
  A.nq = (d + 63) / 64;
  A.nv = (dv + 63) / 64;
  A.max_blocks = max_blocks;
  CUtensorMap m[4];
  const __nv_bfloat16 *cp = (const __nv_bfloat16*)cache, *qp = (const __nv_bfloat16*)q;
  const uint64_t krow = (uint64_t)D.row * 2, slots = (uint64_t)pages * KV_BLOCK, qhead = (uint64_t)D.d16 * maps * 2;
  int r = ft_make_tmap_3d(&m[0], qp, 2, true, D.d16, H, q_rows, qhead, (uint64_t)ldq * 2, 64, A.R, A.tok, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[1], qp + (maps == 2 ? D.d16 : 0), 2, true, D.d16, H, q_rows, qhead, (uint64_t)ldq * 2, 64, A.R, A.tok, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[2], cp, 2, true, D.d16, D.GK, slots, (uint64_t)D.d16 * 2, krow, 64, 1, KV_BLOCK, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[3], cp + (size_t)D.GK * D.d16, 2, true, D.v16, G, slots, (uint64_t)D.v16 * 2, krow, 64, 1, KV_BLOCK, CU_TENSOR_MAP_SWIZZLE_128B);
  if (r) return r;
  A.slack = join ? 1024 : flash_slack(nt, A.nq, A.nv);
  const int smem = join ? flash_diff_smem(A.nq, A.nv) : flash_smem(nt, A.nq, A.nv);
#define FT_GF(T, Q, V) return launch_flash<T, Q, V>(m, tiles, ntiles, block_table, A, out, ldo, smem, st)
#define FT_GFD(Q, V) return launch_flash<2, Q, V, true>(m, tiles, ntiles, block_table, A, out, ldo, smem, st)
  if (join) {
    if (A.nq == 1 && A.nv == 1) FT_GFD(1, 1);
    if (A.nq == 1 && A.nv == 2) FT_GFD(1, 2);
    if (A.nq == 2 && A.nv == 2) FT_GFD(2, 2);
    FT_GFD(0, 0);
  }
  if (nt == 2) FT_GF(2, 0, 0);
  if (A.nq == 1 && A.nv == 1) FT_GF(1, 1, 1);
  if (A.nq == 2 && A.nv == 1) FT_GF(1, 2, 1);
  if (A.nq == 1 && A.nv == 2) FT_GF(1, 1, 2);
  if (A.nq == 2 && A.nv == 2) FT_GF(1, 2, 2);
  FT_GF(1, 0, 0);
#undef FT_GF
#undef FT_GFD
}
