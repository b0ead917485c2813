// Matrix memory (the mLSTM cell of Beck et al., "xLSTM: Extended Long Short-Term Memory", 2024). A head remembers a d x dv matrix S, a vector n of size d and a level m,
// all zero ahead of the first token; S and n are kept divided by e^m. A token with log forget gate f, log input gate i, query q (scaled), key k and value v does
//
//   level   m'   = larger of m + f and i           keep = e^(m + f - m'),  take = e^(i - m')
//   memory  S'   = keep S + take k v^T             n'   = keep n + take k
//   output  S'^T q divided by (1e-6 + larger of |n' . q| and e^(-m'))
//
// followed by an RMS norm of every head's output, a weight, a sigmoid gate and a scale. States live in f32, one slot per sequence: [heads][d16 x v16 | n (d16) |
// m, 3 spare], head sizes padded to multiples of 16 with zeros.
//
// A stretch of tokens can be taken at once. With F the running sum of f and u_s = i_s - F_s inside the stretch, R_t = max(m_in, max_(s <= t) u_s):
//   m_t = F_t + R_t,   weight of key s at t: e^(u_s - R_t),   weight of the state before the stretch: e^(m_in - R_t)
// so nothing but differences of nearby numbers is exponentiated, and every exponent is at most zero.
//
//   ft_mm_walk     prompts (bf16, tcgen05): a CTA walks a segment of a sequence in chunks of 128 tokens with 128 value columns of one head's state in registers.
//                  Long sequences are cut into segments that walk at the same time: a first pass collects every segment's own contribution,
//                  ft_mm_merge chains them into the state ahead of each segment, a second pass produces the outputs. What enters the states meets the
//                  16-bit tensor cores as sums of two bf16 numbers.
//   ft_mm_rows     one token after another, any sizes, f32 or bf16 data (the 32-bit path)
//   ft_mm_finish   norm, gate, scale of the outputs; moves n and m of the finished stretch into the slots
//   ft_mm_decode   one token per sequence from split-K planes: the state is read and written once; the CTAs of a head form a cluster
// Compiled without fast-math.
#include <cooperative_groups.h>

#include "common.cuh"
#include "host_common.h"

namespace {

struct MemDims {
  int H, d, dv, d16, v16;
  int h8;                            // gate columns per kind (heads padded to a multiple of 8)
  float cap;                         // soft limit of the gates' pre-activations
  __host__ __device__ size_t head() const { return (size_t)d16 * v16 + d16 + 4; }
};
constexpr float DEN_EPS = 1e-6f;

FT_DEVICE float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
FT_DEVICE float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
FT_DEVICE float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
template <typename T> FT_DEVICE float one(T v);
template <> FT_DEVICE float one<float>(float v) { return v; }
template <> FT_DEVICE float one<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> FT_DEVICE T to(float v);
template <> FT_DEVICE float to<float>(float v) { return v; }
template <> FT_DEVICE __nv_bfloat16 to<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// A segment of a sequence's new tokens: {first row, rows, state slot, sequence, flags, scratch state}
constexpr int SEG_INTS = 8, SEG_ONLY = 1, SEG_LAST = 2, SEG_ZERO = 4;      // ONLY: state from the slot, not from scratch; ZERO: the sequence starts, its slot's content is void
struct MemIO {
  const void* x;                     // [rows][ld]: queries H x d16 | keys H x d16 | values H x v16 | gates H x v16
  int64_t ld;
  const float* gates;                // [rows][ldg]: input gates (h8 columns), forget gates; pre-activations without bias
  int64_t ldg;
  const float *bi, *bf;              // [H]
  const int* segs;
  float* slots;                      // [slot][slot_stride]
  size_t slot_stride;
  float* nm;                         // [sequence][H][d16 + 4]: n and m after the stretch
  void* o;                           // [rows][H * v16] in the data type
};

// ------------------------------------------------------------------------------------------------------------
// token by token: grid (ceil(v16 / 32), H, sequences), 256 threads: 32 value columns x 8 groups of state rows
// ------------------------------------------------------------------------------------------------------------
constexpr int MR_COLS = 32;
template <typename T>
__global__ void __launch_bounds__(256) mm_rows_kernel(MemIO io, MemDims D) {
  extern __shared__ __align__(16) float sm[];
  float* S = sm;                              // [d16][32]
  float* n = S + D.d16 * MR_COLS;
  float* q = n + D.d16;
  float* k = q + D.d16;
  float* red = k + D.d16;                     // [8][32] + 32
  const int* sg = io.segs + (size_t)blockIdx.z * SEG_INTS;
  const int row0 = sg[0], rows = sg[1], flags = sg[4], hd = blockIdx.y, c = threadIdx.x & 31, rg = threadIdx.x >> 5, col = blockIdx.x * MR_COLS + c;
  float* st = io.slots + (size_t)sg[2] * io.slot_stride + hd * D.head();
  const float* sn = st + (size_t)D.d16 * D.v16;
  const bool zero = flags & SEG_ZERO;
  for (int r = rg; r < D.d16; r += 8) S[r * MR_COLS + c] = zero || col >= D.v16 ? 0.f : st[(size_t)r * D.v16 + col];
  for (int r = threadIdx.x; r < D.d16; r += 256) n[r] = zero ? 0.f : sn[r];
  float m = zero ? 0.f : sn[D.d16];
  const float scale = 1.f / sqrtf((float)D.d);
  const T* x = reinterpret_cast<const T*>(io.x);
  for (int t = 0; t < rows; t++) {
    const T* xr = x + (size_t)(row0 + t) * io.ld;
    const float* gr = io.gates + (size_t)(row0 + t) * io.ldg;
    for (int r = threadIdx.x; r < D.d16; r += 256) {
      q[r] = one(xr[hd * D.d16 + r]) * scale;
      k[r] = one(xr[(D.H + hd) * D.d16 + r]);
    }
    const float v = col < D.v16 ? one(xr[2 * D.H * D.d16 + hd * D.v16 + col]) : 0.f;
    const float ig = soft_cap(gr[hd] + io.bi[hd], D.cap), fg = log_sigmoid(soft_cap(gr[D.h8 + hd] + io.bf[hd], D.cap));
    const float mn = fmaxf(fg + m, ig), keep = expf(fg + m - mn), add = expf(ig - mn);
    m = mn;
    __syncthreads();
    float acc = 0.f, nq = 0.f;
    for (int r = rg; r < D.d16; r += 8) {
      const float s = keep * S[r * MR_COLS + c] + add * k[r] * v;
      S[r * MR_COLS + c] = s;
      acc += s * q[r];
    }
    for (int r = threadIdx.x; r < D.d16; r += 256) {
      n[r] = keep * n[r] + add * k[r];
      nq += n[r] * q[r];
    }
    red[rg * 32 + c] = acc;
    nq = block_sum(nq, red + 256);            // its barriers also publish red
    if (rg == 0) {
      float a = 0.f;
#pragma unroll
      for (int g = 0; g < 8; g++) a += red[g * 32 + c];
      if (col < D.v16) reinterpret_cast<T*>(io.o)[(size_t)(row0 + t) * D.H * D.v16 + hd * D.v16 + col] = to<T>(a / (fmaxf(fabsf(nq), expf(-m)) + DEN_EPS));
    }
    __syncthreads();
  }
  for (int r = rg; r < D.d16; r += 8)
    if (col < D.v16) st[(size_t)r * D.v16 + col] = S[r * MR_COLS + c];
  if (blockIdx.x == 0) {                      // the other CTAs of this head may not have read n yet: it moves into the slot later
    float* d = io.nm + ((size_t)sg[3] * D.H + hd) * (D.d16 + 4);
    for (int r = threadIdx.x; r < D.d16; r += 256) d[r] = n[r];
    if (threadIdx.x == 0) d[D.d16] = m;
  }
}

// ------------------------------------------------------------------------------------------------------------
// chunk walk (tcgen05): grid (segments, H, ceil(v16 / 128)), 384 threads. A chunk is 128 tokens; a CTA keeps 128 value columns of the state, transposed: thread
// (row v, half) of the first eight warps holds S[half of the key dimensions][v] in f32 registers, and as bf16 in TMEM, where it is an operand of the tensor cores.
//
//   scores [t][s]  = Q K^T                                                          (Q, K from shared memory)
//   O1 [v][t]      = S^T Q^T      (S^T from TMEM)                                   the past, scaled per token when it is read
//   nq [t]         = Q n          (n: high + low part)
//   O2 [v][t]      = V^T P^T      (P = masked, weighted scores)                     the chunk itself
//   dS [v][d]      = (w V)^T K    (w V: values times their weight in the next state, high + low);  S <- decay S + dS in f32
//   n <- decay n + sum_t w_t k_t  on the FMA pipes, under dS
//
// What enters the state (w V) and the normaliser meet the 16-bit tensor cores as sums of two bf16 numbers, so that states are exact to 16 mantissa bits per
// addend; the read-out takes P and S in bf16, as attention takes its weights.
//
// Warps 0..7: weights of the keys, outputs, state. Warp 8: issues copies and products. Warps 9..11: w V; warp 9 also the gates of the next chunk. Named barriers separate
// the steps of a chunk, which depend on one another. Shared memory: Q (then w V) | K | V | P (of its second 64 columns only the lower rows exist) | n as an
// operand. TMEM: [scores, then O2 | O1], later dS over both | S^T | nq.
// ------------------------------------------------------------------------------------------------------------
constexpr int MW_C = 128, MW_V = 128, MW_BLK = MW_C * 128;      // chunk, value columns, bytes of a 64-column block of 128 rows
constexpr int MW_THREADS = 384, MW_GATES = 6 * MW_C + 8;        // floats of one chunk's gate arrays
constexpr int MW_VEC = 16 * 128;                                // bytes of a 64-column block of a 16-row operand (rows: high, low, zeros)
constexpr int MW_REGS = 168, MW_REGS_STATE = 208, MW_REGS_HELP = 88;
constexpr uint32_t FT_K_MEMORY = 11;

FT_DEVICE float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
FT_DEVICE float exp_fast(float x) { return ex2(x * 1.4426950408889634f); }
FT_DEVICE bool mw_wait(uint64_t* bar, uint32_t parity) {
  if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = globaltimer_ns();
  for (uint32_t i = 1;; i++) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 0xff) == 0 && globaltimer_ns() - t0 > 2000000000ull) return false;
  }
}
// bar.sync counts whole warps: lanes that a wait has let go one by one come together first
FT_DEVICE void bar_named(int id, int threads) {
  __syncwarp();
  asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory");
}
template <int N> FT_DEVICE void reg_inc() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(N)); }
template <int N> FT_DEVICE void reg_dec() { asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(N)); }
// two neighbouring f32 values as bf16 high parts and bf16 remainders (16 mantissa bits together)
FT_DEVICE uint32_t pack2(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}
FT_DEVICE void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack2(a, b);
  lo = pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
// 16-byte chunk c of row r in a block of 128-byte rows, as TMA and the tensor cores place it
FT_DEVICE uint32_t sw128(int r, int c) { return (uint32_t)(r * 128 + ((c ^ (r & 7)) << 4)); }
// element i of a 16-row operand: high part in row 0, remainder in row 1
FT_DEVICE void put_vec(uint8_t* base, int i, float v) {
  uint8_t* b = base + (i >> 6) * MW_VEC;
  const int e = i & 63;
  const __nv_bfloat16 h = __float2bfloat16(v);
  *reinterpret_cast<__nv_bfloat16*>(b + sw128(0, e >> 3) + (e & 7) * 2) = h;
  *reinterpret_cast<__nv_bfloat16*>(b + sw128(1, e >> 3) + (e & 7) * 2) = __float2bfloat16(v - __bfloat162float(h));
}

__host__ __device__ constexpr int mw_smem(int nq, bool out) {
  return 4 * MW_BLK + nq * MW_BLK + 2 * MW_BLK + (out ? MW_BLK + MW_BLK / 2 : 0) + nq * MW_VEC + (2 * MW_GATES + 4 * MW_C + 64 * nq) * 4 + 64 + 1024;
}

// NQ: 64-column blocks of the key size. OUT: outputs from the state ahead of the segment; else: the segment's own contribution, into scratch state [scratch index + 1],
// with m relative to an empty past and the sum of the forget gates beside it.
template <int NQ, bool OUT>
__global__ void __launch_bounds__(MW_THREADS, 1) mm_walk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                                                                MemIO io, MemDims D, float* __restrict__ scratch, uint32_t* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;                                    // four blocks: queries [NQ]; later w V: high (two blocks), low (two blocks)
  uint8_t* sK = sQ + 4 * MW_BLK;                         // [NQ]
  uint8_t* sV = sK + NQ * MW_BLK;                        // [2]
  uint8_t* sP = sV + 2 * MW_BLK;                         // block of columns 0..63, half block of columns 64..127
  uint8_t* sN = sP + (OUT ? MW_BLK + MW_BLK / 2 : 0);    // [NQ] n as an operand
  // per chunk, two in turn: [128] u = i - F | running maximum R of u and m_in | weight in the next state | weight of the past times the queries' scale | e^(-m), then
  // 1 / denominator | e^(u - largest u of its 32 tokens) | those four maxima | sum of the forget gates
  float* gate_sets = reinterpret_cast<float*>(sN + NQ * MW_VEC);
  float* rs = gate_sets + 2 * MW_GATES;                  // [2][128] sums of the key weights
  float* raw = rs + 2 * MW_C;                            // [2][128] log gates of the next chunk
  float* nf = raw + 2 * MW_C;                            // [64 NQ] n
  uint64_t* bars = reinterpret_cast<uint64_t*>(nf + 64 * NQ);
  uint64_t *b_load = bars, *b_s = bars + 1, *b_o1 = bars + 2, *b_o2 = bars + 3, *b_ds = bars + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);
  volatile int* failed = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int* sg = io.segs + (size_t)blockIdx.x * SEG_INTS;
  const int row0 = sg[0], rows = sg[1], flags = sg[4], hd = blockIdx.y, v0 = blockIdx.z * MW_V;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool zero = !OUT || ((flags & SEG_ONLY) && (flags & SEG_ZERO));
  float* slot = io.slots + (size_t)sg[2] * io.slot_stride + hd * D.head();
  const float* in = (flags & SEG_ONLY) ? slot : scratch + (size_t)sg[5] * D.H * D.head() + hd * D.head();
  const size_t n_at = (size_t)D.d16 * D.v16;

  if (tid == 0) {
    for (int i = 0; i < 5; i++) mbar_init(&bars[i], 1);
    mbar_fence_init();
    *failed = 0;
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
  }
  if (warp == 8) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  for (int i = tid; i < NQ * MW_VEC / 16; i += MW_THREADS) reinterpret_cast<uint4*>(sN)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < 64 * NQ; i += MW_THREADS) nf[i] = zero || i >= D.d16 ? 0.f : in[n_at + i];
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tX = *tmem_slot, tA = tX + 256, tNq = tX + 384;
  float m_in = OUT ? (zero ? 0.f : in[n_at + D.d16 + ((flags & SEG_ONLY) ? 0 : 2)]) : -INFINITY;
  bool ok = true;
  // a wait that ran out: everybody keeps to the barriers and leaves at the next chunk
  auto wait = [&](uint64_t* bar, int par, uint32_t site) {
    if (ok && !mw_wait(bar, par)) {
      ft_set_status(status, FT_K_MEMORY, site, blockIdx.x);
      *failed = 1;
      ok = false;
    }
  };
  // values times their weight in the next state, over the queries: 16-byte pieces first, first + step, ...
  auto weigh_values = [&](const float* w, int first, int step) {
#pragma unroll 2
    for (int i = first; i < 2 * MW_C * 8; i += step) {
      const int r = (i >> 3) & (MW_C - 1);
      const uint32_t at = (i >> 10) * MW_BLK + sw128(r, i & 7);
      const float k = w[r];
      float v8[8];
      bf16x8_to_float(*reinterpret_cast<const bf16x8*>(sV + at), v8);
      uint32_t h[4], l[4];
#pragma unroll
      for (int e = 0; e < 4; e++) split2(v8[2 * e] * k, v8[2 * e + 1] * k, h[e], l[e]);
      *reinterpret_cast<uint4*>(sQ + at) = make_uint4(h[0], h[1], h[2], h[3]);
      *reinterpret_cast<uint4*>(sQ + 2 * MW_BLK + at) = make_uint4(l[0], l[1], l[2], l[3]);
    }
  };
  enum { BAR_CHUNK = 1, BAR_P, BAR_DEN, BAR_STATE, BAR_N, BAR_GATES };

  if (warp >= 8) {
    if constexpr (NQ > 2) reg_dec<MW_REGS_HELP>();
    // gates of a chunk (one warp), four neighbouring tokens a lane: running sum of the forget gates, running maximum
    const float bias_i = io.bi[hd], bias_f = io.bf[hd], scale = rsqrtf((float)D.d);
    auto fetch_gates = [&](int c0) {                     // warps 9..11
      for (int i = tid - 288; i < MW_C; i += 96) {
        const int t = c0 + i;
        float ig = -INFINITY, fg = 0.f;
        if (t < rows) {
          const float* gr = io.gates + (size_t)(row0 + t) * io.ldg;
          ig = soft_cap(gr[hd] + bias_i, D.cap);
          fg = log_sigmoid(soft_cap(gr[D.h8 + hd] + bias_f, D.cap));
        }
        raw[i] = ig;
        raw[MW_C + i] = fg;
      }
    };
    auto make_gates = [&](float m, int set) {
      float* g = gate_sets + set * MW_GATES;
      float F[4], uu[4], s = 0.f;
#pragma unroll
      for (int e = 0; e < 4; e++) {
        s += raw[MW_C + lane * 4 + e];
        F[e] = s;
        uu[e] = raw[lane * 4 + e];
      }
      float tot = s;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, tot, o);
        if (lane >= o) tot += y;
      }
      const float ahead = tot - s;
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < 4; e++) {
        F[e] += ahead;
        uu[e] -= F[e];
        mx = fmaxf(mx, uu[e]);
      }
      float top = mx;                                    // of the 32 tokens that eight lanes hold
#pragma unroll
      for (int o = 1; o < 8; o <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
      if ((lane & 7) == 0) g[6 * MW_C + (lane >> 3)] = top;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, y);
      }
      float before = __shfl_up_sync(0xffffffffu, mx, 1);
      before = fmaxf(lane == 0 ? -INFINITY : before, m);
      const float last = fmaxf(__shfl_sync(0xffffffffu, mx, 31), m);
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = lane * 4 + e;
        before = fmaxf(before, uu[e]);
        g[t] = uu[e];
        g[MW_C + t] = before;
        g[2 * MW_C + t] = exp_fast(uu[e] - last);
        g[3 * MW_C + t] = exp_fast(m - before) * scale;
        g[4 * MW_C + t] = exp_fast(-(F[e] + before));
        g[5 * MW_C + t] = top == -INFINITY ? 0.f : exp_fast(uu[e] - top);
      }
      if (lane == 31) g[6 * MW_C + 4] = F[3];
    };
    auto load_chunk = [&](int c0) {                      // one thread
      mbar_expect_tx(b_load, ((OUT ? NQ : 0) + NQ + 2) * MW_BLK);
      for (int c = 0; c < NQ; c++) {
        if (OUT) tma_load_3d(sQ + c * MW_BLK, &tmQ, b_load, c * 64, hd, row0 + c0);
        tma_load_3d(sK + c * MW_BLK, &tmK, b_load, c * 64, hd, row0 + c0);
      }
      for (int c = 0; c < 2; c++) tma_load_3d(sV + c * MW_BLK, &tmV, b_load, v0 + c * 64, hd, row0 + c0);
    };
    if (warp == 8 && lane == 0) load_chunk(0);
    if (warp > 8) {
      fetch_gates(0);
      bar_named(BAR_GATES, 96);
      if (warp == 9) make_gates(m_in, 0);
    }
    const uint32_t idesc_s = make_idesc_f16(128, 128, 1, 0, 0), idesc_n = make_idesc_f16(128, 16, 1, 0, 0), idesc_o2 = make_idesc_f16(128, 128, 1, 1, 0),
                   idesc_o2h = make_idesc_f16(128, 64, 1, 1, 0), idesc_ds = make_idesc_f16(128, NQ * 64, 1, 1, 1);
    // all descriptors share their upper half (1024 bytes between groups of eight rows, 128-byte swizzle); the lower half counts 16-byte units from the operand's start.
    // K-major operands are rows of 64-column blocks, "mn" is the same memory with the contiguous dimension as M or N
    auto desc = [](uint32_t low) -> uint64_t { return ((uint64_t)((1024 >> 4) | (1u << 14) | (FT_SWZ_128B << 29)) << 32) | low; };
    auto low_k = [](const uint8_t* p) -> uint32_t { return (smem_u32(p) >> 4) | (1u << 16); };
    auto low_mn = [](const uint8_t* p) -> uint32_t { return (smem_u32(p) >> 4) | ((uint32_t)(MW_BLK >> 4) << 16); };
    const uint32_t q_k = low_k(sQ), k_k = low_k(sK), p_k = low_k(sP), n_k = low_k(sN), k_mn = low_mn(sK), v_mn = low_mn(sV), w_mn = low_mn(sQ);
    auto block = [](int k) -> uint32_t { return (k >> 2) * (MW_BLK / 16) + (k & 3) * 2; };      // 16 columns number k of a K-major operand
    int c0 = 0;
    for (int ch = 0; c0 < rows; ch++, c0 += MW_C) {
      const int par = ch & 1;
      const float* g = gate_sets + par * MW_GATES;
      bar_named(BAR_CHUNK, MW_THREADS);                  // gates, state and normaliser are in place
      if (*failed) break;
      tc_fence_after();
      if (warp > 8 && c0 + MW_C < rows) fetch_gates(c0 + MW_C);
      wait(b_load, par, 1);
      if constexpr (OUT) {
        if (warp == 8) {
          if (lane == 0 && ok) {
#pragma unroll
            for (int k = 0; k < NQ * 4; k++) umma_f16_ss(tX, desc(q_k + block(k)), desc(k_k + block(k)), idesc_s, k != 0);
            umma_commit(b_s);
#pragma unroll
            for (int k = 0; k < NQ * 4; k++) {
              umma_f16_ts(tX + 128, tA + k * 8, desc(q_k + block(k)), idesc_s, k != 0);
              umma_f16_ss(tNq, desc(q_k + block(k)), desc(n_k + (k >> 2) * (MW_VEC / 16) + (k & 3) * 2), idesc_n, k != 0);
            }
            umma_commit(b_o1);
          }
          __syncwarp();
          bar_named(BAR_P, 288);                         // P complete, scores read
          tc_fence_after();
          if (lane == 0 && ok) {
#pragma unroll
            for (int k = 0; k < 4; k++) umma_f16_ss(tX, desc(v_mn + k * 128), desc(p_k + k * 2), idesc_o2, k != 0);
#pragma unroll
            for (int k = 0; k < 4; k++) umma_f16_ss(tX + 64, desc(v_mn + (k + 4) * 128), desc(p_k + MW_BLK / 16 + k * 2), idesc_o2h, 1);
            umma_commit(b_o2);
          }
          __syncwarp();
        } else {
          wait(b_o1, par, 3);                            // the queries are consumed
          weigh_values(g + 2 * MW_C, tid - 288, 96);
          fence_proxy_async_smem();
        }
      }
      bar_named(BAR_STATE, MW_THREADS);                  // w V complete, outputs read
      tc_fence_after();
      if (warp == 8) {
        if (lane == 0 && ok) {
#pragma unroll
          for (int k = 0; k < 8; k++) {
            umma_f16_ss(tX, desc(w_mn + k * 128), desc(k_mn + k * 128), idesc_ds, k != 0);
            umma_f16_ss(tX, desc(w_mn + 2 * (MW_BLK / 16) + k * 128), desc(k_mn + k * 128), idesc_ds, 1);
          }
          umma_commit(b_ds);
        }
        __syncwarp();
        bar_named(BAR_N, 288);                           // n is done with the keys
        wait(b_ds, par, 5);
        if (lane == 0 && ok && c0 + MW_C < rows) load_chunk(c0 + MW_C);
        __syncwarp();
      }
      m_in = g[6 * MW_C + 4] + g[2 * MW_C - 1];              // sum of the forget gates + last running maximum
      if (warp == 9 && c0 + MW_C < rows) make_gates(m_in, par ^ 1);
    }
  } else {
    if constexpr (NQ > 2) reg_inc<MW_REGS_STATE>();
    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    const float scale = rsqrtf((float)D.d);
    float S[NQ * 32];                                    // S[half * 32 NQ + i][v0 + row]
#pragma unroll
    for (int i = 0; i < NQ * 32; i++) {
      const int d = half * NQ * 32 + i;
      S[i] = !zero && d < D.d16 && v0 + row < D.v16 ? in[(size_t)d * D.v16 + v0 + row] : 0.f;
    }
    float f_total = 0.f;
    auto publish = [&]() {                               // state and normaliser as operands of the next chunk's outputs
#pragma unroll
      for (int i = 0; i < NQ; i++) {
        uint32_t h[16];
#pragma unroll
        for (int e = 0; e < 16; e++) h[e] = pack2(S[i * 32 + 2 * e], S[i * 32 + 2 * e + 1]);
        tmem_st_32x32b_x16(tA + lanes + half * NQ * 16 + i * 16, h);
      }
      tmem_st_wait();
    };
    if (OUT) {
      publish();
      if (tid < NQ * 64) put_vec(sN, tid, nf[tid]);
      fence_proxy_async_smem();
    }
    int c0 = 0;
    for (int ch = 0; c0 < rows; ch++, c0 += MW_C) {
      const int cnt = min(MW_C, rows - c0), par = ch & 1;
      float* u = gate_sets + par * MW_GATES;
      const float *R = u + MW_C, *ein = u + 3 * MW_C;
      float* inv = u + 4 * MW_C;
      tc_fence_before();
      bar_named(BAR_CHUNK, MW_THREADS);
      if (*failed) break;
      tc_fence_after();
      if constexpr (OUT) {
        wait(b_s, par, 2);
        tc_fence_after();
        float sum = 0.f;
        if (half == 0 || row >= 64) {                    // weights of the keys: thread (token row, half of the keys); the upper right quarter is masked whole
          const float Rt = R[row];
          uint8_t* dst = half == 0 ? sP : sP + MW_BLK;
          const int pr = half == 0 ? row : row - 64;
#pragma unroll
          for (int b = 0; b < 2; b++) {
            const int kb = half * 2 + b, s0 = kb * 32;   // 32 keys: all ahead of this warp's tokens, around them, or behind
            if (kb > (warp & 3)) {
#pragma unroll
              for (int c8 = 0; c8 < 4; c8++) *reinterpret_cast<uint4*>(dst + sw128(pr, b * 4 + c8)) = make_uint4(0, 0, 0, 0);
              continue;
            }
            uint32_t sv[32];
            __syncwarp();
            tmem_ld_32x32b_x32(tX + lanes + s0, sv);
            tmem_ld_wait();
            if (kb < (warp & 3)) {                       // e^(u - R) = e^(u - top) e^(top - R), both at most one
              const float k = scale * exp_fast(u[6 * MW_C + kb] - Rt);
#pragma unroll
              for (int c8 = 0; c8 < 4; c8++) {
                uint32_t h[4];
#pragma unroll
                for (int e = 0; e < 8; e += 4) {
                  const float4 eu = *reinterpret_cast<const float4*>(u + 5 * MW_C + s0 + c8 * 8 + e);
                  const float p0 = __uint_as_float(sv[c8 * 8 + e]) * (eu.x * k), p1 = __uint_as_float(sv[c8 * 8 + e + 1]) * (eu.y * k);
                  const float p2 = __uint_as_float(sv[c8 * 8 + e + 2]) * (eu.z * k), p3 = __uint_as_float(sv[c8 * 8 + e + 3]) * (eu.w * k);
                  sum += (p0 + p1) + (p2 + p3);
                  h[e / 2] = pack2(p0, p1);
                  h[e / 2 + 1] = pack2(p2, p3);
                }
                *reinterpret_cast<uint4*>(dst + sw128(pr, b * 4 + c8)) = make_uint4(h[0], h[1], h[2], h[3]);
              }
            } else {
#pragma unroll
              for (int c8 = 0; c8 < 4; c8++) {
                uint32_t h[4];
#pragma unroll
                for (int e = 0; e < 8; e += 4) {
                  const int i = c8 * 8 + e;                // key, counted from the warp's first token; this thread's is `lane`
                  const float4 us = *reinterpret_cast<const float4*>(u + s0 + i);
                  const float p0 = i <= lane ? __uint_as_float(sv[i]) * (scale * exp_fast(us.x - Rt)) : 0.f;
                  const float p1 = i + 1 <= lane ? __uint_as_float(sv[i + 1]) * (scale * exp_fast(us.y - Rt)) : 0.f;
                  const float p2 = i + 2 <= lane ? __uint_as_float(sv[i + 2]) * (scale * exp_fast(us.z - Rt)) : 0.f;
                  const float p3 = i + 3 <= lane ? __uint_as_float(sv[i + 3]) * (scale * exp_fast(us.w - Rt)) : 0.f;
                  sum += (p0 + p1) + (p2 + p3);
                  h[e / 2] = pack2(p0, p1);
                  h[e / 2 + 1] = pack2(p2, p3);
                }
                *reinterpret_cast<uint4*>(dst + sw128(pr, b * 4 + c8)) = make_uint4(h[0], h[1], h[2], h[3]);
              }
            }
          }
        }
        rs[half * MW_C + row] = sum;
        fence_proxy_async_smem();
        tc_fence_before();
        bar_named(BAR_P, 288);                           // P complete, scores read
        tc_fence_after();
        wait(b_o1, par, 3);
        tc_fence_after();
        if (half == 0) {                                 // denominators: thread = token
          uint32_t x[16];
          __syncwarp();
          tmem_ld_32x32b_x16(tNq + lanes, x);
          tmem_ld_wait();
          const float dot = (__uint_as_float(x[0]) + __uint_as_float(x[1])) * ein[row] + sum + rs[MW_C + row];
          inv[row] = 1.f / (fmaxf(fabsf(dot), inv[row]) + DEN_EPS);
        }
        bar_named(BAR_DEN, 256);
        wait(b_o2, par, 4);
        tc_fence_after();
        // outputs: thread (value row, half of the tokens); four neighbouring lanes turn four tokens around, so that each stores four columns of one token
        const int b0 = lane & 1, b1 = (lane >> 1) & 1, mine = lane & 3, col = v0 + (row & ~3);
        const size_t pitch = (size_t)D.H * D.v16;
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(io.o) + (size_t)(row0 + c0 + half * 64 + mine) * pitch + hd * D.v16 + col;
        const int left = col < D.v16 ? cnt - half * 64 - mine : 0;       // tokens of this thread's that exist, every fourth one counted as four
        uint32_t o1[2][16], o2[2][16];
        auto fetch = [&](int b) {
          tmem_ld_32x32b_x16(tX + 128 + lanes + half * 64 + b * 16, o1[b & 1]);
          tmem_ld_32x32b_x16(tX + lanes + half * 64 + b * 16, o2[b & 1]);
        };
        __syncwarp();
        fetch(0);
#pragma unroll
        for (int b = 0; b < 4; b++) {
          const int t0 = half * 64 + b * 16;
          tmem_ld_wait();
          __syncwarp();
          if (b < 3) fetch(b + 1);
          const uint32_t (&p1)[16] = o1[b & 1];
          const uint32_t (&p2)[16] = o2[b & 1];
#pragma unroll
          for (int e = 0; e < 16; e += 4) {
            const float4 en = *reinterpret_cast<const float4*>(ein + t0 + e), iv = *reinterpret_cast<const float4*>(inv + t0 + e);
            const float a = (__uint_as_float(p1[e]) * en.x + __uint_as_float(p2[e])) * iv.x, bb = (__uint_as_float(p1[e + 1]) * en.y + __uint_as_float(p2[e + 1])) * iv.y;
            const float c = (__uint_as_float(p1[e + 2]) * en.z + __uint_as_float(p2[e + 2])) * iv.z, d = (__uint_as_float(p1[e + 3]) * en.w + __uint_as_float(p2[e + 3])) * iv.w;
            const float g0 = __shfl_xor_sync(0xffffffffu, b0 ? a : bb, 1), g1 = __shfl_xor_sync(0xffffffffu, b0 ? c : d, 1);
            const uint32_t lo = b0 ? pack2(g0, bb) : pack2(a, g0), hi = b0 ? pack2(g1, d) : pack2(c, g1);      // columns of the lane pair: token b0, token 2 + b0
            const uint32_t got = __shfl_xor_sync(0xffffffffu, b1 ? lo : hi, 2);
            if (b * 16 + e < left) *reinterpret_cast<uint2*>(dst) = b1 ? make_uint2(got, hi) : make_uint2(lo, got);
            dst += 4 * pitch;
          }
        }
      } else {
        wait(b_load, par, 1);
        weigh_values(u + 2 * MW_C, tid, 256);
        fence_proxy_async_smem();
      }
      const float r_last = R[MW_C - 1], f_chunk = u[6 * MW_C + 4], decay = exp_fast(m_in - r_last);
      tc_fence_before();
      bar_named(BAR_STATE, MW_THREADS);
      tc_fence_after();
      m_in = f_chunk + r_last;
      f_total += f_chunk;
      {                                                  // n: a lane takes eight columns of every eighth token
        const int tg = lane >> 2;
        const float* w = u + 2 * MW_C;
        for (int j = warp * 4 + (lane & 3); j < NQ * 8; j += 32) {
          float a[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
          for (int i = 0; i < MW_C / 8; i++) {
            const int t = i * 8 + tg;
            float k8[8];
            bf16x8_to_float(*reinterpret_cast<const bf16x8*>(sK + (j >> 3) * MW_BLK + sw128(t, j & 7)), k8);
            const float wt = w[t];
#pragma unroll
            for (int e = 0; e < 8; e++) a[e] += wt * k8[e];
          }
#pragma unroll
          for (int e = 0; e < 8; e++) {
            a[e] += __shfl_xor_sync(0xffffffffu, a[e], 4);
            a[e] += __shfl_xor_sync(0xffffffffu, a[e], 8);
            a[e] += __shfl_xor_sync(0xffffffffu, a[e], 16);
          }
          if (tg == 0) {
#pragma unroll
            for (int e = 0; e < 8; e++) {
              const float v = nf[j * 8 + e] * decay + a[e];
              nf[j * 8 + e] = v;
              if (OUT) put_vec(sN, j * 8 + e, v);        // the products that read the old one are done
            }
          }
        }
        fence_proxy_async_smem();
      }
      bar_named(BAR_N, 288);                             // K may be overwritten from here on
      wait(b_ds, par, 5);
      tc_fence_after();
#pragma unroll
      for (int i = 0; i < NQ; i++) {
        uint32_t x[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tX + lanes + half * NQ * 32 + i * 32, x);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e++) S[i * 32 + e] = S[i * 32 + e] * decay + __uint_as_float(x[e]);
      }
      if (OUT && c0 + MW_C < rows) publish();
    }
    if (ok && !*failed && (!OUT || (flags & SEG_LAST))) {
      float* dst = OUT ? slot : scratch + (size_t)(sg[5] + 1) * D.H * D.head() + hd * D.head();
      if (v0 + row < D.v16) {
#pragma unroll
        for (int i = 0; i < NQ * 32; i++) {
          const int d = half * NQ * 32 + i;
          if (d < D.d16) dst[(size_t)d * D.v16 + v0 + row] = S[i];
        }
      }
      if (blockIdx.z == 0) {
        // a slot's n may still be unread by the other CTAs of this head: it moves there later
        float* to = OUT ? io.nm + ((size_t)sg[3] * D.H + hd) * (D.d16 + 4) : dst + n_at;
        for (int i = tid; i < D.d16; i += 256) to[i] = nf[i];
        if (tid == 0) {
          to[D.d16] = m_in;
          to[D.d16 + 1] = f_total;
        }
      }
    }
  }
  if (*failed)
    for (int i = 0; i < 64; i++) __nanosleep(1000);      // copies in flight land before the shared memory goes away
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tX, 512);
  }
}

// chains the segments of a sequence: scratch state j (the contribution of segment j - 1) becomes the state ahead of segment j; state 0 is the slot's (the outputs' pass
// must not read the slot, which its last segment overwrites). Table per sequence: {first segment's scratch index, segments, slot, zero}. grid (ceil(d16 v16 / 1024), H, sequences)
__global__ void __launch_bounds__(256) mm_merge_kernel(const int4* __restrict__ seqs, const float* __restrict__ slots, size_t slot_stride, MemDims D, float* __restrict__ scratch) {
  const int4 sq = seqs[blockIdx.z];
  if (sq.y < 2) return;
  const int hd = blockIdx.y;
  const size_t elems = (size_t)D.d16 * D.v16, at = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4, step = (size_t)D.H * D.head();
  const float* slot = slots + (size_t)sq.z * slot_stride + hd * D.head();
  float* sc = scratch + (size_t)sq.x * step + hd * D.head();
  const bool zero = sq.w != 0;
  auto chain = [&](size_t off, bool quad) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    float m = zero ? 0.f : slot[elems + D.d16];
    if (!zero && !quad) v = *reinterpret_cast<const float4*>(slot + off);
    if (quad) sc[elems + D.d16 + 2] = m;
    else *reinterpret_cast<float4*>(sc + off) = v;
    for (int j = 1; j < sq.y; j++) {
      float* q = sc + j * step + elems + D.d16;
      const float ml = __ldcg(q), F = __ldcg(q + 1), mo = fmaxf(F + m, ml), keep = expf(F + m - mo), add = expf(ml - mo);
      if (quad) {
        q[2] = mo;
      } else {
        float4* l = reinterpret_cast<float4*>(sc + j * step + off);
        const float4 x = *l;
        v = make_float4(keep * v.x + add * x.x, keep * v.y + add * x.y, keep * v.z + add * x.z, keep * v.w + add * x.w);
        *l = v;
      }
      m = mo;
    }
  };
  if (at < elems) chain(at, false);
  if (blockIdx.x == 0) {
    for (int i = threadIdx.x * 4; i < D.d16; i += 1024) chain(elems + i, false);
    if (threadIdx.x == 0) chain(0, true);
  }
}

// a warp per (row, head), eight columns a lane. CTAs past the rows move n and m of one sequence into its slot.
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

constexpr int FIN_WARPS = 8;
template <typename T>
__global__ void __launch_bounds__(FIN_WARPS * 32) mm_finish_kernel(const T* __restrict__ o, int rows, int ctas, const T* __restrict__ gate, int64_t ldg, const float* __restrict__ norm,
                                                                   float eps, float out_scale, T* __restrict__ out, int64_t ldo, MemDims D, const int4* __restrict__ seqs,
                                                                   const float* __restrict__ nm, float* __restrict__ slots, size_t slot_stride) {
  if ((int)blockIdx.x >= ctas) {
    const int s = blockIdx.x - ctas;
    float* dst = slots + (size_t)seqs[s].z * slot_stride;
    for (int i = threadIdx.x; i < D.H * (D.d16 + 1); i += FIN_WARPS * 32) {
      const int hd = i / (D.d16 + 1), e = i % (D.d16 + 1);
      dst[hd * D.head() + (size_t)D.d16 * D.v16 + e] = nm[((size_t)s * D.H + hd) * (D.d16 + 4) + e];
    }
    return;
  }
  const int unit = blockIdx.x * FIN_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= rows * D.H) return;
  const int r = unit / D.H, hd = unit % D.H;
  const T* src = o + (size_t)unit * D.v16;
  const T* gr = gate + (size_t)r * ldg + hd * D.v16;
  constexpr int KEEP = 2;                                  // vectors of a lane that stay in registers (heads of up to 512 columns)
  float x[KEEP][8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; i++) {
    const int c = lane * 8 + i * 256;
    if (c < D.v16) {
      load8(src + c, x[i]);
#pragma unroll
      for (int e = 0; e < 8; e++) ss += x[i][e] * x[i][e];
    }
  }
  for (int c = lane * 8 + KEEP * 256; c < D.v16; c += 256) {
    float y[8];
    load8(src + c, y);
#pragma unroll
    for (int e = 0; e < 8; e++) ss += y[e] * y[e];
  }
  const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D.dv + eps) * out_scale;
  auto finish = [&](int c, float (&v)[8]) {
    float g[8], w[8];
    load8(gr + c, g);
    load8(norm + hd * D.v16 + c, w);
#pragma unroll
    for (int e = 0; e < 8; e++) v[e] = v[e] * rstd * w[e] * (sizeof(T) == 4 ? sigmoid_exact(g[e]) : 1.f / (1.f + __expf(-g[e])));
    store8(out + (size_t)r * ldo + hd * D.v16 + c, v);
  };
#pragma unroll
  for (int i = 0; i < KEEP; i++)
    if (lane * 8 + i * 256 < D.v16) finish(lane * 8 + i * 256, x[i]);
  for (int c = lane * 8 + KEEP * 256; c < D.v16; c += 256) {
    float y[8];
    load8(src + c, y);
    finish(c, y);
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode: cluster of CTAs per (head, sequence), grid (CTAs, H, B), 256 threads. A CTA takes 4 LPR value columns; LPR lanes read a row of the state, 256 / LPR rows at a
// time. The state's lines are requested before the wait for the predecessor (the last kernel that wrote them is a whole step back).
// ------------------------------------------------------------------------------------------------------------
struct MemDecode {
  const float* planes;
  int splits;
  int64_t ldp;
  size_t pstride;
  int col, gate_col;                 // columns of the queries (keys, values, gates behind them) and of the input gates
  const float *bi, *bf, *norm;
  float eps, out_scale;
  const int *positions, *slot_of;
  float* slots;
  size_t slot_stride;
};
FT_DEVICE float4 plane_sum4(const float* __restrict__ p, int splits, size_t stride) {
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int s = 0; s < splits; s++) {
    const float4 t = __ldcg(reinterpret_cast<const float4*>(p + s * stride));
    a.x += t.x; a.y += t.y; a.z += t.z; a.w += t.w;
  }
  return a;
}

template <int LPR>
__global__ void __launch_bounds__(256) mm_decode_kernel(MemDecode A, MemDims D, __nv_bfloat16* __restrict__ out, int64_t ldo) {
  namespace cg = cooperative_groups;
  constexpr int VC = 4 * LPR, RG = 256 / LPR, UN = 4;
  extern __shared__ __align__(16) float sm[];
  float* q = sm;                     // [d16] scaled
  float* k = q + D.d16;
  float* n = k + D.d16;
  float* v = n + D.d16;              // [VC]
  float* gt = v + VC;                // [VC]
  float* part = gt + VC;             // [RG][VC]
  __shared__ float red[32];
  __shared__ float gate_sh[2], cta_ss;
  cg::cluster_group cluster = cg::this_cluster();
  const int cta = blockIdx.x, ncta = gridDim.x, hd = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lc = tid % LPR, rg = tid / LPR, c0 = cta * VC, col = c0 + lc * 4;
  const bool zero = A.positions[b] == 0, live = col < D.v16;
  float* S = A.slots + (size_t)A.slot_of[b] * A.slot_stride + hd * D.head();
  float* sn = S + (size_t)D.d16 * D.v16;
  if (!zero && live && (lc % 8) == 0)
    for (int r = rg; r < D.d16; r += RG) asm volatile("prefetch.global.L2 [%0];" ::"l"(S + (size_t)r * D.v16 + col));
  pdl_wait();
  pdl_launch_dependents();
  const float* src = A.planes + (size_t)b * A.ldp;
  const float scale = rsqrtf((float)D.d), m_old = zero ? 0.f : sn[D.d16];
  for (int i = tid; i < D.d16 / 2; i += 256) {             // queries, then keys, four at a time
    const bool is_q = i < D.d16 / 4;
    const int r = (is_q ? i : i - D.d16 / 4) * 4;
    const float4 x = plane_sum4(src + A.col + ((is_q ? 0 : D.H) + hd) * D.d16 + r, A.splits, A.pstride);
    *reinterpret_cast<float4*>((is_q ? q : k) + r) = is_q ? make_float4(x.x * scale, x.y * scale, x.z * scale, x.w * scale) : x;
  }
  if (tid >= 256 - 2 * LPR) {                              // values and output gates of this CTA's columns
    const int i = tid - (256 - 2 * LPR), c = c0 + (i % LPR) * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D.v16) x = plane_sum4(src + A.col + 2 * D.H * D.d16 + (i < LPR ? 0 : D.H * D.v16) + hd * D.v16 + c, A.splits, A.pstride);
    *reinterpret_cast<float4*>((i < LPR ? v : gt) + (i % LPR) * 4) = x;
  }
  for (int i = tid; i < D.d16; i += 256) n[i] = zero ? 0.f : sn[i];
  if (warp < 2) {                                          // input and forget gate
    float x = 0.f;
    for (int s = lane; s < A.splits; s += 32) x += __ldcg(src + s * A.pstride + A.gate_col + warp * D.h8 + hd);
    x = warp_sum(x);
    if (lane == 0) gate_sh[warp] = soft_cap(x + (warp ? A.bf : A.bi)[hd], D.cap);
  }
  __syncthreads();
  const float ig = gate_sh[0], fg = log_sigmoid(gate_sh[1]), m_new = fmaxf(fg + m_old, ig), keep = expf(fg + m_old - m_new), add = expf(ig - m_new);
  float nq = 0.f;
  for (int i = tid; i < D.d16; i += 256) {
    const float x = keep * n[i] + add * k[i];
    n[i] = x;
    nq += x * q[i];
  }
  nq = block_sum(nq, red);
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m_new)) + DEN_EPS);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (live) {
    const float4 vv = *reinterpret_cast<const float4*>(v + lc * 4);
    for (int r0 = rg; r0 < D.d16; r0 += RG * UN) {
      float4 s[UN];
#pragma unroll
      for (int i = 0; i < UN; i++) {
        const int r = r0 + i * RG;
        s[i] = zero || r >= D.d16 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (size_t)r * D.v16 + col);
      }
#pragma unroll
      for (int i = 0; i < UN; i++) {
        const int r = r0 + i * RG;
        if (r < D.d16) {
          const float ak = add * k[r], qr = q[r];
          s[i] = make_float4(keep * s[i].x + ak * vv.x, keep * s[i].y + ak * vv.y, keep * s[i].z + ak * vv.z, keep * s[i].w + ak * vv.w);
          *reinterpret_cast<float4*>(S + (size_t)r * D.v16 + col) = s[i];
          acc.x += s[i].x * qr; acc.y += s[i].y * qr; acc.z += s[i].z * qr; acc.w += s[i].w * qr;
        }
      }
    }
  }
  *reinterpret_cast<float4*>(part + rg * VC + lc * 4) = acc;
  __syncthreads();
  float y = 0.f;
  if (tid < VC) {
#pragma unroll 8
    for (int g = 0; g < RG; g++) y += part[g * VC + tid];
    y *= inv;
  }
  const float ss = block_sum(y * y, red);
  if (tid == 0) cta_ss = ss;
  cluster.sync();                                          // from here on every CTA of the head has read n and m
  float tot = 0.f;
  for (int r = 0; r < ncta; r++) tot += *cluster.map_shared_rank(&cta_ss, r);
  const float rstd = 1.f / sqrtf(tot / (float)D.dv + A.eps) * A.out_scale;
  if (tid < VC && c0 + tid < D.v16)
    out[(size_t)b * ldo + hd * D.v16 + c0 + tid] = __float2bfloat16(y * rstd * A.norm[hd * D.v16 + c0 + tid] * sigmoid_exact(gt[tid]));
  if (cta == 0) {
    for (int i = tid; i < D.d16; i += 256) sn[i] = n[i];
    if (tid == 0) sn[D.d16] = m_new;
  }
  cluster.sync();                                          // nobody leaves while a partner may still read its shared memory
}

bool make_dims(MemDims& D, int H, int d, int dv, float cap) {
  if (H < 1 || H > 65535 || d < 1 || dv < 1 || !(cap > 0.f)) return false;
  D = MemDims{H, d, dv, (d + 15) & ~15, (dv + 15) & ~15, (H + 7) & ~7, cap};
  return true;
}
constexpr int SMEM_MAX = 232448;
int rows_smem(int d16) { return (d16 * MR_COLS + 3 * d16 + 8 * 32 + 32) * 4; }

template <int NQ, bool OUT>
int launch_walk(const CUtensorMap (&m)[3], dim3 grid, cudaStream_t st, const MemIO& io, const MemDims& D, float* scratch) {
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    // the warps trade registers (NQ > 2) out of what the block was launched with
    cudaFuncAttributes fa;
    FT_CUDA_TRY(cudaFuncGetAttributes(&fa, mm_walk_kernel<NQ, OUT>));
    static_assert(MW_REGS_STATE * 256 + MW_REGS_HELP * 128 <= MW_REGS * MW_THREADS, "register split");
    if (NQ > 2 && fa.numRegs < MW_REGS) return FT_ERR_ARG;
    FT_CUDA_TRY(cudaFuncSetAttribute(mm_walk_kernel<NQ, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, mw_smem(NQ, OUT)));
    done[dev] = true;
  }
  mm_walk_kernel<NQ, OUT><<<grid, MW_THREADS, mw_smem(NQ, OUT), st>>>(m[0], m[1], m[2], io, D, scratch, ft_status_ptr());
  return (int)cudaGetLastError();
}

template <int LPR>
int launch_decode(int ctas, int B, cudaStream_t st, const MemDecode& A, const MemDims& D, void* out, int64_t ldo) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(ctas, D.H, B);
  cfg.blockDim = dim3(256);
  cfg.dynamicSmemBytes = (3 * D.d16 + 2 * 4 * LPR + 1024) * 4;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = ctas;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ft_pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, mm_decode_kernel<LPR>, A, D, (__nv_bfloat16*)out, ldo);
}

}  // namespace

// Whether ft_mm_walk takes these head sizes.
FT_EXPORT int ft_mm_walk_fits(int d, int dv) { return d >= 1 && dv >= 1 && d <= 256; }

// Prompt stretches of a ragged batch in bf16. x [rows][ld]: queries H x d16 | keys H x d16 | values H x v16 (16-byte aligned, ld a multiple of 8); gates f32 [rows][ldg]: input
// gates, at column h8 = H rounded up to 8 forget gates; biases f32 [H]. segs int[nsegs][8] {first row, rows, slot, sequence, flags, scratch state, 0, 0}, flags 1: the only segment
// of its stretch (its state comes from the slot), 2: last, 4: the sequence starts (zero state). out = 0: contributions of the segments into scratch states [scratch state + 1] (f32 [H][d16 v16 + d16 + 4]
// each); out = 1: outputs o bf16 [rows][H * v16], last segments leave S in their slot (f32 slots of slot_stride) and n, m in nm f32 [sequence][H][d16 + 4].
FT_EXPORT int ft_mm_walk(const void* x, int64_t ld, int rows, const float* gates, int64_t ldg, const float* bias_i, const float* bias_f, float cap, const int* segs, int nsegs, int H, int d,
                         int dv, float* slots, int64_t slot_stride, float* scratch, float* nm, void* o, int out, cudaStream_t st) {
  MemDims D;
  if (nsegs < 1 || rows < 1 || !make_dims(D, H, d, dv, cap) || (ld & 7) || (reinterpret_cast<uintptr_t>(x) & 15) || (!out && !scratch) || (out && (!o || !nm))) return FT_ERR_ARG;
  if (!ft_mm_walk_fits(d, dv)) return FT_ERR_TOO_LARGE;
  const MemIO io{x, ld, gates, ldg, bias_i, bias_f, segs, slots, (size_t)slot_stride, nm, o};
  const dim3 grid(nsegs, H, (D.v16 + MW_V - 1) / MW_V);
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  FT_CUDA_TRY(ft_bind_context(dev));
  CUtensorMap m[3];
  const __nv_bfloat16* xp = (const __nv_bfloat16*)x;
  const uint64_t dp = (uint64_t)D.d16 * 2, vp = (uint64_t)D.v16 * 2, lp = (uint64_t)ld * 2;
  int r = ft_make_tmap_3d(&m[0], xp, 2, true, D.d16, H, rows, dp, lp, 64, 1, MW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[1], xp + (size_t)H * D.d16, 2, true, D.d16, H, rows, dp, lp, 64, 1, MW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[2], xp + (size_t)2 * H * D.d16, 2, true, D.v16, H, rows, vp, lp, 64, 1, MW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (r) return r;
#define FT_MW(N) return out ? launch_walk<N, true>(m, grid, st, io, D, scratch) : launch_walk<N, false>(m, grid, st, io, D, scratch)
  if (D.d16 <= 64) FT_MW(1);
  if (D.d16 <= 128) FT_MW(2);
  if (D.d16 <= 192) FT_MW(3);
  FT_MW(4);
#undef FT_MW
}

// seqs int4[nseq] {scratch state of the first segment, segments, slot, 1 if the sequence starts}: turns the contributions left by ft_mm_walk into the states ahead of
// the segments.
FT_EXPORT int ft_mm_merge(const int* seqs, int nseq, int H, int d, int dv, const float* slots, int64_t slot_stride, float* scratch, cudaStream_t st) {
  MemDims D;
  if (nseq < 1 || nseq > 65535 || !make_dims(D, H, d, dv, 1.f)) return FT_ERR_ARG;
  mm_merge_kernel<<<dim3((D.d16 * D.v16 + 1023) / 1024, H, nseq), 256, 0, st>>>(reinterpret_cast<const int4*>(seqs), slots, (size_t)slot_stride, D, scratch);
  return (int)cudaGetLastError();
}

// The same stretches token by token, bf16 or f32 (is_f32), one segment per sequence (flags 3, or 7 where the sequence starts). Key sizes up to 1600.
FT_EXPORT int ft_mm_rows(const void* x, int64_t ld, const float* gates, int64_t ldg, const float* bias_i, const float* bias_f, float cap, const int* segs, int nsegs, int H, int d,
                         int dv, float* slots, int64_t slot_stride, float* nm, void* o, int is_f32, cudaStream_t st) {
  MemDims D;
  if (nsegs < 1 || nsegs > 65535 || !make_dims(D, H, d, dv, cap)) return FT_ERR_ARG;
  const int smem = rows_smem(D.d16);
  if (smem > SMEM_MAX) return FT_ERR_TOO_LARGE;
  const MemIO io{x, ld, gates, ldg, bias_i, bias_f, segs, slots, (size_t)slot_stride, nm, o};
  const dim3 grid((D.v16 + MR_COLS - 1) / MR_COLS, H, nsegs);
  if (is_f32) {
    FT_CUDA_TRY(cudaFuncSetAttribute(mm_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    mm_rows_kernel<float><<<grid, 256, smem, st>>>(io, D);
  } else {
    FT_CUDA_TRY(cudaFuncSetAttribute(mm_rows_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    mm_rows_kernel<__nv_bfloat16><<<grid, 256, smem, st>>>(io, D);
  }
  return (int)cudaGetLastError();
}

// out [rows][ldo] (heads of v16; o, gate and out in one type) = o / rms(o of the head) * norm (f32 [H * v16]) * sigmoid(gate [rows][ldg]) * out_scale; moves n and m of every sequence of seqs (as for
// ft_mm_merge) from nm into its slot.
FT_EXPORT int ft_mm_finish(const void* o, int rows, const void* gate, int64_t ldg, const float* norm, float eps, float out_scale, void* out, int64_t ldo, int H, int d, int dv,
                           const int* seqs, int nseq, const float* nm, float* slots, int64_t slot_stride, int is_f32, cudaStream_t st) {
  MemDims D;
  if (rows < 1 || nseq < 1 || !make_dims(D, H, d, dv, 1.f) || (ldg & 7) || (ldo & 7)) return FT_ERR_ARG;
  const int4* sq = reinterpret_cast<const int4*>(seqs);
  const int ctas = (int)(((int64_t)rows * H + FIN_WARPS - 1) / FIN_WARPS);
#define FT_FIN(T) mm_finish_kernel<T><<<ctas + nseq, FIN_WARPS * 32, 0, st>>>((const T*)o, rows, ctas, (const T*)gate, ldg, norm, eps, out_scale, (T*)out, ldo, D, sq, nm, slots, \
                                                                              (size_t)slot_stride)
  if (is_f32) FT_FIN(float); else FT_FIN(__nv_bfloat16);
#undef FT_FIN
  return (int)cudaGetLastError();
}

// One token of B <= 16 sequences from split-K planes: columns as x of ft_mm_walk from `col` on (output gates H x v16 behind the values), input and forget gates from gate_col
// on. The state of slot slot_of[b] is advanced in place (taken as zero where positions[b] is 0); out bf16 [B][ldo], finished. Sizes up to 1024.
FT_EXPORT int ft_mm_decode(const float* planes, int splits, int64_t ldp, int64_t plane_stride, int B, int H, int d, int dv, int col, int gate_col, const float* bias_i,
                           const float* bias_f, float cap, const float* norm, float eps, float out_scale, const int* positions, const int* slot_of, float* slots,
                           int64_t slot_stride, void* out, int64_t ldo, cudaStream_t st) {
  MemDims D;
  if (B < 1 || B > 16 || splits < 1 || !make_dims(D, H, d, dv, cap) || (ldp & 3) || (plane_stride & 3) || (col & 3)) return FT_ERR_ARG;
  if (D.d16 > 1024 || D.v16 > 1024) return FT_ERR_TOO_LARGE;
  const MemDecode A{planes, splits, ldp, (size_t)plane_stride, col, gate_col, bias_i, bias_f, norm, eps, out_scale, positions, slot_of, slots, (size_t)slot_stride};
  const int lpr = D.v16 <= 256 ? 8 : D.v16 <= 512 ? 16 : 32, want = (D.v16 + 4 * lpr - 1) / (4 * lpr);
  int ctas = 1;
  while (ctas < want) ctas *= 2;
  if (lpr == 8) return launch_decode<8>(ctas, B, st, A, D, out, ldo);
  if (lpr == 16) return launch_decode<16>(ctas, B, st, A, D, out, ldo);
  return launch_decode<32>(ctas, B, st, A, D, out, ldo);
}
