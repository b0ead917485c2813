// Selective state space (the recurrence of Mamba-2; Dao and Gu, "Transformers are SSMs", 2024) with its short convolution and gated norm. A head remembers an N x dv matrix S,
// zero ahead of the first token; with step size d = softplus(dt + bias) and rate a = -e^A_log a token with vectors B, C (shared by the heads of a group) and value x does
//
//   S' = e^(a d) S + d B x^T        y = S'^T C + D x
//
// B, C and x are outputs of a causal convolution per channel with silu; y is gated with silu(z) and RMS-normed in equal parts of its columns.
//
// Sizes are padded with zeros: n16, v16 (multiples of 16). Channels of the convolution: x H x v16 | B G x n16 | C G x n16. A sequence's slot holds f32 [H][n16][v16] states, then
// the last taps - 1 inputs of the convolution, oldest first, [taps - 1][channels].
//
// A stretch of tokens can be taken at once. With F the running sum of a d inside the stretch (falling, so that every exponent below is at most zero):
//   y_t = e^(F_t) S_in^T C_t + sum_(s <= t) (C_t . B_s) e^(F_t - F_s) d_s x_s + D x_t,      S_out = e^(F_L) S_in + sum_s e^(F_L - F_s) d_s B_s x_s^T
//
//   ft_ssm_conv         convolution and silu of the new tokens of a ragged batch
//   ft_ssm_walk         prompts (bf16, tcgen05): a CTA walks a segment of a sequence in chunks of 128 tokens with 64 value columns of one head's state in registers. Long
//                       sequences are cut into segments that walk at the same time: a first pass collects every segment's own contribution, ft_ssm_merge chains them
//                       into the state ahead of each segment, a second pass produces the outputs
//   ft_ssm_rows         one token after another, any sizes, f32 or bf16 data (the 32-bit path)
//   ft_ssm_finish       gate and norm of the outputs; moves the last inputs of the convolution into the slots
//   ft_ssm_decode       one token per sequence from split-K planes: convolution, then state update, read-out, gate and norm
// Compiled without fast-math.
#include "common.cuh"
#include "host_common.h"

namespace {

struct SsmDims {
  int H, G, N, dv, n16, v16, taps;
  __host__ __device__ size_t head() const { return (size_t)n16 * v16; }
  __host__ __device__ int b_col() const { return H * v16; }
  __host__ __device__ int c_col() const { return H * v16 + G * n16; }
  __host__ __device__ int channels() const { return H * v16 + 2 * G * n16; }
  __host__ __device__ size_t conv_at() const { return H * head(); }
};

FT_DEVICE float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
FT_DEVICE float silu(float z) { return z / (1.f + expf(-z)); }
FT_DEVICE float silu_fast(float z) { return z / (1.f + __expf(-z)); }
template <typename T> FT_DEVICE float silu_for(float z) { return sizeof(T) == 4 ? silu(z) : silu_fast(z); }
template <typename T> FT_DEVICE float one(T v);
template <> FT_DEVICE float one<float>(float v) { return v; }
template <> FT_DEVICE float one<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> FT_DEVICE T to(float v);
template <> FT_DEVICE float to<float>(float v) { return v; }
template <> FT_DEVICE __nv_bfloat16 to<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
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

// ------------------------------------------------------------------------------------------------------------
// convolution: grid (channel blocks, row blocks), 128 threads, eight channels a thread. spans int4[sequence] {first row, rows, slot, 1 if the sequence starts}. TAPS: number
// of taps with the window of earlier inputs in registers, or 0 to read it again for every row.
// ------------------------------------------------------------------------------------------------------------
constexpr int CONV_ROWS = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const T* __restrict__ x, int64_t ld, int rows, const int* __restrict__ seq_of, const int4* __restrict__ spans,
                                                       const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ slots, size_t slot_stride, SsmDims D,
                                                       T* __restrict__ out) {
  const int cc = D.channels(), c = (blockIdx.x * 128 + threadIdx.x) * 8, taps = TAPS > 0 ? TAPS : D.taps;
  if (c >= cc) return;
  const int r0 = blockIdx.y * CONV_ROWS, r1 = min(rows, r0 + CONV_ROWS);
  // input of row r - back of the sequence of row r
  auto input = [&](const int4& sp, int r, int back, float (&v)[8]) {
    const int src = r - back;
    if (src >= sp.x) {
      load8(x + (size_t)src * ld + c, v);
    } else if (!sp.w) {
      load8(slots + (size_t)sp.z * slot_stride + D.conv_at() + (size_t)(taps - 1 + src - sp.x) * cc + c, v);
    } else {
#pragma unroll
      for (int e = 0; e < 8; e++) v[e] = 0.f;
    }
  };
  float b[8];
  load8(bias + c, b);
  if constexpr (TAPS > 0) {
    float wt[TAPS][8], win[TAPS][8];
#pragma unroll
    for (int k = 0; k < TAPS; k++) load8(w + (size_t)k * cc + c, wt[k]);
    auto tap = [&](T* dst) {
      float a[8];
#pragma unroll
      for (int e = 0; e < 8; e++) {
        float t = b[e];
#pragma unroll
        for (int k = 0; k < TAPS; k++) t += wt[k][e] * win[k][e];
        a[e] = silu_for<T>(t);
      }
      store8(dst, a);
#pragma unroll
      for (int k = 0; k < TAPS - 1; k++)
#pragma unroll
        for (int e = 0; e < 8; e++) win[k][e] = win[k + 1][e];
    };
    const int first = seq_of[r0];
    if (r1 - r0 == CONV_ROWS && seq_of[r1 - 1] == first) {      // rows of one sequence: all of them on their way at once
      const int4 sp = spans[first];
      uint4 raw[CONV_ROWS];
      static_assert(sizeof(T) == 2, "eight channels in 16 bytes");
#pragma unroll
      for (int j = 0; j < CONV_ROWS; j++) raw[j] = *reinterpret_cast<const uint4*>(x + (size_t)(r0 + j) * ld + c);
#pragma unroll
      for (int k = 0; k < TAPS - 1; k++) input(sp, r0, TAPS - 1 - k, win[k]);
#pragma unroll
      for (int j = 0; j < CONV_ROWS; j++) {
        bf16x8_to_float(*reinterpret_cast<const bf16x8*>(&raw[j]), win[TAPS - 1]);
        tap(out + (size_t)(r0 + j) * cc + c);
      }
      return;
    }
    int cur = -1;
    for (int r = r0; r < r1; r++) {
      const int s = seq_of[r];
      const int4 sp = spans[s];
      if (s != cur) {
#pragma unroll
        for (int k = 0; k < TAPS - 1; k++) input(sp, r, TAPS - 1 - k, win[k]);
        cur = s;
      }
      load8(x + (size_t)r * ld + c, win[TAPS - 1]);
      tap(out + (size_t)r * cc + c);
    }
  } else {
    for (int r = r0; r < r1; r++) {
      const int4 sp = spans[seq_of[r]];
      float a[8];
#pragma unroll
      for (int e = 0; e < 8; e++) a[e] = b[e];
      for (int k = 0; k < taps; k++) {
        float v[8], wk[8];
        input(sp, r, taps - 1 - k, v);
        load8(w + (size_t)k * cc + c, wk);
#pragma unroll
        for (int e = 0; e < 8; e++) a[e] += wk[e] * v[e];
      }
#pragma unroll
      for (int e = 0; e < 8; e++) a[e] = silu_for<T>(a[e]);
      store8(out + (size_t)r * cc + c, a);
    }
  }
}

// A segment of a sequence's new tokens: {first row, rows, state slot, sequence, flags, scratch state}
constexpr int SEG_INTS = 8, SEG_ONLY = 1, SEG_LAST = 2, SEG_ZERO = 4;      // ONLY: state from the slot, not from scratch; ZERO: the sequence starts, its slot's content is void
struct SsmIO {
  const void* u;                     // [rows][channels]: output of the convolution
  const float* dt;                   // [rows][ldt]: pre-activations without bias
  int64_t ldt;
  const float *dt_bias, *rate, *skip;      // [H]: bias of dt, -e^A_log, D
  const int* segs;
  float* slots;                      // [slot][slot_stride]
  size_t slot_stride;
  void* o;                           // [rows][H * v16] in the data type
};

// ------------------------------------------------------------------------------------------------------------
// token by token: grid (ceil(v16 / 32), H, sequences), 256 threads: 32 value columns x 8 groups of state rows
// ------------------------------------------------------------------------------------------------------------
constexpr int SR_COLS = 32;
template <typename T>
__global__ void __launch_bounds__(256) ssm_rows_kernel(SsmIO io, SsmDims D) {
  extern __shared__ __align__(16) float sm[];
  float* S = sm;                              // [n16][32]
  float* vec = S + D.n16 * SR_COLS;           // [2][2][n16]: B and C of a token, two tokens in turn
  float* red = vec + 4 * D.n16;               // [2][8][32]
  const int* sg = io.segs + (size_t)blockIdx.z * SEG_INTS;
  const int row0 = sg[0], rows = sg[1], hd = blockIdx.y, c = threadIdx.x & 31, rg = threadIdx.x >> 5, col = blockIdx.x * SR_COLS + c, g = hd / (D.H / D.G);
  float* st = io.slots + (size_t)sg[2] * io.slot_stride + hd * D.head();
  const bool zero = sg[4] & SEG_ZERO, live = col < D.v16;
  for (int r = rg; r < D.n16; r += 8) S[r * SR_COLS + c] = zero || !live ? 0.f : st[(size_t)r * D.v16 + col];
  const T* u = reinterpret_cast<const T*>(io.u);
  const size_t cc = D.channels();
  const float bias = io.dt_bias[hd], rate = io.rate[hd], skip = io.skip[hd];
  for (int t = 0; t < rows; t++) {
    const T* ur = u + (size_t)(row0 + t) * cc;
    float* b = vec + (t & 1) * 2 * D.n16;
    for (int r = threadIdx.x; r < 2 * D.n16; r += 256) b[r] = one(ur[(r < D.n16 ? D.b_col() : D.c_col()) + g * D.n16 + (r < D.n16 ? r : r - D.n16)]);
    const float v = live ? one(ur[hd * D.v16 + col]) : 0.f;
    const float d = softplus(io.dt[(size_t)(row0 + t) * io.ldt + hd] + bias), keep = expf(rate * d), dv = d * v;
    __syncthreads();
    float acc = 0.f;
    for (int r = rg; r < D.n16; r += 8) {
      const float s = keep * S[r * SR_COLS + c] + b[r] * dv;
      S[r * SR_COLS + c] = s;
      acc += s * b[D.n16 + r];
    }
    float* rd = red + (t & 1) * 256;
    rd[rg * 32 + c] = acc;
    __syncthreads();
    if (rg == 0 && live) {
      float a = skip * v;
#pragma unroll
      for (int k = 0; k < 8; k++) a += rd[k * 32 + c];
      reinterpret_cast<T*>(io.o)[(size_t)(row0 + t) * D.H * D.v16 + hd * D.v16 + col] = to<T>(a);
    }
  }
  if (live)
    for (int r = rg; r < D.n16; r += 8) st[(size_t)r * D.v16 + col] = S[r * SR_COLS + c];
}

// ------------------------------------------------------------------------------------------------------------
// chunk walk (tcgen05): grid (segments, H, ceil(v16 / 64)), 288 threads. A chunk is 128 tokens; a CTA keeps 64 value columns of a head's state: thread (row n, half) of the first
// eight warps holds S[n][half of the columns] in f32 registers (two rows where N is above 128), and all of them as bf16 in shared memory, an operand of the read-out.
//
//   G  [t][s] = C B^T          (from shared memory)
//   Y1 [t][v] = C S            the past, scaled per token when it is read
//   Y2 [t][v] = P X            P = masked, weighted scores with D on the diagonal, bf16 in TMEM
//   dS [n][v] = B^T (w X)      w X: values times their weight in the next state, as a sum of two bf16 numbers (16 mantissa bits); S <- decay S + dS in f32
//
// Warp 8 issues copies and products and makes the weights of the next chunk. Two CTAs share an SM (N <= 128): one's products run under the other's exponentials.
// Shared memory: C, later w X | B | X | S as an operand | weights. TMEM: [G, then Y2 in its first half | Y1 | P, then dS].
// ------------------------------------------------------------------------------------------------------------
constexpr int SW_C = 128, SW_V = 64, SW_BLK = SW_C * 128;       // chunk, value columns, bytes of a 64-column block of 128 rows
constexpr int SW_THREADS = 288, SW_GATES = 5 * SW_C + 4;        // floats of one chunk's weights
constexpr uint32_t FT_K_SSM = 12;

FT_DEVICE float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
FT_DEVICE float exp_fast(float x) { return ex2(x * 1.4426950408889634f); }
FT_DEVICE bool sw_wait(uint64_t* bar, uint32_t parity) {
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
FT_DEVICE uint32_t pack2(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}
// two neighbouring f32 values as bf16 high parts and bf16 remainders
FT_DEVICE void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack2(a, b);
  lo = pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
// 16-byte chunk c of row r in a block of 128-byte rows, as TMA and the tensor cores place it
FT_DEVICE uint32_t sw128(int r, int c) { return (uint32_t)(r * 128 + ((c ^ (r & 7)) << 4)); }

__host__ __device__ constexpr int sw_first(int nm, bool out) { return out ? 2 * nm : 2; }       // blocks that C takes, and w X after it
__host__ __device__ constexpr int sw_smem(int nm, bool out) {
  return (sw_first(nm, out) + 2 * nm + 1 + (out ? nm : 0)) * SW_BLK + 2 * SW_GATES * 4 + 64 + 1024;
}

// NM: 128-row blocks of the state. OUT: outputs from the state ahead of the segment; else: the segment's own contribution, into scratch state [scratch index + 1] ([H][n16 v16 + 4],
// the sum of a d behind the matrix).
template <int NM, bool OUT>
__global__ void __launch_bounds__(SW_THREADS, NM == 1 ? 2 : 1) ssm_walk_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmB,
                                                                               const __grid_constant__ CUtensorMap tmX, SsmIO io, SsmDims D, float* __restrict__ scratch,
                                                                               uint32_t* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sC = smem;
  uint8_t* sB = sC + sw_first(NM, OUT) * SW_BLK;         // [2 NM]
  uint8_t* sX = sB + 2 * NM * SW_BLK;
  uint8_t* sS = sX + SW_BLK;                             // [NM] rows n of 64 columns
  // per chunk, two in turn: [128] F | d e^(F of the last token of its 32 - F) | d | d e^(F_L - F) | e^F | F_L
  float* weight_sets = reinterpret_cast<float*>(sS + (OUT ? NM : 0) * SW_BLK);
  uint64_t* bars = reinterpret_cast<uint64_t*>(weight_sets + 2 * SW_GATES);
  uint64_t *b_load = bars, *b_g = bars + 1, *b_y1 = bars + 2, *b_y2 = bars + 3, *b_ds = bars + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 5);
  volatile int* failed = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int* sg = io.segs + (size_t)blockIdx.x * SEG_INTS;
  const int row0 = sg[0], rows = sg[1], flags = sg[4], hd = blockIdx.y, g = hd / (D.H / D.G), v0 = blockIdx.z * SW_V;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool zero = !OUT || ((flags & SEG_ONLY) && (flags & SEG_ZERO));
  const size_t scratch_head = D.head() + 4;
  float* slot = io.slots + (size_t)sg[2] * io.slot_stride + hd * D.head();
  const float* in = (flags & SEG_ONLY) ? slot : scratch + ((size_t)sg[5] * D.H + hd) * scratch_head;

  if (tid == 0) {
    for (int i = 0; i < 5; i++) mbar_init(&bars[i], 1);
    mbar_fence_init();
    *failed = 0;
    tma_prefetch_desc(&tmC); tma_prefetch_desc(&tmB); tma_prefetch_desc(&tmX);
  }
  constexpr uint32_t TMEM = NM == 1 ? 256 : 512;
  if (warp == 8) { tmem_alloc(tmem_slot, TMEM); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tG = *tmem_slot, tY1 = tG + 128, tP = tG + 192;
  bool ok = true;
  // a wait that ran out: everybody keeps to the barriers and leaves at the next chunk
  auto wait = [&](uint64_t* bar, int par, uint32_t site) {
    if (ok && !sw_wait(bar, par)) {
      ft_set_status(status, FT_K_SSM, site, blockIdx.x);
      *failed = 1;
      ok = false;
    }
    __syncwarp();
  };
  enum { BAR_CHUNK = 1, BAR_P, BAR_W };

  if (warp == 8) {
    const float bias = io.dt_bias[hd], rate = io.rate[hd];
    auto fetch = [&](int c0, float (&raw)[4]) {
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = c0 + lane * 4 + e;
        raw[e] = t < rows ? io.dt[(size_t)(row0 + t) * io.ldt + hd] : 0.f;
      }
    };
    auto make_weights = [&](int c0, const float (&raw)[4], int set) {      // four neighbouring tokens a lane
      float* w = weight_sets + set * SW_GATES;
      float d[4], F[4], s = 0.f;
#pragma unroll
      for (int e = 0; e < 4; e++) {
        d[e] = c0 + lane * 4 + e < rows ? softplus(raw[e] + bias) : 0.f;
        s += rate * d[e];
        F[e] = s;
      }
      float tot = s;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, tot, o);
        if (lane >= o) tot += y;
      }
      const float ahead = tot - s;
#pragma unroll
      for (int e = 0; e < 4; e++) F[e] += ahead;
      const float Fb = __shfl_sync(0xffffffffu, F[3], lane | 7), FL = __shfl_sync(0xffffffffu, F[3], 31);
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = lane * 4 + e;
        w[t] = F[e];
        w[SW_C + t] = d[e] * expf(Fb - F[e]);
        w[2 * SW_C + t] = d[e];
        w[3 * SW_C + t] = d[e] * expf(FL - F[e]);
        w[4 * SW_C + t] = expf(F[e]);
      }
      if (lane == 31) w[5 * SW_C] = FL;
    };
    auto load_chunk = [&](int c0) {                      // one thread; columns past the state's size arrive as zeros
      mbar_expect_tx(b_load, ((OUT ? 4 : 2) * NM + 1) * SW_BLK);
      for (int c = 0; c < 2 * NM; c++) {
        if (OUT) tma_load_3d(sC + c * SW_BLK, &tmC, b_load, c * 64, g, row0 + c0);
        tma_load_3d(sB + c * SW_BLK, &tmB, b_load, c * 64, g, row0 + c0);
      }
      tma_load_3d(sX, &tmX, b_load, v0, hd, row0 + c0);
    };
    if (lane == 0) load_chunk(0);
    float raw[4];
    fetch(0, raw);
    make_weights(0, raw, 0);
    const uint32_t idesc_g = make_idesc_f16(128, 128, 1, 0, 0), idesc_y = make_idesc_f16(128, SW_V, 1, 0, 1), idesc_ds = make_idesc_f16(128, SW_V, 1, 1, 1);
    // all descriptors share their upper half (1024 bytes between groups of eight rows, 128-byte swizzle); the lower half counts 16-byte units from the operand's start.
    // K-major operands are rows of 64-column blocks, "mn" is the same memory with the contiguous dimension as M or N
    auto desc = [](uint32_t low) -> uint64_t { return ((uint64_t)((1024 >> 4) | (1u << 14) | (FT_SWZ_128B << 29)) << 32) | low; };
    auto low_k = [](const uint8_t* p) -> uint32_t { return (smem_u32(p) >> 4) | (1u << 16); };
    auto low_mn = [](const uint8_t* p) -> uint32_t { return (smem_u32(p) >> 4) | ((uint32_t)(SW_BLK >> 4) << 16); };
    auto block = [](int k) -> uint32_t { return (k >> 2) * (SW_BLK / 16) + (k & 3) * 2; };      // 16 columns number k of a K-major operand
    const uint32_t c_k = low_k(sC), b_k = low_k(sB), b_mn = low_mn(sB), x_mn = low_mn(sX), w_mn = low_mn(sC), s_mn = low_mn(sS);
    int c0 = 0;
    for (int ch = 0; c0 < rows; ch++, c0 += SW_C) {
      const int par = ch & 1;
      const bool more = c0 + SW_C < rows;
      bar_named(BAR_CHUNK, SW_THREADS);                  // weights and state are in place
      if (*failed) break;
      tc_fence_after();
      if (more) fetch(c0 + SW_C, raw);
      wait(b_load, par, 1);
      if constexpr (OUT) {
        if (lane == 0 && ok) {
#pragma unroll
          for (int k = 0; k < NM * 8; k++) umma_f16_ss(tG, desc(c_k + block(k)), desc(b_k + block(k)), idesc_g, k != 0);
          umma_commit(b_g);
#pragma unroll
          for (int k = 0; k < NM * 8; k++) umma_f16_ss(tY1, desc(c_k + block(k)), desc(s_mn + k * 128), idesc_y, k != 0);
          umma_commit(b_y1);
        }
        __syncwarp();
        bar_named(BAR_P, SW_THREADS);                    // P complete, G read
        tc_fence_after();
        if (lane == 0 && ok) {
#pragma unroll
          for (int k = 0; k < 8; k++) umma_f16_ts(tG, tP + k * 8, desc(x_mn + k * 128), idesc_y, k != 0);
          umma_commit(b_y2);
        }
        __syncwarp();
      }
      bar_named(BAR_W, SW_THREADS);                      // w X complete
      if (OUT) wait(b_y2, par, 4);                       // dS takes the place of P
      tc_fence_after();
      if (lane == 0 && ok) {
#pragma unroll
        for (int m = 0; m < NM; m++)
#pragma unroll
          for (int k = 0; k < 8; k++) {
            umma_f16_ss(tP + m * SW_V, desc(b_mn + m * 2 * (SW_BLK / 16) + k * 128), desc(w_mn + k * 128), idesc_ds, k != 0);
            umma_f16_ss(tP + m * SW_V, desc(b_mn + m * 2 * (SW_BLK / 16) + k * 128), desc(w_mn + SW_BLK / 16 + k * 128), idesc_ds, 1);
          }
        umma_commit(b_ds);
      }
      __syncwarp();
      if (more) make_weights(c0 + SW_C, raw, par ^ 1);
      wait(b_ds, par, 5);
      if (lane == 0 && ok && more) load_chunk(c0 + SW_C);
      __syncwarp();
    }
  } else {
    const int row = (warp & 3) * 32 + lane, half = warp >> 2;
    const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
    const float skip = io.skip[hd];
    float S[NM * 32];                                    // S[m * 128 + row][v0 + half * 32 + i]
#pragma unroll
    for (int i = 0; i < NM * 32; i++) {
      const int n = (i >> 5) * 128 + row, v = v0 + half * 32 + (i & 31);
      S[i] = !zero && n < D.n16 && v < D.v16 ? in[(size_t)n * D.v16 + v] : 0.f;
    }
    float f_total = 0.f;
    auto publish = [&]() {                               // the state as an operand of the next chunk's outputs
#pragma unroll
      for (int m = 0; m < NM; m++)
#pragma unroll
        for (int c = 0; c < 4; c++) {
          const float* s = S + m * 32 + c * 8;
          *reinterpret_cast<uint4*>(sS + m * SW_BLK + sw128(row, half * 4 + c)) = make_uint4(pack2(s[0], s[1]), pack2(s[2], s[3]), pack2(s[4], s[5]), pack2(s[6], s[7]));
        }
      fence_proxy_async_smem();
    };
    if (OUT) publish();
    int c0 = 0;
    for (int ch = 0; c0 < rows; ch++, c0 += SW_C) {
      const int cnt = min(SW_C, rows - c0), par = ch & 1;
      const float* F = weight_sets + par * SW_GATES;
      tc_fence_before();
      bar_named(BAR_CHUNK, SW_THREADS);
      if (*failed) break;
      tc_fence_after();
      if constexpr (OUT) {
        wait(b_g, par, 2);
        tc_fence_after();
        const float Ft = F[row];
#pragma unroll
        for (int b = 0; b < 2; b++) {
          const int kb = half * 2 + b, s0 = kb * 32;     // 32 tokens: all ahead of this warp's, around them, or behind
          uint32_t h[16];
          if (kb > (warp & 3)) {
#pragma unroll
            for (int e = 0; e < 16; e++) h[e] = 0;
          } else {
            uint32_t sv[32];
            __syncwarp();
            tmem_ld_32x32b_x32(tG + lanes + s0, sv);
            tmem_ld_wait();
            if (kb < (warp & 3)) {                       // e^(F_t - F_s) = e^(F_t - F_b) e^(F_b - F_s), both at most one
              const float k = exp_fast(Ft - F[s0 + 31]);
#pragma unroll
              for (int e = 0; e < 32; e += 4) {
                const float4 w = *reinterpret_cast<const float4*>(F + SW_C + s0 + e);
                h[e / 2] = pack2(__uint_as_float(sv[e]) * (w.x * k), __uint_as_float(sv[e + 1]) * (w.y * k));
                h[e / 2 + 1] = pack2(__uint_as_float(sv[e + 2]) * (w.z * k), __uint_as_float(sv[e + 3]) * (w.w * k));
              }
            } else {
#pragma unroll
              for (int e = 0; e < 32; e += 4) {          // key, counted from the warp's first token; this thread's is `lane`
                const float4 f = *reinterpret_cast<const float4*>(F + s0 + e), d = *reinterpret_cast<const float4*>(F + 2 * SW_C + s0 + e);
                float p[4] = {__uint_as_float(sv[e]) * (d.x * exp_fast(Ft - f.x)), __uint_as_float(sv[e + 1]) * (d.y * exp_fast(Ft - f.y)),
                              __uint_as_float(sv[e + 2]) * (d.z * exp_fast(Ft - f.z)), __uint_as_float(sv[e + 3]) * (d.w * exp_fast(Ft - f.w))};
#pragma unroll
                for (int j = 0; j < 4; j++) p[j] = e + j < lane ? p[j] : e + j == lane ? p[j] + skip : 0.f;
                h[e / 2] = pack2(p[0], p[1]);
                h[e / 2 + 1] = pack2(p[2], p[3]);
              }
            }
          }
          __syncwarp();
          tmem_st_32x32b_x16(tP + lanes + kb * 16, h);
        }
        tmem_st_wait();
        tc_fence_before();
        bar_named(BAR_P, SW_THREADS);                    // P complete, G read
        tc_fence_after();
        wait(b_y1, par, 3);                              // C is consumed
      }
      wait(b_load, par, 6);
      {                                                  // values times their weight in the next state, over C
        const float* w = F + 3 * SW_C;
#pragma unroll
        for (int i = tid; i < SW_C * 8; i += 256) {
          const int r = i >> 3;
          const uint32_t at = sw128(r, i & 7);
          const float k = w[r];
          float v8[8];
          bf16x8_to_float(*reinterpret_cast<const bf16x8*>(sX + at), v8);
          uint32_t h[4], l[4];
#pragma unroll
          for (int e = 0; e < 4; e++) split2(v8[2 * e] * k, v8[2 * e + 1] * k, h[e], l[e]);
          *reinterpret_cast<uint4*>(sC + at) = make_uint4(h[0], h[1], h[2], h[3]);
          *reinterpret_cast<uint4*>(sC + SW_BLK + at) = make_uint4(l[0], l[1], l[2], l[3]);
        }
      }
      fence_proxy_async_smem();
      const float f_chunk = F[5 * SW_C], decay = exp_fast(f_chunk);
      f_total += f_chunk;
      bar_named(BAR_W, SW_THREADS);
      if constexpr (OUT) {
        wait(b_y2, par, 4);
        tc_fence_after();
        const float ef = F[4 * SW_C + row];
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(io.o) + (size_t)(row0 + c0 + row) * D.H * D.v16 + hd * D.v16 + v0 + half * 32;
        const int left = row < cnt ? D.v16 - v0 - half * 32 : 0;       // columns of this thread's that exist
#pragma unroll
        for (int b = 0; b < 2; b++) {
          uint32_t y1[16], y2[16];
          __syncwarp();
          tmem_ld_32x32b_x16(tY1 + lanes + half * 32 + b * 16, y1);
          tmem_ld_32x32b_x16(tG + lanes + half * 32 + b * 16, y2);
          tmem_ld_wait();
          float y[16];
#pragma unroll
          for (int e = 0; e < 16; e++) y[e] = __uint_as_float(y1[e]) * ef + __uint_as_float(y2[e]);
          if (b * 16 < left) {
            *reinterpret_cast<uint4*>(dst + b * 16) = make_uint4(pack2(y[0], y[1]), pack2(y[2], y[3]), pack2(y[4], y[5]), pack2(y[6], y[7]));
            *reinterpret_cast<uint4*>(dst + b * 16 + 8) = make_uint4(pack2(y[8], y[9]), pack2(y[10], y[11]), pack2(y[12], y[13]), pack2(y[14], y[15]));
          }
        }
      }
      wait(b_ds, par, 5);
      tc_fence_after();
#pragma unroll
      for (int m = 0; m < NM; m++) {
        uint32_t x[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tP + lanes + m * SW_V + half * 32, x);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 32; e++) S[m * 32 + e] = S[m * 32 + e] * decay + __uint_as_float(x[e]);
      }
      if (OUT && c0 + SW_C < rows) publish();
    }
    if (ok && !*failed && (!OUT || (flags & SEG_LAST))) {
      float* dst = OUT ? slot : scratch + ((size_t)(sg[5] + 1) * D.H + hd) * scratch_head;
#pragma unroll
      for (int i = 0; i < NM * 32; i++) {
        const int n = (i >> 5) * 128 + row, v = v0 + half * 32 + (i & 31);
        if (n < D.n16 && v < D.v16) dst[(size_t)n * D.v16 + v] = S[i];
      }
      if (!OUT && tid == 0 && blockIdx.z == 0) dst[D.head()] = f_total;
    }
  }
  if (*failed)
    for (int i = 0; i < 64; i++) __nanosleep(1000);      // copies in flight land before the shared memory goes away
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tG, TMEM);
  }
}

// chains the segments of a sequence: scratch state j (the contribution of segment j - 1) becomes the state ahead of segment j; state 0 is the slot's (the outputs' pass
// must not read the slot, which its last segment overwrites). Table per sequence: {first segment's scratch index, segments, slot, zero}. grid (ceil(n16 v16 / 1024), H, sequences)
__global__ void __launch_bounds__(256) ssm_merge_kernel(const int4* __restrict__ seqs, const float* __restrict__ slots, size_t slot_stride, SsmDims D, float* __restrict__ scratch) {
  const int4 sq = seqs[blockIdx.z];
  const size_t at = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4, elems = D.head(), step = (size_t)D.H * (elems + 4);
  if (sq.y < 2 || at >= elems) return;
  float* sc = scratch + (size_t)sq.x * step + blockIdx.y * (elems + 4);
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!sq.w) v = *reinterpret_cast<const float4*>(slots + (size_t)sq.z * slot_stride + blockIdx.y * elems + at);
  *reinterpret_cast<float4*>(sc + at) = v;
  for (int j = 1; j < sq.y; j++) {
    const float keep = expf(__ldcg(sc + j * step + elems));
    float4* l = reinterpret_cast<float4*>(sc + j * step + at);
    const float4 x = *l;
    v = make_float4(keep * v.x + x.x, keep * v.y + x.y, keep * v.z + x.z, keep * v.w + x.w);
    *l = v;
  }
}

// ------------------------------------------------------------------------------------------------------------
// gate and norm: a CTA per row; CTAs past the rows move the last inputs of the convolution of 1024 channels of one sequence. The norm's parts are `part` columns of the unpadded row.
// ALIGNED: parts and heads are multiples of eight columns, so that a vector of eight belongs to one part.
// ------------------------------------------------------------------------------------------------------------
struct NormParts {
  int parts, part;
  float eps;
  const float* w;                    // [H * v16]
};
struct ConvTail {                    // inputs of the convolution, and where their last ones go
  const void* x;
  int64_t ld;
  const int4* spans;
  float* slots;
  size_t slot_stride;
};
FT_DEVICE int padded_column(const SsmDims& D, int i) { return D.dv == D.v16 ? i : i / D.dv * D.v16 + i % D.dv; }

constexpr int FIN_T = 256;
// KV: vectors of eight columns a thread keeps
template <typename T, bool ALIGNED, int KV>
__global__ void __launch_bounds__(FIN_T) ssm_finish_kernel(const T* __restrict__ y, int rows, const T* __restrict__ z, int64_t ldz, NormParts P, T* __restrict__ out, int64_t ldo,
                                                           SsmDims D, ConvTail C, int tails) {
  extern __shared__ __align__(16) float fsm[];
  __shared__ float red[32];
  const int cols = D.H * D.v16, tid = threadIdx.x;
  if ((int)blockIdx.x >= rows) {
    const int s = (blockIdx.x - rows) / tails, cc = D.channels(), last = D.taps - 1;
    const int4 sp = C.spans[s];
    float* st = C.slots + (size_t)sp.z * C.slot_stride + D.conv_at();
    const int c1 = min(cc, ((int)(blockIdx.x - rows) % tails + 1) * 1024);
    for (int c = (int)(blockIdx.x - rows) % tails * 1024 + tid; c < c1; c += FIN_T)
      for (int k = 0; k < last; k++) {               // ascending: an old input moves to a lower place before that is overwritten
        const int j = sp.y - last + k;
        float v = 0.f;
        if (j >= 0) v = one(reinterpret_cast<const T*>(C.x)[(size_t)(sp.x + j) * C.ld + c]);
        else if (!sp.w) v = st[(size_t)(k + sp.y) * cc + c];
        st[(size_t)k * cc + c] = v;
      }
    return;
  }
  const int r = blockIdx.x, nvec = cols / 8;
  float* inv = fsm;                                      // [parts]
  float* keep = fsm + ((P.parts + 3) & ~3);              // ALIGNED: [nvec] sums of squares, else [cols] gated outputs
  float g[KV][8];
#pragma unroll
  for (int i = 0; i < KV; i++) {
    const int v = i * FIN_T + tid;
    float ss = 0.f;
    if (v < nvec) {
      float zz[8];
      load8(y + (size_t)r * cols + v * 8, g[i]);
      load8(z + (size_t)r * ldz + v * 8, zz);
#pragma unroll
      for (int e = 0; e < 8; e++) {
        g[i][e] *= silu_for<T>(zz[e]);
        ss += g[i][e] * g[i][e];
      }
      if constexpr (ALIGNED) keep[v] = ss;
      else store8(keep + v * 8, g[i]);
    }
  }
  __syncthreads();
  if constexpr (ALIGNED) {
    const int warp = tid >> 5, lane = tid & 31;
    for (int p = warp; p < P.parts; p += FIN_T / 32) {
      const int a = padded_column(D, p * P.part) / 8, b = padded_column(D, p * P.part + P.part - 8) / 8;      // padding in between holds zeros
      float s = 0.f;
      for (int v = a + lane; v <= b; v += 32) s += keep[v];
      s = warp_sum(s);
      if (lane == 0) inv[p] = 1.f / sqrtf(s / (float)P.part + P.eps);
    }
  } else {
    for (int p = 0; p < P.parts; p++) {
      float s = 0.f;
      for (int i = tid; i < P.part; i += FIN_T) {
        const float v = keep[padded_column(D, p * P.part + i)];
        s += v * v;
      }
      s = block_sum(s, red);
      if (tid == 0) inv[p] = 1.f / sqrtf(s / (float)P.part + P.eps);
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < KV; i++) {
    const int v = i * FIN_T + tid;
    if (v < nvec) {
      float w[8];
      load8(P.w + v * 8, w);
      const int hd = v * 8 / D.v16, in = v * 8 % D.v16;
#pragma unroll
      for (int e = 0; e < 8; e++) {
        const int p = (hd * D.dv + in + (ALIGNED ? 0 : e)) / P.part;       // padding may point past the last part: its weight is zero
        g[i][e] *= inv[min(p, P.parts - 1)] * w[e];
      }
      store8(out + (size_t)r * ldo + v * 8, g[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------------------------
constexpr int DEC_TOK = 16;
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
struct SsmDecode {
  const float* planes;
  int splits;
  int64_t ldp;
  size_t pstride;
  int z_col, x_col, dt_col;          // columns of the gate z, the convolution's inputs and the step sizes
  const float *conv_w, *conv_b, *dt_bias, *rate, *skip;
  const int *positions, *slot_of;
  float* slots;
  size_t slot_stride;
  float *u, *gz, *step;              // [16][channels], [16][H * v16], [16][2][H] (d, e^(a d))
};

// grid (blocks of 128 quads over gate | channels | step sizes, B), 128 threads, four columns a thread
__global__ void __launch_bounds__(128) ssm_decode_conv_kernel(SsmDecode A, SsmDims D) {
  const int b = blockIdx.y, cols = D.H * D.v16, cc = D.channels(), i = (blockIdx.x * 128 + threadIdx.x) * 4, c = i - cols;
  const bool conv = c >= 0 && c < cc;
  const float* wp = A.conv_w + (conv ? c : 0);
  const float4 bias = *reinterpret_cast<const float4*>(A.conv_b + (conv ? c : 0)), wl = *reinterpret_cast<const float4*>(wp + (size_t)(D.taps - 1) * cc);
  const bool zero = A.positions[b] == 0;
  float* st = A.slots + (size_t)A.slot_of[b] * A.slot_stride + D.conv_at() + (conv ? c : 0);
  pdl_wait();
  pdl_launch_dependents();
  const float* src = A.planes + (size_t)b * A.ldp;
  if (i < cols) {
    const float4 z = plane_sum4(src + A.z_col + i, A.splits, A.pstride);
    *reinterpret_cast<float4*>(A.gz + (size_t)b * cols + i) = make_float4(silu(z.x), silu(z.y), silu(z.z), silu(z.w));
  } else if (conv) {
    const float4 x = plane_sum4(src + A.x_col + c, A.splits, A.pstride);
    float4 a = make_float4(bias.x + wl.x * x.x, bias.y + wl.y * x.y, bias.z + wl.z * x.z, bias.w + wl.w * x.w);
    float4 old = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!zero && D.taps > 1) old = *reinterpret_cast<const float4*>(st);
    for (int k = 0; k + 1 < D.taps; k++) {
      const float4 w = *reinterpret_cast<const float4*>(wp + (size_t)k * cc);
      a.x += w.x * old.x; a.y += w.y * old.y; a.z += w.z * old.z; a.w += w.w * old.w;
      float4 next = x;
      if (k + 2 < D.taps) next = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st + (size_t)(k + 1) * cc);
      *reinterpret_cast<float4*>(st + (size_t)k * cc) = next;
      old = next;
    }
    *reinterpret_cast<float4*>(A.u + (size_t)b * cc + c) = make_float4(silu(a.x), silu(a.y), silu(a.z), silu(a.w));
  } else if (c - cc < D.H) {
    const int h0 = c - cc;
    const float4 v = plane_sum4(src + A.dt_col + h0, A.splits, A.pstride);        // columns past the heads: readable, not stored
    const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int j = 0; j < 4; j++)
      if (h0 + j < D.H) {
        const float d = softplus(e[j] + A.dt_bias[h0 + j]);
        A.step[(size_t)b * 2 * D.H + h0 + j] = d;
        A.step[(size_t)b * 2 * D.H + D.H + h0 + j] = expf(A.rate[h0 + j] * d);
      }
  }
}

// grid (H * ceil(v16 / 64), B), 256 threads: sixteen lanes read 64 columns of a state row, sixteen rows at a time. The state's first rows are read before the wait for the predecessor
// (the last kernel that wrote them is a whole step back). The last CTA of a token norms its row.
constexpr int SD_ROWS = 8;           // rows of a thread that wait in registers
__global__ void __launch_bounds__(256) ssm_decode_kernel(SsmDecode A, SsmDims D, NormParts P, float* __restrict__ gated, int* __restrict__ counters, __nv_bfloat16* __restrict__ out,
                                                         int64_t ldo) {
  __shared__ float part[16][SW_V];
  __shared__ float red[32];
  __shared__ int is_last;
  extern __shared__ __align__(16) float dsm[];           // [2 n16] B and C; later [parts]
  const int vb = (D.v16 + SW_V - 1) / SW_V, hd = blockIdx.x / vb, b = blockIdx.y, tid = threadIdx.x, lc = tid & 15, rg = tid >> 4, v0 = blockIdx.x % vb * SW_V, col = v0 + lc * 4;
  const int g = hd / (D.H / D.G), cols = D.H * D.v16;
  const bool zero = A.positions[b] == 0, live = col < D.v16;
  float* S = A.slots + (size_t)A.slot_of[b] * A.slot_stride + hd * D.head();
  float4 s[SD_ROWS];
#pragma unroll
  for (int i = 0; i < SD_ROWS; i++) {
    const int r = rg + i * 16;
    s[i] = zero || !live || r >= D.n16 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (size_t)r * D.v16 + col);
  }
  const float skip = A.skip[hd];
  pdl_wait();
  pdl_launch_dependents();
  const float* u = A.u + (size_t)b * D.channels();
  for (int i = tid; i < D.n16 / 2; i += 256) {            // B, then C, four at a time
    const int r = i * 4, is_c = r >= D.n16;
    *reinterpret_cast<float4*>(dsm + r) = __ldcg(reinterpret_cast<const float4*>(u + (is_c ? D.c_col() - D.n16 : D.b_col()) + g * D.n16 + r));
  }
  const float d = __ldcg(A.step + (size_t)b * 2 * D.H + hd), keep = __ldcg(A.step + (size_t)b * 2 * D.H + D.H + hd);
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
  if (live) x = __ldcg(reinterpret_cast<const float4*>(u + hd * D.v16 + col));
  const float4 dx = make_float4(d * x.x, d * x.y, d * x.z, d * x.w);
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  auto update = [&](int r, float4 v) {
    const float bk = dsm[r], ck = dsm[D.n16 + r];
    v = make_float4(keep * v.x + bk * dx.x, keep * v.y + bk * dx.y, keep * v.z + bk * dx.z, keep * v.w + bk * dx.w);
    *reinterpret_cast<float4*>(S + (size_t)r * D.v16 + col) = v;
    acc.x += v.x * ck; acc.y += v.y * ck; acc.z += v.z * ck; acc.w += v.w * ck;
  };
  if (live) {
#pragma unroll
    for (int i = 0; i < SD_ROWS; i++)
      if (rg + i * 16 < D.n16) update(rg + i * 16, s[i]);
    for (int r = rg + SD_ROWS * 16; r < D.n16; r += 16)
      update(r, zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (size_t)r * D.v16 + col));
  }
  *reinterpret_cast<float4*>(&part[rg][lc * 4]) = acc;
  __syncthreads();
  if (tid < SW_V && v0 + tid < D.v16) {
    float y = skip * __ldcg(u + hd * D.v16 + v0 + tid);
#pragma unroll
    for (int k = 0; k < 16; k++) y += part[k][tid];
    const size_t at = (size_t)b * cols + hd * D.v16 + v0 + tid;
    gated[at] = y * __ldcg(A.gz + at);
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    is_last = atomicAdd(counters + b, 1) == (int)gridDim.x - 1;
    if (is_last) counters[b] = 0;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  const float* row = gated + (size_t)b * cols;
  float* inv = dsm;
  for (int p = 0; p < P.parts; p++) {
    float ss = 0.f;
    if (D.dv == D.v16 && (P.part & 3) == 0) {
#pragma unroll 4
      for (int i = tid * 4; i < P.part; i += 1024) {
        const float4 v = __ldcg(reinterpret_cast<const float4*>(row + p * P.part + i));
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
    } else {
      for (int i = tid; i < P.part; i += 256) {
        const float v = __ldcg(row + padded_column(D, p * P.part + i));
        ss += v * v;
      }
    }
    ss = block_sum(ss, red);
    if (tid == 0) inv[p] = 1.f / sqrtf(ss / (float)P.part + P.eps);
  }
  __syncthreads();
  for (int c = tid * 4; c < cols; c += 1024) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(row + c)), w = *reinterpret_cast<const float4*>(P.w + c);
    const float e[4] = {v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w};
    float f[4];
    const int h = c / D.v16, in = c % D.v16;
#pragma unroll
    for (int j = 0; j < 4; j++) f[j] = e[j] * inv[min((h * D.dv + in + j) / P.part, P.parts - 1)];      // padding has weight zero
    uint2 pk;
    pk.x = pack2(f[0], f[1]);
    pk.y = pack2(f[2], f[3]);
    *reinterpret_cast<uint2*>(out + (size_t)b * ldo + c) = pk;
  }
}

bool make_dims(SsmDims& D, int H, int G, int N, int dv, int taps) {
  if (G < 1 || H < G || H % G || H > 65535 || N < 1 || dv < 1 || taps < 1) return false;
  D = SsmDims{H, G, N, dv, (N + 15) & ~15, (dv + 15) & ~15, taps};
  return true;
}
bool make_parts(NormParts& P, const SsmDims& D, int parts, float eps, const float* w) {
  if (parts < 1 || parts > 4096 || (D.H * D.dv) % parts) return false;
  P = NormParts{parts, D.H * D.dv / parts, eps, w};
  return true;
}
constexpr int SMEM_MAX = 232448;
int rows_smem(int n16) { return (n16 * SR_COLS + 4 * n16 + 512) * 4; }

template <int NM, bool OUT>
int launch_walk(const CUtensorMap (&m)[3], dim3 grid, cudaStream_t st, const SsmIO& io, const SsmDims& D, float* scratch) {
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    FT_CUDA_TRY(cudaFuncSetAttribute(ssm_walk_kernel<NM, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, sw_smem(NM, OUT)));
    done[dev] = true;
  }
  ssm_walk_kernel<NM, OUT><<<grid, SW_THREADS, sw_smem(NM, OUT), st>>>(m[0], m[1], m[2], io, D, scratch, ft_status_ptr());
  return (int)cudaGetLastError();
}

template <typename T, bool ALIGNED, int KV>
int launch_finish(int ctas, int smem, cudaStream_t st, const void* y, int rows, const void* z, int64_t ldz, const NormParts& P, void* out, int64_t ldo, const SsmDims& D,
                  const ConvTail& C, int tails) {
  if (smem > 48 * 1024) FT_CUDA_TRY(cudaFuncSetAttribute(ssm_finish_kernel<T, ALIGNED, KV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX - 1024));
  ssm_finish_kernel<T, ALIGNED, KV><<<ctas, FIN_T, smem, st>>>((const T*)y, rows, (const T*)z, ldz, P, (T*)out, ldo, D, C, tails);
  return (int)cudaGetLastError();
}
template <typename T>
int dispatch_finish(int ctas, cudaStream_t st, const void* y, int rows, const void* z, int64_t ldz, const NormParts& P, void* out, int64_t ldo, const SsmDims& D, const ConvTail& C,
                    int tails) {
  const int nvec = D.H * D.v16 / 8, kv = (nvec + FIN_T - 1) / FIN_T;
  const bool aligned = P.part % 8 == 0 && D.dv % 8 == 0;
  const int smem = (((P.parts + 3) & ~3) + (aligned ? nvec : nvec * 8)) * 4;
  if (kv > 8 || smem > SMEM_MAX - 1024) return FT_ERR_TOO_LARGE;
#define FT_SF(A, K) return launch_finish<T, A, K>(ctas, smem, st, y, rows, z, ldz, P, out, ldo, D, C, tails)
  if (aligned) {
    if (kv <= 1) FT_SF(true, 1);
    if (kv <= 2) FT_SF(true, 2);
    if (kv <= 4) FT_SF(true, 4);
    FT_SF(true, 8);
  }
  if (kv <= 2) FT_SF(false, 2);
  FT_SF(false, 8);
#undef FT_SF
}

}  // namespace

// Causal convolution per channel and silu of a ragged batch's new tokens: x [rows][ld] (channels x H x v16 | B G x n16 | C G x n16, ld a multiple of 8) -> out [rows][channels], bf16
// or (is_f32) f32. w f32 [taps][channels], the current token's last; bias f32 [channels]. seq_of int[rows]; spans int4[sequence] {first row, rows, slot, 1 if the sequence
// starts}: inputs ahead of the first row come from the slot's last taps - 1 inputs (f32 slots of slot_stride), or are zero.
FT_EXPORT int ft_ssm_conv(const void* x, int64_t ld, int rows, const int* seq_of, const int* spans, const float* w, const float* bias, const float* slots, int64_t slot_stride, int H,
                          int G, int N, int dv, int taps, void* out, int is_f32, cudaStream_t st) {
  SsmDims D;
  if (rows < 1 || !make_dims(D, H, G, N, dv, taps) || (ld & 7) || ld < D.channels() || (slot_stride & 7)) return FT_ERR_ARG;
  const dim3 grid((D.channels() / 8 + 127) / 128, (rows + CONV_ROWS - 1) / CONV_ROWS);
#define FT_SC(T, K) ssm_conv_kernel<T, K><<<grid, 128, 0, st>>>((const T*)x, ld, rows, seq_of, reinterpret_cast<const int4*>(spans), w, bias, slots, (size_t)slot_stride, D, (T*)out)
  if (is_f32) FT_SC(float, 0);
  else if (taps == 4) FT_SC(__nv_bfloat16, 4);
  else FT_SC(__nv_bfloat16, 0);
#undef FT_SC
  return (int)cudaGetLastError();
}

// Whether ft_ssm_walk takes this state size.
FT_EXPORT int ft_ssm_walk_fits(int N) { return N >= 1 && N <= 256; }

// Prompt stretches of a ragged batch in bf16. u [rows][channels] as left by ft_ssm_conv (16-byte aligned); dt f32 [rows][ldt]: step sizes ahead of bias and softplus; dt_bias, rate
// (-e^A_log), skip (D) f32 [H]. segs int[nsegs][8] {first row, rows, slot, sequence, flags, scratch state, 0, 0}, flags 1: the only segment of its stretch (its state comes from the
// slot), 2: last, 4: the sequence starts (zero state). out = 0: contributions of the segments into scratch states [scratch state + 1] (f32 [H][n16 v16 + 4] each); out = 1: outputs
// o bf16 [rows][H * v16], last segments leave their state in the slot (f32 slots of slot_stride).
FT_EXPORT int ft_ssm_walk(const void* u, int rows, const float* dt, int64_t ldt, const float* dt_bias, const float* rate, const float* skip, const int* segs, int nsegs, int H, int G,
                          int N, int dv, float* slots, int64_t slot_stride, float* scratch, void* o, int out, cudaStream_t st) {
  SsmDims D;
  if (nsegs < 1 || rows < 1 || !make_dims(D, H, G, N, dv, 1) || (reinterpret_cast<uintptr_t>(u) & 15) || (!out && !scratch) || (out && !o)) return FT_ERR_ARG;
  if (!ft_ssm_walk_fits(N)) return FT_ERR_TOO_LARGE;
  const SsmIO io{u, dt, ldt, dt_bias, rate, skip, segs, slots, (size_t)slot_stride, o};
  const dim3 grid(nsegs, H, (D.v16 + SW_V - 1) / SW_V);
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  FT_CUDA_TRY(ft_bind_context(dev));
  CUtensorMap m[3];
  const __nv_bfloat16* up = (const __nv_bfloat16*)u;
  const uint64_t np = (uint64_t)D.n16 * 2, vp = (uint64_t)D.v16 * 2, lp = (uint64_t)D.channels() * 2;
  int r = ft_make_tmap_3d(&m[0], up + D.c_col(), 2, true, D.n16, G, rows, np, lp, 64, 1, SW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[1], up + D.b_col(), 2, true, D.n16, G, rows, np, lp, 64, 1, SW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (!r) r = ft_make_tmap_3d(&m[2], up, 2, true, D.v16, H, rows, vp, lp, 64, 1, SW_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (r) return r;
  if (D.n16 <= 128) return out ? launch_walk<1, true>(m, grid, st, io, D, scratch) : launch_walk<1, false>(m, grid, st, io, D, scratch);
  return out ? launch_walk<2, true>(m, grid, st, io, D, scratch) : launch_walk<2, false>(m, grid, st, io, D, scratch);
}

// seqs int4[nseq] {scratch state of the first segment, segments, slot, 1 if the sequence starts}: turns the contributions left by ft_ssm_walk into the states ahead of the segments.
FT_EXPORT int ft_ssm_merge(const int* seqs, int nseq, int H, int G, int N, int dv, const float* slots, int64_t slot_stride, float* scratch, cudaStream_t st) {
  SsmDims D;
  if (nseq < 1 || nseq > 65535 || !make_dims(D, H, G, N, dv, 1) || (slot_stride & 3)) return FT_ERR_ARG;
  ssm_merge_kernel<<<dim3((D.n16 * D.v16 + 1023) / 1024, H, nseq), 256, 0, st>>>(reinterpret_cast<const int4*>(seqs), slots, (size_t)slot_stride, D, scratch);
  return (int)cudaGetLastError();
}

// The same stretches token by token, bf16 or f32 (is_f32), one segment per sequence (flags 3, or 7 where the sequence starts). State sizes up to 1600.
FT_EXPORT int ft_ssm_rows(const void* u, const float* dt, int64_t ldt, const float* dt_bias, const float* rate, const float* skip, const int* segs, int nsegs, int H, int G, int N,
                          int dv, float* slots, int64_t slot_stride, void* o, int is_f32, cudaStream_t st) {
  SsmDims D;
  if (nsegs < 1 || nsegs > 65535 || !make_dims(D, H, G, N, dv, 1)) return FT_ERR_ARG;
  const int smem = rows_smem(D.n16);
  if (smem > SMEM_MAX) return FT_ERR_TOO_LARGE;
  const SsmIO io{u, dt, ldt, dt_bias, rate, skip, segs, slots, (size_t)slot_stride, o};
  const dim3 grid((D.v16 + SR_COLS - 1) / SR_COLS, H, nsegs);
  if (is_f32) {
    FT_CUDA_TRY(cudaFuncSetAttribute(ssm_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    ssm_rows_kernel<float><<<grid, 256, smem, st>>>(io, D);
  } else {
    FT_CUDA_TRY(cudaFuncSetAttribute(ssm_rows_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    ssm_rows_kernel<__nv_bfloat16><<<grid, 256, smem, st>>>(io, D);
  }
  return (int)cudaGetLastError();
}

// out [rows][ldo] (heads of v16) = y silu(z), normed in `parts` equal parts of the H * dv columns (RMS, eps), times norm (f32 [H * v16], zero in the padding); y [rows][H * v16],
// z [rows][ldz], all in one type. The last taps - 1 inputs of the convolution (x [rows][ldx], as for ft_ssm_conv) of every sequence of spans move into its slot. H * v16 up to 16384.
FT_EXPORT int ft_ssm_finish(const void* y, int rows, const void* z, int64_t ldz, int parts, float eps, const float* norm, void* out, int64_t ldo, int H, int G, int N, int dv, int taps,
                            const void* x, int64_t ldx, const int* spans, int nseq, float* slots, int64_t slot_stride, int is_f32, cudaStream_t st) {
  SsmDims D;
  NormParts P;
  if (rows < 1 || nseq < 1 || !make_dims(D, H, G, N, dv, taps) || !make_parts(P, D, parts, eps, norm) || (ldz & 7) || (ldo & 7)) return FT_ERR_ARG;
  const ConvTail C{x, ldx, reinterpret_cast<const int4*>(spans), slots, (size_t)slot_stride};
  const int tails = (D.channels() + 1023) / 1024, ctas = rows + (taps > 1 ? nseq * tails : 0);
  if (is_f32) return dispatch_finish<float>(ctas, st, y, rows, z, ldz, P, out, ldo, D, C, tails);
  return dispatch_finish<__nv_bfloat16>(ctas, st, y, rows, z, ldz, P, out, ldo, D, C, tails);
}

// One token of B <= 16 sequences from split-K planes: gate z H x v16 from column z_col, inputs of the convolution from x_col (channels as in ft_ssm_conv), step sizes from dt_col on
// (readable up to H rounded up to 4). State and last inputs of slot slot_of[b] are advanced in place (taken as zero where positions[b] is 0). u f32 [16][channels], gz and gated
// f32 [16][H * v16], step f32 [16][2 H]: scratch; counters int[16], zero before the first launch (the kernel leaves them zero). out bf16 [B][ldo], finished. State sizes up to 4096.
FT_EXPORT int ft_ssm_decode(const float* planes, int splits, int64_t ldp, int64_t plane_stride, int B, int H, int G, int N, int dv, int taps, int z_col, int x_col, int dt_col,
                            const float* conv_w, const float* conv_b, const float* dt_bias, const float* rate, const float* skip, int parts, float eps, const float* norm,
                            const int* positions, const int* slot_of, float* slots, int64_t slot_stride, float* u, float* gz, float* step, float* gated, int* counters, void* out,
                            int64_t ldo, cudaStream_t st) {
  SsmDims D;
  NormParts P;
  if (B < 1 || B > DEC_TOK || splits < 1 || !make_dims(D, H, G, N, dv, taps) || !make_parts(P, D, parts, eps, norm) || (ldp & 3) || (plane_stride & 3) || (z_col & 3) || (x_col & 3) ||
      (dt_col & 3) || (slot_stride & 3) || (ldo & 3))
    return FT_ERR_ARG;
  if (D.n16 > 4096) return FT_ERR_TOO_LARGE;
  const SsmDecode A{planes, splits, ldp, (size_t)plane_stride, z_col, x_col, dt_col, conv_w, conv_b, dt_bias, rate, skip, positions, slot_of, slots, (size_t)slot_stride, u, gz, step};
  const int quads = (H * D.v16 + D.channels() + ((H + 3) & ~3)) / 4;
  const int r = (int)ft_launch_pdl(ssm_decode_conv_kernel, dim3((quads + 127) / 128, B), dim3(128), 0, st, A, D);
  if (r) return r;
  const int words = 2 * D.n16 > parts ? 2 * D.n16 : parts;
  return (int)ft_launch_pdl(ssm_decode_kernel, dim3(H * ((D.v16 + SW_V - 1) / SW_V), B), dim3(256), (size_t)words * 4, st, A, D, P, gated, counters, (__nv_bfloat16*)out, ldo);
}
