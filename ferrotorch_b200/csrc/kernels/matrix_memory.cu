// Matrix memory (the mLSTM cell of xLSTM, Beck et al. 2024): per head a d x dv matrix S and a vector n that decay by a forget gate and take in k v^T and k with an
// input gate, both gates in the log domain against a running maximum m that starts at zero:
//
//   m_t = max(f_t + m_(t-1), i_t);   S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T;   n_t alike with k_t
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
//
// followed by an RMS norm of every head's output, a weight, a sigmoid gate and a scale. States live in f32, one slot per sequence: [heads][d16 x v16 | n (d16) |
// m, 3 spare], head sizes padded to multiples of 16 with zeros.
//
// A stretch of tokens can be taken at once. With F the running sum of f and u_s = i_s - F_s inside the stretch, R_t = max(m_in, max_(s <= t) u_s):
//   m_t = F_t + R_t,   weight of key s at t: e^(u_s - R_t),   weight of the state before the stretch: e^(m_in - R_t)
// so nothing but differences of nearby numbers is exponentiated, and every exponent is at most zero.
//
//   ft_mm_walk     prompts (bf16): a CTA walks a segment of a sequence in chunks of 64 tokens with 64 value columns of one head's state in registers. Long
//                  sequences are cut into segments that walk at the same time: a first pass collects every segment's own contribution,
//                  ft_mm_merge chains them into the state ahead of each segment, a second pass produces the outputs. f32 quantities (weighted values, state, weights
//                  of the keys) meet the 16-bit tensor cores as sums of two bf16 numbers.
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
  float* o;                          // [rows][H * v16] f32
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
      if (col < D.v16) io.o[(size_t)(row0 + t) * D.H * D.v16 + hd * D.v16 + col] = a / (fmaxf(fabsf(nq), expf(-m)) + DEN_EPS);
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
// chunk walk: grid (segments, H, ceil(v16 / 64)), 256 threads
// ------------------------------------------------------------------------------------------------------------
constexpr int MW_C = 64, MW_V = 64, MW_VP = MW_V * 2 + 16;      // chunk, value columns, pitch of 64-column bf16 rows in bytes

FT_DEVICE void cp_async16z(uint32_t dst, const void* src, bool live) {       // 16 bytes, or zeros
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
FT_DEVICE void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
FT_DEVICE void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
FT_DEVICE void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two neighbouring f32 values as bf16 high parts and bf16 remainders (16 mantissa bits together)
FT_DEVICE void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__host__ __device__ inline int mw_pitch(int d16) { return d16 * 2 + 16; }
inline int mw_smem(int d16, bool out) {
  const int rows = MW_C * MW_VP;
  return MW_C * mw_pitch(d16) * (out ? 2 : 1) + rows * (out ? 5 : 3) + (out ? 2 * d16 * MW_VP : 0) + (8 * MW_C + d16) * 4;
}

// MT: 16-row tiles of the state per warp (d16 <= 128 MT). OUT: outputs from the state ahead of the segment; else: the segment's own contribution, into
// scratch state [scratch index + 1], with m relative to an empty past and the sum of the forget gates beside it.
template <int MT, bool OUT>
__global__ void __launch_bounds__(256, 1) mm_walk_kernel(MemIO io, MemDims D, float* __restrict__ scratch) {
  extern __shared__ __align__(128) uint8_t smem[];
  const int pd = mw_pitch(D.d16);
  uint8_t* p = smem;
  uint8_t* sK = p;              p += MW_C * pd;
  uint8_t* sV = p;              p += MW_C * MW_VP;
  uint8_t* sWh = p;             p += MW_C * MW_VP;      // values times their weight in the state, high and low parts
  uint8_t* sWl = p;             p += MW_C * MW_VP;
  uint8_t* sQ = p;              p += OUT ? MW_C * pd : 0;
  uint8_t* sPh = p;             p += OUT ? MW_C * MW_VP : 0;      // weights of the keys
  uint8_t* sPl = p;             p += OUT ? MW_C * MW_VP : 0;
  uint8_t* sSh = p;             p += OUT ? D.d16 * MW_VP : 0;     // state ahead of the chunk
  uint8_t* sSl = p;             p += OUT ? D.d16 * MW_VP : 0;
  float* u = reinterpret_cast<float*>(p);     // [64] i - F
  float* R = u + MW_C;                        // [64] running maximum of u and m_in
  float* Fs = R + MW_C;                       // [64] running sum of f
  float* w = Fs + MW_C;                       // [64] weight in the next state
  float* rs = w + MW_C;                       // [2][64] row sums of the key weights
  float* nq = rs + 2 * MW_C;                  // [64] n . q
  float* n = nq + 2 * MW_C;                   // [d16]
  const int* sg = io.segs + (size_t)blockIdx.x * SEG_INTS;
  const int row0 = sg[0], rows = sg[1], flags = sg[4], hd = blockIdx.y, v0 = blockIdx.z * MW_V;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int rt = warp & 3, ch = warp >> 2, mtiles = D.d16 / 16, ksteps = D.d16 / 16;
  const float scale = rsqrtf((float)D.d);
  const bool zero = !OUT || ((flags & SEG_ONLY) && (flags & SEG_ZERO));
  float* slot = io.slots + (size_t)sg[2] * io.slot_stride + hd * D.head();
  const float* in = (flags & SEG_ONLY) ? slot : scratch + (size_t)sg[5] * D.H * D.head() + hd * D.head();
  const size_t n_at = (size_t)D.d16 * D.v16;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(io.x);

  float S[MT][8][4];
#pragma unroll
  for (int a = 0; a < MT; a++)
#pragma unroll
    for (int b = 0; b < 8; b++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int r = (warp * MT + a) * 16 + g + 8 * e, c = v0 + b * 8 + t2;
        float2 v = make_float2(0.f, 0.f);
        if (!zero && r < D.d16 && c < D.v16) v = *reinterpret_cast<const float2*>(in + (size_t)r * D.v16 + c);
        S[a][b][2 * e] = v.x;
        S[a][b][2 * e + 1] = v.y;
      }
  for (int i = tid; i < D.d16; i += 256) n[i] = zero ? 0.f : in[n_at + i];
  float m_in = OUT ? (zero ? 0.f : in[n_at + D.d16 + ((flags & SEG_ONLY) ? 0 : 2)]) : -INFINITY, f_total = 0.f;
  auto publish = [&]() {                      // state registers -> shared memory, as the operand of the next chunk's outputs
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
      for (int b = 0; b < 8; b++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int r = (warp * MT + a) * 16 + g + 8 * e;
          if (r < D.d16) {
            uint32_t h, l;
            split2(S[a][b][2 * e], S[a][b][2 * e + 1], h, l);
            *reinterpret_cast<uint32_t*>(sSh + r * MW_VP + (b * 8 + t2) * 2) = h;
            *reinterpret_cast<uint32_t*>(sSl + r * MW_VP + (b * 8 + t2) * 2) = l;
          }
        }
  };
  auto load_chunk = [&](int c0, int cnt) {
    const int kv = D.d16 / 8;
    for (int i = tid; i < MW_C * kv; i += 256) {
      const int r = i / kv, v = i % kv;
      const bool live = r < cnt;
      const __nv_bfloat16* xr = x + (size_t)(row0 + c0 + (live ? r : 0)) * io.ld + v * 8;
      cp_async16z(smem_u32(sK + r * pd + v * 16), xr + (D.H + hd) * D.d16, live);
      if (OUT) cp_async16z(smem_u32(sQ + r * pd + v * 16), xr + hd * D.d16, live);
    }
    for (int i = tid; i < MW_C * 8; i += 256) {
      const int r = i >> 3, v = i & 7;
      const bool live = r < cnt && v0 + v * 8 < D.v16;
      cp_async16z(smem_u32(sV + r * MW_VP + v * 16), x + (size_t)(row0 + c0 + (live ? r : 0)) * io.ld + 2 * D.H * D.d16 + hd * D.v16 + (live ? v0 + v * 8 : 0), live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  bool have_state = !zero;
  if (OUT && have_state) publish();
  load_chunk(0, min(MW_C, rows));
  for (int c0 = 0; c0 < rows; c0 += MW_C) {
    const int cnt = min(MW_C, rows - c0);
    if (warp == 0) {                          // gates of two neighbouring tokens per lane, running sum and running maximum
      float f[2], ig[2];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int t = lane * 2 + e;
        f[e] = 0.f;
        ig[e] = -INFINITY;
        if (t < cnt) {
          const float* gr = io.gates + (size_t)(row0 + c0 + t) * io.ldg;
          ig[e] = soft_cap(gr[hd] + io.bi[hd], D.cap);
          f[e] = log_sigmoid(soft_cap(gr[D.h8 + hd] + io.bf[hd], D.cap));
        }
      }
      float s = f[0] + f[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += y;
      }
      const float F0 = s - f[1], F1 = s, u0 = ig[0] - F0, u1 = ig[1] - F1;
      float mx = fmaxf(u0, u1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, y);
      }
      float before = __shfl_up_sync(0xffffffffu, mx, 1);
      before = fmaxf(lane == 0 ? -INFINITY : before, m_in);
      const float R0 = fmaxf(before, u0), R1 = fmaxf(R0, u1), Rl = __shfl_sync(0xffffffffu, R1, 31);
      const int t = lane * 2;
      u[t] = u0; u[t + 1] = u1;
      R[t] = R0; R[t + 1] = R1;
      Fs[t] = F0; Fs[t + 1] = F1;
      w[t] = __expf(u0 - Rl); w[t + 1] = __expf(u1 - Rl);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float R_last = R[MW_C - 1], decay = __expf(m_in - R_last);
    // weighted values
    for (int i = tid; i < MW_C * MW_V / 2; i += 256) {
      const int t = i >> 5, c = (i & 31) * 4;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sV + t * MW_VP + c));
      uint32_t h, l;
      split2(v.x * w[t], v.y * w[t], h, l);
      *reinterpret_cast<uint32_t*>(sWh + t * MW_VP + c) = h;
      *reinterpret_cast<uint32_t*>(sWl + t * MW_VP + c) = l;
    }
    if constexpr (OUT) {
      // weights of the keys: rows 16 rt, tokens 32 ch
      float s[4][4];
#pragma unroll
      for (int b = 0; b < 4; b++) s[b][0] = s[b][1] = s[b][2] = s[b][3] = 0.f;
      if (ch * 32 <= rt * 16 + 15) {
        const uint32_t qa = smem_u32(sQ) + (rt * 16 + (lane & 15)) * pd + (lane >> 4) * 16;
        const uint32_t ka = smem_u32(sK) + (ch * 32 + (lane & 7) + ((lane >> 4) << 3)) * pd + ((lane >> 3) & 1) * 16;
        for (int ks = 0; ks < ksteps; ks++) {
          uint32_t a[4], b0[4], b1[4];
          ldmatrix_x4(a, qa + ks * 32);
          ldmatrix_x4(b0, ka + ks * 32);
          ldmatrix_x4(b1, ka + 16 * pd + ks * 32);
          mma_16816(s[0], a, b0[0], b0[1]);
          mma_16816(s[1], a, b0[2], b0[3]);
          mma_16816(s[2], a, b1[0], b1[1]);
          mma_16816(s[3], a, b1[2], b1[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int r = rt * 16 + g + 8 * e;
        const float Rr = R[r];
        float sum = 0.f;
#pragma unroll
        for (int b = 0; b < 4; b++) {
          const int c = ch * 32 + b * 8 + t2;
          const float p0 = c <= r ? s[b][2 * e] * scale * __expf(u[c] - Rr) : 0.f, p1 = c + 1 <= r ? s[b][2 * e + 1] * scale * __expf(u[c + 1] - Rr) : 0.f;
          sum += p0 + p1;
          uint32_t h, l;
          split2(p0, p1, h, l);
          *reinterpret_cast<uint32_t*>(sPh + r * MW_VP + c * 2) = h;
          *reinterpret_cast<uint32_t*>(sPl + r * MW_VP + c * 2) = l;
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        if ((lane & 3) == 0) rs[ch * MW_C + r] = sum;
      }
      // n . q: four threads per token
      {
        const int t = tid >> 2;
        float a = 0.f;
        if (have_state)
          for (int v = tid & 3; v < D.d16 / 8; v += 4) {
            float q8[8];
            bf16x8_to_float(*reinterpret_cast<const bf16x8*>(sQ + t * pd + v * 16), q8);
#pragma unroll
            for (int e = 0; e < 8; e++) a += q8[e] * n[v * 8 + e];
          }
        a += __shfl_xor_sync(0xffffffffu, a, 1);
        a += __shfl_xor_sync(0xffffffffu, a, 2);
        if ((tid & 3) == 0) nq[t] = a;
      }
    }
    __syncthreads();
    if constexpr (OUT) {
      // outputs: rows 16 rt, value columns 32 ch
      float o[4][4];
#pragma unroll
      for (int b = 0; b < 4; b++) o[b][0] = o[b][1] = o[b][2] = o[b][3] = 0.f;
      const uint32_t bofs = ((lane & 7) + (((lane >> 3) & 1) << 3)) * MW_VP + (ch * 32 + (lane >> 4) * 8) * 2;
      const int r0 = rt * 16 + g;
      const float e0 = __expf(m_in - R[r0]) * scale, e1 = __expf(m_in - R[r0 + 8]) * scale;
      if (have_state) {
        const uint32_t qa = smem_u32(sQ) + (rt * 16 + (lane & 15)) * pd + (lane >> 4) * 16;
        const uint32_t sh = smem_u32(sSh) + bofs, sl = smem_u32(sSl) + bofs;
        for (int ks = 0; ks < ksteps; ks++) {
          uint32_t a[4];
          ldmatrix_x4(a, qa + ks * 32);
#pragma unroll
          for (int b = 0; b < 2; b++) {
            uint32_t h[4], l[4];
            ldmatrix_x4_trans(h, sh + ks * 16 * MW_VP + b * 32);
            ldmatrix_x4_trans(l, sl + ks * 16 * MW_VP + b * 32);
            mma_16816(o[2 * b], a, h[0], h[1]);
            mma_16816(o[2 * b + 1], a, h[2], h[3]);
            mma_16816(o[2 * b], a, l[0], l[1]);
            mma_16816(o[2 * b + 1], a, l[2], l[3]);
          }
        }
#pragma unroll
        for (int b = 0; b < 4; b++) { o[b][0] *= e0; o[b][1] *= e0; o[b][2] *= e1; o[b][3] *= e1; }
      }
      const uint32_t pofs = (rt * 16 + (lane & 15)) * MW_VP + (lane >> 4) * 16;
      for (int kt = 0; kt <= rt; kt++) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, smem_u32(sPh) + pofs + kt * 32);
        ldmatrix_x4(al, smem_u32(sPl) + pofs + kt * 32);
#pragma unroll
        for (int b = 0; b < 2; b++) {
          uint32_t v[4];
          ldmatrix_x4_trans(v, smem_u32(sV) + bofs + kt * 16 * MW_VP + b * 32);
          mma_16816(o[2 * b], ah, v[0], v[1]);
          mma_16816(o[2 * b + 1], ah, v[2], v[3]);
          mma_16816(o[2 * b], al, v[0], v[1]);
          mma_16816(o[2 * b + 1], al, v[2], v[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int r = r0 + 8 * e;
        const float dot = nq[r] * (e ? e1 : e0) + rs[r] + rs[MW_C + r];
        const float inv = 1.f / (fmaxf(fabsf(dot), __expf(-(Fs[r] + R[r]))) + DEN_EPS);
        float* dst = io.o + (size_t)(row0 + c0 + r) * D.H * D.v16 + hd * D.v16;
#pragma unroll
        for (int b = 0; b < 4; b++) {
          const int c = v0 + ch * 32 + b * 8 + t2;
          if (r < cnt && c < D.v16) *reinterpret_cast<float2*>(dst + c) = make_float2(o[b][2 * e] * inv, o[b][2 * e + 1] * inv);
        }
      }
    }
    // the state after the chunk
    if (warp * MT < mtiles) {
#pragma unroll
      for (int a = 0; a < MT; a++)
#pragma unroll
        for (int b = 0; b < 8; b++)
#pragma unroll
          for (int e = 0; e < 4; e++) S[a][b][e] *= decay;
      const uint32_t bofs = ((lane & 7) + (((lane >> 3) & 1) << 3)) * MW_VP + (lane >> 4) * 16;
      for (int kt = 0; kt < MW_C / 16; kt++) {
        uint32_t a[MT][4];
#pragma unroll
        for (int i = 0; i < MT; i++) {
          const int m0 = min(warp * MT + i, mtiles - 1) * 16;
          ldmatrix_x4_trans(a[i], smem_u32(sK) + (kt * 16 + ((lane >> 4) << 3) + (lane & 7)) * pd + (m0 + ((lane >> 3) & 1) * 8) * 2);
        }
#pragma unroll
        for (int b = 0; b < 4; b++) {
          uint32_t h[4], l[4];
          ldmatrix_x4_trans(h, smem_u32(sWh) + bofs + kt * 16 * MW_VP + b * 32);
          ldmatrix_x4_trans(l, smem_u32(sWl) + bofs + kt * 16 * MW_VP + b * 32);
#pragma unroll
          for (int i = 0; i < MT; i++) {
            mma_16816(S[i][2 * b], a[i], h[0], h[1]);
            mma_16816(S[i][2 * b + 1], a[i], h[2], h[3]);
            mma_16816(S[i][2 * b], a[i], l[0], l[1]);
            mma_16816(S[i][2 * b + 1], a[i], l[2], l[3]);
          }
        }
      }
    }
    for (int i = tid; i < D.d16; i += 256) {
      float a = 0.f;
#pragma unroll 8
      for (int t = 0; t < MW_C; t++) a += w[t] * __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sK + t * pd + i * 2));
      n[i] = n[i] * decay + a;                // read by the next chunk only: the barrier below and the one after its loads lie in between
    }
    const float f_last = Fs[MW_C - 1];
    m_in = f_last + R_last;
    f_total += f_last;
    have_state = true;
    __syncthreads();
    if (c0 + MW_C < rows) {
      load_chunk(c0 + MW_C, min(MW_C, rows - c0 - MW_C));
      if (OUT) publish();
    }
  }
  if (OUT && !(flags & SEG_LAST)) return;
  float* dst = OUT ? slot : scratch + (size_t)(sg[5] + 1) * D.H * D.head() + hd * D.head();
#pragma unroll
  for (int a = 0; a < MT; a++)
#pragma unroll
    for (int b = 0; b < 8; b++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int r = (warp * MT + a) * 16 + g + 8 * e, c = v0 + b * 8 + t2;
        if (r < D.d16 && c < D.v16) *reinterpret_cast<float2*>(dst + (size_t)r * D.v16 + c) = make_float2(S[a][b][2 * e], S[a][b][2 * e + 1]);
      }
  if (blockIdx.z == 0) {
    // a slot's n may still be unread by the other CTAs of this head: it moves there later
    float* nd = OUT ? io.nm + ((size_t)sg[3] * D.H + hd) * (D.d16 + 4) : dst + n_at;
    for (int i = tid; i < D.d16; i += 256) nd[i] = n[i];
    if (tid == 0) {
      nd[D.d16] = m_in;
      nd[D.d16 + 1] = f_total;
    }
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

// rows: warp per head. CTAs past the rows move n and m of one sequence into its slot.
template <typename T>
__global__ void __launch_bounds__(128) mm_finish_kernel(const float* __restrict__ o, int rows, const T* __restrict__ gate, int64_t ldg, const float* __restrict__ norm, float eps,
                                                        float out_scale, T* __restrict__ out, int64_t ldo, MemDims D, const int4* __restrict__ seqs,
                                                        const float* __restrict__ nm, float* __restrict__ slots, size_t slot_stride) {
  if ((int)blockIdx.x >= rows) {
    const int s = blockIdx.x - rows;
    float* dst = slots + (size_t)seqs[s].z * slot_stride;
    for (int i = threadIdx.x; i < D.H * (D.d16 + 1); i += 128) {
      const int hd = i / (D.d16 + 1), e = i % (D.d16 + 1);
      dst[hd * D.head() + (size_t)D.d16 * D.v16 + e] = nm[((size_t)s * D.H + hd) * (D.d16 + 4) + e];
    }
    return;
  }
  const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int hd = warp; hd < D.H; hd += 4) {
    const float* src = o + (size_t)r * D.H * D.v16 + hd * D.v16;
    float ss = 0.f;
    for (int c = lane * 4; c < D.v16; c += 128) {
      const float4 v = *reinterpret_cast<const float4*>(src + c);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)D.dv + eps) * out_scale;
    for (int c = lane * 4; c < D.v16; c += 128) {
      const float4 v = *reinterpret_cast<const float4*>(src + c), w = *reinterpret_cast<const float4*>(norm + hd * D.v16 + c);
      const float x[4] = {v.x * w.x, v.y * w.y, v.z * w.z, v.w * w.w};
      const T* gr = gate + (size_t)r * ldg + hd * D.v16 + c;
      T* dst = out + (size_t)r * ldo + hd * D.v16 + c;
      float y[4];
      if constexpr (sizeof(T) == 4) {
        const float4 gv = *reinterpret_cast<const float4*>(gr);
        y[0] = gv.x; y[1] = gv.y; y[2] = gv.z; y[3] = gv.w;
      } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(gr);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        y[0] = a.x; y[1] = a.y; y[2] = b.x; y[3] = b.y;
      }
#pragma unroll
      for (int e = 0; e < 4; e++) y[e] = x[e] * rstd * (sizeof(T) == 4 ? sigmoid_exact(y[e]) : 1.f / (1.f + __expf(-y[e])));
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(y[0], y[1]), b = __floats2bfloat162_rn(y[2], y[3]);
        uint2 pk;
        pk.x = *reinterpret_cast<uint32_t*>(&a);
        pk.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(dst) = pk;
      }
    }
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

template <int MT, bool OUT>
int launch_walk(dim3 grid, cudaStream_t st, const MemIO& io, const MemDims& D, float* scratch) {
  static bool done[64] = {};
  int dev = 0;
  FT_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 64 && !done[dev]) {
    FT_CUDA_TRY(cudaFuncSetAttribute(mm_walk_kernel<MT, OUT>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX));
    done[dev] = true;
  }
  mm_walk_kernel<MT, OUT><<<grid, 256, mw_smem(D.d16, OUT), st>>>(io, D, scratch);
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
FT_EXPORT int ft_mm_walk_fits(int d, int dv) {
  const int d16 = (d + 15) & ~15;
  return d >= 1 && dv >= 1 && d16 <= 256 && mw_smem(d16, true) <= SMEM_MAX;
}

// Prompt stretches of a ragged batch in bf16. x [rows][ld]: queries H x d16 | keys H x d16 | values H x v16 (16-byte aligned, ld a multiple of 8); gates f32 [rows][ldg]: input
// gates, at column h8 = H rounded up to 8 forget gates; biases f32 [H]. segs int[nsegs][8] {first row, rows, slot, sequence, flags, scratch state, 0, 0}, flags 1: the only segment
// of its stretch (its state comes from the slot), 2: last, 4: the sequence starts (zero state). out = 0: contributions of the segments into scratch states [scratch state + 1] (f32 [H][d16 v16 + d16 + 4]
// each); out = 1: outputs o f32 [rows][H * v16], last segments leave S in their slot (f32 slots of slot_stride) and n, m in nm f32 [sequence][H][d16 + 4].
FT_EXPORT int ft_mm_walk(const void* x, int64_t ld, const float* gates, int64_t ldg, const float* bias_i, const float* bias_f, float cap, const int* segs, int nsegs, int H, int d,
                         int dv, float* slots, int64_t slot_stride, float* scratch, float* nm, float* o, int out, cudaStream_t st) {
  MemDims D;
  if (nsegs < 1 || !make_dims(D, H, d, dv, cap) || (ld & 7) || (reinterpret_cast<uintptr_t>(x) & 15) || (!out && !scratch) || (out && (!o || !nm))) return FT_ERR_ARG;
  if (!ft_mm_walk_fits(d, dv)) return FT_ERR_TOO_LARGE;
  const MemIO io{x, ld, gates, ldg, bias_i, bias_f, segs, slots, (size_t)slot_stride, nm, o};
  const dim3 grid(nsegs, H, (D.v16 + MW_V - 1) / MW_V);
  if (D.d16 <= 128) return out ? launch_walk<1, true>(grid, st, io, D, scratch) : launch_walk<1, false>(grid, st, io, D, scratch);
  return out ? launch_walk<2, true>(grid, st, io, D, scratch) : launch_walk<2, false>(grid, st, io, D, scratch);
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
                         int dv, float* slots, int64_t slot_stride, float* nm, float* o, int is_f32, cudaStream_t st) {
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

// out [rows][ldo] (heads of v16) = o / rms(o of the head) * norm (f32 [H * v16]) * sigmoid(gate [rows][ldg]) * out_scale; moves n and m of every sequence of seqs (as for
// ft_mm_merge) from nm into its slot.
FT_EXPORT int ft_mm_finish(const float* o, int rows, const void* gate, int64_t ldg, const float* norm, float eps, float out_scale, void* out, int64_t ldo, int H, int d, int dv,
                           const int* seqs, int nseq, const float* nm, float* slots, int64_t slot_stride, int is_f32, cudaStream_t st) {
  MemDims D;
  if (rows < 1 || nseq < 1 || !make_dims(D, H, d, dv, 1.f) || (ldg & 3) || (ldo & 3)) return FT_ERR_ARG;
  const int4* sq = reinterpret_cast<const int4*>(seqs);
  if (is_f32) mm_finish_kernel<float><<<rows + nseq, 128, 0, st>>>(o, rows, (const float*)gate, ldg, norm, eps, out_scale, (float*)out, ldo, D, sq, nm, slots, (size_t)slot_stride);
  else mm_finish_kernel<__nv_bfloat16><<<rows + nseq, 128, 0, st>>>(o, rows, (const __nv_bfloat16*)gate, ldg, norm, eps, out_scale, (__nv_bfloat16*)out, ldo, D, sq, nm, slots,
                                                                   (size_t)slot_stride);
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
