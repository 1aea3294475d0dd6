// Chunk-parallel form of the linear-attention recurrences whose decay is ONE number per head - fixed (RecurArgs mode 0)
// or a new one for every token (mode 2 with g_head: the state-space mixer) - for prompts.
//
//   S_t = lam S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
//
// (written below for a fixed lam; with a decay a_t per token every power lam^(i-j) becomes the product a_(j+1) .. a_i,
// formed as exp(c_i - c_j) from the running sums c of the decays' logarithms inside the chunk, so that no product of
// many small numbers is ever divided by another one.)
//
// Inside a chunk of CH tokens that starts from the state P, token i (0-based) reads
//   o_i = lam^(i+1) P^T q_i + sum_{j <= i} lam^(i-j) (q_i . k_j) v_j
// and the chunk leaves  lam^n P + sum_j lam^(n-1-j) k_j v_j^T  behind (n = tokens in the chunk).  Nothing in the two
// sums depends on another chunk, so a prompt runs as three launches over all (sequence, head, chunk) at once instead
// of one dependent chain over its tokens:
//   1. lin_chunk_state_kernel   D_c = sum_j lam^(n-1-j) k_j v_j^T           one CTA per (chunk, head, sequence)
//   2. lin_chunk_scan_kernel    P_c = state before chunk c, in place of D_c; the slot's state after the last chunk
//   3. lin_chunk_out_kernel     A = (Q K^T) .* lam^(i-j) (causal), o = lam^(i+1) Q P_c + A V
// Every product is an fp32 FFMA chain over shared-memory tiles (4 x 4 outputs per thread, operands stored with the
// summed index outermost so that both are read as 16-byte vectors); the powers of lam come from double precision.
// With a normaliser (NRM: RecurArgs::n_state, the mLSTM) a column n of the state with values 1 runs along: a chunk adds
// the column sums of its scaled keys, and n . q is q . P_n plus the row sums of A.  Keys carry a factor per token
// (k_scale), and the decays' running sums are kept in double precision: a log decay can be as large as -30, and the
// difference of two sums of 64 of them is what enters the exponential.
// In bf16 mode (RecurArgs::bf16_ops, mLSTM) steps 1 and 3 run on warp-level tensor products with fp32 accumulation: queries,
// keys and values, which are outputs of bf16 projections, are operands as they are (bf16), while everything the recurrence
// itself makes - decayed keys, decayed scores, the states - enters as a pair hi + lo of bf16 values (16 significant bits).
// A chunk's products are 64 x 64 tiles with 64 .. 256 summed terms, and their operands are built in the kernel.
// The sums run in another order than the token-by-token kernel, so the two agree to fp32 rounding, not bit for bit.
#include <stdint.h>

#include "common.cuh"
#include "mixer.h"

namespace {

constexpr int CH = 64;       // tokens per chunk
constexpr int LDT = CH + 4;  // row length of a transposed [channel][token] tile: 16-byte rows, 4-bank skew

__device__ __forceinline__ float act_silu(int act_in, float x) {
  return act_in == 0 ? x : act_in == 2 ? __fdividef(x, 1.0f + __expf(-x)) : silu_ref(x);
}

// acc[r][c] += sum_kk X[kk * ldx + r] * Y[kk * ldy + c]; X, Y already point at this thread's four rows / columns
__device__ __forceinline__ void mm44(const float* __restrict__ X, int ldx, const float* __restrict__ Y, int ldy, int K,
                                     float (&acc)[4][4]) {
#pragma unroll 8
  for (int kk = 0; kk < K; ++kk) {
    const float4 x = *reinterpret_cast<const float4*>(X + (size_t)kk * ldx);
    const float4 y = *reinterpret_cast<const float4*>(Y + (size_t)kk * ldy);
    acc[0][0] += x.x * y.x; acc[0][1] += x.x * y.y; acc[0][2] += x.x * y.z; acc[0][3] += x.x * y.w;
    acc[1][0] += x.y * y.x; acc[1][1] += x.y * y.y; acc[1][2] += x.y * y.z; acc[1][3] += x.y * y.w;
    acc[2][0] += x.z * y.x; acc[2][1] += x.z * y.y; acc[2][2] += x.z * y.z; acc[2][3] += x.z * y.w;
    acc[3][0] += x.w * y.x; acc[3][1] += x.w * y.y; acc[3][2] += x.w * y.z; acc[3][3] += x.w * y.w;
  }
}

__device__ __forceinline__ void zero44(float (&acc)[4][4]) {
#pragma unroll
  for (int r = 0; r < 4; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[r][c] = 0.f;
}

// powers lam^0 .. lam^CH of this head's decay, from double precision
__device__ __forceinline__ void fill_powers(float* pw, float lam) {
  for (int p = threadIdx.x; p <= CH; p += blockDim.x) pw[p] = (float)pow((double)lam, (double)p);
}

// cl[j] = sum over t <= j of the chunk's log decays (tokens >= n add nothing): warp 0 scans, 32 tokens at a time
template <typename T>
__device__ __forceinline__ void fill_cumlog(T* cl, const float* __restrict__ lg, size_t stride, int n) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  T carry = 0;
  for (int j0 = 0; j0 < CH; j0 += 32) {
    const int j = j0 + lane;
    T v = j < n ? (T)lg[(size_t)j * stride] : (T)0;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const T t = __shfl_up_sync(L3_FULL, v, o);
      if (lane >= o) v += t;
    }
    v += carry;
    cl[j] = v;
    carry = __shfl_sync(L3_FULL, v, 31);
  }
}

// where the chunks' total decays live inside the workspace: behind the chunk states
__device__ __forceinline__ float* chunk_decays(const RecurArgs& a, int NC) { return a.ws + (size_t)a.B * a.H * NC * a.DK * a.DV; }
// and the chunks' normaliser columns [B, H, NC, DK] behind those (on a multiple of four floats)
__device__ __forceinline__ float* chunk_norms(const RecurArgs& a, int NC) {
  return a.ws + (size_t)a.B * a.H * NC * a.DK * a.DV + (((size_t)a.B * a.H * NC + 3) & ~(size_t)3);
}

// rows [n, CH) of a natural [token][cols] tile and tokens >= n of the operands are zero: they add nothing
__device__ __forceinline__ void load_natural(float* dst, int ld_dst, const float* src, size_t ld_src, int n, int cols, int act_in,
                                             const float* row_scale) {
  const int c4 = cols / 4;
  for (int idx = threadIdx.x; idx < CH * c4; idx += blockDim.x) {
    const int j = idx / c4, c = (idx - j * c4) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < n) {
      v = *reinterpret_cast<const float4*>(src + (size_t)j * ld_src + c);
      const float s = row_scale ? row_scale[j] : 1.f;
      v.x = act_silu(act_in, v.x) * s; v.y = act_silu(act_in, v.y) * s;
      v.z = act_silu(act_in, v.z) * s; v.w = act_silu(act_in, v.w) * s;
    }
    *reinterpret_cast<float4*>(dst + (size_t)j * ld_dst + c) = v;
  }
}

// dst[channel][token] from rows [token][channel]: a lane takes four channels of one token (one 16-byte load), and
// adjacent lanes take adjacent tokens, so the four scalar stores of a warp fall into distinct banks
__device__ __forceinline__ void load_transposed(float* dst, const float* src, size_t ld_src, int n, int cols, int act_in, float mul = 1.f) {
  const int c4 = cols / 4;
  for (int idx = threadIdx.x; idx < CH * c4; idx += blockDim.x) {
    const int j = idx % CH, c = (idx / CH) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < n) {
      v = *reinterpret_cast<const float4*>(src + (size_t)j * ld_src + c);
      v.x = act_silu(act_in, v.x); v.y = act_silu(act_in, v.y); v.z = act_silu(act_in, v.z); v.w = act_silu(act_in, v.w);
      v.x *= mul; v.y *= mul; v.z *= mul; v.w *= mul;
    }
    dst[(size_t)(c + 0) * LDT + j] = v.x;
    dst[(size_t)(c + 1) * LDT + j] = v.y;
    dst[(size_t)(c + 2) * LDT + j] = v.z;
    dst[(size_t)(c + 3) * LDT + j] = v.w;
  }
}

// ---------------------------------------------------------------------------- 1. what a chunk adds to the state
template <bool DEC, bool NRM>
__global__ void __launch_bounds__(256) lin_chunk_state_kernel(RecurArgs a, int NC) {
  extern __shared__ __align__(16) float sm[];
  __shared__ double pd[NRM ? CH : 1];
  float* pw = sm;                 // [CH + 1] + scale per token [CH]
  float* sc = pw + CH + 4;        // lam^(n - 1 - j)
  float* Ks = sc + CH;            // [CH][DK]
  float* Vs = Ks + (size_t)CH * a.DK;  // [CH][DV]
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int n = min(CH, a.L - c * CH);
  const size_t row0 = (size_t)b * a.L + (size_t)c * CH;
  if (NRM) fill_cumlog(pd, a.log_g + row0 * a.H + h, a.H, n);
  else if (DEC) fill_cumlog(pw, a.log_g + row0 * a.H + h, a.H, n);
  else fill_powers(pw, a.head_decay[h]);
  __syncthreads();
  if (NRM) {
    for (int j = tid; j < CH; j += blockDim.x) sc[j] = j < n ? expf((float)(pd[n - 1] - pd[j])) * a.k_scale[(row0 + j) * a.H + h] : 0.f;
    if (tid == 0) chunk_decays(a, NC)[((size_t)b * a.H + h) * NC + c] = expf((float)pd[n - 1]);
  } else {
    for (int j = tid; j < CH; j += blockDim.x) sc[j] = j < n ? (DEC ? expf(pw[n - 1] - pw[j]) : pw[n - 1 - j]) : 0.f;
    if (DEC && tid == 0) chunk_decays(a, NC)[((size_t)b * a.H + h) * NC + c] = expf(pw[n - 1]);
  }
  __syncthreads();
  load_natural(Ks, a.DK, a.k + row0 * a.ld_k + (size_t)(h / a.rep) * a.DK, a.ld_k, n, a.DK, a.act_in, sc);
  load_natural(Vs, a.DV, a.v + row0 * a.ld_v + (size_t)h * a.DV, a.ld_v, n, a.DV, a.act_in, nullptr);
  __syncthreads();
  if (NRM)
    for (int d = tid; d < a.DK; d += blockDim.x) {
      float t = 0.f;
#pragma unroll 8
      for (int j = 0; j < CH; ++j) t += Ks[(size_t)j * a.DK + d];
      chunk_norms(a, NC)[(((size_t)b * a.H + h) * NC + c) * a.DK + d] = t;
    }
  const int tx = tid & 15, ty = tid >> 4;
  float* D = a.ws + (((size_t)b * a.H + h) * NC + c) * a.DK * a.DV;
  for (int d0 = 0; d0 < a.DK; d0 += 64)
    for (int e0 = 0; e0 < a.DV; e0 += 64) {
      float acc[4][4];
      zero44(acc);
      mm44(Ks + d0 + ty * 4, a.DK, Vs + e0 + tx * 4, a.DV, CH, acc);
#pragma unroll
      for (int r = 0; r < 4; ++r)
        *reinterpret_cast<float4*>(D + (size_t)(d0 + ty * 4 + r) * a.DV + e0 + tx * 4) =
            make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
    }
}

// ---------------------------------------------------------------------------- 2. the states between the chunks
template <bool DEC, bool NRM>
__global__ void __launch_bounds__(256) lin_chunk_scan_kernel(RecurArgs a, int NC) {
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z;
  size_t n4 = (size_t)a.DK * a.DV / 4;
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const bool is_n = NRM && i >= n4;  // the normaliser's column, behind the matrix
  if (i >= n4 + (NRM ? a.DK / 4 : 0)) return;
  const float lam = DEC ? 0.f : a.head_decay[h];
  const float full = DEC ? 0.f : (float)pow((double)lam, (double)CH);
  const float last = DEC ? 0.f : (float)pow((double)lam, (double)(a.L - (NC - 1) * CH));
  const float* cdec = DEC ? chunk_decays(a, NC) + ((size_t)b * a.H + h) * NC : nullptr;
  float4* st;
  float4* W;
  if (is_n) {
    i -= n4;
    n4 = a.DK / 4;
    st = reinterpret_cast<float4*>(a.n_state + ((size_t)b * a.H + h) * a.DK) + i;
    W = reinterpret_cast<float4*>(chunk_norms(a, NC) + ((size_t)b * a.H + h) * NC * a.DK) + i;
  } else {
    st = reinterpret_cast<float4*>(a.state + ((size_t)b * a.H + h) * a.DK * a.DV) + i;
    W = reinterpret_cast<float4*>(a.ws + ((size_t)b * a.H + h) * NC * a.DK * a.DV) + i;
  }
  float4 S = *st;
  // the chunk sums do not depend on S: four loads stay in flight ahead of the chain
  constexpr int AHEAD = 4;
  float4 d[AHEAD];
#pragma unroll
  for (int u = 0; u < AHEAD; ++u) d[u] = u < NC ? W[(size_t)u * n4] : make_float4(0.f, 0.f, 0.f, 0.f);
  for (int c0 = 0; c0 < NC; c0 += AHEAD) {
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int c = c0 + u;
      if (c < NC) {
        const float4 cur = d[u];
        if (c + AHEAD < NC) d[u] = W[(size_t)(c + AHEAD) * n4];
        W[(size_t)c * n4] = S;
        const float f = DEC ? cdec[c] : c == NC - 1 ? last : full;
        S.x = f * S.x + cur.x; S.y = f * S.y + cur.y; S.z = f * S.z + cur.z; S.w = f * S.w + cur.w;
      }
    }
  }
  *st = S;
}

// ---------------------------------------------------------------------------- 3. the outputs of a chunk
template <bool DEC, bool NRM>
__global__ void __launch_bounds__(256) lin_chunk_out_kernel(RecurArgs a, int NC) {
  extern __shared__ __align__(16) float sm[];
  __shared__ double pd[NRM ? CH : 1];
  __shared__ float ks[NRM ? CH : 1];
  float* pw = sm;                            // [CH + 1]
  float* Qt = pw + CH + 4;                   // [DK][LDT]
  float* Kt = Qt + (size_t)a.DK * LDT;       // [DK][LDT]
  float* At = Kt + (size_t)a.DK * LDT;       // [CH][LDT]: At[j][i] = lam^(i-j) q_i . k_j for j <= i
  float* Vs = At + (size_t)CH * LDT;         // [CH][64]
  float* Ps = Kt;                            // [DK][64]: the keys are done with once A stands
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int n = min(CH, a.L - c * CH);
  const size_t row0 = (size_t)b * a.L + (size_t)c * CH;
  if (NRM) {
    fill_cumlog(pd, a.log_g + row0 * a.H + h, a.H, n);
    if (tid >= 32 && tid < 32 + CH) ks[tid - 32] = tid - 32 < n ? a.k_scale[(row0 + tid - 32) * a.H + h] : 0.f;
  } else if (DEC) fill_cumlog(pw, a.log_g + row0 * a.H + h, a.H, n);
  else fill_powers(pw, a.head_decay[h]);
  load_transposed(Qt, a.q + row0 * a.ld_q + (size_t)(h / a.rep) * a.DK, a.ld_q, n, a.DK, a.act_in, NRM ? a.q_mul : 1.f);
  load_transposed(Kt, a.k + row0 * a.ld_k + (size_t)(h / a.rep) * a.DK, a.ld_k, n, a.DK, a.act_in);
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  {
    float acc[4][4];  // acc[r][cc]: query i = ty * 4 + r, key j = tx * 4 + cc
    zero44(acc);
    mm44(Qt + ty * 4, LDT, Kt + tx * 4, LDT, a.DK, acc);
#pragma unroll
    for (int cc = 0; cc < 4; ++cc) {
      const int j = tx * 4 + cc;
      float4 o;
      float* op = &o.x;
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int i = ty * 4 + r;
        if (NRM) op[r] = j <= i ? acc[r][cc] * (expf((float)(pd[i] - pd[j])) * ks[j]) : 0.f;
        else op[r] = j <= i ? acc[r][cc] * (DEC ? expf(pw[i] - pw[j]) : pw[i - j]) : 0.f;
      }
      *reinterpret_cast<float4*>(At + (size_t)j * LDT + ty * 4) = o;
    }
  }
  if (NRM) {  // n . q of every token: four threads per row
    const float* Pn = chunk_norms(a, NC) + (((size_t)b * a.H + h) * NC + c) * a.DK;
    __syncthreads();  // At is written
    const int i = tid >> 2, part = tid & 3;
    float t = 0.f;
    for (int d = part; d < a.DK; d += 4) t = fmaf(Qt[(size_t)d * LDT + i], Pn[d], t);
    t *= expf((float)pd[i]);
    for (int j = part; j <= i; j += 4) t += At[(size_t)j * LDT + i];
    t += __shfl_xor_sync(L3_FULL, t, 1);
    t += __shfl_xor_sync(L3_FULL, t, 2);
    if (part == 0 && i < n) a.nq[(row0 + i) * a.H + h] = t;
  }
  const float* P = a.ws + (((size_t)b * a.H + h) * NC + c) * a.DK * a.DV;
  const int O = a.H * a.DV;
  for (int e0 = 0; e0 < a.DV; e0 += 64) {
    __syncthreads();  // At is written; the previous tile's Vs / Ps are no longer read
    load_natural(Vs, 64, a.v + row0 * a.ld_v + (size_t)h * a.DV + e0, a.ld_v, n, 64, a.act_in, nullptr);
    for (int idx = tid; idx < a.DK * 16; idx += blockDim.x) {
      const int d = idx >> 4, e = (idx & 15) * 4;
      *reinterpret_cast<float4*>(Ps + (size_t)d * 64 + e) = *reinterpret_cast<const float4*>(P + (size_t)d * a.DV + e0 + e);
    }
    __syncthreads();
    float acc[4][4];
    zero44(acc);
    mm44(Qt + ty * 4, LDT, Ps + tx * 4, 64, a.DK, acc);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const float f = NRM ? expf((float)pd[ty * 4 + r]) : DEC ? expf(pw[ty * 4 + r]) : pw[ty * 4 + r + 1];
#pragma unroll
      for (int cc = 0; cc < 4; ++cc) acc[r][cc] *= f;
    }
    mm44(At + ty * 4, LDT, Vs + tx * 4, 64, CH, acc);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int i = ty * 4 + r;
      if (i < n)
        *reinterpret_cast<float4*>(a.out + (row0 + i) * O + (size_t)h * a.DV + e0 + tx * 4) =
            make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
    }
  }
}

// ---------------------------------------------------------------------------- bf16 mode: the same two kernels on mma.sync
constexpr int LDE = 64 + 8;  // row length of a 64-wide bf16 tile: rows 144 bytes apart fall into distinct banks

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint2 pack4(const float4& v) {
  union { __nv_bfloat162 h[2]; uint2 u; } o;
  o.h[0] = __floats2bfloat162_rn(v.x, v.y);
  o.h[1] = __floats2bfloat162_rn(v.z, v.w);
  return o.u;
}
// v = hi + lo up to 2^-17 of v
__device__ __forceinline__ void split4(const float4& v, uint2& hi, uint2& lo) {
  hi = pack4(v);
  lo = pack4(make_float4(v.x - __uint_as_float(hi.x << 16), v.y - __uint_as_float(hi.x & 0xffff0000u), v.z - __uint_as_float(hi.y << 16),
                         v.w - __uint_as_float(hi.y & 0xffff0000u)));
}

// A [ROWS][COLS] block of floats on its way into bf16 tiles: fetch() issues every load of the thread's share at once, put() /
// put_split() converts and stores it; between the two a thread can work on the previous block.  Rows >= n are zeros.
template <int ROWS, int COLS>
struct Block {
  static constexpr int C4 = COLS / 4, N = ROWS * C4 / 256;
  static_assert(ROWS * C4 % 256 == 0, "a whole number of vectors per thread");
  float4 v[N];
  __device__ __forceinline__ void fetch(const float* src, size_t ld, int n) {
#pragma unroll
    for (int u = 0; u < N; ++u) {
      const int idx = threadIdx.x + u * 256, j = idx / C4, c = (idx % C4) * 4;
      v[u] = j < n ? *reinterpret_cast<const float4*>(src + (size_t)j * ld + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  __device__ __forceinline__ void put(bf16* dst, int ld_dst, float mul) const {
#pragma unroll
    for (int u = 0; u < N; ++u) {
      const int idx = threadIdx.x + u * 256, j = idx / C4, c = (idx % C4) * 4;
      *reinterpret_cast<uint2*>(dst + (size_t)j * ld_dst + c) = pack4(make_float4(v[u].x * mul, v[u].y * mul, v[u].z * mul, v[u].w * mul));
    }
  }
  // a (hi, lo) pair of tiles, row j times row_mul[j] (null: 1)
  __device__ __forceinline__ void put_split(bf16* hi, bf16* lo, int ld_dst, const float* row_mul) const {
#pragma unroll
    for (int u = 0; u < N; ++u) {
      const int idx = threadIdx.x + u * 256, j = idx / C4, c = (idx % C4) * 4;
      const float m = row_mul ? row_mul[j] : 1.f;
      uint2 h, l;
      split4(make_float4(v[u].x * m, v[u].y * m, v[u].z * m, v[u].w * m), h, l);
      *reinterpret_cast<uint2*>(hi + (size_t)j * ld_dst + c) = h;
      *reinterpret_cast<uint2*>(lo + (size_t)j * ld_dst + c) = l;
    }
  }
};

// grid (NC * NE, H, B): the chunk's D, value columns [e_lo, e_hi) of it.  8 warps on a 64 x 64 tile: 16 rows x 32 columns each
template <int DK>
__global__ void __launch_bounds__(256) lin_chunk_state_mma_kernel(RecurArgs a, int NC, int NE) {
  extern __shared__ __align__(16) uint8_t smb[];
  __shared__ double pd[CH];
  __shared__ float sc[CH];
  constexpr int LDK = DK + 8;
  bf16* Kh = reinterpret_cast<bf16*>(smb);           // [CH][LDK] decayed keys, hi and lo
  bf16* Kl = Kh + (size_t)CH * LDK;
  bf16* Vs = Kl + (size_t)CH * LDK;                  // [CH][LDE]
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x / NE, ne = blockIdx.x - c * NE, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int lane = tid & 31, warp = tid >> 5, wm = warp & 3, wn = warp >> 2;
  const int n = min(CH, a.L - c * CH);
  const size_t row0 = (size_t)b * a.L + (size_t)c * CH;
  const int per = a.DV / 64 / NE, e_lo = ne * per * 64, e_hi = e_lo + per * 64;
  const float* vsrc = a.v + row0 * a.ld_v + (size_t)h * a.DV;
  Block<CH, DK> kb;
  Block<CH, 64> vb;
  kb.fetch(a.k + row0 * a.ld_k + (size_t)(h / a.rep) * DK, a.ld_k, n);
  vb.fetch(vsrc + e_lo, a.ld_v, n);
  fill_cumlog(pd, a.log_g + row0 * a.H + h, a.H, n);
  __syncthreads();
  for (int j = tid; j < CH; j += 256) sc[j] = j < n ? expf((float)(pd[n - 1] - pd[j])) * a.k_scale[(row0 + j) * a.H + h] : 0.f;
  if (ne == 0 && tid == 0) chunk_decays(a, NC)[((size_t)b * a.H + h) * NC + c] = expf((float)pd[n - 1]);
  __syncthreads();
  kb.put_split(Kh, Kl, LDK, sc);
  float* D = a.ws + (((size_t)b * a.H + h) * NC + c) * a.DK * a.DV;
  for (int e0 = e_lo; e0 < e_hi; e0 += 64) {
    if (e0 > e_lo) __syncthreads();  // the previous tile's values are no longer read
    vb.put(Vs, LDE, 1.f);
    __syncthreads();
    if (e0 + 64 < e_hi) vb.fetch(vsrc + e0 + 64, a.ld_v, n);  // in flight during the products
    if (ne == 0 && e0 == 0)
      for (int d = tid; d < DK; d += 256) {
        float t = 0.f;
#pragma unroll 8
        for (int j = 0; j < CH; ++j) t += __bfloat162float(Kh[(size_t)j * LDK + d]) + __bfloat162float(Kl[(size_t)j * LDK + d]);
        chunk_norms(a, NC)[(((size_t)b * a.H + h) * NC + c) * DK + d] = t;
      }
#pragma unroll 1
    for (int d0 = 0; d0 < DK; d0 += 64) {
      float acc[4][4];
      zero44(acc);
#pragma unroll
      for (int k0 = 0; k0 < CH; k0 += 16) {
        uint32_t ah[4], al[4], v0[4], v1[4];
        // A = K^T: tokens are rows of the tile, so both operands are read transposed
        const size_t ka = (size_t)(k0 + (lane & 7) + ((lane >> 4) << 3)) * LDK + d0 + wm * 16 + ((lane >> 3) & 1) * 8;
        ldsm4t(ah, smem_addr(Kh + ka));
        ldsm4t(al, smem_addr(Kl + ka));
        const bf16* vp = Vs + (size_t)(k0 + (lane & 15)) * LDE + wn * 32 + (lane >> 4) * 8;
        ldsm4t(v0, smem_addr(vp));
        ldsm4t(v1, smem_addr(vp + 16));
        mma16816(acc[0], ah, v0[0], v0[1]); mma16816(acc[1], ah, v0[2], v0[3]);
        mma16816(acc[2], ah, v1[0], v1[1]); mma16816(acc[3], ah, v1[2], v1[3]);
        mma16816(acc[0], al, v0[0], v0[1]); mma16816(acc[1], al, v0[2], v0[3]);
        mma16816(acc[2], al, v1[0], v1[1]); mma16816(acc[3], al, v1[2], v1[3]);
      }
      float* dp = D + (size_t)(d0 + wm * 16 + (lane >> 2)) * a.DV + e0 + wn * 32 + (lane & 3) * 2;
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        *reinterpret_cast<float2*>(dp + t * 8) = make_float2(acc[t][0], acc[t][1]);
        *reinterpret_cast<float2*>(dp + (size_t)8 * a.DV + t * 8) = make_float2(acc[t][2], acc[t][3]);
      }
    }
  }
}

// grid (NC * NE, H, B): the chunk's outputs, value columns as above
template <int DK>
__global__ void __launch_bounds__(256) lin_chunk_out_mma_kernel(RecurArgs a, int NC, int NE) {
  extern __shared__ __align__(16) uint8_t smb[];
  __shared__ double pd[CH];
  __shared__ float ks[CH], s_nq[2][CH];
  constexpr int LDK = DK + 8;
  bf16* Qs = reinterpret_cast<bf16*>(smb);           // [CH][LDK]
  bf16* Ks = Qs + (size_t)CH * LDK;                  // [CH][LDK]
  bf16* Ah = Ks + (size_t)CH * LDK;                  // [CH][LDE] decayed scores, hi and lo
  bf16* Al = Ah + (size_t)CH * LDE;
  bf16* Vs = Al + (size_t)CH * LDE;                  // [CH][LDE]
  bf16* Ph = Vs + (size_t)CH * LDE;                  // [DK][LDE] the state ahead of the chunk, hi and lo
  bf16* Pl = Ph + (size_t)DK * LDE;
  pdl_launch();
  pdl_wait();
  const int c = blockIdx.x / NE, ne = blockIdx.x - c * NE, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int lane = tid & 31, warp = tid >> 5, wm = warp & 3, wn = warp >> 2;
  const int n = min(CH, a.L - c * CH);
  const size_t row0 = (size_t)b * a.L + (size_t)c * CH;
  fill_cumlog(pd, a.log_g + row0 * a.H + h, a.H, n);
  if (tid >= 32 && tid < 32 + CH) ks[tid - 32] = tid - 32 < n ? a.k_scale[(row0 + tid - 32) * a.H + h] : 0.f;
  {
    Block<CH, DK> qb, kb;
    qb.fetch(a.q + row0 * a.ld_q + (size_t)(h / a.rep) * DK, a.ld_q, n);
    kb.fetch(a.k + row0 * a.ld_k + (size_t)(h / a.rep) * DK, a.ld_k, n);
    qb.put(Qs, LDK, a.q_mul);
    kb.put(Ks, LDK, 1.f);
  }
  const float* P = a.ws + (((size_t)b * a.H + h) * NC + c) * DK * a.DV;
  const float* vsrc = a.v + row0 * a.ld_v + (size_t)h * a.DV;
  const int O = a.H * a.DV;
  const int per = a.DV / 64 / NE, e_lo = ne * per * 64, e_hi = e_lo + per * 64;
  Block<CH, 64> vb;
  Block<DK, 64> pb;
  vb.fetch(vsrc + e_lo, a.ld_v, n);  // the first tile's values and state columns: in flight during the scores
  pb.fetch(P + e_lo, a.DV, DK);
  __syncthreads();
  const int r0 = wm * 16 + (lane >> 2);              // this lane's accumulator rows: r0 and r0 + 8
  const size_t qa = (size_t)(wm * 16 + (lane & 15)) * LDK + (lane >> 4) * 8;
  {
    float acc[4][4];
    zero44(acc);
    const bf16* kp = Ks + (size_t)(wn * 32 + (lane & 7) + ((lane >> 4) << 3)) * LDK + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int k0 = 0; k0 < DK; k0 += 16) {
      uint32_t q[4], k_0[4], k_1[4];
      ldsm4(q, smem_addr(Qs + qa + k0));
      ldsm4(k_0, smem_addr(kp + k0));
      ldsm4(k_1, smem_addr(kp + (size_t)16 * LDK + k0));
      mma16816(acc[0], q, k_0[0], k_0[1]); mma16816(acc[1], q, k_0[2], k_0[3]);
      mma16816(acc[2], q, k_1[0], k_1[1]); mma16816(acc[3], q, k_1[2], k_1[3]);
    }
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int t = 0; t < 4; ++t)
#pragma unroll
      for (int u = 0; u < 2; ++u) {                  // rows r0, r0 + 8
        const int i = r0 + u * 8, j = wn * 32 + t * 8 + (lane & 3) * 2;
        const float x = j <= i ? acc[t][2 * u] * (expf((float)(pd[i] - pd[j])) * ks[j]) : 0.f;
        const float y = j + 1 <= i ? acc[t][2 * u + 1] * (expf((float)(pd[i] - pd[j + 1])) * ks[j + 1]) : 0.f;
        sum[u] += x + y;
        const __nv_bfloat162 hi = __floats2bfloat162_rn(x, y);
        *reinterpret_cast<__nv_bfloat162*>(Ah + (size_t)i * LDE + j) = hi;
        *reinterpret_cast<__nv_bfloat162*>(Al + (size_t)i * LDE + j) = __floats2bfloat162_rn(x - __low2float(hi), y - __high2float(hi));
      }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      sum[u] += __shfl_xor_sync(L3_FULL, sum[u], 1);
      sum[u] += __shfl_xor_sync(L3_FULL, sum[u], 2);
      if ((lane & 3) == 0) s_nq[wn][r0 + u * 8] = sum[u];
    }
  }
  __syncthreads();
  if (ne == 0) {  // n . q of every token: four threads per row
    const float* Pn = chunk_norms(a, NC) + (((size_t)b * a.H + h) * NC + c) * DK;
    const int i = tid >> 2, part = tid & 3;
    float t = 0.f;
#pragma unroll 4
    for (int d = part * 2; d < DK; d += 8) {
      const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Qs + (size_t)i * LDK + d));
      t = fmaf(q.x, Pn[d], t);
      t = fmaf(q.y, Pn[d + 1], t);
    }
    t += __shfl_xor_sync(L3_FULL, t, 1);
    t += __shfl_xor_sync(L3_FULL, t, 2);
    if (part == 0 && i < n) a.nq[(row0 + i) * a.H + h] = fmaf(t, expf((float)pd[i]), s_nq[0][i] + s_nq[1][i]);
  }
  const float f0 = expf((float)pd[r0]), f1 = expf((float)pd[r0 + 8]);
  const size_t va = (size_t)(lane & 15) * LDE + wn * 32 + (lane >> 4) * 8, aa = (size_t)(wm * 16 + (lane & 15)) * LDE + (lane >> 4) * 8;
  for (int e0 = e_lo; e0 < e_hi; e0 += 64) {
    if (e0 > e_lo) __syncthreads();  // the previous tile's Vs / P are no longer read
    vb.put(Vs, LDE, 1.f);
    pb.put_split(Ph, Pl, LDE, nullptr);
    __syncthreads();
    if (e0 + 64 < e_hi) { vb.fetch(vsrc + e0 + 64, a.ld_v, n); pb.fetch(P + e0 + 64, a.DV, DK); }
    float acc[4][4];
    zero44(acc);
#pragma unroll 4
    for (int k0 = 0; k0 < DK; k0 += 16) {
      uint32_t q[4], p0[4], p1[4];
      ldsm4(q, smem_addr(Qs + qa + k0));
      const size_t o = (size_t)k0 * LDE + va;
      ldsm4t(p0, smem_addr(Ph + o));
      ldsm4t(p1, smem_addr(Ph + o + 16));
      mma16816(acc[0], q, p0[0], p0[1]); mma16816(acc[1], q, p0[2], p0[3]);
      mma16816(acc[2], q, p1[0], p1[1]); mma16816(acc[3], q, p1[2], p1[3]);
      ldsm4t(p0, smem_addr(Pl + o));
      ldsm4t(p1, smem_addr(Pl + o + 16));
      mma16816(acc[0], q, p0[0], p0[1]); mma16816(acc[1], q, p0[2], p0[3]);
      mma16816(acc[2], q, p1[0], p1[1]); mma16816(acc[3], q, p1[2], p1[3]);
    }
#pragma unroll
    for (int t = 0; t < 4; ++t) { acc[t][0] *= f0; acc[t][1] *= f0; acc[t][2] *= f1; acc[t][3] *= f1; }
#pragma unroll
    for (int k0 = 0; k0 < CH; k0 += 16) {
      uint32_t ah[4], al[4], v0[4], v1[4];
      ldsm4(ah, smem_addr(Ah + aa + k0));
      ldsm4(al, smem_addr(Al + aa + k0));
      const size_t o = (size_t)k0 * LDE + va;
      ldsm4t(v0, smem_addr(Vs + o));
      ldsm4t(v1, smem_addr(Vs + o + 16));
      mma16816(acc[0], ah, v0[0], v0[1]); mma16816(acc[1], ah, v0[2], v0[3]);
      mma16816(acc[2], ah, v1[0], v1[1]); mma16816(acc[3], ah, v1[2], v1[3]);
      mma16816(acc[0], al, v0[0], v0[1]); mma16816(acc[1], al, v0[2], v0[3]);
      mma16816(acc[2], al, v1[0], v1[1]); mma16816(acc[3], al, v1[2], v1[3]);
    }
    float* op = a.out + (row0 + r0) * O + (size_t)h * a.DV + e0 + wn * 32 + (lane & 3) * 2;
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      if (r0 < n) *reinterpret_cast<float2*>(op + t * 8) = make_float2(acc[t][0], acc[t][1]);
      if (r0 + 8 < n) *reinterpret_cast<float2*>(op + (size_t)8 * O + t * 8) = make_float2(acc[t][2], acc[t][3]);
    }
  }
}

// CTAs per chunk along the value columns: a divisor of the 64-column tiles, enough that `want` CTAs run
int value_splits(int ctas, int tiles, int want) {
  int ne = 1;
  for (int d = 1; d <= tiles; ++d)
    if (tiles % d == 0) { ne = d; if (ctas * d >= want) break; }
  return ne;
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

size_t recur_chunk_ws_floats(int B, int L, int H, int DK, int DV) {
  const size_t NC = (L + CH - 1) / CH;
  return (size_t)B * H * NC * DK * DV + (size_t)B * H * NC + 4 + (size_t)B * H * NC * DK;  // chunk states, total decays, normalisers
}

bool recur_chunk_shape(int DK, int DV) { return DK % 64 == 0 && DK <= 256 && DV % 64 == 0 && DV >= 64 && DV <= 512; }

bool recur_chunk_supported(const RecurArgs& a) {
  const bool per_token = a.mode == 2 && a.g_head && a.log_g;  // one decay per head and token
  if ((a.mode != 0 && !per_token) || !a.ws || a.L < 2 * CH) return false;
  if (!recur_chunk_shape(a.DK, a.DV)) return false;
  if (a.ld_q % 4 || a.ld_k % 4 || a.ld_v % 4 || (a.H * a.DV) % 4) return false;
  if (!aligned16(a.q) || !aligned16(a.k) || !aligned16(a.v) || !aligned16(a.out) || !aligned16(a.ws) || !aligned16(a.state)) return false;
  return recur_chunk_ws_floats(a.B, a.L, a.H, a.DK, a.DV) <= a.ws_floats;
}

cudaError_t launch_recur_chunk(const RecurArgs& a, cudaStream_t s) {
  if (!recur_chunk_supported(a)) return cudaErrorInvalidValue;
  const int NC = (a.L + CH - 1) / CH;
  const dim3 grid(NC, a.H, a.B);
  const size_t sm1 = (size_t)(CH + 4 + CH + CH * a.DK + CH * a.DV) * sizeof(float);
  const size_t sm3 = (size_t)(CH + 4 + 2 * a.DK * LDT + CH * LDT + CH * 64) * sizeof(float);
  const int n4 = (a.DK * a.DV + (a.n_state ? a.DK : 0)) / 4;
  auto go = [&](auto k_state, auto k_scan, auto k_out) {
    cudaError_t e;
    if ((e = cudaFuncSetAttribute(k_state, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1)) != cudaSuccess) return e;
    if ((e = cudaFuncSetAttribute(k_out, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm3)) != cudaSuccess) return e;
    if ((e = launch_k(k_state, grid, dim3(256), sm1, s, a, NC)) != cudaSuccess) return e;
    if ((e = launch_k(k_scan, dim3((n4 + 255) / 256, a.H, a.B), dim3(256), 0, s, a, NC)) != cudaSuccess) return e;
    return launch_k(k_out, grid, dim3(256), sm3, s, a, NC);
  };
  if (a.n_state && a.bf16_ops) {
    const size_t sb1 = ((size_t)2 * CH * (a.DK + 8) + CH * LDE) * 2, sb3 = ((size_t)2 * CH * (a.DK + 8) + 3 * CH * LDE + 2 * (size_t)a.DK * LDE) * 2;
    const int ctas = NC * a.H * a.B, tiles = a.DV / 64;
    const int ne1 = value_splits(ctas, tiles, 100), ne3 = value_splits(ctas, tiles, 100);  // measured: only short prompts of few heads gain
    auto go_mma = [&](auto k_state, auto k_out) {
      cudaError_t e;
      if ((e = cudaFuncSetAttribute(k_state, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sb1)) != cudaSuccess) return e;
      if ((e = cudaFuncSetAttribute(k_out, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sb3)) != cudaSuccess) return e;
      if ((e = launch_k(k_state, dim3(NC * ne1, a.H, a.B), dim3(256), sb1, s, a, NC, ne1)) != cudaSuccess) return e;
      if ((e = launch_k(lin_chunk_scan_kernel<true, true>, dim3((n4 + 255) / 256, a.H, a.B), dim3(256), 0, s, a, NC)) != cudaSuccess) return e;
      return launch_k(k_out, dim3(NC * ne3, a.H, a.B), dim3(256), sb3, s, a, NC, ne3);
    };
    switch (a.DK) {
      case 64: return go_mma(lin_chunk_state_mma_kernel<64>, lin_chunk_out_mma_kernel<64>);
      case 128: return go_mma(lin_chunk_state_mma_kernel<128>, lin_chunk_out_mma_kernel<128>);
      case 192: return go_mma(lin_chunk_state_mma_kernel<192>, lin_chunk_out_mma_kernel<192>);
      default: return go_mma(lin_chunk_state_mma_kernel<256>, lin_chunk_out_mma_kernel<256>);
    }
  }
  if (a.n_state) return go(lin_chunk_state_kernel<true, true>, lin_chunk_scan_kernel<true, true>, lin_chunk_out_kernel<true, true>);
  if (a.mode == 2) return go(lin_chunk_state_kernel<true, false>, lin_chunk_scan_kernel<true, false>, lin_chunk_out_kernel<true, false>);
  return go(lin_chunk_state_kernel<false, false>, lin_chunk_scan_kernel<false, false>, lin_chunk_out_kernel<false, false>);
}
