// Attention over a sliding window or inside chunks of the sequence, which may keep the first tokens (L3_MIX_WINDOW): GQA
// with key size DK and value size DV, the weight of a visible key either a softmax term - plain, or with a per-head sink
// in the denominator - or sigmoid(score + per-head bias) without any normalisation over keys; an optional sigmoid gate per
// head on the output.  Everything fp32 (FFMA): scores, weights, accumulation.
//
//  * win_prep_kernel     a warp per head vector of a token: biases, optional RMS norm per head with a weight, rotary turn
//                        of the leading rot_dims entries at the token's position (pairs (2i, 2i + 1) or (i, i + rot_dims / 2); angle = position * frequency in fp32,
//                        sincosf), optional division by the turned vector's root mean square, q to the query buffer, k and
//                        the value row to the caches
//  * win_attn_kernel     a CTA holds 32 query rows of ONE key head - row = (token, query head of the group), token-major,
//                        so the heads of a group share every key / value tile - and walks the keys the tile can see, 64 at
//                        a time: first the kept tokens that lie ahead of the window, then the window.  A
//                        warp owns 4 rows; in the score phase a lane holds two keys (16-byte shared loads, key rows padded by
//                        4 floats), in the output phase a lane owns value columns read as 16-byte pieces while the weights
//                        arrive as 16-byte broadcasts.  Softmax rows run the online form,
//                        started at (max = sink, sum = 1) so that the sink needs no key; sigmoid rows just accumulate.
//                        Calls of few tokens split the key tiles over CTAs (win_attn_combine_kernel merges).
//  * win_decode_kernel   one token per sequence, groups of 1, 2, 4 or 8 query heads: a CTA per (key split, key head, sequence).
//                        Four threads per key score it for all heads of the group, a warp per head turns the scores into
//                        weights, and the values - requested together with the keys - are summed by (16-byte column piece,
//                        key part) threads.  Other sizes run win_attn_kernel.
#include <stdlib.h>

#include <algorithm>

#include "common.cuh"
#include "mixer.h"
#include "../../include/llama3_b200.h"

namespace {

constexpr int WA_SPLIT_MAX = 32;
constexpr int WA_ROWS = 32, WA_KEYS = 64, WA_WARPS = 8, WA_QW = WA_ROWS / WA_WARPS;

// four consecutive values to a row of floats / bf16
__device__ __forceinline__ void put4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void put4(bf16* p, float a, float b, float c, float d) {
  union { __nv_bfloat162 h[2]; uint2 u; } o;
  o.h[0] = __floats2bfloat162_rn(a, b);
  o.h[1] = __floats2bfloat162_rn(c, d);
  *reinterpret_cast<uint2*>(p) = o.u;
}

// grid (rows, y): the row's H + G head vectors and G value rows over the CTA's warps and over y CTAs
template <typename KVT>
__global__ void __launch_bounds__(256) win_prep_kernel(WinPrepArgs a) {
  extern __shared__ __align__(16) float sm[];  // [warps][DK padded to 4] | cosines and sines of the row's angles [rot_dims / 2] each
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x;
  const int b = r / a.L, t = r - b * a.L;
  const int pos = *a.pos_ptr + t;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const float* row = a.proj + (size_t)r * a.ld;
  const int DKP = (a.DK + 3) & ~3, half = a.rot_dims / 2;
  float* buf = sm + (size_t)warp * DKP;
  float* cs = sm + (size_t)nw * DKP;
  float* sn = cs + half;
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &sn[i], &cs[i]);  // once per CTA, its heads read them
  __syncthreads();
  for (int v = blockIdx.y * nw + warp; v < a.H + 2 * a.G; v += gridDim.y * nw) {
    const bool is_q = v < a.H, is_v = v >= a.H + a.G;
    const int g = is_q ? 0 : is_v ? v - a.H - a.G : v - a.H;  // key head
    const int n = is_v ? a.DV : a.DK;
    const size_t col = is_q ? a.q_off + (size_t)v * a.DK : is_v ? a.v_off + (size_t)g * a.DV : a.k_off + (size_t)g * a.DK;
    const float* src = row + col;
    const float* bias = a.bias ? a.bias + col : nullptr;
    const bool vec = n % 4 == 0 && col % 4 == 0 && a.ld % 4 == 0;
    if (is_v) {
      KVT* dst = (KVT*)a.cache_v + (((size_t)b * a.G + g) * a.M + pos) * a.DV;
      if (vec) {
        for (int i = lane * 4; i < n; i += 128) {
          float4 x = *reinterpret_cast<const float4*>(src + i);
          if (bias) { const float4 c = *reinterpret_cast<const float4*>(bias + i); x.x += c.x; x.y += c.y; x.z += c.z; x.w += c.w; }
          put4(dst + i, x.x, x.y, x.z, x.w);
        }
      } else
        for (int i = lane; i < n; i += 32) dst[i] = from_f32<KVT>(src[i] + (bias ? bias[i] : 0.f));
      continue;
    }
    float ss = 0.f;
    if (vec) {
      for (int i = lane * 4; i < n; i += 128) {
        float4 x = *reinterpret_cast<const float4*>(src + i);
        if (bias) { const float4 c = *reinterpret_cast<const float4*>(bias + i); x.x += c.x; x.y += c.y; x.z += c.z; x.w += c.w; }
        ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
        *reinterpret_cast<float4*>(buf + i) = x;
      }
    } else {
      for (int i = lane; i < n; i += 32) { const float x = src[i] + (bias ? bias[i] : 0.f); ss = fmaf(x, x, ss); buf[i] = x; }
    }
    const float* w = is_q ? a.wq : a.wk;
    // a rotation changes no length: the root mean square is the same ahead of it and behind it
    const float rinv = w || a.unit_norm ? 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps) : 1.0f;
    __syncwarp();
    auto in = [&](int i) { return w ? buf[i] * rinv * w[i] : buf[i] * rinv; };
    auto out = [&](int i) {
      const float x = in(i);
      if (i >= a.rot_dims) return x;
      const bool second = a.rot_layout ? i >= half : i & 1;
      const int p = a.rot_layout ? (second ? i - half : i) : i >> 1;
      const float y = in(a.rot_layout ? (second ? i - half : i + half) : i ^ 1);
      return second ? x * cs[p] + y * sn[p] : x * cs[p] - y * sn[p];
    };
    KVT* ck = (KVT*)a.cache_k + (((size_t)b * a.G + g) * a.M + pos) * a.DK;
    float* qf = a.q_out ? a.q_out + ((size_t)r * a.H + v) * a.DK : nullptr;
    bf16* qp = a.q16 ? a.q16 + ((size_t)r * a.H + v) * a.q16_ld : nullptr;
    if (n % 4 == 0 && a.rot_layout == 1 && half % 4 == 0) {  // a group of four turns with the group half a rotation away
      for (int i = lane * 4; i < n; i += 128) {
        auto in4 = [&](int c) {
          float4 x = *reinterpret_cast<const float4*>(buf + c);
          x.x *= rinv; x.y *= rinv; x.z *= rinv; x.w *= rinv;
          if (w) { const float4 k = *reinterpret_cast<const float4*>(w + c); x.x *= k.x; x.y *= k.y; x.z *= k.z; x.w *= k.w; }
          return x;
        };
        float4 x = in4(i);
        if (i < a.rot_dims) {
          const bool second = i >= half;
          const int p = second ? i - half : i;
          const float4 y = in4(second ? i - half : i + half);
          const float4 c = *reinterpret_cast<const float4*>(cs + p);
          float4 n4 = *reinterpret_cast<const float4*>(sn + p);
          if (!second) { n4.x = -n4.x; n4.y = -n4.y; n4.z = -n4.z; n4.w = -n4.w; }
          x.x = x.x * c.x + y.x * n4.x; x.y = x.y * c.y + y.y * n4.y; x.z = x.z * c.z + y.z * n4.z; x.w = x.w * c.w + y.w * n4.w;
        }
        if (!is_q) put4(ck + i, x.x, x.y, x.z, x.w);
        else {
          if (qf) put4(qf + i, x.x, x.y, x.z, x.w);
          if (qp) put4(qp + i, x.x, x.y, x.z, x.w);
        }
      }
    } else if (n % 4 == 0) {
      for (int i = lane * 4; i < n; i += 128) {
        const float x0 = out(i), x1 = out(i + 1), x2 = out(i + 2), x3 = out(i + 3);
        if (!is_q) put4(ck + i, x0, x1, x2, x3);
        else {
          if (qf) put4(qf + i, x0, x1, x2, x3);
          if (qp) put4(qp + i, x0, x1, x2, x3);
        }
      }
    } else {
      for (int i = lane; i < n; i += 32) {
        const float x = out(i);
        if (!is_q) ck[i] = from_f32<KVT>(x);
        else {
          if (qf) qf[i] = x;
          if (qp) qp[i] = __float2bfloat16_rn(x);
        }
      }
    }
    if (is_q && qp)
      for (int i = n + lane; i < a.q16_ld; i += 32) qp[i] = __float2bfloat16_rn(0.f);
    __syncwarp();
  }
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// One row of a key / value tile from the cache into shared memory as floats: `n` values (dst padded with zeros up to np).
// 16-byte global loads where the row length allows them.
template <typename KVT>
__device__ __forceinline__ void stage_row(const KVT* __restrict__ src, int n, int np, float* __restrict__ dst, int part, int nparts) {
  constexpr int VEC = 16 / (int)sizeof(KVT);
  if (src && n % VEC == 0) {
    for (int c = part; c < n / VEC; c += nparts) {
      float v[VEC];
      Vec16<KVT>::load(src + c * VEC, v);
#pragma unroll
      for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(dst + c * VEC + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
    for (int i = n + part; i < np; i += nparts) dst[i] = 0.f;
  } else {
    for (int i = part; i < np; i += nparts) dst[i] = (src && i < n) ? to_f32(src[i]) : 0.f;
  }
}

// value column j (< NJ) of a lane: lanes read 16-byte (8-byte, 4-byte) pieces that tile a row without bank conflicts
template <int NJ>
__device__ __forceinline__ int win_col(int lane, int j) {
  return NJ == 1 ? lane : NJ == 2 ? 2 * lane + j : (j >> 2) * 128 + 4 * lane + (j & 3);
}

// NJ: value columns per lane (DV <= 32 NJ)
template <typename KVT, int NJ>
__global__ void __launch_bounds__(256) win_attn_kernel(WinAttnArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int DKP = (a.DK + 3) & ~3, KS = DKP + 4, DVP = 32 * NJ;
  float* sQ = sm;                                  // [32][DKP]
  float* sK = sQ + (size_t)WA_ROWS * DKP;          // [64][DKP + 4]
  float* sV = sK + (size_t)WA_KEYS * KS;           // [64][DVP]
  float* sP = sV + (size_t)WA_KEYS * DVP;          // [warps][QW][64]
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rep = a.H / a.G;
  const int g = blockIdx.y;
  const int b = blockIdx.z / a.nsplit, split = blockIdx.z - b * a.nsplit;
  const int nrows = a.L * rep;                     // rows of this (sequence, key head): row = t * rep + head in group
  const int row0 = (gridDim.x - 1 - blockIdx.x) * WA_ROWS;  // late tokens see the most keys: their tiles start first
  const int pos0 = *a.pos_ptr;
  const int t_lo = row0 / rep, t_hi = min(a.L - 1, (row0 + WA_ROWS - 1) / rep);
  const int p_lo = pos0 + t_lo, p_hi = pos0 + t_hi;
  // keys the tile can see: [0, ka) kept tokens ahead of the window, then [w_lo, p_hi]
  auto first_key = [&](int p) { return a.window <= 0 ? 0 : a.chunked ? p - p % a.window : max(0, p - a.window + 1); };
  const int w_lo = first_key(p_lo);
  const int ka = min(a.keep_first, w_lo);
  const int nkeys = ka + (p_hi + 1 - w_lo);
  const int ntiles = (nkeys + WA_KEYS - 1) / WA_KEYS;
  const int per = (ntiles + a.nsplit - 1) / a.nsplit;
  const int tile_lo = split * per, tile_hi = min(ntiles, tile_lo + per);

  // queries: 8 threads per row
  for (int rr = tid >> 3; rr < WA_ROWS; rr += 32) {
    const int row = row0 + rr;
    const float* src = nullptr;
    if (row < nrows) {
      const int t = row / rep, h = g * rep + (row - t * rep);
      src = a.q + (((size_t)b * a.L + t) * a.H + h) * a.DK;
    }
    stage_row<float>(src, a.DK, DKP, sQ + (size_t)rr * DKP, tid & 7, 8);
  }
  // per-row state: rows warp, warp + 8, warp + 16, warp + 24 of the tile
  float o[WA_QW][NJ], mx[WA_QW], sum[WA_QW], hv[WA_QW];
  int rpos[WA_QW], rlo[WA_QW];  // a row's position and the first key of its window / chunk
#pragma unroll
  for (int qi = 0; qi < WA_QW; ++qi) {
    const int row = row0 + warp + qi * WA_WARPS;
    const bool live = row < nrows;
    const int t = live ? row / rep : 0, h = g * rep + (live ? row - t * rep : 0);
    rpos[qi] = live ? pos0 + t : -1;
    rlo[qi] = live ? first_key(pos0 + t) : 0;
    hv[qi] = a.head_vec ? a.head_vec[h] : 0.f;
    const bool sink_here = a.kind == L3_ATTN_SINK && a.head_vec && split == 0;
    mx[qi] = sink_here ? hv[qi] : -INFINITY;
    sum[qi] = sink_here ? 1.f : 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) o[qi][j] = 0.f;
  }
  const KVT* ck = (const KVT*)a.cache_k + ((size_t)b * a.G + g) * a.M * a.DK;
  const KVT* cv = (const KVT*)a.cache_v + ((size_t)b * a.G + g) * a.M * a.DV;
  float* myP = sP + (size_t)warp * WA_QW * WA_KEYS;

  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    __syncthreads();  // the previous tile has been used (and sQ is complete)
    const int v0 = tile * WA_KEYS;
    for (int kk = tid >> 3; kk < WA_KEYS; kk += 32) {  // 8 threads per key / value row
      const int vi = v0 + kk;
      const int j = vi < nkeys ? (vi < ka ? vi : w_lo + (vi - ka)) : -1;
      stage_row<KVT>(j >= 0 ? ck + (size_t)j * a.DK : nullptr, a.DK, DKP, sK + (size_t)kk * KS, tid & 7, 8);
      stage_row<KVT>(j >= 0 ? cv + (size_t)j * a.DV : nullptr, a.DV, DVP, sV + (size_t)kk * DVP, tid & 7, 8);
    }
    __syncthreads();
    // scores: a lane holds keys lane and lane + 32 of the tile
    int kj[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int vi = v0 + lane + 32 * u;
      kj[u] = vi < nkeys ? (vi < ka ? vi : w_lo + (vi - ka)) : -1;
    }
    float sc[WA_QW][2];
#pragma unroll
    for (int qi = 0; qi < WA_QW; ++qi) sc[qi][0] = sc[qi][1] = 0.f;
    const float4* kA = reinterpret_cast<const float4*>(sK + (size_t)lane * KS);
    const float4* kB = reinterpret_cast<const float4*>(sK + (size_t)(lane + 32) * KS);
#pragma unroll 2
    for (int d4 = 0; d4 < DKP / 4; ++d4) {
      const float4 ka4 = kA[d4], kb4 = kB[d4];
#pragma unroll
      for (int qi = 0; qi < WA_QW; ++qi) {
        const float4 qv = reinterpret_cast<const float4*>(sQ + (size_t)(warp + qi * WA_WARPS) * DKP)[d4];
        sc[qi][0] = fmaf(qv.x, ka4.x, sc[qi][0]); sc[qi][1] = fmaf(qv.x, kb4.x, sc[qi][1]);
        sc[qi][0] = fmaf(qv.y, ka4.y, sc[qi][0]); sc[qi][1] = fmaf(qv.y, kb4.y, sc[qi][1]);
        sc[qi][0] = fmaf(qv.z, ka4.z, sc[qi][0]); sc[qi][1] = fmaf(qv.z, kb4.z, sc[qi][1]);
        sc[qi][0] = fmaf(qv.w, ka4.w, sc[qi][0]); sc[qi][1] = fmaf(qv.w, kb4.w, sc[qi][1]);
      }
    }
#pragma unroll
    for (int qi = 0; qi < WA_QW; ++qi) {
      const int p = rpos[qi];
      bool vis[2];
      float s2[2], w[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        vis[u] = kj[u] >= 0 && kj[u] <= p && (kj[u] >= rlo[qi] || kj[u] < a.keep_first);
        s2[u] = sc[qi][u] * a.scale;
      }
      if (a.kind == L3_ATTN_SIGMOID) {
        w[0] = vis[0] ? sigmoid_f(s2[0] + hv[qi]) : 0.f;
        w[1] = vis[1] ? sigmoid_f(s2[1] + hv[qi]) : 0.f;
      } else {
        const float mnew = fmaxf(mx[qi], warp_max(fmaxf(vis[0] ? s2[0] : -INFINITY, vis[1] ? s2[1] : -INFINITY)));
        const float alpha = mnew == -INFINITY ? 1.f : expf(mx[qi] - mnew);
        w[0] = vis[0] ? expf(s2[0] - mnew) : 0.f;
        w[1] = vis[1] ? expf(s2[1] - mnew) : 0.f;
        sum[qi] = sum[qi] * alpha + warp_sum(w[0] + w[1]);
        mx[qi] = mnew;
#pragma unroll
        for (int j = 0; j < NJ; ++j) o[qi][j] *= alpha;
      }
      myP[qi * WA_KEYS + lane] = w[0];
      myP[qi * WA_KEYS + lane + 32] = w[1];
    }
    __syncwarp();
    // outputs: a lane owns NJ value columns (win_col), read as 16-byte pieces
    for (int k0 = 0; k0 < WA_KEYS; k0 += 4) {
      float4 pw[WA_QW];
#pragma unroll
      for (int qi = 0; qi < WA_QW; ++qi) pw[qi] = *reinterpret_cast<const float4*>(myP + qi * WA_KEYS + k0);
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        float vv[NJ];
        const float* vr = sV + (size_t)(k0 + kk) * DVP;
        if (NJ == 1) vv[0] = vr[lane];
        else if (NJ == 2) { const float2 t2 = *reinterpret_cast<const float2*>(vr + 2 * lane); vv[0] = t2.x; vv[1] = t2.y; }
        else {
#pragma unroll
          for (int c = 0; c < NJ / 4; ++c) {
            const float4 t4 = *reinterpret_cast<const float4*>(vr + c * 128 + 4 * lane);
            vv[4 * c] = t4.x; vv[4 * c + 1] = t4.y; vv[4 * c + 2] = t4.z; vv[4 * c + 3] = t4.w;
          }
        }
#pragma unroll
        for (int qi = 0; qi < WA_QW; ++qi) {
          const float pk = kk == 0 ? pw[qi].x : kk == 1 ? pw[qi].y : kk == 2 ? pw[qi].z : pw[qi].w;
#pragma unroll
          for (int j = 0; j < NJ; ++j) o[qi][j] = fmaf(pk, vv[j], o[qi][j]);
        }
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int qi = 0; qi < WA_QW; ++qi) {
    const int row = row0 + warp + qi * WA_WARPS;
    if (row >= nrows) continue;
    const int t = row / rep, h = g * rep + (row - t * rep);
    const size_t r = (size_t)b * a.L + t;
    if (a.nsplit > 1) {  // partial (o, max, sum) of this split
      const size_t pi = (r * a.H + h) * a.nsplit + split;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int d = win_col<NJ>(lane, j);
        if (d < a.DV) a.part_o[pi * a.DV + d] = o[qi][j];
      }
      if (lane == 0) { a.part_ml[pi * 2] = mx[qi]; a.part_ml[pi * 2 + 1] = sum[qi]; }
      continue;
    }
    float mul = a.out_scale * (a.kind == L3_ATTN_SIGMOID ? 1.f : (sum[qi] > 0.f ? 1.0f / sum[qi] : 0.f));
    if (a.gate) mul *= sigmoid_f(a.gate[r * a.ld_gate + h]);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int d = win_col<NJ>(lane, j);
      if (d < a.DV) {
        const float v = o[qi][j] * mul;
        const size_t oi = r * a.ld_out + (size_t)h * a.DV + d;
        if (a.out) a.out[oi] = v;
        if (a.out16) a.out16[oi] = __float2bfloat16_rn(v);
      }
    }
  }
}

constexpr int WD_KEYS = 64, WD_KV = 8, WD_VV = 8;  // keys per tile; 16-byte pieces of a key / keys of a value part per thread

template <typename KVT, int REP>
__global__ void __launch_bounds__(256) win_decode_kernel(WinAttnArgs a) {
  constexpr int VEC = Vec16<KVT>::N;
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;                          // [REP][DK]
  float* sS = sQ + (size_t)REP * a.DK;     // [REP][WD_KEYS] scores, then weights
  float* sA = sS + REP * WD_KEYS;          // [REP] rescaling of the sums so far
  float* sM = sA + REP;                    // [REP] maximum | [REP] sum, at the end
  float* sR = sM + 2 * REP + (4 - 3 * REP % 4) % 4;  // [parts][REP][DV]
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = blockIdx.y, b = blockIdx.z, split = blockIdx.x;
  const int p = *a.pos_ptr;                // the token's position; L == 1
  const int lo = a.window <= 0 ? 0 : a.chunked ? p - p % a.window : max(0, p - a.window + 1);
  const int ka = min(a.keep_first, lo), nkeys = ka + p + 1 - lo;
  const int per = ((nkeys + a.nsplit - 1) / a.nsplit + 7) & ~7;
  const int k_lo = min(nkeys, split * per), k_hi = min(nkeys, k_lo + per);
  const KVT* ck = (const KVT*)a.cache_k + ((size_t)b * a.G + g) * a.M * a.DK;
  const KVT* cv = (const KVT*)a.cache_v + ((size_t)b * a.G + g) * a.M * a.DV;
  auto key_of = [&](int vi) { return vi < ka ? vi : lo + (vi - ka); };
  const float* qrow = a.q + ((size_t)b * a.H + (size_t)g * REP) * a.DK;
  for (int i = tid; i < REP * a.DK; i += 256) sQ[i] = qrow[i];
  const int nkv = a.DK / VEC, nvv = a.DV / VEC, parts = 256 / nvv;  // pieces of a key, of a value; key parts of the output phase
  const int kk = tid >> 2, kp = tid & 3;                            // score phase: key, quarter of its pieces
  const int vc = tid % nvv, vp = tid / nvv;                         // output phase: column piece, key part
  float m_run = -INFINITY, l_run = 0.f, hv = 0.f;
  if (warp < REP) {  // warp r keeps head r's maximum and sum
    hv = a.head_vec ? a.head_vec[g * REP + warp] : 0.f;
    if (a.kind == L3_ATTN_SINK && a.head_vec && split == 0) { m_run = hv; l_run = 1.f; }
  }
  float acc[REP][VEC];
#pragma unroll
  for (int r = 0; r < REP; ++r)
#pragma unroll
    for (int x = 0; x < VEC; ++x) acc[r][x] = 0.f;

  for (int t0 = k_lo; t0 < k_hi; t0 += WD_KEYS) {
    uint4 kreg[WD_KV], vreg[WD_VV];
    const bool k_ok = t0 + kk < k_hi;
    const KVT* krow = ck + (size_t)key_of(k_ok ? t0 + kk : t0) * a.DK;
#pragma unroll
    for (int i = 0; i < WD_KV; ++i)
      if (kp + 4 * i < nkv) kreg[i] = ldg_stream16(krow + (size_t)(kp + 4 * i) * VEC);
#pragma unroll
    for (int i = 0; i < WD_VV; ++i) {
      const int vi = t0 + vp + i * parts;
      if (vp + i * parts < WD_KEYS && vi < k_hi) vreg[i] = ldg_stream16(cv + (size_t)key_of(vi) * a.DV + (size_t)vc * VEC);
    }
    __syncthreads();  // sQ stands; the previous tile's weights have been used
    float sc[REP];
#pragma unroll
    for (int r = 0; r < REP; ++r) sc[r] = 0.f;
#pragma unroll
    for (int i = 0; i < WD_KV; ++i)
      if (kp + 4 * i < nkv) {
        float f[VEC];
        Vec16<KVT>::unpack(kreg[i], f);
#pragma unroll
        for (int r = 0; r < REP; ++r) {
          const float* q = sQ + (size_t)r * a.DK + (kp + 4 * i) * VEC;
#pragma unroll
          for (int x = 0; x < VEC; x += 4) {
            const float4 q4 = *reinterpret_cast<const float4*>(q + x);
            sc[r] = fmaf(f[x], q4.x, sc[r]); sc[r] = fmaf(f[x + 1], q4.y, sc[r]);
            sc[r] = fmaf(f[x + 2], q4.z, sc[r]); sc[r] = fmaf(f[x + 3], q4.w, sc[r]);
          }
        }
      }
#pragma unroll
    for (int r = 0; r < REP; ++r) {
      float s = sc[r];
      s += __shfl_xor_sync(L3_FULL, s, 1);
      s += __shfl_xor_sync(L3_FULL, s, 2);
      if (kp == 0) sS[r * WD_KEYS + kk] = k_ok ? s * a.scale : -INFINITY;
    }
    __syncthreads();
    if (warp < REP) {
      float* s = sS + warp * WD_KEYS;
      const float s0 = s[lane], s1 = s[lane + 32];
      float w0, w1, alpha = 1.f;
      if (a.kind == L3_ATTN_SIGMOID) {
        w0 = s0 == -INFINITY ? 0.f : sigmoid_f(s0 + hv);
        w1 = s1 == -INFINITY ? 0.f : sigmoid_f(s1 + hv);
      } else {
        const float mnew = fmaxf(m_run, warp_max(fmaxf(s0, s1)));  // a tile holds a key: finite
        alpha = expf(m_run - mnew);
        w0 = expf(s0 - mnew);
        w1 = expf(s1 - mnew);
        l_run = l_run * alpha + warp_sum(w0 + w1);
        m_run = mnew;
      }
      s[lane] = w0;
      s[lane + 32] = w1;
      if (lane == 0) sA[warp] = alpha;
    }
    __syncthreads();
    if (t0 > k_lo) {
#pragma unroll
      for (int r = 0; r < REP; ++r)
#pragma unroll
        for (int x = 0; x < VEC; ++x) acc[r][x] *= sA[r];
    }
#pragma unroll
    for (int i = 0; i < WD_VV; ++i) {
      const int vk = vp + i * parts;
      if (vk < WD_KEYS && t0 + vk < k_hi) {
        float f[VEC];
        Vec16<KVT>::unpack(vreg[i], f);
#pragma unroll
        for (int r = 0; r < REP; ++r) {
          const float w = sS[r * WD_KEYS + vk];
#pragma unroll
          for (int x = 0; x < VEC; ++x) acc[r][x] = fmaf(w, f[x], acc[r][x]);
        }
      }
    }
  }
  if (warp < REP && lane == 0) { sM[warp] = m_run; sM[REP + warp] = l_run; }
#pragma unroll
  for (int r = 0; r < REP; ++r)
#pragma unroll
    for (int x = 0; x < VEC; x += 4)
      *reinterpret_cast<float4*>(sR + ((size_t)vp * REP + r) * a.DV + vc * VEC + x) = make_float4(acc[r][x], acc[r][x + 1], acc[r][x + 2], acc[r][x + 3]);
  __syncthreads();
  for (int i = tid; i < REP * a.DV; i += 256) {
    const int r = i / a.DV, d = i - r * a.DV, h = g * REP + r;
    float t = 0.f;
#pragma unroll 8
    for (int q = 0; q < parts; ++q) t += sR[((size_t)q * REP + r) * a.DV + d];
    const size_t rh = (size_t)b * a.H + h;
    if (a.nsplit > 1) {
      const size_t pi = rh * a.nsplit + split;
      a.part_o[pi * a.DV + d] = t;
      if (d == 0) { a.part_ml[pi * 2] = sM[r]; a.part_ml[pi * 2 + 1] = sM[REP + r]; }
      continue;
    }
    float mul = a.out_scale * (a.kind == L3_ATTN_SIGMOID ? 1.f : (sM[REP + r] > 0.f ? 1.0f / sM[REP + r] : 0.f));
    if (a.gate) mul *= sigmoid_f(a.gate[(size_t)b * a.ld_gate + h]);
    const size_t oi = (size_t)b * a.ld_out + (size_t)h * a.DV + d;
    if (a.out) a.out[oi] = t * mul;
    if (a.out16) a.out16[oi] = __float2bfloat16_rn(t * mul);
  }
}

// a CTA per (row, head): the splits' weights once, then a thread per value column
__global__ void __launch_bounds__(128) win_attn_combine_kernel(WinAttnArgs a) {
  __shared__ float s_f[WA_SPLIT_MAX];
  __shared__ float s_den;
  pdl_launch();
  pdl_wait();
  const size_t rh = blockIdx.x, r = rh / a.H;
  const int h = (int)(rh - r * a.H), lane = threadIdx.x & 31;
  if (threadIdx.x < 32) {  // nsplit <= 32: a lane per split
    const bool on = lane < a.nsplit;
    const float m = on ? a.part_ml[(rh * a.nsplit + lane) * 2] : -INFINITY, l = on ? a.part_ml[(rh * a.nsplit + lane) * 2 + 1] : 0.f;
    float f = 1.f, den = 1.f;
    if (a.kind != L3_ATTN_SIGMOID) {
      const float M = warp_max(m);
      f = m == -INFINITY ? 0.f : expf(m - M);
      den = warp_sum(f * l);
    }
    if (on) s_f[lane] = f;
    if (lane == 0) s_den = den;
  }
  __syncthreads();
  float mul = a.out_scale * (s_den > 0.f ? 1.0f / s_den : 0.f);
  if (a.gate) mul *= sigmoid_f(a.gate[r * a.ld_gate + h]);
  const float* po = a.part_o + rh * a.nsplit * a.DV;
  for (int d = threadIdx.x; d < a.DV; d += blockDim.x) {
    float acc = 0.f;
#pragma unroll 8
    for (int s = 0; s < a.nsplit; ++s) acc = fmaf(po[(size_t)s * a.DV + d], s_f[s], acc);
    const float v = acc * mul;
    const size_t oi = r * a.ld_out + (size_t)h * a.DV + d;
    if (a.out) a.out[oi] = v;
    if (a.out16) a.out16[oi] = __float2bfloat16_rn(v);
  }
}

size_t win_attn_smem(int DK, int NJ) {
  const int DKP = (DK + 3) & ~3;
  return ((size_t)WA_ROWS * DKP + (size_t)WA_KEYS * (DKP + 4) + (size_t)WA_KEYS * 32 * NJ + (size_t)WA_WARPS * WA_QW * WA_KEYS) * sizeof(float);
}

int win_nj(int DV) { return DV <= 32 ? 1 : DV <= 64 ? 2 : DV <= 128 ? 4 : DV <= 256 ? 8 : 16; }

template <typename KVT, int NJ>
cudaError_t launch_win_nj(const WinAttnArgs& a, dim3 grid, cudaStream_t s) {
  const size_t smem = win_attn_smem(a.DK, NJ);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(win_attn_kernel<KVT, NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_k(win_attn_kernel<KVT, NJ>, grid, dim3(256), smem, s, a);
}

// decode sizes: whole 16-byte pieces, a tile's keys and values in registers
template <typename KVT>
bool win_decode_supported(const WinAttnArgs& a) {
  constexpr int VEC = Vec16<KVT>::N;
  const int rep = a.H / a.G, nvv = a.DV / VEC;
  return a.L == 1 && (rep == 1 || rep == 2 || rep == 4 || rep == 8) && a.DK % VEC == 0 && a.DV % VEC == 0 && a.DK <= 4 * WD_KV * VEC &&
         256 % nvv == 0 && WD_KEYS * nvv <= 256 * WD_VV;
}

template <typename KVT, int REP>
cudaError_t launch_win_decode(const WinAttnArgs& a, cudaStream_t s) {
  const int parts = 256 / (a.DV / Vec16<KVT>::N);
  const size_t smem = ((size_t)REP * a.DK + REP * WD_KEYS + 3 * REP + 4 + (size_t)parts * REP * a.DV) * sizeof(float);
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(win_decode_kernel<KVT, REP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_k(win_decode_kernel<KVT, REP>, dim3(a.nsplit, a.G, a.B), dim3(256), smem, s, a);
}

template <typename KVT>
cudaError_t launch_win_t(const WinAttnArgs& a, dim3 grid, cudaStream_t s) {
  static const bool decode_on = !(getenv("L3_WINDOW_DECODE") && atoi(getenv("L3_WINDOW_DECODE")) == 0);
  if (decode_on && win_decode_supported<KVT>(a)) {
    switch (a.H / a.G) {
      case 1: return launch_win_decode<KVT, 1>(a, s);
      case 2: return launch_win_decode<KVT, 2>(a, s);
      case 4: return launch_win_decode<KVT, 4>(a, s);
      default: return launch_win_decode<KVT, 8>(a, s);
    }
  }
  switch (win_nj(a.DV)) {
    case 1: return launch_win_nj<KVT, 1>(a, grid, s);
    case 2: return launch_win_nj<KVT, 2>(a, grid, s);
    case 4: return launch_win_nj<KVT, 4>(a, grid, s);
    case 8: return launch_win_nj<KVT, 8>(a, grid, s);
    default: return launch_win_nj<KVT, 16>(a, grid, s);
  }
}

}  // namespace

bool win_attn_supported(int DK, int DV) {
  return DK >= 1 && DV >= 1 && DV <= 512 && win_attn_smem(DK, win_nj(DV)) <= 220 * 1024;
}

int win_attn_splits(int B, int L, int H, int G, int window, int keep_first, int max_keys, int max_split) {
  if (L > 8) return 1;
  const int rep = H / G;
  const int ctas = B * G * ((L * rep + WA_ROWS - 1) / WA_ROWS);
  int keys = max_keys;
  if (window > 0) keys = std::min(keys, window + L + keep_first);
  const int tiles = (keys + WA_KEYS - 1) / WA_KEYS;
  // a key tile or more per split, aimed at two CTAs per SM
  return std::max(1, std::min(std::min(max_split, tiles), (2 * 148) / std::max(1, ctas)));
}

size_t win_attn_part_floats(int max_rows, int H, int DV, int max_split) { return (size_t)max_rows * H * max_split * DV; }

cudaError_t launch_win_prep(const WinPrepArgs& a, int rows, bool kv_bf16, cudaStream_t s) {
  if (a.unit_norm && (a.wq || a.wk)) return cudaErrorInvalidValue;
  const int items = a.H + 2 * a.G;
  const int warps = std::min(8, items);
  const size_t smem = ((size_t)warps * ((a.DK + 3) & ~3) + a.rot_dims) * sizeof(float);
  const dim3 grid(rows, rows <= 64 ? (items + warps - 1) / warps : 1);  // few rows: their head vectors over CTAs, too
  if (kv_bf16) return launch_k(win_prep_kernel<bf16>, grid, dim3(32 * warps), smem, s, a);
  return launch_k(win_prep_kernel<float>, grid, dim3(32 * warps), smem, s, a);
}

cudaError_t launch_win_attn(const WinAttnArgs& a, bool kv_bf16, cudaStream_t s) {
  if (!win_attn_supported(a.DK, a.DV) || a.H % a.G != 0 || a.nsplit < 1 || a.nsplit > WA_SPLIT_MAX) return cudaErrorInvalidValue;
  if (a.nsplit > 1 && (!a.part_o || !a.part_ml)) return cudaErrorInvalidValue;
  const int rep = a.H / a.G;
  const dim3 grid((a.L * rep + WA_ROWS - 1) / WA_ROWS, a.G, a.B * a.nsplit);
  cudaError_t e = kv_bf16 ? launch_win_t<bf16>(a, grid, s) : launch_win_t<float>(a, grid, s);
  if (e != cudaSuccess || a.nsplit == 1) return e;
  return launch_k(win_attn_combine_kernel, dim3((unsigned)(a.B * a.L * a.H)), dim3(128), 0, s, a);
}
