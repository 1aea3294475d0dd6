// Latent attention of layer-list decoders (layerlist.cu): every token caches ONE row [c | k_r] - a normed latent c
// (kv_rank) and a rotated key part k_r (rot_dim) shared by all heads.  Head j's key is [Wuk_j c | k_r] and its
// value Wuv_j c, so with the query folded onto the latent, q~_j = [Wuk_j^T q_c | rot(q_r)], the score is
// q~_j . [c | k_r] and the output Wuv_j (sum_i p_i c_i): attention runs on the cache rows themselves, all heads
// of a token against the same rows, the value of a row being its first kv_rank entries.
//
//  * latent_prep_kernel        norms of the two latents, rotation of k_r, cache append (a CTA per token and latent); the
//                              query latent alone for a layer that reads another layer's cache
//  * head_gemm_kernel          batched per-head product (Wuk_j^T q_c and Wuv_j ctx): 64 x 64 FFMA tiles, 4 x 4 per thread;
//                              head_gemv_kernel for up to 8 rows (decode).  The launch that folds the queries also turns
//                              their rotated part; the one that expands the values also applies an element-wise gate
//  * attn_latent_kernel        flash-style exact attention: a CTA holds up to 32 (token, head) query rows in shared
//                              memory and walks the visible cache rows 32 at a time; a lane scores one key for its warp's
//                              query rows, then the lanes own output columns.  Scores, weights and sums fp32.
//                              Calls with few rows spread them over all warps and split the keys over CTAs;
//                              attn_latent_combine_kernel merges the parts.  A sink
//                              (one logit per head without a value) joins the denominator once, at the very end.
#include <algorithm>

#include "common.cuh"
#include "mixer.h"

namespace {

__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < nw; ++w) t += red[w];
  return t;
}

// dst = src with its first `dims` entries turned at position pos: the pair (u, v) of entries (2i, 2i + 1) (layout 0) or
// (i, i + dims / 2) (layout 1) becomes (u cos a - v sin a, v cos a + u sin a), a = pos * f_i in fp32.  Work item i: pair i,
// or for i >= dims / 2 the unchanged entry i + dims / 2.
template <typename T>
__device__ __forceinline__ void rotate_item(const float* src, T* dst, int i, int dims, int layout, int pos, const float* __restrict__ freq) {
  const int half = dims >> 1;
  if (i >= half) { dst[i + half] = from_f32<T>(src[i + half]); return; }
  const int iu = layout ? i : 2 * i, iv = layout ? i + half : 2 * i + 1;
  const float u = src[iu], v = src[iv];
  float sn, cs;
  sincosf((float)pos * freq[i], &sn, &cs);
  dst[iu] = from_f32<T>(u * cs - v * sn);
  dst[iv] = from_f32<T>(v * cs + u * sn);
}

// blockIdx.y 0: the query latent of a token; 1: its cache row
template <typename KVT>
__global__ void __launch_bounds__(256) latent_prep_kernel(LatentPrepArgs a) {
  __shared__ float red[32];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x;
  const bool query = blockIdx.y == 0;
  const int n = query ? a.q_rank : a.kv_rank;
  const float* row = a.proj + (size_t)r * a.ld + (query ? 0 : a.k_off);
  const float* w = query ? a.wq : a.wk;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = row[i]; ss = fmaf(v, v, ss); }
  const float rinv = 1.0f / sqrtf(block_sum(ss, red) / (float)n + a.eps);
  if (query) {
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const float v = row[i] * rinv * w[i];
      if (a.cq) a.cq[(size_t)r * n + i] = v;
      if (a.cq16) a.cq16[(size_t)r * n + i] = __float2bfloat16_rn(v);
    }
    return;
  }
  const int b = r / a.L, pos = *a.pos_ptr + r - b * a.L;
  KVT* dst = (KVT*)a.cache + ((size_t)b * a.M + pos) * (a.kv_rank + a.rot_dim);
  for (int i = threadIdx.x; i < n; i += blockDim.x) dst[i] = from_f32<KVT>(row[i] * rinv * w[i]);
  for (int i = threadIdx.x; i < a.rot_dim - a.rot_dims / 2; i += blockDim.x)
    rotate_item(row + n, dst + n, i, a.rot_dims, a.rot_layout, pos, a.inv_freq);
}

// ---------------------------------------------------------------- batched per-head product
constexpr int HG_BM = 64, HG_BN = 64, HG_BK = 16;

// rotated query part of rows [r0, r1), head h: C[r, h, J ..] = rot(A[r, h, K ..])
__device__ __forceinline__ void head_rotate(const HeadGemmArgs& a, int h, int r0, int r1) {
  const int items = a.rot_dim - a.rot_dims / 2;
  for (int e = threadIdx.x; e < (r1 - r0) * items; e += blockDim.x) {
    const int r = r0 + e / items, i = e % items;
    rotate_item(a.A + (size_t)r * a.lda + (size_t)h * a.a_hs + a.K, a.C + (size_t)r * a.ldc + (size_t)h * a.c_hs + a.J, i, a.rot_dims,
                a.rot_layout, *a.pos_ptr + r % a.L, a.inv_freq);
  }
}

__device__ __forceinline__ float head_gate(const HeadGemmArgs& a, int r, int h, int j) {
  return a.gate ? 1.0f / (1.0f + expf(-a.gate[(size_t)r * a.ld_gate + (size_t)h * a.c_hs + j])) : 1.0f;
}

template <typename WT>
__global__ void __launch_bounds__(256) head_gemm_kernel(HeadGemmArgs a) {
  __shared__ __align__(16) float As[HG_BK][HG_BM + 4];
  __shared__ __align__(16) float Bs[HG_BK][HG_BN + 4];
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.z, r0 = blockIdx.x * HG_BM, j0 = blockIdx.y * HG_BN;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const float* A = a.A + (size_t)h * a.a_hs;
  const WT* W = (const WT*)a.W + (size_t)h * a.w_hs;
  float acc[4][4] = {};
  // a thread moves 4 elements of each tile; the next tile's global loads are issued ahead of this tile's products
  float ra[4], rb[4];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int e = tid + u * 256;
      const int k = e & (HG_BK - 1), rr = e >> 4;
      const int r = r0 + rr, kk = k0 + k;
      ra[u] = (r < a.rows && kk < a.K) ? A[(size_t)r * a.lda + kk] : 0.f;
      int kb, jj;
      if (a.w_js == 1) { jj = e & (HG_BN - 1); kb = e >> 6; } else { kb = e & (HG_BK - 1); jj = e >> 4; }
      const int j = j0 + jj, kw = k0 + kb;
      rb[u] = (j < a.J && kw < a.K) ? to_f32(W[(size_t)kw * a.w_ks + (size_t)j * a.w_js]) : 0.f;
    }
  };
  fetch(0);
  for (int k0 = 0; k0 < a.K; k0 += HG_BK) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int e = tid + u * 256;
      As[e & (HG_BK - 1)][e >> 4] = ra[u];
      if (a.w_js == 1) Bs[e >> 6][e & (HG_BN - 1)] = rb[u]; else Bs[e & (HG_BK - 1)][e >> 4] = rb[u];
    }
    __syncthreads();
    if (k0 + HG_BK < a.K) fetch(k0 + HG_BK);
#pragma unroll
    for (int k = 0; k < HG_BK; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&Bs[k][tx * 4]);
      const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + ty * 4 + i;
    if (r >= a.rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int jj = j0 + tx * 4 + j;
      if (jj >= a.J) continue;
      const size_t o = (size_t)r * a.ldc + (size_t)h * a.c_hs + jj;
      const float v = acc[i][j] * head_gate(a, r, h, jj);
      if (a.C) a.C[o] = v;
      if (a.C16) a.C16[o] = __float2bfloat16_rn(v);
    }
  }
  if (a.rot_dim > 0 && blockIdx.y == 0) head_rotate(a, h, r0, min(r0 + HG_BM, a.rows));
}

// ---------------------------------------------------------------- attention over the latent cache
constexpr int LA_KT = 32, LA_RW_MAX = 4, LA_WARPS = 8, LA_PF = 10;
constexpr int LA_CTAS = 2 * 148;  // splits stop at two CTAs per SM

__host__ __device__ inline int la_kstride(int Dk) {
  // 16-byte loads by 8 lanes at a time want an odd stride in 16-byte units; scalar loads an odd stride in words
  if (Dk % 4 == 0) return ((Dk / 4) & 1) ? Dk : Dk + 4;
  return (Dk & 1) ? Dk : Dk + 1;
}

// What the weighted sum of values is multiplied by at the end: 1 / denominator, the sink's term included, times the head's
// gate.  m, l: maximum and sum of exp(score - m) over the visible keys (never empty: a token sees itself).
__device__ __forceinline__ float latent_out_scale(const LatentAttnArgs& a, size_t tok, int head, float m, float l) {
  const float g = a.gate ? 1.0f / (1.0f + expf(-a.gate[tok * a.ld_gate + head])) : 1.0f;
  if (!a.sink) return g / l;
  const float sk = a.sink[head];
  if (sk <= m) return g / (l + expf(sk - m));
  const float c = expf(m - sk);  // the sink is the largest logit
  return g * c / fmaf(l, c, 1.0f);
}

// ND: output columns per lane (Dv <= 32 * ND); RW: query rows per warp
template <typename KVT, int ND, int LA_RW>
__global__ void __launch_bounds__(256) attn_latent_kernel(LatentAttnArgs a) {
  extern __shared__ __align__(16) float sm[];
  constexpr int LA_ROWS = LA_WARPS * LA_RW;
  const int Dk = a.Dk, Dv = a.Dv, KS = la_kstride(Dk), QS = (Dk + 3) & ~3;
  float* Qs = sm;                                    // [LA_ROWS][QS]
  float* Ks = Qs + LA_ROWS * QS;                     // [LA_KT][KS]
  float* Ps = Ks + LA_KT * KS;                       // [LA_WARPS][LA_KT][LA_RW]
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int b = blockIdx.y, split = blockIdx.z;
  const int nrow = a.L * a.H;                        // query rows of this sequence, (t, h) flattened
  const int row0 = blockIdx.x * LA_ROWS;
  const int pos0 = *a.pos_ptr;
  const int rows_here = min(LA_ROWS, nrow - row0);
  const int t_last = (row0 + rows_here - 1) / a.H;   // last token this CTA serves
  int k_begin = 0, k_end = pos0 + t_last + 1;        // visible keys of that token
  if (a.nsplit > 1) {
    const int per = ((k_end + a.nsplit - 1) / a.nsplit + LA_KT - 1) / LA_KT * LA_KT;
    k_begin = split * per;
    k_end = min(k_end, k_begin + per);
    if (k_begin >= k_end) {  // no keys for this split: weight zero, and the merge does not read the partial outputs
      for (int rr = threadIdx.x; rr < rows_here; rr += blockDim.x) {
        float* ml = a.part_ml + (((size_t)b * nrow + row0 + rr) * a.nsplit + split) * 2;
        ml[0] = -INFINITY; ml[1] = 0.f;
      }
      return;
    }
  }
  const float* qg = a.q + ((size_t)b * nrow + row0) * Dk;
  if (Dk % 4 == 0) {
    const int nv = LA_ROWS * Dk / 4;
#pragma unroll 4
    for (int v = threadIdx.x; v < nv; v += 256) {
      const int rr = (v * 4) / Dk, d = v * 4 - rr * Dk;
      float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
      if (rr < rows_here) q4 = *reinterpret_cast<const float4*>(qg + (size_t)v * 4);
      *reinterpret_cast<float4*>(Qs + rr * QS + d) = make_float4(q4.x * a.scale, q4.y * a.scale, q4.z * a.scale, q4.w * a.scale);
    }
  } else {
#pragma unroll 8
    for (int e = threadIdx.x; e < LA_ROWS * Dk; e += 256) {
      const int rr = e / Dk, d = e - rr * Dk;
      Qs[rr * QS + d] = rr < rows_here ? qg[e] * a.scale : 0.f;
    }
  }
  // this warp's rows and their last visible key
  int lim[LA_RW];
#pragma unroll
  for (int i = 0; i < LA_RW; ++i) {
    const int rr = warp * LA_RW + i;
    lim[i] = rr < rows_here ? pos0 + (row0 + rr) / a.H : -1;
  }
  float mrun[LA_RW], lrun[LA_RW], acc[LA_RW][ND];
#pragma unroll
  for (int i = 0; i < LA_RW; ++i) {
    mrun[i] = -INFINITY; lrun[i] = 0.f;
#pragma unroll
    for (int c = 0; c < ND; ++c) acc[i][c] = 0.f;
  }
  const KVT* cb = (const KVT*)a.cache + (size_t)b * a.M * Dk;
  const bool vec4 = (Dk % 4) == 0;
  float* Pw = Ps + warp * LA_KT * LA_RW;
  // A tile of cache rows is one contiguous block.  With rows that are a whole number of 16-byte vectors every thread
  // keeps up to LA_PF vectors of the NEXT tile in registers: their loads are in flight while this tile is used.
  constexpr int VEC = 16 / (int)sizeof(KVT);
  const bool kvec = (Dk % VEC) == 0 && vec4;
  uint4 pf[LA_PF];
  auto issue = [&](int k0n) {
    const int nvec = min(LA_KT, k_end - k0n) * Dk / VEC;
    const KVT* srcn = cb + (size_t)k0n * Dk;
#pragma unroll
    for (int u = 0; u < LA_PF; ++u) {
      const int v = threadIdx.x + u * 256;
      if (v < nvec) pf[u] = ldg_stream16(srcn + (size_t)v * VEC);
    }
  };
  auto put = [&](const uint4& r, int v) {  // vector v of the tile: VEC entries of one row
    const int e = v * VEC, j = e / Dk, d = e - j * Dk;
    float f[VEC];
    Vec16<KVT>::unpack(r, f);
#pragma unroll
    for (int x = 0; x < VEC; x += 4) *reinterpret_cast<float4*>(Ks + j * KS + d + x) = make_float4(f[x], f[x + 1], f[x + 2], f[x + 3]);
  };
  if (kvec && k_begin < k_end) issue(k_begin);
  for (int k0 = k_begin; k0 < k_end; k0 += LA_KT) {
    const int nk = min(LA_KT, k_end - k0);
    __syncthreads();  // the previous tile is consumed (first pass: Qs is complete)
    const KVT* src = cb + (size_t)k0 * Dk;
    if (kvec) {
      const int nvec = nk * Dk / VEC;
#pragma unroll
      for (int u = 0; u < LA_PF; ++u) {
        const int v = threadIdx.x + u * 256;
        if (v < nvec) put(pf[u], v);
      }
      for (int v0 = threadIdx.x + LA_PF * 256; v0 < nvec; v0 += 4 * 256) {  // rows too long for the registers
        uint4 r[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) if (v0 + u * 256 < nvec) r[u] = ldg_stream16(src + (size_t)(v0 + u * 256) * VEC);
#pragma unroll
        for (int u = 0; u < 4; ++u) if (v0 + u * 256 < nvec) put(r[u], v0 + u * 256);
      }
    } else {
#pragma unroll 8
      for (int e = threadIdx.x; e < nk * Dk; e += 256) {
        const int j = e / Dk, d = e - j * Dk;
        Ks[j * KS + d] = to_f32(src[e]);
      }
    }
    __syncthreads();
    if (kvec && k0 + LA_KT < k_end) issue(k0 + LA_KT);
    // scores: lane = key
    float s[LA_RW] = {};
    if (lane < nk) {
      const float* kr = Ks + lane * KS;
      const float* q0 = Qs + (warp * LA_RW) * QS;
      if (vec4) {
        for (int d = 0; d < Dk; d += 4) {
          const float4 kv = *reinterpret_cast<const float4*>(kr + d);
#pragma unroll
          for (int i = 0; i < LA_RW; ++i) {
            const float4 qv = *reinterpret_cast<const float4*>(q0 + i * QS + d);
            s[i] = fmaf(qv.x, kv.x, s[i]); s[i] = fmaf(qv.y, kv.y, s[i]);
            s[i] = fmaf(qv.z, kv.z, s[i]); s[i] = fmaf(qv.w, kv.w, s[i]);
          }
        }
      } else {
        for (int d = 0; d < Dk; ++d) {
          const float kv = kr[d];
#pragma unroll
          for (int i = 0; i < LA_RW; ++i) s[i] = fmaf(q0[i * QS + d], kv, s[i]);
        }
      }
    }
    float p[LA_RW];
#pragma unroll
    for (int i = 0; i < LA_RW; ++i) {
      const bool vis = lane < nk && k0 + lane <= lim[i];
      const float sc = vis ? s[i] : -INFINITY;
      const float mnew = fmaxf(mrun[i], warp_max(sc));
      // a row that sees nothing yet keeps m = -inf: weights 0, no rescale
      p[i] = vis ? expf(sc - mnew) : 0.f;
      const float alpha = mnew == -INFINITY ? 1.f : expf(mrun[i] - mnew);
      lrun[i] = lrun[i] * alpha + warp_sum(p[i]);
      mrun[i] = mnew;
#pragma unroll
      for (int c = 0; c < ND; ++c) acc[i][c] *= alpha;
    }
    if constexpr (LA_RW == 4) *reinterpret_cast<float4*>(Pw + lane * LA_RW) = make_float4(p[0], p[1], p[2], p[3]);
    else if constexpr (LA_RW == 2) *reinterpret_cast<float2*>(Pw + lane * LA_RW) = make_float2(p[0], p[1]);
    else Pw[lane] = p[0];
    __syncwarp();
    for (int j = 0; j < nk; ++j) {
      float pj[LA_RW];
      if constexpr (LA_RW == 4) { const float4 t = *reinterpret_cast<const float4*>(Pw + j * LA_RW); pj[0] = t.x; pj[1] = t.y; pj[2] = t.z; pj[3] = t.w; }
      else if constexpr (LA_RW == 2) { const float2 t = *reinterpret_cast<const float2*>(Pw + j * LA_RW); pj[0] = t.x; pj[1] = t.y; }
      else pj[0] = Pw[j];
      const float* vr = Ks + j * KS;
#pragma unroll
      for (int c = 0; c < ND; ++c) {
        const int d = lane + 32 * c;
        const float v = d < Dv ? vr[d] : 0.f;
#pragma unroll
        for (int i = 0; i < LA_RW; ++i) acc[i][c] = fmaf(pj[i], v, acc[i][c]);
      }
    }
    __syncwarp();
  }
#pragma unroll
  for (int i = 0; i < LA_RW; ++i) {
    const int rr = warp * LA_RW + i;
    if (rr >= rows_here) continue;
    const size_t row = (size_t)b * nrow + row0 + rr;           // = token row * H + head
    if (a.nsplit > 1) {
      float* po = a.part_o + (row * a.nsplit + split) * Dv;
#pragma unroll
      for (int c = 0; c < ND; ++c) { const int d = lane + 32 * c; if (d < Dv) po[d] = acc[i][c]; }
      if (lane == 0) { a.part_ml[(row * a.nsplit + split) * 2] = mrun[i]; a.part_ml[(row * a.nsplit + split) * 2 + 1] = lrun[i]; }
    } else {
      const size_t tok = row / a.H;
      const int head = (int)(row - tok * a.H);
      const float inv = latent_out_scale(a, tok, head, mrun[i], lrun[i]);
#pragma unroll
      for (int c = 0; c < ND; ++c) { const int d = lane + 32 * c; if (d < Dv) a.out[row * Dv + d] = acc[i][c] * inv; }
    }
  }
}

// merge of the splits: a CTA per (query row, 128 output columns)
__global__ void __launch_bounds__(128) attn_latent_combine_kernel(LatentAttnArgs a) {
  __shared__ float wsplit[LA_CTAS], red[8];
  pdl_launch();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* ml = a.part_ml + row * a.nsplit * 2;
  float mx = -INFINITY;
  for (int s = threadIdx.x; s < a.nsplit; s += 128) mx = fmaxf(mx, ml[2 * s]);
  mx = warp_max(mx);
  if (lane == 0) red[warp] = mx;
  __syncthreads();
  mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  float l = 0.f;
  for (int s = threadIdx.x; s < a.nsplit; s += 128) {
    const float w = ml[2 * s] == -INFINITY ? 0.f : expf(ml[2 * s] - mx);
    wsplit[s] = w;
    l = fmaf(w, ml[2 * s + 1], l);
  }
  l = warp_sum(l);
  if (lane == 0) red[4 + warp] = l;
  __syncthreads();
  l = (red[4] + red[5]) + (red[6] + red[7]);
  const int d = blockIdx.y * 128 + threadIdx.x;
  if (d >= a.Dv) return;
  const size_t tok = row / a.H;
  const float* po = a.part_o + row * a.nsplit * a.Dv + d;
  float o = 0.f;
#pragma unroll 16
  for (int s = 0; s < a.nsplit; ++s) {
    const float w = wsplit[s];
    const float v = w != 0.f ? __ldg(po + (size_t)s * a.Dv) : 0.f;  // a split without keys left nothing here
    o = fmaf(w, v, o);
  }
  a.out[row * a.Dv + d] = o * latent_out_scale(a, tok, (int)(row - tok * a.H), mx, l);
}

// Few rows (decode): the per-head product as matrix-vector products that stream the head's weights once.
// w_ks == 1 (an output's weights are contiguous): a warp per output; w_js == 1: a CTA per 64 outputs, two to a lane, its
// warps each taking an eighth of the k range.
constexpr int HV_OUT = 64;
template <typename WT>
__global__ void __launch_bounds__(256) head_gemv_kernel(HeadGemmArgs a) {
  __shared__ float part[8][HV_OUT];
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.y, r = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* A = a.A + (size_t)r * a.lda + (size_t)h * a.a_hs;
  const WT* W = (const WT*)a.W + (size_t)h * a.w_hs;
  if (a.rot_dim > 0 && blockIdx.x == 0) head_rotate(a, h, r, r + 1);
  float v;
  int j;
  if (a.w_ks == 1) {
    j = blockIdx.x * 8 + warp;
    if (j >= a.J) return;
    const WT* wr = W + (size_t)j * a.w_js;
    float acc = 0.f;
#pragma unroll 4
    for (int k = lane; k < a.K; k += 32) acc = fmaf(to_f32(wr[k]), A[k], acc);
    v = warp_sum(acc);
    if (lane != 0) return;
  } else {
    const int per = (a.K + 7) / 8, k0 = warp * per, k1 = min(a.K, k0 + per);
    const int j0 = blockIdx.x * HV_OUT + lane, j1 = j0 + 32;
    const int c0 = min(j0, a.J - 1), c1 = min(j1, a.J - 1);  // lanes past the last output repeat it
    float acc0 = 0.f, acc1 = 0.f;
#pragma unroll 16
    for (int k = k0; k < k1; ++k) {
      const WT* wk = W + (size_t)k * a.w_ks;
      const float x = A[k];
      acc0 = fmaf(to_f32(wk[c0]), x, acc0);
      acc1 = fmaf(to_f32(wk[c1]), x, acc1);
    }
    part[warp][lane] = acc0;
    part[warp][lane + 32] = acc1;
    __syncthreads();
    if (threadIdx.x >= HV_OUT) return;
    j = blockIdx.x * HV_OUT + threadIdx.x;
    if (j >= a.J) return;
    v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) v += part[w][threadIdx.x];
  }
  const size_t o = (size_t)r * a.ldc + (size_t)h * a.c_hs + j;
  v *= head_gate(a, r, h, j);
  if (a.C) a.C[o] = v;
  if (a.C16) a.C16[o] = __float2bfloat16_rn(v);
}

// query rows per warp: few rows spread over all warps of a CTA
int la_rw(int L, int H) { return L * H <= LA_WARPS ? 1 : L * H <= 2 * LA_WARPS ? 2 : LA_RW_MAX; }

size_t la_smem(int Dk, int rw) {
  return ((size_t)LA_WARPS * rw * ((Dk + 3) & ~3) + (size_t)LA_KT * la_kstride(Dk) + LA_WARPS * LA_KT * rw) * sizeof(float);
}

template <typename KVT, int ND, int RW>
cudaError_t launch_la_t(const LatentAttnArgs& a, cudaStream_t s) {
  static bool set = false;
  if (!set) {
    const cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<KVT, ND, RW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return e;
    set = true;
  }
  const int rows = LA_WARPS * RW;
  const dim3 grid((a.L * a.H + rows - 1) / rows, a.B, std::max(1, a.nsplit));
  return launch_k(attn_latent_kernel<KVT, ND, RW>, grid, dim3(256), la_smem(a.Dk, RW), s, a);
}

template <typename KVT, int ND>
cudaError_t launch_la_n(const LatentAttnArgs& a, cudaStream_t s) {
  switch (la_rw(a.L, a.H)) {
    case 1: return launch_la_t<KVT, ND, 1>(a, s);
    case 2: return launch_la_t<KVT, ND, 2>(a, s);
    default: return launch_la_t<KVT, ND, 4>(a, s);
  }
}

template <typename KVT>
cudaError_t launch_la(const LatentAttnArgs& a, cudaStream_t s) {
  const int nd = (a.Dv + 31) / 32;
  if (nd <= 1) return launch_la_n<KVT, 1>(a, s);
  if (nd <= 2) return launch_la_n<KVT, 2>(a, s);
  if (nd <= 4) return launch_la_n<KVT, 4>(a, s);
  if (nd <= 8) return launch_la_n<KVT, 8>(a, s);
  if (nd <= 16) return launch_la_n<KVT, 16>(a, s);
  if (nd <= 32) return launch_la_n<KVT, 32>(a, s);
  return cudaErrorInvalidValue;
}

}  // namespace

size_t latent_attn_smem(int Dk) { return la_smem(Dk, LA_RW_MAX); }

int latent_attn_splits(int B, int L, int H, int max_keys) {
  const int rows = LA_WARPS * la_rw(L, H), ctas = B * ((L * H + rows - 1) / rows);
  return std::max(1, std::min((max_keys + LA_KT - 1) / LA_KT, LA_CTAS / ctas));
}

size_t latent_attn_part_rows() { return (size_t)LA_CTAS * LA_WARPS * LA_RW_MAX; }

bool latent_attn_supported(int Dk, int Dv) { return Dv >= 1 && Dv <= Dk && Dv <= 1024 && latent_attn_smem(Dk) <= 220 * 1024; }

cudaError_t launch_latent_attn(const LatentAttnArgs& a, bool kv_bf16, cudaStream_t s) {
  cudaError_t e = kv_bf16 ? launch_la<bf16>(a, s) : launch_la<float>(a, s);
  if (e != cudaSuccess || a.nsplit <= 1) return e;
  return launch_k(attn_latent_combine_kernel, dim3(a.B * a.L * a.H, (a.Dv + 127) / 128), dim3(128), 0, s, a);
}

cudaError_t launch_latent_prep(const LatentPrepArgs& a, int rows, bool kv_bf16, cudaStream_t s) {
  const dim3 grid(rows, a.k_off < 0 ? 1 : 2);
  if (kv_bf16) return launch_k(latent_prep_kernel<bf16>, grid, dim3(256), 0, s, a);
  return launch_k(latent_prep_kernel<float>, grid, dim3(256), 0, s, a);
}

cudaError_t launch_head_gemm(const HeadGemmArgs& a, bool w_bf16, cudaStream_t s) {
  if (a.rows <= 8) {
    const dim3 g(a.w_ks == 1 ? (a.J + 7) / 8 : (a.J + HV_OUT - 1) / HV_OUT, a.H, a.rows);
    if (w_bf16) return launch_k(head_gemv_kernel<bf16>, g, dim3(256), 0, s, a);
    return launch_k(head_gemv_kernel<float>, g, dim3(256), 0, s, a);
  }
  const dim3 grid((a.rows + HG_BM - 1) / HG_BM, (a.J + HG_BN - 1) / HG_BN, a.H);
  if (w_bf16) return launch_k(head_gemm_kernel<bf16>, grid, dim3(256), 0, s, a);
  return launch_k(head_gemm_kernel<float>, grid, dim3(256), 0, s, a);
}
