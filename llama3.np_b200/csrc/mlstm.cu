// Matrix memory with exponential gates (the mLSTM of xLSTM), beside the recurrences of recurrent.cu / recur_chunk.cu.
//
//   i = cap tanh((z_i + b_i) / cap),  f = logsigmoid(cap tanh((z_f + b_f) / cap)),  m_t = max(f + m_(t-1), i)
//   S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,  n_t likewise with k alone,
//   o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)
//
// The running maximum m makes this a linear recurrence with ONE decay per (token, head) and scaled keys, so prompts run
// on the kernels the state-space mixer uses: mlstm_gates_kernel forms decays, their logarithms, key factors and the floor
// e^(-m) of every token, the recurrence carries n as one more column, and the output stage (mix_out_kernel) divides.
//
//  * mlstm_gates_kernel   a CTA per (head, sequence).  m_t as a function of m_0 is x -> max(a + x, b); such maps compose
//                         ((a1 + a2, max(b1 + a2, b2))), so a tile of 256 or 1024 tokens is one block-wide scan, tiles in a row.
//                         b stays of the order of the gates however long the tile, and a alone never survives against it.
//  * mlstm_step_kernel    one token per sequence: gates, state update, normaliser, norm per head, output gate and scale in
//                         one launch.  A cluster of CTAs shares a head by value columns; the square sum of the head's
//                         outputs crosses the cluster through distributed shared memory.
// Everything fp32.
#include <cooperative_groups.h>

#include <algorithm>

#include "common.cuh"
#include "mixer.h"

namespace cg = cooperative_groups;

namespace {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// GT: tokens per tile of the gate scan, a thread each
template <int GT>
__global__ void __launch_bounds__(GT) mlstm_gates_kernel(MlstmGateArgs a) {
  __shared__ float s_m[GT + 1];
  __shared__ float w_a[GT / 32], w_b[GT / 32];
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float bi = a.bias[h], bf = a.bias[a.H + h];
  float m0 = a.m[(size_t)b * a.H + h];
  for (int t0 = 0; t0 < a.L; t0 += GT) {
    const int n = min(GT, a.L - t0);
    const size_t row = (size_t)b * a.L + t0 + tid;
    float ig = 0.f, fg = 0.f;
    float ca = 0.f, cb = -INFINITY;  // the identity map
    if (tid < n) {
      const float* p = a.proj + row * a.ld;
      ig = soft_cap(p[a.i_off + h] + bi, a.cap);
      fg = log_sigmoid(soft_cap(p[a.f_off + h] + bf, a.cap));
      ca = fg; cb = ig;
    }
    // inclusive scan: (ca, cb) becomes the map of tokens t0 .. t0 + tid
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(L3_FULL, ca, o), pb = __shfl_up_sync(L3_FULL, cb, o);
      if (lane >= o) { cb = fmaxf(pb + ca, cb); ca += pa; }
    }
    if (lane == 31) { w_a[warp] = ca; w_b[warp] = cb; }
    __syncthreads();
    float mw = m0;  // m ahead of this warp's first token
    for (int w = 0; w < warp; ++w) mw = fmaxf(w_a[w] + mw, w_b[w]);
    const float m = fmaxf(ca + mw, cb);
    s_m[tid + 1] = m;
    if (tid == 0) s_m[0] = m0;
    __syncthreads();
    if (tid < n) {
      const float ld = fg + s_m[tid] - m;
      const size_t o = row * a.H + h;
      a.log_decay[o] = ld;
      a.decay[o] = expf(ld);
      a.k_scale[o] = expf(ig - m);
      a.floor[o] = expf(-m);
    }
    m0 = s_m[n];
    __syncthreads();  // s_m, w_a, w_b are written again by the next tile
  }
  if (tid == 0) a.m[(size_t)b * a.H + h] = m0;
}

// V: value columns per thread (DV a multiple of V * CL); grid (CL, H, B).  A thread owns V columns of every RL-th key row.
template <int V, int CL>
__global__ void __cluster_dims__(CL, 1, 1) __launch_bounds__(256) mlstm_step_kernel(MlstmStepArgs a) {
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                 // [DK] scaled query
  float* sk = sq + a.DK;          // [DK] scaled key
  float* so = sk + a.DK;          // [cols of this CTA] outputs
  float* red = so + ((a.DV / CL + 3) & ~3);  // [256 * V] partial outputs
  __shared__ float s_red[8];
  __shared__ float s_ssq;
  pdl_launch();
  pdl_wait();
  const int rank = CL > 1 ? blockIdx.x : 0;
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float* row = a.proj + (size_t)b * a.ld;
  const size_t bh = (size_t)b * a.H + h;
  // gates: every thread the same arithmetic
  const float ig = soft_cap(row[a.i_off + h] + a.bias[h], a.cap);
  const float fg = log_sigmoid(soft_cap(row[a.f_off + h] + a.bias[a.H + h], a.cap));
  const float m_old = a.m[bh];
  const float m = fmaxf(fg + m_old, ig);
  const float dec = expf(fg + m_old - m), ks = expf(ig - m);
  float nq = 0.f;
  float* n_row = a.n + bh * a.DK;
  for (int d = tid; d < a.DK; d += 256) {
    const float q = row[a.q_off + (size_t)h * a.DK + d] * a.q_mul, k = row[a.k_off + (size_t)h * a.DK + d] * ks;
    sq[d] = q;
    sk[d] = k;
    nq = fmaf(fmaf(dec, n_row[d], k), q, nq);
  }
  nq = warp_sum(nq);
  if (lane == 0) s_red[warp] = nq;
  __syncthreads();
  nq = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) nq += s_red[w];
  const float dinv = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
  const int cols = a.DV / CL, c_base = rank * cols;
  const int groups = cols / V;                       // column groups of this CTA
  float* S = a.S + bh * a.DK * a.DV + c_base;
  float ssq = 0.f;
  for (int g0 = 0; g0 < groups; g0 += 256) {
    const int cg_n = min(256, groups - g0), RL = 256 / cg_n;
    const int g = tid % cg_n, rl = tid / cg_n;
    const int c = (g0 + g) * V;
    float acc[V];
#pragma unroll
    for (int u = 0; u < V; ++u) acc[u] = 0.f;
    if (rl < RL) {
      float vv[V];
#pragma unroll
      for (int u = 0; u < V; ++u) vv[u] = row[a.v_off + (size_t)h * a.DV + c_base + c + u];
#pragma unroll 4
      for (int d = rl; d < a.DK; d += RL) {
        float* p = S + (size_t)d * a.DV + c;
        const float k = sk[d], q = sq[d];
        if (V == 4) {
          float4 s4 = *reinterpret_cast<const float4*>(p);
          s4.x = fmaf(dec, s4.x, k * vv[0]); s4.y = fmaf(dec, s4.y, k * vv[1 % V]);
          s4.z = fmaf(dec, s4.z, k * vv[2 % V]); s4.w = fmaf(dec, s4.w, k * vv[3 % V]);
          acc[0] = fmaf(s4.x, q, acc[0]); acc[1 % V] = fmaf(s4.y, q, acc[1 % V]);
          acc[2 % V] = fmaf(s4.z, q, acc[2 % V]); acc[3 % V] = fmaf(s4.w, q, acc[3 % V]);
          *reinterpret_cast<float4*>(p) = s4;
        } else {
          const float s1 = fmaf(dec, *p, k * vv[0]);
          acc[0] = fmaf(s1, q, acc[0]);
          *p = s1;
        }
      }
#pragma unroll
      for (int u = 0; u < V; ++u) red[(size_t)rl * cg_n * V + g * V + u] = acc[u];
    }
    __syncthreads();
    for (int j = tid; j < cg_n * V; j += 256) {
      float t = 0.f;
      for (int r = 0; r < RL; ++r) t += red[(size_t)r * cg_n * V + j];
      t *= dinv;
      so[g0 * V + j] = t;
      ssq = fmaf(t, t, ssq);
    }
    __syncthreads();  // red is written again by the next block of columns
  }
  ssq = warp_sum(ssq);
  if (lane == 0) s_red[warp] = ssq;
  __syncthreads();
  if (tid == 0) {
    float t = 0.f;
    for (int w = 0; w < 8; ++w) t += s_red[w];
    s_ssq = t;
  }
  float tot;
  if constexpr (CL > 1) {
    cg::cluster_group cl = cg::this_cluster();
    cl.sync();  // every CTA of the head has read n and m and published its square sum
    tot = 0.f;
#pragma unroll
    for (int r = 0; r < CL; ++r) tot += *cl.map_shared_rank(&s_ssq, r);
    cl.sync();  // no CTA leaves while another still reads its square sum
  } else {
    __syncthreads();
    tot = s_ssq;
  }
  if (rank == 0) {
    for (int d = tid; d < a.DK; d += 256) n_row[d] = fmaf(dec, n_row[d], sk[d]);
    if (tid == 0) a.m[bh] = m;
  }
  const float rinv = 1.0f / sqrtf(tot / (float)a.DV + a.eps);
  for (int j = tid; j < cols; j += 256) {
    const int c = h * a.DV + c_base + j;
    const float v = so[j] * rinv * a.w[c] * sigmoid_f(row[a.g_off + c]) * a.out_scale;
    const size_t o = (size_t)b * a.ld_out + c;
    if (a.out) a.out[o] = v;
    if (a.out16) a.out16[o] = __float2bfloat16_rn(v);
  }
}

template <int V, int CL>
cudaError_t launch_step(const MlstmStepArgs& a, int B, cudaStream_t s) {
  const size_t smem = ((size_t)2 * a.DK + ((a.DV / CL + 3) & ~3) + 256 * V) * sizeof(float);
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(mlstm_step_kernel<V, CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_k(mlstm_step_kernel<V, CL>, dim3(CL, a.H, B), dim3(256), smem, s, a);
}

}  // namespace

cudaError_t launch_mlstm_gates(const MlstmGateArgs& a, int B, cudaStream_t s) {
  if (a.L > 256) return launch_k(mlstm_gates_kernel<1024>, dim3(a.H, B), dim3(1024), 0, s, a);
  return launch_k(mlstm_gates_kernel<256>, dim3(a.H, B), dim3(256), 0, s, a);
}

cudaError_t launch_mlstm_step(const MlstmStepArgs& a, int B, cudaStream_t s) {
  // 16-byte accesses need whole groups of four columns in every CTA; a CTA of the cluster keeps at least 16 columns
  if (a.DV % 128 == 0) return launch_step<4, 8>(a, B, s);
  if (a.DV % 64 == 0) return launch_step<4, 4>(a, B, s);
  if (a.DV % 32 == 0) return launch_step<4, 2>(a, B, s);
  if (a.DV % 4 == 0) return launch_step<4, 1>(a, B, s);
  return launch_step<1, 1>(a, B, s);
}
