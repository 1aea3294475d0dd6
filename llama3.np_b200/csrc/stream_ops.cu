// Residual streams of pre-norm layer-list decoders (layerlist.cu, L3StackConfig::streams): instead of one residual row per
// token there are S of them.  Sublayer q reads u = sum_s in[s] X_s (normed) and its result y re-mixes all of them at once:
// X_t <- sum_s mix[s, t] X_s + out[t] (ls * y).  Everything fp32.
//
// The tail of one sublayer and the head of the next are ONE launch: the S rows are read once, the new ones are written, and
// the next sublayer's input (or, after the last sublayer, the sum of the streams) leaves in the same pass.
//
//  * stream_rows_kernel    a CTA per token: the next input with its RMS norm and the bf16 mirror the GEMMs read
//  * stream_slices_kernel  few tokens: a row spread over CTAs; the un-normed input goes out, the row-streaming GEMV norms it
//                          while staging (LinearArgs::norm_w)
#include "common.cuh"
#include "mixer.h"

namespace {

template <int VEC> struct Row;
template <> struct Row<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void store16(bf16* p) const {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
};
template <> struct Row<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
  __device__ __forceinline__ void store16(bf16* p) const { *p = __float2bfloat16_rn(v[0]); }
};

// the stream weights of one launch in shared memory: mix [from][to], then out, then in
struct StreamWeights {
  float mix[STREAMS_MAX * STREAMS_MAX], out[STREAMS_MAX], in[STREAMS_MAX];
};

__device__ __forceinline__ void load_weights(const StreamArgs& a, StreamWeights& w) {
  const int S = a.S;
  if (a.y)
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) w.mix[i] = a.mix[i];
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    w.out[i] = a.y ? a.out_w[i] : 0.f;
    w.in[i] = a.in_w ? a.in_w[i] : 0.f;
  }
  __syncthreads();
}

// Entries [i, i + VEC) of token r: the streams move on by the pending sublayer result (if any); returns the next input, and
// the sum of the streams in `total`.  NS: streams held in registers (a.S <= NS; EXACT: a.S == NS, known to the compiler).
template <int NS, bool EXACT, int VEC>
__device__ __forceinline__ Row<VEC> advance(const StreamArgs& a, const StreamWeights& w, size_t r, int i, Row<VEC>& total) {
  const int S = EXACT ? NS : a.S, D = a.D;
  Row<VEC> x[NS];
  float* Xr = a.X + r * (size_t)S * D + i;
  if (a.x0) {  // every stream starts as the embedding output
    x[0].load(a.x0 + r * (size_t)D + i);
#pragma unroll
    for (int k = 0; k < VEC; ++k) x[0].v[k] *= a.x_mul;
#pragma unroll
    for (int s = 1; s < NS; ++s) x[s] = x[0];
  } else {
#pragma unroll
    for (int s = 0; s < NS; ++s)
      if (EXACT || s < S) x[s].load(Xr + (size_t)s * D);
  }
  Row<VEC> u, y;
#pragma unroll
  for (int k = 0; k < VEC; ++k) { u.v[k] = 0.f; total.v[k] = 0.f; }
  if (a.y) {
    y.load(a.y + r * (size_t)D + i);
    if (a.ls) {
      Row<VEC> l;
      l.load(a.ls + i);
#pragma unroll
      for (int k = 0; k < VEC; ++k) y.v[k] *= l.v[k];
    }
  }
  if (!a.y) {
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      if (!EXACT && s >= S) break;
#pragma unroll
      for (int k = 0; k < VEC; ++k) { u.v[k] = fmaf(w.in[s], x[s].v[k], u.v[k]); total.v[k] += x[s].v[k]; }
    }
    return u;
  }
#pragma unroll (EXACT ? NS : 1)
  for (int t = 0; t < S; ++t) {
    Row<VEC> n;
#pragma unroll
    for (int k = 0; k < VEC; ++k) n.v[k] = w.out[t] * y.v[k];
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      if (!EXACT && s >= S) break;
      const float c = w.mix[s * S + t];
#pragma unroll
      for (int k = 0; k < VEC; ++k) n.v[k] = fmaf(c, x[s].v[k], n.v[k]);
    }
    if (a.store) n.store(Xr + (size_t)t * D);
    const float in = w.in[t];
#pragma unroll
    for (int k = 0; k < VEC; ++k) { u.v[k] = fmaf(in, n.v[k], u.v[k]); total.v[k] += n.v[k]; }
  }
  return u;
}

template <int NS, bool EXACT, int VEC>
__global__ void __launch_bounds__(256) stream_rows_kernel(StreamArgs a) {
  extern __shared__ __align__(16) float us[];  // [D] the next input ahead of its norm
  __shared__ StreamWeights w;
  __shared__ float red[8];
  pdl_launch();
  load_weights(a, w);  // weights do not depend on the previous kernel
  pdl_wait();
  const size_t r = blockIdx.x;
  const int D = a.D;
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < D; i += blockDim.x * VEC) {
    Row<VEC> total;
    const Row<VEC> u = advance<NS, EXACT, VEC>(a, w, r, i, total);
    if (a.sum) total.store(a.sum + r * (size_t)D + i);
    if (a.in_w) {
      u.store(us + i);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(u.v[k], u.v[k], ss);
    }
  }
  if (!a.in_w) return;
  float rinv = 1.f;
  if (a.norm_w) {
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += red[i];
    rinv = 1.0f / sqrtf(tot / (float)D + a.eps);
  }
  for (int i = threadIdx.x * VEC; i < D; i += blockDim.x * VEC) {  // each thread finishes what it stored
    Row<VEC> u;
    u.load(us + i);
    if (a.norm_w) {
      Row<VEC> g;
      g.load(a.norm_w + i);
#pragma unroll
      for (int k = 0; k < VEC; ++k) u.v[k] = u.v[k] * rinv * g.v[k];
    }
    if (a.h) u.store(a.h + r * (size_t)D + i);
    if (a.h16) u.store16(a.h16 + r * (size_t)D + i);
  }
}

template <int NS, bool EXACT, int VEC>
__global__ void __launch_bounds__(128) stream_slices_kernel(StreamArgs a) {
  __shared__ StreamWeights w;
  pdl_launch();
  load_weights(a, w);
  pdl_wait();
  const size_t r = blockIdx.y;
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= a.D) return;
  Row<VEC> total;
  const Row<VEC> u = advance<NS, EXACT, VEC>(a, w, r, i, total);
  if (a.sum) total.store(a.sum + r * (size_t)a.D + i);
  if (a.in_w) u.store(a.h + r * (size_t)a.D + i);
}

template <int NS, bool EXACT, int VEC>
cudaError_t launch_stream_t(const StreamArgs& a, int rows, cudaStream_t s) {
  const bool sliced = rows <= 8 && !a.norm_w && !a.h16;
  if (sliced) {
    const int per = 128 * VEC;
    return launch_k(stream_slices_kernel<NS, EXACT, VEC>, dim3((a.D + per - 1) / per, rows), dim3(128), 0, s, a);
  }
  auto kern = stream_rows_kernel<NS, EXACT, VEC>;
  const size_t smem = a.in_w ? (size_t)a.D * sizeof(float) : 0;
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  const int threads = a.D >= 1024 ? 256 : a.D >= 256 ? 128 : 64;
  return launch_k(kern, dim3(rows), dim3(threads), smem, s, a);
}

template <int VEC>
cudaError_t launch_stream_v(const StreamArgs& a, int rows, cudaStream_t s) {
  switch (a.S) {
    case 1: return launch_stream_t<1, true, VEC>(a, rows, s);
    case 2: return launch_stream_t<2, true, VEC>(a, rows, s);
    case 3: return launch_stream_t<3, true, VEC>(a, rows, s);
    case 4: return launch_stream_t<4, true, VEC>(a, rows, s);
    default: break;
  }
  if (a.S <= 8) return launch_stream_t<8, false, VEC>(a, rows, s);
  return launch_stream_t<STREAMS_MAX, false, 1>(a, rows, s);
}

}  // namespace

bool streams_supported(int S, int D) { return S >= 1 && S <= STREAMS_MAX && (size_t)D * sizeof(float) <= 160 * 1024; }

cudaError_t launch_streams(const StreamArgs& a, int rows, cudaStream_t s) {
  if (!streams_supported(a.S, a.D)) return cudaErrorInvalidValue;
  return a.D % 4 == 0 ? launch_stream_v<4>(a, rows, s) : launch_stream_v<1>(a, rows, s);
}
