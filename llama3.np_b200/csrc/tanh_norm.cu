// Element-wise norms of layer-list decoders (dynamic tanh):  n(x) = tanh(alpha x) * w + b  with one alpha per norm and a
// weight and a bias per coordinate.  Nothing is reduced over the row, so one pass over the stream forms everything a layer
// needs from it: what joins the stream ahead of the layer (embedding multiplier, a looped block's step vector, the
// embedding output), the inputs of up to two sublayers with their bf16 mirrors, and the stream that goes on (plus a vector
// the output projections would otherwise have to add: their biases).  Everything fp32.
#include "common.cuh"
#include "mixer.h"

namespace {

template <int V>
struct Pack;
template <>
struct Pack<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
  __device__ __forceinline__ void store16(bf16* p) const { *p = __float2bfloat16_rn(v[0]); }
};
template <>
struct Pack<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void store16(bf16* p) const {
    union { __nv_bfloat162 h[2]; uint2 u; } o;
    o.h[0] = __floats2bfloat162_rn(v[0], v[1]);
    o.h[1] = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = o.u;
  }
};

// a thread per V consecutive coordinates of a row
template <int V>
__global__ void __launch_bounds__(256) tanh_norm_kernel(TanhNormArgs a, int64_t n) {
  pdl_launch();
  pdl_wait();
  const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= n) return;
  const int64_t r = i / a.D;
  const int c = (int)(i - r * a.D);
  const int64_t src = (a.src_rows ? (int64_t)a.src_rows[r] : r * a.src_mul + a.src_add) * a.D + c;
  Pack<V> x, t;
  x.load(a.x + src);
#pragma unroll
  for (int u = 0; u < V; ++u) x.v[u] *= a.mul;
  if (a.x0_out) x.store(a.x0_out + i);
  if (a.rows) {
    t.load(a.rows + i);
#pragma unroll
    for (int u = 0; u < V; ++u) x.v[u] += t.v[u];
  }
  if (a.vec) {
    t.load(a.vec + c);
#pragma unroll
    for (int u = 0; u < V; ++u) x.v[u] += t.v[u];
  }
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    if (q >= a.n_norm) break;
    Pack<V> w, b, o;
    w.load(a.w[q] + c);
    b.load(a.b[q] + c);
    const float alpha = *a.alpha[q];
#pragma unroll
    for (int u = 0; u < V; ++u) o.v[u] = tanhf(alpha * x.v[u]) * w.v[u] + b.v[u];
    if (a.out[q]) o.store(a.out[q] + i);
    if (a.out16[q]) o.store16(a.out16[q] + i);
  }
  if (a.write) {
    if (a.post) {
      t.load(a.post + c);
#pragma unroll
      for (int u = 0; u < V; ++u) x.v[u] += t.v[u];
    }
    x.store(a.x + i);
  }
}

}  // namespace

cudaError_t launch_tanh_norms(const TanhNormArgs& a, int rows, cudaStream_t s) {
  const bool gathered = a.src_rows || a.src_mul != 1 || a.src_add != 0;
  if (a.n_norm < 0 || a.n_norm > 2 || (gathered && (a.write || a.rows || a.x0_out))) return cudaErrorInvalidValue;
  const int64_t n = (int64_t)rows * a.D;
  if (a.D % 4 == 0) return launch_k(tanh_norm_kernel<4>, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, s, a, n);
  return launch_k(tanh_norm_kernel<1>, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, a, n);
}
