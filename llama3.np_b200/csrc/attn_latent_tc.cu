// Latent attention of prompts on the 5th-generation tensor cores (bf16 mode): the cached rows [c | k_r] of a sequence are
// EXPANDED once per call by a tcgen05 GEMM into per-head keys and values ([Wuk; Wuv] c, bf16; layerlist.cu) and attention
// runs per head on those - 2 (dim + rot_dim + vdim) FLOPs per (query, key, head) instead of the folded form's
// 2 (2 kv_rank + rot_dim) - as a flash-style kernel.  Decode keeps the folded form (attn_latent.cu): it reads the small
// cache rows only.
//
//  * latent_q_pack_kernel    the queries as a bf16 TMA operand: per head [q_c | 0 | rot(q_r) | 0], both parts padded to whole
//                            64-entry slices, so that what a key slice holds beyond its head's entries meets zeros
//  * attn_latent_tc_kernel   one CTA = 128 queries of one (sequence, head), keys in blocks of 64:
//      warp 0     TMA: the query tile, then the key blocks - the head's slice of the expansion, and the rotated part straight
//                 from the cache rows (shared by all heads)
//      warp 1     issues S_j = Q K_j^T into one of two TMEM score buffers
//      warp 11    issues O_w += P_j V_j, V as an MN-major operand (a thread of its own: the waits and the operand descriptors of
//                 the two products would otherwise queue behind one another in one instruction stream)
//      warps 2-9  two groups of four softmax warps taking alternate key blocks (w = j & 1), each with its own running
//                 maximum, sum and TMEM output; a thread is a query row.  The weights leave as TWO bf16 tiles, p = hi + lo
//                 (16 significant bits), and O takes both: scores, weights and sums are fp32 in effect.  The outputs are
//                 rescaled lazily, only when a maximum has grown by more than 2^8.  At the end the two groups merge, add the
//                 sink's term to the denominator, and apply the output gate.
//      warp 10    TMA: the value blocks
// Window and chunk attention (attn_window.cu) of prompts runs the same kernel with its caches as the key and value operands: the
// key blocks then start at the first key the tile's first query sees, and scores outside a row's window are masked.
// Every wait is bounded: one that runs out sets a flag, the CTA drains and the host reports an error.
#include <cuda.h>

#include <algorithm>

#include "common.cuh"
#include "gemm_tc.h"
#include "mixer.h"
#include "../../include/llama3_b200.h"

namespace {

constexpr int BQ = 128, BKV = 64;
constexpr int SLICE_Q = BQ * 128, SLICE_K = BKV * 128;   // bytes of one 64-entry slice of a query tile / key or value block
constexpr int P_TILE = BQ * BKV * 2;                     // one bf16 weight tile; a group owns two (hi, lo)
constexpr int STAGES_MAX = 3;
constexpr int THREADS = 384;
constexpr int TMEM_COLS = 512;                           // 2 score buffers of 64 columns, 2 outputs of up to 192
constexpr int TAIL = 512 + 2 * BQ * 8;                   // barriers, TMEM slot, flag; (maximum, sum) of both groups' rows
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
// false: the wait ran out (here or in another thread of the CTA); the caller goes on without touching what it waited for
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* fail) {
  for (uint32_t spins = 0; spins < (1u << 20); ++spins) {
    uint32_t ok;
    asm volatile(
        "{\n.reg .pred p;\n"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
        "selp.u32 %0, 1, 0, p;\n}"
        : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
    if (ok) return true;
    if ((spins & 63) == 63 && *fail) return false;
  }
  *fail = 1;
  return false;
}
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* tm, int c0, int c1, uint32_t bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
      ::"r"(dst), "l"(tm), "r"(c0), "r"(c1), "r"(bar) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void mma_bf16(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accum) {
  asm volatile(
      "{\n.reg .pred p;\nsetp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}"
      ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accum) : "memory");
}
__device__ __forceinline__ void tmem_ld32_issue(uint32_t taddr, float* v) {
  uint32_t* r = reinterpret_cast<uint32_t*>(v);
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const float* v) {
  const uint32_t* r = reinterpret_cast<const uint32_t*>(v);
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
        "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
        "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&t);
}
// K-major, 128-byte-swizzled operand tile: rows of 128 bytes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t desc_k_sw128(uint32_t smem_addr) {
  return (uint64_t)((smem_addr & 0x3FFFF) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) |
         ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}
// MN-major, 128-byte-swizzled operand (V: rows = keys = the MMA's K dimension): 8-key groups 1024 bytes apart, 64-entry
// slices of the value dimension lbo_bytes apart
__device__ __forceinline__ uint64_t desc_mn_sw128(uint32_t smem_addr, uint32_t lbo_bytes) {
  return (uint64_t)((smem_addr & 0x3FFFF) >> 4) | ((uint64_t)((lbo_bytes >> 4) & 0x3FFF) << 16) |
         ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}
// bf16 x bf16 -> fp32, M = 128
constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((128u >> 4) << 24);
constexpr uint32_t IDESC_S = IDESC | ((uint32_t)(BKV >> 3) << 17);
constexpr uint32_t IDESC_PV = IDESC | (1u << 16);  // B operand MN-major; N is added at run time

}  // namespace

namespace {

// ---------------------------------------------------------------- queries as an operand
__global__ void __launch_bounds__(256) latent_q_pack_kernel(LatentQPackArgs a) {
  extern __shared__ float trig[];  // cosines, then sines, of this row's position
  pdl_launch();
  pdl_wait();
  const size_t r = blockIdx.x;
  const int half = a.rot_dims >> 1;
  const int pos = *a.pos_ptr + (int)(r % a.L);
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * a.inv_freq[i], &trig[half + i], &trig[i]);
  __syncthreads();
  const int dpad = (a.dim + 63) & ~63, DQ = dpad + ((a.rot_dim + 63) & ~63);
  const int hd = a.dim + a.rot_dim, n8 = a.H * DQ / 8;
  const float* src = a.q + r * (size_t)a.H * hd;
  bf16* dst = a.q16 + r * (size_t)a.H * DQ;
  for (int g = threadIdx.x; g < n8; g += blockDim.x) {
    const int h = g * 8 / DQ, d0 = g * 8 - h * DQ;
    const float* qh = src + (size_t)h * hd;
    __align__(16) float v[8];
    const int i0 = d0 - dpad;  // sizes are multiples of 8: a group of 8 lies wholly inside a part or wholly in its padding
    if (d0 < dpad ? d0 >= a.dim : i0 >= a.rot_dim) {
      *reinterpret_cast<uint4*>(dst + (size_t)g * 8) = make_uint4(0, 0, 0, 0);
      continue;
    }
    const float* qr = qh + a.dim;
    const float* s8 = d0 < dpad ? qh + d0 : qr + i0;
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(s8);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(s8 + 4);
    if (d0 >= dpad) {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = i0 + k;
        if (i >= a.rot_dims) continue;
        const int p = a.rot_layout ? (i < half ? i : i - half) : i >> 1;           // pair
        const bool second = a.rot_layout ? i >= half : i & 1;
        const float other = qr[a.rot_layout ? (second ? i - half : i + half) : i ^ 1];
        v[k] = second ? v[k] * trig[p] + other * trig[half + p] : v[k] * trig[p] - other * trig[half + p];
      }
    }
    *reinterpret_cast<uint4*>(dst + (size_t)g * 8) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  }
}

// ---------------------------------------------------------------- attention
struct Shape {
  int nks, nrs, nqs, nvs;  // 64-entry slices of the un-rotated keys, the rotated part, both, the values
  int kst, vst;            // depths of the key and value rings
  __host__ __device__ int q_bytes() const { return nqs * SLICE_Q; }
  __host__ __device__ int k_bytes() const { return nqs * SLICE_K; }
  __host__ __device__ int v_bytes() const { return nvs * SLICE_K; }
  __host__ __device__ int smem() const { return 1024 + q_bytes() + kst * k_bytes() + vst * v_bytes() + 4 * P_TILE + TAIL; }
};

__host__ __device__ inline Shape make_shape(int dim, int rot_dim, int vdim) {
  Shape s;
  s.nks = (dim + 63) / 64; s.nrs = (rot_dim + 63) / 64; s.nqs = s.nks + s.nrs; s.nvs = (vdim + 63) / 64;
  // a key block is refilled from L2 while the other ones of the ring are used: the keys, needed first, get the spare stage
  s.kst = s.vst = STAGES_MAX;
  while (s.smem() > 227 * 1024 && s.kst + s.vst > 2) { if (s.vst >= s.kst) --s.vst; else --s.kst; }
  return s;
}

__global__ void __launch_bounds__(THREADS, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmE,
                      const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmV, LatentTcArgs a) {
  extern __shared__ uint8_t smem_raw[];
  const Shape sh = make_shape(a.dim, a.rot_dim, a.vdim);
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t sQ = (raw + 1023u) & ~1023u;
  const uint32_t sK = sQ + sh.q_bytes(), sV = sK + sh.kst * sh.k_bytes(), sP = sV + sh.vst * sh.v_bytes();
  const uint32_t bars = sP + 4 * P_TILE;
  const uint32_t q_full = bars, k_full = bars + 8, k_empty = k_full + 8 * STAGES_MAX, v_full = k_empty + 8 * STAGES_MAX,
                 v_empty = v_full + 8 * STAGES_MAX, s_full = v_empty + 8 * STAGES_MAX, s_empty = s_full + 16,
                 p_full = s_empty + 16, p_empty = p_full + 16, tmem_slot = p_empty + 16;
  uint8_t* sP_ptr = smem_raw + (sP - raw);
  uint32_t* tmem_slot_ptr = reinterpret_cast<uint32_t*>(smem_raw + (tmem_slot - raw));
  volatile int* fail = reinterpret_cast<volatile int*>(tmem_slot_ptr + 1);
  float2* ml = reinterpret_cast<float2*>(smem_raw + (bars + 512 - raw));  // [group][row] (maximum, sum)

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = gridDim.y - 1 - blockIdx.y;  // longest tiles (latest queries) of every head first
  const int head = blockIdx.x, bl = blockIdx.z, b = a.b0 + bl;
  const int q0 = qt * BQ;
  pdl_launch();

  if (warp == 0 && lane == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmQ));
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmE));
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmC));
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmV));
    *fail = 0;
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES_MAX; ++s) {
      mbar_init(k_full + 8 * s, 1); mbar_init(k_empty + 8 * s, 1);
      mbar_init(v_full + 8 * s, 1); mbar_init(v_empty + 8 * s, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(s_full + 8 * i, 1); mbar_init(s_empty + 8 * i, 128);
      mbar_init(p_full + 8 * i, 128); mbar_init(p_empty + 8 * i, 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tmem_slot), "n"(TMEM_COLS));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot_ptr;
  pdl_wait();
  const int start = *a.pos_ptr;
  const int last_q = min(q0 + BQ, a.L) - 1;                // last real query row of this tile
  auto first_key = [&](int p) { return a.window <= 0 ? 0 : a.chunked ? p - p % a.window : max(0, p - a.window + 1); };
  const int key_lo = first_key(start + q0);                // first key of the tile's blocks
  const int nb = (start + last_q - key_lo) / BKV + 1;      // key blocks holding a visible key
  const int kv_head = head / a.rep;
  const int kv_row = bl * a.seq_rows + kv_head * a.head_rows + key_lo;
  const uint32_t tS = tmem_base, tO = tmem_base + 2 * BKV; // two score buffers, then the two groups' outputs
  const int o_cols = (a.vdim + 31) & ~31;
  const int kcol0 = a.k_col + kv_head * a.k_cols, vcol0 = a.v_col + kv_head * a.v_cols;

  if (warp == 0) {
    if (lane == 0) {  // ---------------- queries and keys
      const int DQ = sh.nqs * 64;
      mbar_expect_tx(q_full, sh.q_bytes());
      for (int s = 0; s < sh.nqs; ++s) tma_load_2d(sQ + s * SLICE_Q, &tmQ, head * DQ + s * 64, b * a.L + q0, q_full);
      for (int j = 0; j < nb; ++j) {
        const int st = j % sh.kst, use = j / sh.kst;
        if (use > 0 && !mbar_wait(k_empty + 8 * st, (use - 1) & 1, fail)) break;
        const uint32_t kb = sK + st * sh.k_bytes(), bar = k_full + 8 * st;
        mbar_expect_tx(bar, sh.k_bytes());
        for (int s = 0; s < sh.nks; ++s) tma_load_2d(kb + s * SLICE_K, &tmE, kcol0 + s * 64, kv_row + j * BKV, bar);
        for (int s = 0; s < sh.nrs; ++s) tma_load_2d(kb + (sh.nks + s) * SLICE_K, &tmC, a.kv_rank + s * 64, b * a.M + j * BKV, bar);
      }
    }
  } else if (warp == 10) {
    if (lane == 0) {  // ---------------- values
      for (int j = 0; j < nb; ++j) {
        const int st = j % sh.vst, use = j / sh.vst;
        if (use > 0 && !mbar_wait(v_empty + 8 * st, (use - 1) & 1, fail)) break;
        mbar_expect_tx(v_full + 8 * st, sh.v_bytes());
        for (int s = 0; s < sh.nvs; ++s)
          tma_load_2d(sV + st * sh.v_bytes() + s * SLICE_K, &tmV, vcol0 + s * 64, kv_row + j * BKV, v_full + 8 * st);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {  // ---------------- scores
      uint32_t steps = 0;  // 16-entry steps of every slice, four bits each
      for (int s = 0; s < sh.nqs; ++s) {
        const int n = s < sh.nks ? a.dim - s * 64 : a.rot_dim - (s - sh.nks) * 64;
        steps |= (uint32_t)((min(n, 64) + 15) >> 4) << (4 * s);
      }
      const uint64_t dq = desc_k_sw128(sQ), dk0 = desc_k_sw128(sK);
      bool ok = mbar_wait(q_full, 0, fail);
      int st = 0, ph = 0;
      for (int j = 0; j < nb && ok; ++j) {
        const int w = j & 1;
        ok = mbar_wait(k_full + 8 * st, ph, fail) && (j < 2 || mbar_wait(s_empty + 8 * w, ((j >> 1) - 1) & 1, fail));
        if (!ok) break;
        tc_fence_after();
        const uint64_t dk = dk0 + (uint64_t)((st * sh.k_bytes()) >> 4);
        const uint32_t td = tS + w * BKV;
        for (int s = 0; s < sh.nqs; ++s) {
          const uint64_t ad = dq + (uint64_t)(s * (SLICE_Q >> 4)), bd = dk + (uint64_t)(s * (SLICE_K >> 4));
          const int n = (steps >> (4 * s)) & 15;
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk < n) mma_bf16(td, ad + kk * 2, bd + kk * 2, IDESC_S, (s | kk) ? 1u : 0u);
        }
        tc_commit(k_empty + 8 * st);
        tc_commit(s_full + 8 * w);
        if (++st == sh.kst) { st = 0; ph ^= 1; }
      }
    }
  } else if (warp == 11) {
    if (lane == 0) {  // ---------------- outputs
      const uint32_t idesc_pv = IDESC_PV | ((uint32_t)(((a.vdim + 15) & ~15) >> 3) << 17);
      const uint64_t dp0 = desc_k_sw128(sP), dv0 = desc_mn_sw128(sV, SLICE_K);
      int st = 0, ph = 0;
      for (int j = 0; j < nb; ++j) {
        const int w = j & 1;
        if (!mbar_wait(v_full + 8 * st, ph, fail) || !mbar_wait(p_full + 8 * w, (j >> 1) & 1, fail)) break;
        tc_fence_after();
        const uint64_t dv = dv0 + (uint64_t)((st * sh.v_bytes()) >> 4), dp = dp0 + (uint64_t)(w * (2 * P_TILE >> 4));
        const uint32_t td = tO + w * o_cols;
#pragma unroll
        for (int part = 0; part < 2; ++part)  // high part, then low part
#pragma unroll
          for (int kk = 0; kk < BKV / 16; ++kk)  // 16 keys per MMA
            mma_bf16(td, dp + part * (P_TILE >> 4) + kk * 2, dv + kk * (2048 >> 4), idesc_pv, (part | kk) ? 1u : (j < 2 ? 0u : 1u));
        tc_commit(v_empty + 8 * st);
        tc_commit(p_empty + 8 * w);
        if (++st == sh.vst) { st = 0; ph ^= 1; }
      }
    }
  } else {  // ---------------- softmax and output: thread = query row
    const int w = (warp - 2) >> 2, quarter = warp & 3;       // group; TMEM lanes this warp may read
    const int r = quarter * 32 + lane;
    const int qpos = start + q0 + r;                         // keys [qlo, qpos] are visible
    const int qlo = first_key(qpos);
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const float sc = a.scale * LOG2E;                        // p = 2^((s - m) * sc)
    const uint32_t tOw = tO + w * o_cols + lane_off;
    uint8_t* pw = sP_ptr + (2 * w) * P_TILE + r * 128;
    float m_used = -INFINITY, l_run = 0.f;
    int it = 0;
    bool ok = true;
    for (int j = w; j < nb; j += 2, ++it) {
      ok = mbar_wait(s_full + 8 * w, it & 1, fail);
      ok = __all_sync(L3_FULL, ok);
      if (!ok) break;
      tc_fence_after();
      float v[BKV];
      tmem_ld32_issue(tS + w * BKV + lane_off, v);
      tmem_ld32_issue(tS + w * BKV + lane_off + 32, v + 32);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(s_empty + 8 * w);                          // S_j is in registers
      const int key0 = key_lo + j * BKV;
      if (key0 + BKV - 1 > qpos) {
#pragma unroll
        for (int i = 0; i < BKV; ++i)
          if (key0 + i > qpos) v[i] = -INFINITY;
      }
      if (key0 < qlo) {
#pragma unroll
        for (int i = 0; i < BKV; ++i)
          if (key0 + i < qlo) v[i] = -INFINITY;
      }
      float mx4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
      for (int i = 4; i < BKV; i += 4) {
        mx4[0] = fmaxf(mx4[0], v[i]); mx4[1] = fmaxf(mx4[1], v[i + 1]);
        mx4[2] = fmaxf(mx4[2], v[i + 2]); mx4[3] = fmaxf(mx4[3], v[i + 3]);
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      bool waited = false;
      if (it == 0) {
        m_used = mx;                                         // may stay -inf: this row sees no key of the block
      } else {
        const bool grow = (mx - m_used) * sc > 8.0f;         // false for two -inf (NaN)
        if (__any_sync(L3_FULL, grow)) {
          ok = __all_sync(L3_FULL, mbar_wait(p_empty + 8 * w, (it - 1) & 1, fail));  // the group's last PV is done: O is stable
          if (!ok) break;
          waited = true;
          tc_fence_after();
          const float alpha = grow ? fast_exp2((m_used - mx) * sc) : 1.0f;
          if (grow) { m_used = mx; l_run *= alpha; }
          for (int c = 0; c < o_cols; c += 32) {
            float ov[32];
            tmem_ld32_issue(tOw + c, ov);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) ov[i] *= alpha;
            tmem_st32(tOw + c, ov);
          }
          tc_fence_before();
        }
      }
      const float moff = m_used == -INFINITY ? 0.f : m_used * sc;
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t hi[BKV / 2], lo[BKV / 2];
#pragma unroll
      for (int i = 0; i < BKV; i += 2) {
        const float p0 = fast_exp2(fmaf(v[i], sc, -moff)), p1 = fast_exp2(fmaf(v[i + 1], sc, -moff));  // 2^-inf = 0
        rs4[(i >> 1) & 3] += p0 + p1;
        const uint32_t t = pack_bf16(p0, p1);
        hi[i >> 1] = t;
        lo[i >> 1] = pack_bf16(p0 - __uint_as_float(t << 16), p1 - __uint_as_float(t & 0xffff0000u));
      }
      l_run += (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);
      if (it > 0 && !waited) {                               // the group's last PV has consumed the previous P
        ok = __all_sync(L3_FULL, mbar_wait(p_empty + 8 * w, (it - 1) & 1, fail));
        if (!ok) break;
      }
#pragma unroll
      for (int q = 0; q < BKV / 8; ++q) {                    // 16-byte chunks, swizzled inside the 128-byte row
        const int o = (q ^ (r & 7)) << 4;
        *reinterpret_cast<uint4*>(pw + o) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
        *reinterpret_cast<uint4*>(pw + P_TILE + o) = make_uint4(lo[4 * q], lo[4 * q + 1], lo[4 * q + 2], lo[4 * q + 3]);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // P (generic proxy) -> tensor core (async proxy)
      mbar_arrive(p_full + 8 * w);
    }
    if (ok && it > 0) ok = mbar_wait(p_empty + 8 * w, (it - 1) & 1, fail);  // the group's last PV has landed in O
    ml[w * BQ + r] = make_float2(m_used == -INFINITY ? -INFINITY : m_used * sc, l_run);
    tc_fence_before();
    __syncwarp();
    asm volatile("bar.sync 1, 256;" ::: "memory");           // both groups are done
    tc_fence_after();
    if (*fail == 0) {
      const float2 g0 = ml[r], g1 = ml[BQ + r];
      const float sk = a.sink ? a.sink[head] * LOG2E : -INFINITY;
      const float mm = fmaxf(fmaxf(g0.x, g1.x), sk);
      float f0 = fast_exp2(g0.x - mm), f1 = fast_exp2(g1.x - mm);  // a real row sees at least its own key: mm is finite
      const float den = g0.y * f0 + g1.y * f1 + fast_exp2(sk - mm);
      const bool real = q0 + r < a.L;
      const size_t row = (size_t)b * a.L + q0 + r;
      float inv = a.out_scale / den;
      if (real && a.gate && !a.gate_wide) inv *= 1.0f / (1.0f + __expf(-a.gate[row * a.ld_gate + head]));
      f0 *= inv; f1 *= inv;
      const size_t out0 = row * (size_t)a.ld_out + (size_t)head * a.vdim;
      for (int c = w * 32; c < o_cols; c += 64) {            // the groups share the output columns
        float o0[32], o1[32];
        tmem_ld32_issue(tO + lane_off + c, o0);
        if (nb > 1) tmem_ld32_issue(tO + o_cols + lane_off + c, o1);
        tmem_ld_wait();
#pragma unroll
        for (int d = 0; d < 32; d += 8) {
          if (!real || c + d >= a.vdim) break;
          float o[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) o[i] = nb > 1 ? fmaf(o0[d + i], f0, o1[d + i] * f1) : o0[d + i] * f0;
          if (a.gate && a.gate_wide) {
            const float* gp = a.gate + row * a.ld_gate + (size_t)head * a.vdim + c + d;
#pragma unroll
            for (int i = 0; i < 8; i += 4) {
              const float4 g = *reinterpret_cast<const float4*>(gp + i);
              o[i] *= 1.0f / (1.0f + __expf(-g.x)); o[i + 1] *= 1.0f / (1.0f + __expf(-g.y));
              o[i + 2] *= 1.0f / (1.0f + __expf(-g.z)); o[i + 3] *= 1.0f / (1.0f + __expf(-g.w));
            }
          }
          if (a.out16) *reinterpret_cast<uint4*>(a.out16 + out0 + c + d) = make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]), pack_bf16(o[6], o[7]));
          if (a.out) {
            *reinterpret_cast<float4*>(a.out + out0 + c + d) = make_float4(o[0], o[1], o[2], o[3]);
            *reinterpret_cast<float4*>(a.out + out0 + c + d + 4) = make_float4(o[4], o[5], o[6], o[7]);
          }
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0 && *fail) {
    *a.err = 1;
    __nanosleep(1000000);  // copies still in flight land before the shared memory is given up
  }
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "n"(TMEM_COLS));
  }
}

}  // namespace

int latent_tc_q_ld(int dim, int rot_dim) { return ((dim + 63) & ~63) + ((rot_dim + 63) & ~63); }

bool latent_tc_supported(int dim, int rot_dim, int vdim, int kv_rank) {
  if (dim % 8 || rot_dim % 8 || vdim % 8 || kv_rank % 8 || dim < 8 || vdim < 8 || vdim > 192 || !tc_gemm_supported(kv_rank + rot_dim)) return false;
  return make_shape(dim, rot_dim, vdim).smem() <= 227 * 1024;
}

cudaError_t launch_latent_q_pack(const LatentQPackArgs& a, int rows, cudaStream_t s) {
  return launch_k(latent_q_pack_kernel, dim3(rows), dim3(256), (size_t)std::max(1, a.rot_dims) * sizeof(float), s, a);
}

static cudaError_t launch_tc(const CUtensorMap* mq, const CUtensorMap* mk, const CUtensorMap* mc, const CUtensorMap* mv, const LatentTcArgs& a,
                             int n_seq, cudaStream_t s) {
  static bool done[16] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!done[dev & 15]) {
    const cudaError_t e = cudaFuncSetAttribute(attn_latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return e;
    done[dev & 15] = true;
  }
  if (!mq || !mk || !mc || !mv) return cudaErrorInvalidValue;
  const dim3 grid(a.H, (a.L + BQ - 1) / BQ, n_seq);
  return launch_k(attn_latent_tc_kernel, grid, dim3(THREADS), (size_t)make_shape(a.dim, a.rot_dim, a.vdim).smem(), s, *mq, *mk, *mc, *mv, a);
}

cudaError_t launch_attn_latent_tc(const LatentTcArgs& args, int n_seq, cudaStream_t s) {
  LatentTcArgs a = args;
  a.rep = 1; a.seq_rows = a.e_rows; a.head_rows = 0;
  a.k_col = 0; a.k_cols = a.dim; a.v_col = a.H * a.dim; a.v_cols = a.vdim;
  a.window = 0; a.chunked = 0; a.ld_out = a.H * a.vdim; a.out_scale = 1.f;
  const CUtensorMap* me = tc_get_map(a.expand, true, a.e_seqs * a.e_rows, a.H * (a.dim + a.vdim), BKV);
  return launch_tc(tc_get_map(a.q16, true, a.n_rows, a.H * latent_tc_q_ld(a.dim, a.rot_dim), BQ), me,
                   tc_get_map(a.cache, true, a.c_seqs * a.M, a.kv_rank + a.rot_dim, BKV), me, a, n_seq, s);
}

bool win_attn_tc_supported(int DK, int DV, int kind, int keep_first, float scale, int ld_out) {
  // 16-byte rows in the caches and in the output; the map's box is one 64-entry slice wide
  if (kind == L3_ATTN_SIGMOID || keep_first > 0 || !(scale > 0.f) || DK % 8 || DV % 8 || ld_out % 8 || DK < 64 || DV < 64 || DV > 192) return false;
  return tc_gemm_supported(DK) && make_shape(DK, 0, DV).smem() <= 227 * 1024;
}

cudaError_t launch_win_attn_tc(const WinAttnArgs& w, const bf16* q16, int cache_seqs, int* err, cudaStream_t s) {
  if (!win_attn_tc_supported(w.DK, w.DV, w.kind, w.keep_first, w.scale, w.ld_out) || w.H % w.G) return cudaErrorInvalidValue;
  if (((uintptr_t)w.out | (uintptr_t)w.out16) & 15) return cudaErrorInvalidValue;
  LatentTcArgs a{};
  a.q16 = q16; a.out = w.out; a.out16 = w.out16; a.gate = w.gate; a.ld_gate = w.ld_gate; a.sink = w.head_vec; a.pos_ptr = w.pos_ptr;
  a.scale = w.scale; a.err = err; a.n_rows = w.B * w.L; a.L = w.L; a.H = w.H; a.dim = w.DK; a.vdim = w.DV; a.M = w.M;
  a.rep = w.H / w.G; a.seq_rows = w.G * w.M; a.head_rows = w.M;
  a.window = w.window; a.chunked = w.chunked; a.ld_out = w.ld_out; a.out_scale = w.out_scale;
  const int rows = cache_seqs * w.G * w.M;
  const CUtensorMap* mk = tc_get_map(w.cache_k, true, rows, w.DK, BKV);
  return launch_tc(tc_get_map(q16, true, a.n_rows, a.H * latent_tc_q_ld(w.DK, 0), BQ), mk, mk, tc_get_map(w.cache_v, true, rows, w.DV, BKV), a, w.B, s);
}
