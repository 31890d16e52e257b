// Device helpers shared by the kernels of the layer-list decoders: bf16 tensor-core fragments, asynchronous copies, and the
// ordering rule of their launches.
//
// Every kernel here is launched with programmatic dependent launch and runs `pdl_wait` and then `pdl_trigger`, in that
// order: a kernel starts only after every CTA of its predecessor has passed its own wait, so what kernels before the
// predecessor wrote may be read ahead of `pdl_wait`; what the predecessor writes may not.  Pointers to data of earlier
// kernels carry no `__restrict__`: the compiler could otherwise move their loads ahead of the wait.
#pragma once
#include <cuda_bf16.h>

#include "cuda/common.cuh"

namespace bonsai {
namespace lay {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_addr(p)));
}
// c (16x8, f32) += a (16x16, bf16, row) * b (16x8, bf16, col)
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Lane addresses of the three fragment loads the kernels use, for a tile stored row-major with `ld` elements per row:
// A operand (rows x k), 16x16 at (r0, k0)
__device__ __forceinline__ const bf16* frag_a(const bf16* s, int ld, int r0, int k0, int lane) {
  return s + (r0 + (lane & 15)) * ld + k0 + (lane >> 4) * 8;
}
// two 8-column B operands whose columns are the tile's rows (n x k): columns n0..n0+15, k0..k0+15; registers {0,1} and {2,3}
__device__ __forceinline__ const bf16* frag_b_rows(const bf16* s, int ld, int n0, int k0, int lane) {
  return s + (n0 + (lane & 7) + ((lane >> 4) << 3)) * ld + k0 + ((lane >> 3) & 1) * 8;
}
// two 8-column B operands whose k runs along the tile's rows (k x n), loaded with .trans: k0..k0+15, columns n0..n0+15
__device__ __forceinline__ const bf16* frag_b_cols(const bf16* s, int ld, int k0, int n0, int lane) {
  return s + (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + n0 + (lane >> 4) * 8;
}
// A operand stored transposed (k x rows), loaded with .trans: rows r0..r0+15, k0..k0+15
__device__ __forceinline__ const bf16* frag_a_cols(const bf16* s, int ld, int r0, int k0, int lane) {
  return s + (k0 + (lane & 7) + ((lane >> 4) << 3)) * ld + r0 + ((lane >> 3) & 1) * 8;
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

constexpr float kLog2e = 1.4426950408889634f;

// The same with the approximate exponential and division (some 2^-22 of the result), for kernels that would wait for the accurate ones.
template <bool EXACT>
__device__ __forceinline__ float sigmoid_as(float x) {
  return EXACT ? sigmoid(x) : __fdividef(1.0f, 1.0f + ex2(-x * kLog2e));
}
template <bool EXACT>
__device__ __forceinline__ float silu_as(float x) {
  return x * sigmoid_as<EXACT>(x);
}
// max(x, 0) + log(1 + e) with e = exp(-|x|); the approximate form sums the series of log(1 + e) where e is small, so that small results
// keep their digits
template <bool EXACT>
__device__ __forceinline__ float softplus_as(float x) {
  if (EXACT) return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x)));
  const float e = ex2(-fabsf(x) * kLog2e);
  const float series = e * (1.0f - e * (1.0f / 2 - e * (1.0f / 3 - e * (1.0f / 4 - e * (1.0f / 5 - e * (1.0f / 6))))));
  return fmaxf(x, 0.0f) + (e < 0.0625f ? series : __logf(1.0f + e));
}

__device__ __forceinline__ void store_act(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_act(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_act4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }
__device__ __forceinline__ void store_act4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ float load_act(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load_act(const float* p) { return *p; }

// Element d of a head v(0), v(1), ... whose first `dims` dimensions are turned by the angles of `rot` (cosine, sine per pair; null: no
// rotation); pairs are (2i, 2i + 1), or (i, i + dims / 2).
template <typename V>
__device__ __forceinline__ float rotated(V v, int d, const float2* rot, int dims, int pairs) {
  if (d >= dims || rot == nullptr) return v(d);
  const int half = dims >> 1;
  const bool first = pairs ? (d & 1) == 0 : d < half;
  const float2 cs = rot[pairs ? d >> 1 : (first ? d : d - half)];
  const float own = v(d), other = v(pairs ? d ^ 1 : (first ? d + half : d - half));
  return first ? own * cs.x - other * cs.y : own * cs.x + other * cs.y;
}

__device__ __forceinline__ float rotated(const float* v, int d, const float2* rot, int dims, int pairs) {
  return rotated([&](int j) { return v[j]; }, d, rot, dims, pairs);
}

// Clamped gated unit: g * sigmoid(alpha (g + cubic g^3)) * (u + up_offset) with g = min(gate, limit), u = clamp(up, -limit, limit).  With
// alpha = 2 sqrt(2 / pi) and cubic = 0.044715 the first two factors are the tanh form of gelu: (1 + tanh(y)) / 2 = sigmoid(2 y).
struct Glu {
  float limit, alpha, up_offset, cubic;
};
__device__ __forceinline__ float glu(const Glu& a, float g, float u) {
  g = fminf(g, a.limit);
  u = fminf(fmaxf(u, -a.limit), a.limit);
  return g * sigmoid(a.alpha * fmaf(a.cubic * g * g, g, g)) * (u + a.up_offset);
}

// chunked recurrences: tokens per chunk, value columns per CTA, row length of a staged value tile
constexpr int kL = 64;
constexpr int kVT = 64;
constexpr int kVLD = kVT + 8;
// a portion as a whole, the local states of its segments, the segments from the states they start from
enum ChunkMode { kWhole, kLocal, kResume };

// One launch with programmatic dependent launch and, for cluster > 1, thread-block clusters of that many CTAs along
// dimension `dim` (0 = x, 1 = y) of the grid.
template <typename Kern, typename... Args>
static inline int launch(Kern kernel, dim3 grid, int threads, size_t smem, cudaStream_t stream, int cluster, int dim, Args... args) {
  if (smem > 24 * 1024 &&     // 48 KB with the static part
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return BONSAI_CUDA_LAUNCH_FAILED;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = dim == 0 ? cluster : 1;
  attr[1].val.clusterDim.y = dim == 1 ? cluster : 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = cluster > 1 ? 2 : 1;
  const cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, args...);
  return e == cudaSuccess ? BONSAI_CUDA_OK : BONSAI_CUDA_LAUNCH_FAILED;
}

}  // namespace lay
}  // namespace bonsai
