// Projections with dense bf16 weights: out[t][n] = sum_k x[t][k] W[n][k].
//
// `few_rows_kernel` serves decode batches and short portions (up to 64 rows): the weights are streamed once, a warp's lane
// loads 16 contiguous bytes of a weight row and uses them directly as `mma.sync.m16n8k16` A registers.  That is the
// fragment layout up to a permutation of k inside every 32 inputs, and the activations are loaded through the same
// permutation (16 contiguous bytes of an activation row as the B registers), so neither operand passes through shared
// memory.  The eight warps of a CTA split K and meet in shared memory once; matrices of few rows are split further, over the CTAs of a
// cluster, which meet in distributed shared memory.  More activation rows go to the tcgen05 GEMM
// (cuda/bitgemm_prefill.cu, dense bf16 operands).
//
// `f32_kernel` is the 32-bit mode: f32 activations, the same bf16 weights (exact in f32), f32 FMA throughout.
//
// Epilogues: 0 = f32 store, 1 = clamped gated unit over interleaved gate / up rows, 2 = squared relu, 3 = the product itself in the
// activations' type, 4 = f32 store of limit * tanh(product / limit).
#include <cooperative_groups.h>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

__device__ __forceinline__ float squared_relu(float v) {
  v = fmaxf(v, 0.0f);
  return v * v;
}

// the f32 outputs of epilogues 0 and 4
__device__ __forceinline__ float capped(float v, int epi, const Glu& a) { return epi == 4 ? a.limit * tanhf(v / a.limit) : v; }

constexpr int kWarps = 8;

// NT: 8-row groups of activations; grid (16 weight rows, CTAs that split K, a cluster)
template <int NT, bool SPLIT>
__global__ void __launch_bounds__(kWarps * 32) few_rows_kernel(const bf16* __restrict__ W, int n, int kp, const bf16* x, int ldx, int T,
                                                              float* out, bf16* out16, int ldo, int epi, Glu act) {
  constexpr int LD = 8 * NT + 1;
  __shared__ float red[kWarps][16][LD];
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int row0 = blockIdx.x * 16, split = SPLIT ? gridDim.y : 1, rank = SPLIT ? blockIdx.y : 0;
  const bf16* w0 = W + (size_t)min(row0 + g, n - 1) * kp + 8 * t4;
  const bf16* w1 = W + (size_t)min(row0 + g + 8, n - 1) * kp + 8 * t4;
  const int chunks = kp >> 7, first = rank * kWarps + warp, step = split * kWarps;   // 128 inputs each
  uint4 a[4], b[4];
  auto load_w = [&](int c) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      a[i] = __ldcs(reinterpret_cast<const uint4*>(w0 + c * 128 + i * 32));
      b[i] = __ldcs(reinterpret_cast<const uint4*>(w1 + c * 128 + i * 32));
    }
  };
  if (first < chunks) load_w(first);   // weights depend on no earlier kernel
  pdl_wait();
  pdl_trigger();
  const bf16* xr[NT];
#pragma unroll
  for (int j = 0; j < NT; ++j) xr[j] = x + (size_t)min(8 * j + g, T - 1) * ldx + 8 * t4;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
  for (int c = first; c < chunks; c += step) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const uint32_t lo[4] = {a[i].x, b[i].x, a[i].y, b[i].y}, hi[4] = {a[i].z, b[i].z, a[i].w, b[i].w};
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const uint4 v = *reinterpret_cast<const uint4*>(xr[j] + c * 128 + i * 32);
        mma_bf16(acc[j], lo, v.x, v.y);
        mma_bf16(acc[j], hi, v.z, v.w);
      }
    }
    if (c + step < chunks) load_w(c + step);
  }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    red[warp][g][8 * j + 2 * t4] = acc[j][0];
    red[warp][g][8 * j + 2 * t4 + 1] = acc[j][1];
    red[warp][g + 8][8 * j + 2 * t4] = acc[j][2];
    red[warp][g + 8][8 * j + 2 * t4 + 1] = acc[j][3];
  }
  __syncthreads();
  auto warps_sum = [&](int r, int t) {
    float v = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) v += red[w][r][t];
    return v;
  };
  if constexpr (SPLIT) {               // this CTA's sums, where the others find them
    constexpr int PER = 16 * 8 * NT / (kWarps * 32) > 0 ? 16 * 8 * NT / (kWarps * 32) : 1;
    float own[PER];
#pragma unroll
    for (int p = 0; p < PER; ++p) {
      const int i = threadIdx.x + p * kWarps * 32;
      own[p] = i < 16 * T ? warps_sum(i & 15, i >> 4) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int p = 0; p < PER; ++p) {
      const int i = threadIdx.x + p * kWarps * 32;
      if (i < 16 * T) red[0][i & 15][i >> 4] = own[p];
    }
    cluster.sync();
  }
  auto total = [&](int r, int t) {
    if (!SPLIT) return warps_sum(r, t);
    float v = 0.0f;
    for (int s = 0; s < split; ++s) v += *cluster.map_shared_rank(&red[0][r][t], s);
    return v;
  };
  if (epi != 1) {
    for (int i = rank * kWarps * 32 + threadIdx.x; i < 16 * T; i += step * 32) {
      const int r = i & 15, t = i >> 4;
      const float v = total(r, t);
      if (row0 + r >= n) continue;
      if (epi == 0 || epi == 4) out[(size_t)t * ldo + row0 + r] = capped(v, epi, act);
      else out16[(size_t)t * ldo + row0 + r] = __float2bfloat16_rn(epi == 2 ? squared_relu(v) : v);
    }
  } else {
    for (int i = rank * kWarps * 32 + threadIdx.x; i < 8 * T; i += step * 32) {
      const int r = i & 7, t = i >> 3;
      const float gv = total(2 * r, t), uv = total(2 * r + 1, t);
      if (row0 + 2 * r + 1 < n) out16[(size_t)t * ldo + (row0 >> 1) + r] = __float2bfloat16_rn(glu(act, gv, uv));
    }
  }
  if (SPLIT) cluster.sync();           // nobody leaves while its sums are being read
}

// 64 weight rows x 64 activation rows per CTA, 256 threads with 4 x 4 outputs each
__global__ void __launch_bounds__(256) f32_kernel(const bf16* __restrict__ W, int n, int k, int kp, const float* x, int ldx, int T,
                                                  float* out, int ldo, int epi, Glu act) {
  __shared__ float sw[16][68], sx[16][68];
  pdl_wait();
  pdl_trigger();
  const int n0 = blockIdx.x * 64, t0 = blockIdx.y * 64;
  const int tn = threadIdx.x & 15, tt = threadIdx.x >> 4;
  float acc[4][4] = {};   // [activation row][weight row]
  for (int k0 = 0; k0 < k; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256, r = idx >> 4, c = idx & 15;
      const bool kin = k0 + c < k;
      sw[c][r] = kin && n0 + r < n ? __bfloat162float(W[(size_t)(n0 + r) * kp + k0 + c]) : 0.0f;
      sx[c][r] = kin && t0 + r < T ? x[(size_t)(t0 + r) * ldx + k0 + c] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      float wv[4], xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        wv[i] = sw[c][tn * 4 + i];
        xv[i] = sx[c][tt * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + tt * 4 + i;
    if (t >= T) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = n0 + tn * 4 + j;
      if (epi != 1) {
        if (r < n) out[(size_t)t * ldo + r] = epi == 2 ? squared_relu(acc[i][j]) : capped(acc[i][j], epi, act);
      } else if ((j & 1) == 0 && r + 1 < n) {
        out[(size_t)t * ldo + (r >> 1)] = glu(act, acc[i][j], acc[i][j + 1]);
      }
    }
  }
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// W bf16 [n][kp] (kp a multiple of 128, columns past the layer's width zero), x bf16 [T][ldx] (ldx >= kp, finite in the
// padding), T <= 64.  epi 0 and 4: out f32 [T][ldo]; epi 1: out16 bf16 [T][ldo] of n / 2 columns; epi 2 and 3: out16 bf16 [T][ldo].
int bonsai_lay_linear_few(const void* W, int n, int kp, const void* x, int ldx, int T, float* out, void* out16, int ldo, int epi, float limit,
                          float alpha, float up_offset, float cubic, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (n < 1 || kp < 128 || kp % 128 != 0 || ldx < kp || ldx % 8 != 0 || T < 1 || T > 64 || epi < 0 || epi > 4) return BONSAI_CUDA_BAD_ARG;
  const bool f32_out = epi == 0 || epi == 4;
  if ((f32_out && out == nullptr) || (!f32_out && out16 == nullptr) || (epi == 4 && !(limit > 0.0f)) || (epi == 1 && n % 2 != 0)) return BONSAI_CUDA_BAD_ARG;
  const Glu act{limit, alpha, up_offset, cubic};
  // few CTAs: K is split until they cover the GPU, or a warp has one chunk
  int split = 1;
  while (split < 8 && (n + 15) / 16 * split * 2 <= 148 && split * 2 * kWarps <= kp / 128) split *= 2;
  const dim3 grid((n + 15) / 16, split);
#define BONSAI_FEW(NT)                                                                                                                                  \
  (split > 1 ? launch(few_rows_kernel<NT, true>, grid, kWarps * 32, 0, stream, split, 1, (const bf16*)W, n, kp, (const bf16*)x, ldx, T, out,            \
                      (bf16*)out16, ldo, epi, act)                                                                                                      \
             : launch(few_rows_kernel<NT, false>, grid, kWarps * 32, 0, stream, 1, 0, (const bf16*)W, n, kp, (const bf16*)x, ldx, T, out, (bf16*)out16, \
                      ldo, epi, act))
  return T <= 8 ? BONSAI_FEW(1) : (T <= 16 ? BONSAI_FEW(2) : (T <= 32 ? BONSAI_FEW(4) : BONSAI_FEW(8)));
#undef BONSAI_FEW
}

int bonsai_lay_linear_f32(const void* W, int n, int k, int kp, const float* x, int ldx, int T, float* out, int ldo, int epi, float limit, float alpha,
                          float up_offset, float cubic, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (n < 1 || k < 1 || kp < k || ldx < k || T < 1 || out == nullptr || epi < 0 || epi > 4 || (epi == 1 && n % 2 != 0) || (epi == 4 && !(limit > 0.0f))) return BONSAI_CUDA_BAD_ARG;
  return launch(f32_kernel, dim3((n + 63) / 64, (T + 63) / 64), 256, 0, stream, 1, 0, (const bf16*)W, n, k, kp, x, ldx, T, out, ldo, epi,
                Glu{limit, alpha, up_offset, cubic});
}

}  // extern "C"
