// Row-wise steps of the layer-list decoders: embedding lookup, norm-of-the-output residual add, final norm of selected rows,
// and the per-head norm with output gate of the recurrent mixers.  The residual stream is f32; every kernel that changes it
// also leaves the bf16 copy that the next projection reads (null in the f32 mode, where projections read the stream).
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

__global__ void embed_kernel(const bf16* __restrict__ table, int ld_table, const int* tokens, int width, float* x,
                             bf16* x16, int ld16) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const bf16* src = table + (size_t)tokens[t] * ld_table;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const bf16 v = src[c];
    x[(size_t)t * width + c] = __bfloat162float(v);
    if (x16 != nullptr) x16[(size_t)t * ld16 + c] = v;
  }
}

constexpr int kKeep = 4;   // float4 chunks of a row that a thread keeps in registers

// x += y / sqrt(mean(y^2) + eps) * w
__global__ void norm_add_kernel(float* x, const float* y, int ldy, const float* __restrict__ w, float eps, int width,
                                bf16* x16, int ld16) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  float* xr = x + (size_t)blockIdx.x * width;
  const float* yr = y + (size_t)blockIdx.x * ldy;
  bf16* hr = x16 == nullptr ? nullptr : x16 + (size_t)blockIdx.x * ld16;
  float ss = 0.0f;
  if ((width & 3) == 0 && width <= 4 * kKeep * (int)blockDim.x) {
    const int nch = width >> 2;
    float4 v[kKeep], r[kKeep];
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      v[i] = c < nch ? reinterpret_cast<const float4*>(yr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      r[i] = c < nch ? reinterpret_cast<const float4*>(xr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, s32) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nch) {
        const float4 g = reinterpret_cast<const float4*>(w)[c];
        r[i].x += v[i].x * inv * g.x;
        r[i].y += v[i].y * inv * g.y;
        r[i].z += v[i].z * inv * g.z;
        r[i].w += v[i].w * inv * g.w;
        reinterpret_cast<float4*>(xr)[c] = r[i];
        if (hr != nullptr) reinterpret_cast<uint2*>(hr)[c] = make_uint2(pack_bf16(r[i].x, r[i].y), pack_bf16(r[i].z, r[i].w));
      }
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) ss += yr[c] * yr[c];
  const float inv = 1.0f / sqrtf(block_sum(ss, s32) / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    const float v = xr[c] + yr[c] * inv * w[c];
    xr[c] = v;
    if (hr != nullptr) hr[c] = __float2bfloat16_rn(v);
  }
}

// out[i] = norm(x[rows[i]]) * w; rows == null: row i
template <typename OUT>
__global__ void norm_rows_kernel(const float* x, const int* rows, const float* __restrict__ w, float eps, int width,
                                 OUT* out, int ld) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  const int row = rows == nullptr ? blockIdx.x : rows[blockIdx.x];
  const float* xr = x + (size_t)row * width;
  float ss = 0.0f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) ss += xr[c] * xr[c];
  const float inv = 1.0f / sqrtf(block_sum(ss, s32) / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += blockDim.x) store_act(out + (size_t)blockIdx.x * ld + c, xr[c] * inv * w[c]);
}

// One warp per (row, head): o / rms(o over the head) * w * sigmoid(gate)
template <typename OUT>
__global__ void __launch_bounds__(256) gated_head_norm_kernel(const float* o, int ldo, const float* gate, int ldg, const float* __restrict__ w,
                                                              float eps, int T, int heads, int vdim, OUT* out, int ld, int vec) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, item = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= T * heads) return;
  const int t = item / heads, c0 = (item % heads) * vdim;
  const float* orow = o + (size_t)t * ldo + c0;
  const float* grow = gate + (size_t)t * ldg + c0;
  OUT* dst = out + (size_t)t * ld + c0;
  w += c0;
  if (vec) {                 // rows of float4, up to kKeep per lane
    const int nch = vdim >> 2;
    float4 v[kKeep], g[kKeep];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = lane + 32 * i;
      v[i] = c < nch ? reinterpret_cast<const float4*>(orow)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      g[i] = c < nch ? reinterpret_cast<const float4*>(grow)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = lane + 32 * i;
      if (c < nch) {
        const float4 ww = reinterpret_cast<const float4*>(w)[c];
        const float y[4] = {v[i].x * inv * ww.x * sigmoid(g[i].x), v[i].y * inv * ww.y * sigmoid(g[i].y), v[i].z * inv * ww.z * sigmoid(g[i].z),
                            v[i].w * inv * ww.w * sigmoid(g[i].w)};
        if constexpr (sizeof(OUT) == 2) reinterpret_cast<uint2*>(dst)[c] = make_uint2(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]));
        else reinterpret_cast<float4*>(dst)[c] = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
    return;
  }
  float ss = 0.0f;
  for (int c = lane; c < vdim; c += 32) ss += orow[c] * orow[c];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int c = lane; c < vdim; c += 32) store_act(dst + c, orow[c] * inv * w[c] * sigmoid(grow[c]));
}

static int row_threads(int width) {
  const int want = (width + 15) / 16;   // kKeep float4 per thread
  const int t = (want + 31) / 32 * 32;
  return t < 64 ? 64 : (t > 1024 ? 1024 : (width >= 2048 && t < 512 ? 512 : t));
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// x f32 [T][width] = table[tokens[t]] (bf16 rows of ld_table elements); x16 (may be null) bf16 [T][ld16]
int bonsai_lay_embed(const void* table, int ld_table, const int* tokens, int T, int width, float* x, void* x16, int ld16, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || width < 1 || ld_table < width) return BONSAI_CUDA_BAD_ARG;
  return launch(embed_kernel, dim3(T), 256, 0, stream, 1, 0, (const bf16*)table, ld_table, tokens, width, x, (bf16*)x16, ld16);
}

int bonsai_lay_norm_add(float* x, const float* y, int ldy, const float* w, float eps, int T, int width, void* x16, int ld16, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || width < 1 || ldy < width || (ldy & 3) != 0 || (ld16 & 3) != 0) return BONSAI_CUDA_BAD_ARG;
  return launch(norm_add_kernel, dim3(T), row_threads(width), 0, stream, 1, 0, x, y, ldy, w, eps, width, (bf16*)x16, ld16);
}

// out: bf16 when f32_out == 0, f32 otherwise
int bonsai_lay_norm_rows(const float* x, const int* rows, const float* w, float eps, int R, int width, void* out, int ld, int f32_out,
                         cudaStream_t stream) {
  using namespace bonsai::lay;
  if (R < 1 || width < 1 || ld < width) return BONSAI_CUDA_BAD_ARG;
  const int th = row_threads(width);
  if (f32_out) return launch(norm_rows_kernel<float>, dim3(R), th, 0, stream, 1, 0, x, rows, w, eps, width, (float*)out, ld);
  return launch(norm_rows_kernel<bf16>, dim3(R), th, 0, stream, 1, 0, x, rows, w, eps, width, (bf16*)out, ld);
}

int bonsai_lay_gated_head_norm(const float* o, int ldo, const float* gate, int ldg, const float* w, float eps, int T, int heads, int vdim, void* out,
                               int ld, int f32_out, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || heads < 1 || vdim < 1 || ld < heads * vdim || (long long)T * heads >= (1ll << 30)) return BONSAI_CUDA_BAD_ARG;
  const dim3 grid((T * heads + 7) / 8);
  const uintptr_t at = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out);
  const int vec = vdim % 4 == 0 && vdim <= 128 * kKeep && ldo % 4 == 0 && ldg % 4 == 0 && ld % 4 == 0 && at % 16 == 0;
  if (f32_out)
    return launch(gated_head_norm_kernel<float>, grid, 256, 0, stream, 1, 0, o, ldo, gate, ldg, w, eps, T, heads, vdim, (float*)out, ld, vec);
  return launch(gated_head_norm_kernel<bf16>, grid, 256, 0, stream, 1, 0, o, ldo, gate, ldg, w, eps, T, heads, vdim, (bf16*)out, ld, vec);
}

}  // extern "C"
