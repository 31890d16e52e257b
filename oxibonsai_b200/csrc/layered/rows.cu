// Row-wise steps of the layer-list decoders: embedding lookup, residual adds (of a normed output, or of sublayers side by side with
// the chosen experts' outputs), final norm of selected rows, and the gated norms of the recurrent mixers.  The residual stream is
// f32; every kernel that changes it also leaves the input of the next projection: the stream itself, or, in designs with a norm
// ahead of each sublayer, its norm.
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {


__device__ __forceinline__ float4 load_act4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load_act4(const bf16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}

__device__ __forceinline__ float sum_sq(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// The norm that follows a step: x / rms(x) * w, or with `center` the same of x - mean(x); w == null: none
struct Norm {
  const float* w;
  float eps;
  int center;
};

// mean (0 unless centered) and reciprocal deviation of a row that the CTA's threads hold in registers
template <int KEEP>
__device__ __forceinline__ float2 row_stats(const float4 (&v)[KEEP], int nch, int width, const Norm& n, float* s32) {
  float mean = 0.0f, ss = 0.0f;
  if (n.center) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (threadIdx.x + i * blockDim.x < nch) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    mean = block_sum(s, s32) / (float)width;
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if (threadIdx.x + i * blockDim.x < nch) ss += sum_sq(make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean));
  return make_float2(mean, 1.0f / sqrtf(block_sum(ss, s32) / (float)width + n.eps));
}
// the same of a row read through `value(c)`
template <typename V>
__device__ __forceinline__ float2 row_stats(V value, int width, const Norm& n, float* s32) {
  float mean = 0.0f, ss = 0.0f;
  if (n.center) {
    float s = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) s += value(c);
    mean = block_sum(s, s32) / (float)width;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) ss += (value(c) - mean) * (value(c) - mean);
  return make_float2(mean, 1.0f / sqrtf(block_sum(ss, s32) / (float)width + n.eps));
}
__device__ __forceinline__ float4 apply_norm(float4 v, float2 st, float4 g) {
  return make_float4((v.x - st.x) * st.y * g.x, (v.y - st.x) * st.y * g.y, (v.z - st.x) * st.y * g.z, (v.w - st.x) * st.y * g.w);
}

// KEEP in the kernels below: float4 of a row that a thread keeps in registers (0: rows of any width, read again instead).

// x[t] = table[tokens[t]] * scale; h[t] = x[t], or its norm when `next` has a weight.  h may be null.
template <int KEEP, typename H>
__global__ void __launch_bounds__(1024) embed_kernel(const bf16* __restrict__ table, int ld_table, const int* tokens, float scale, int width, float* x,
                                                     H* h, int ldh, Norm next) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const bf16* src = table + (size_t)tokens[t] * ld_table;
  float* xr = x + (size_t)t * width;
  H* hr = h == nullptr ? nullptr : h + (size_t)t * ldh;
  if constexpr (KEEP > 0) {
    const int nch = width >> 2;
    float4 v[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      const uint2 q = c < nch ? reinterpret_cast<const uint2*>(src)[c] : make_uint2(0u, 0u);
      const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
      v[i] = make_float4(lo.x * scale, lo.y * scale, hi.x * scale, hi.y * scale);
      if (c < nch) reinterpret_cast<float4*>(xr)[c] = v[i];
    }
    if (hr == nullptr) return;
    const float2 st = next.w == nullptr ? make_float2(0.0f, 1.0f) : row_stats(v, nch, width, next, s32);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c >= nch) continue;
      if (next.w != nullptr) v[i] = apply_norm(v[i], st, reinterpret_cast<const float4*>(next.w)[c]);
      store_act4(hr + 4 * c, v[i]);
    }
  } else {
    auto value = [&](int c) { return __bfloat162float(src[c]) * scale; };
    const float2 st = next.w == nullptr ? make_float2(0.0f, 1.0f) : row_stats(value, width, next, s32);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const float v = value(c);
      xr[c] = v;
      if (hr != nullptr) store_act(hr + c, next.w != nullptr ? (v - st.x) * st.y * next.w[c] : v);
    }
  }
}

// x += y / sqrt(mean(y^2) + eps) * w; h = x, or its norm with weight `next`
template <int KEEP, typename H>
__global__ void __launch_bounds__(1024) norm_add_kernel(float* x, const float* y, int ldy, const float* __restrict__ w, float eps, int width, H* h, int ldh,
                                                        const float* __restrict__ next) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  float* xr = x + (size_t)blockIdx.x * width;
  const float* yr = y + (size_t)blockIdx.x * ldy;
  H* hr = h == nullptr ? nullptr : h + (size_t)blockIdx.x * ldh;
  float ss = 0.0f, sx = 0.0f;
  if constexpr (KEEP > 0) {
    const int nch = width >> 2;
    float4 v[KEEP], r[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      v[i] = c < nch ? reinterpret_cast<const float4*>(yr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      r[i] = c < nch ? reinterpret_cast<const float4*>(xr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, s32) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nch) {
        const float4 g = reinterpret_cast<const float4*>(w)[c];
        r[i].x += v[i].x * inv * g.x;
        r[i].y += v[i].y * inv * g.y;
        r[i].z += v[i].z * inv * g.z;
        r[i].w += v[i].w * inv * g.w;
        reinterpret_cast<float4*>(xr)[c] = r[i];
        sx += r[i].x * r[i].x + r[i].y * r[i].y + r[i].z * r[i].z + r[i].w * r[i].w;
      }
    }
    if (hr == nullptr) return;
    const float nx = next == nullptr ? 1.0f : 1.0f / sqrtf(block_sum(sx, s32) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c >= nch) continue;
      if (next != nullptr) {
        const float4 g = reinterpret_cast<const float4*>(next)[c];
        r[i] = make_float4(r[i].x * nx * g.x, r[i].y * nx * g.y, r[i].z * nx * g.z, r[i].w * nx * g.w);
      }
      store_act4(hr + 4 * c, r[i]);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += blockDim.x) ss += yr[c] * yr[c];
    const float inv = 1.0f / sqrtf(block_sum(ss, s32) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const float v = xr[c] + yr[c] * inv * w[c];
      xr[c] = v;
      sx += v * v;
    }
    if (hr == nullptr) return;
    const float nx = next == nullptr ? 1.0f : 1.0f / sqrtf(block_sum(sx, s32) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) store_act(hr + c, next == nullptr ? xr[c] : xr[c] * nx * next[c]);
  }
}

// Sublayers side by side: x += mult * (y + sum of the `top` expert rows of the token), h = x or its norm.  at[t * top + k]: row of
// the token's k-th expert in e (their weights are already in them).  counts [experts]: the router's counters, left zero for the
// next layer; may be null.
struct SideBySide {
  float* x;
  const float* y;
  const void* e;
  const int* at;
  int* counts;
  int ldy, lde, top, experts, width;
  float mult;
};

template <int KEEP, typename H, typename E>
__global__ void __launch_bounds__(1024) side_by_side_kernel(SideBySide a, H* h, int ldh, Norm next) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  if (t == 0 && a.counts != nullptr)
    for (int i = threadIdx.x; i < a.experts; i += blockDim.x) a.counts[i] = 0;
  float* xr = a.x + (size_t)t * a.width;
  const float* yr = a.y + (size_t)t * a.ldy;
  H* hr = h == nullptr ? nullptr : h + (size_t)t * ldh;
  const int* at = a.at + (size_t)t * a.top;
  const E* e = static_cast<const E*>(a.e);
  if constexpr (KEEP > 0) {
    const int nch = a.width >> 2;
    float4 v[KEEP], r[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      v[i] = c < nch ? reinterpret_cast<const float4*>(yr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      r[i] = c < nch ? reinterpret_cast<const float4*>(xr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int k = 0; k < a.top; ++k) {
      const E* er = e + (size_t)at[k] * a.lde;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c >= nch) continue;
        const float4 u = load_act4(er + 4 * c);
        v[i].x += u.x; v[i].y += u.y; v[i].z += u.z; v[i].w += u.w;
      }
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      r[i].x += a.mult * v[i].x;
      r[i].y += a.mult * v[i].y;
      r[i].z += a.mult * v[i].z;
      r[i].w += a.mult * v[i].w;
      if (c < nch) reinterpret_cast<float4*>(xr)[c] = r[i];
    }
    if (hr == nullptr) return;
    const float2 st = next.w == nullptr ? make_float2(0.0f, 1.0f) : row_stats(r, nch, a.width, next, s32);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c >= nch) continue;
      if (next.w != nullptr) r[i] = apply_norm(r[i], st, reinterpret_cast<const float4*>(next.w)[c]);
      store_act4(hr + 4 * c, r[i]);
    }
  } else {
    for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
      float v = yr[c];
      for (int k = 0; k < a.top; ++k) v += load_act(e + (size_t)at[k] * a.lde + c);
      xr[c] += a.mult * v;
    }
    if (hr == nullptr) return;
    auto value = [&](int c) { return xr[c]; };     // a thread reads what it wrote
    const float2 st = next.w == nullptr ? make_float2(0.0f, 1.0f) : row_stats(value, a.width, next, s32);
    for (int c = threadIdx.x; c < a.width; c += blockDim.x) store_act(hr + c, next.w == nullptr ? xr[c] : (xr[c] - st.x) * st.y * next.w[c]);
  }
}

// out[i] = norm(x[rows[i]]) * w; rows == null: row i
template <int KEEP, typename OUT>
__global__ void __launch_bounds__(1024) norm_rows_kernel(const float* x, const int* rows, Norm norm, int width, OUT* out, int ld) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  const int row = rows == nullptr ? blockIdx.x : rows[blockIdx.x];
  const float* xr = x + (size_t)row * width;
  OUT* dst = out + (size_t)blockIdx.x * ld;
  if constexpr (KEEP > 0) {
    const int nch = width >> 2;
    float4 v[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      v[i] = c < nch ? reinterpret_cast<const float4*>(xr)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float2 st = row_stats(v, nch, width, norm, s32);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nch) store_act4(dst + 4 * c, apply_norm(v[i], st, reinterpret_cast<const float4*>(norm.w)[c]));
    }
  } else {
    const float2 st = row_stats([&](int c) { return xr[c]; }, width, norm, s32);
    for (int c = threadIdx.x; c < width; c += blockDim.x) store_act(dst + c, (xr[c] - st.x) * st.y * norm.w[c]);
  }
}

// Norm of a recurrent mixer's output in parts of `width` columns (a head, a group of heads, or all of them), with a gate before
// or after it:
//   after:  out = o / rms(o) [* w] * act(gate) * scale          before:  u = o * act(gate), out = u / rms(u) [* w] * scale
// act: sigmoid, or silu.  GT threads per (row, part); KEEP: float4 a thread keeps in registers (0: any width and alignment).
struct GatedNorm {
  const float* o;
  const float* gate;
  const float* w;           // null: no weight
  int ldo, ldg, T, parts, width, ld, silu, before;
  float eps, scale;
};

__device__ __forceinline__ float gate_act(const GatedNorm& a, float g) {
  const float s = sigmoid(g);
  return a.silu ? g * s : s;
}

template <int GT, int KEEP, typename OUT>
__global__ void __launch_bounds__(256) gated_norm_kernel(GatedNorm a, OUT* out) {
  __shared__ float s32[32];
  pdl_wait();
  pdl_trigger();
  constexpr int PER = 256 / GT;
  const int lane = threadIdx.x % GT, item = blockIdx.x * PER + threadIdx.x / GT;
  if (item >= a.T * a.parts) return;       // with GT = 256 the whole CTA
  const int t = item / a.parts, c0 = (item % a.parts) * a.width;
  const float* orow = a.o + (size_t)t * a.ldo + c0;
  const float* grow = a.gate + (size_t)t * a.ldg + c0;
  OUT* dst = out + (size_t)t * a.ld + c0;
  const float* w = a.w == nullptr ? nullptr : a.w + c0;
  auto sum = [&](float v) { return GT == 32 ? warp_sum(v) : block_sum(v, s32); };
  if constexpr (KEEP > 0) {
    const int nch = a.width >> 2;
    float4 v[KEEP], g[KEEP];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = lane + GT * i;
      v[i] = c < nch ? reinterpret_cast<const float4*>(orow)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      g[i] = c < nch ? reinterpret_cast<const float4*>(grow)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      g[i] = make_float4(gate_act(a, g[i].x), gate_act(a, g[i].y), gate_act(a, g[i].z), gate_act(a, g[i].w));
      if (a.before) {
        v[i].x *= g[i].x; v[i].y *= g[i].y; v[i].z *= g[i].z; v[i].w *= g[i].w;
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = a.scale / sqrtf(sum(ss) / (float)a.width + a.eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = lane + GT * i;
      if (c >= nch) continue;
      float4 y = make_float4(v[i].x * inv, v[i].y * inv, v[i].z * inv, v[i].w * inv);
      if (!a.before) {
        y.x *= g[i].x; y.y *= g[i].y; y.z *= g[i].z; y.w *= g[i].w;
      }
      if (w != nullptr) {
        const float4 ww = reinterpret_cast<const float4*>(w)[c];
        y.x *= ww.x; y.y *= ww.y; y.z *= ww.z; y.w *= ww.w;
      }
      store_act4(dst + 4 * c, y);
    }
    return;
  }
  auto value = [&](int c) { return a.before ? orow[c] * gate_act(a, grow[c]) : orow[c]; };
  float ss = 0.0f;
  for (int c = lane; c < a.width; c += GT) {
    const float v = value(c);
    ss += v * v;
  }
  const float inv = a.scale / sqrtf(sum(ss) / (float)a.width + a.eps);
  for (int c = lane; c < a.width; c += GT) {
    float y = value(c) * inv;
    if (!a.before) y *= gate_act(a, grow[c]);
    store_act(dst + c, w == nullptr ? y : y * w[c]);
  }
}

template <typename OUT>
static int run_gated_norm(const GatedNorm& a, OUT* out, cudaStream_t stream) {
  const uintptr_t at = reinterpret_cast<uintptr_t>(a.o) | reinterpret_cast<uintptr_t>(a.gate) | reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(out);
  const bool vec = a.width % 4 == 0 && a.ldo % 4 == 0 && a.ldg % 4 == 0 && a.ld % 4 == 0 && at % 16 == 0;
  const int items = a.T * a.parts;
#define BONSAI_GATED(GT, KEEP) launch(gated_norm_kernel<GT, KEEP, OUT>, dim3((items + 256 / GT - 1) / (256 / GT)), 256, 0, stream, 1, 0, a, out)
  if (a.width <= 512) {
    if (!vec) return BONSAI_GATED(32, 0);
    return a.width <= 128 ? BONSAI_GATED(32, 1) : (a.width <= 256 ? BONSAI_GATED(32, 2) : BONSAI_GATED(32, 4));
  }
  if (!vec || a.width > 4096) return BONSAI_GATED(256, 0);
  return a.width <= 1024 ? BONSAI_GATED(256, 1) : (a.width <= 2048 ? BONSAI_GATED(256, 2) : BONSAI_GATED(256, 4));
#undef BONSAI_GATED
}

static int row_threads(int width) {
  const int t = ((width + 7) / 8 + 31) / 32 * 32;   // two float4 per thread
  return t < 64 ? 64 : (t > 1024 ? 1024 : t);
}

// float4 a thread keeps for rows of `width`, 0 where rows or pointers (or-ed together) are not made of float4
static int row_keep(int width, int ld, uintptr_t pointers) {
  const int th = row_threads(width);
  return width % 4 != 0 || ld % 4 != 0 || pointers % 16 != 0 ? 0 : (width <= 8 * th ? 2 : (width <= 16 * th ? 4 : 0));
}
template <typename... P>
static uintptr_t bits(const P*... p) { return (reinterpret_cast<uintptr_t>(p) | ...); }

#define BONSAI_ROWS(KEEP, KERNEL, H, GRID, ...)                                                       \
  (KEEP == 2 ? launch(KERNEL<2, H>, dim3(GRID), th, 0, stream, 1, 0, __VA_ARGS__)                     \
             : (KEEP == 4 ? launch(KERNEL<4, H>, dim3(GRID), th, 0, stream, 1, 0, __VA_ARGS__)        \
                          : launch(KERNEL<0, H>, dim3(GRID), th, 0, stream, 1, 0, __VA_ARGS__)))

}  // namespace lay
}  // namespace bonsai

extern "C" {

// x f32 [T][width] = table[tokens[t]] * scale (bf16 rows of ld_table elements); h (may be null) [T][ldh], bf16 or f32 = x or, with
// `next`, its norm (center: layer norm)
int bonsai_lay_embed(const void* table, int ld_table, const int* tokens, float scale, int T, int width, float* x, void* h, int ldh, int h_f32,
                     const float* next, float eps, int center, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || width < 1 || ld_table < width || (h != nullptr && ldh < width)) return BONSAI_CUDA_BAD_ARG;
  const int th = row_threads(width), keep = row_keep(width, ld_table | ldh, bits((const char*)table, x, (const char*)h, next));
  const Norm n{next, eps, center};
  return h_f32 ? BONSAI_ROWS(keep, embed_kernel, float, T, (const bf16*)table, ld_table, tokens, scale, width, x, (float*)h, ldh, n)
               : BONSAI_ROWS(keep, embed_kernel, bf16, T, (const bf16*)table, ld_table, tokens, scale, width, x, (bf16*)h, ldh, n);
}

// x += norm(y) * w; h (may be null) = x or, with `next`, its norm
int bonsai_lay_norm_add(float* x, const float* y, int ldy, const float* w, float eps, int T, int width, void* h, int ldh, int h_f32, const float* next,
                        cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || width < 1 || ldy < width || (ldy & 3) != 0 || (h != nullptr && (ldh < width || (ldh & 3) != 0))) return BONSAI_CUDA_BAD_ARG;
  const int th = row_threads(width), keep = row_keep(width, ldy | ldh, bits(x, y, w, (const char*)h, next));
  return h_f32 ? BONSAI_ROWS(keep, norm_add_kernel, float, T, x, y, ldy, w, eps, width, (float*)h, ldh, next)
               : BONSAI_ROWS(keep, norm_add_kernel, bf16, T, x, y, ldy, w, eps, width, (bf16*)h, ldh, next);
}

// x += mult * (y + sum over k < top of e[at[t * top + k]]); e (rows of lde elements) bf16 or f32; h (may be null) = x or, with
// `next`, its norm; counts [experts] (may be null) is left zero
int bonsai_lay_side_by_side(float* x, const float* y, int ldy, const void* e, int lde, int e_f32, const int* at, int top, int* counts, int experts, float mult,
                            int T, int width, void* h, int ldh, int h_f32, const float* next, float eps, int center, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || width < 1 || ldy < width || (h != nullptr && ldh < width) || top < 0 || (top > 0 && (e == nullptr || at == nullptr || lde < width)))
    return BONSAI_CUDA_BAD_ARG;
  const int th = row_threads(width), keep = row_keep(width, ldy | ldh | lde, bits(x, y, (const char*)h, next, (const char*)e));
  const Norm n{next, eps, center};
  const SideBySide a{x, y, e, at, counts, ldy, lde, top, experts, width, mult};
#define BONSAI_SIDE(KEEP, H, E) launch(side_by_side_kernel<KEEP, H, E>, dim3(T), th, 0, stream, 1, 0, a, (H*)h, ldh, n)
#define BONSAI_SIDE_KEEP(H, E) (keep == 2 ? BONSAI_SIDE(2, H, E) : (keep == 4 ? BONSAI_SIDE(4, H, E) : BONSAI_SIDE(0, H, E)))
  if (h_f32) return e_f32 ? BONSAI_SIDE_KEEP(float, float) : BONSAI_SIDE_KEEP(float, bf16);
  return e_f32 ? BONSAI_SIDE_KEEP(bf16, float) : BONSAI_SIDE_KEEP(bf16, bf16);
#undef BONSAI_SIDE_KEEP
#undef BONSAI_SIDE
}

// out: bf16 when f32_out == 0, f32 otherwise
int bonsai_lay_norm_rows(const float* x, const int* rows, const float* w, float eps, int center, int R, int width, void* out, int ld, int f32_out,
                         cudaStream_t stream) {
  using namespace bonsai::lay;
  if (R < 1 || width < 1 || ld < width) return BONSAI_CUDA_BAD_ARG;
  const int th = row_threads(width), keep = row_keep(width, ld, bits(x, w, (const char*)out));
  const Norm n{w, eps, center};
  return f32_out ? BONSAI_ROWS(keep, norm_rows_kernel, float, R, x, rows, n, width, (float*)out, ld)
                 : BONSAI_ROWS(keep, norm_rows_kernel, bf16, R, x, rows, n, width, (bf16*)out, ld);
}

// Gated norm: o and gate f32 [T][ld..] with `parts` parts of `width` columns, w [parts * width] or null; act 0 =
// sigmoid, 1 = silu; before: the gate comes before the norm
int bonsai_lay_gated_norm(const float* o, int ldo, const float* gate, int ldg, const float* w, float eps, int T, int parts, int width, int act, int before,
                          float scale, void* out, int ld, int f32_out, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (T < 1 || parts < 1 || width < 1 || ld < parts * width || (long long)T * parts >= (1ll << 30)) return BONSAI_CUDA_BAD_ARG;
  const GatedNorm a{o, gate, w, ldo, ldg, T, parts, width, ld, act, before, eps, scale};
  return f32_out ? run_gated_norm(a, (float*)out, stream) : run_gated_norm(a, (bf16*)out, stream);
}

}  // extern "C"
