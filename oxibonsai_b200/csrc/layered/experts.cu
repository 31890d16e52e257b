// Mixture of experts: the router's choice, and the experts' projections over the tokens that chose them.
//
//   s = sigmoid(z) or softmax(z), choice = s [+ correction]; only the experts of the `keep` groups with the largest sums of their two
//   best choices are eligible; the `top` best of them get the weights s [/ (sum of the chosen s + den_eps)] * scale.
//
// The pairs (token, chosen expert) are laid out expert by expert: expert e has the sorted rows offsets[e] .. offsets[e + 1] - 1, `token`
// names the token of a sorted row, `weight` its weight and `at` the sorted row of each pair.  A step of few tokens is routed and sorted
// by one CTA; otherwise `route_kernel` counts and `arrange_kernel` sorts and copies the tokens' rows into that order.
//
// Projections: `few_kernel` streams each chosen expert's weights once for up to 32 of its rows (the fragment layout of linear.cu);
// many rows go to the grouped tcgen05 GEMM (cuda/bitgemm_prefill.cu); `f32_kernel` is the 32-bit mode.  The weights are multiplied
// into the experts' hidden units, so the sum over a token's experts is a plain one.
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

constexpr int kMaxExperts = 512, kMaxTop = 32, kSmallPairs = 1024, kSmallTokens = 64;

struct Router {
  const float* z;           // [T][ld], logits at col
  const float* correction;  // [experts]; null: none
  int* counts;              // [experts], zero before a large step's routing
  int* pair;                // [T * top][2]: expert, place among its rows (large steps)
  float* pair_weight;       // [T * top]
  int* lists;               // offsets [experts + 1], number of chosen experts, their list [experts]
  int* token;               // [T * top] by sorted row
  float* weight;            // [T * top] by sorted row
  int* at;                  // [T * top] by pair
  int ld, col, experts, top, groups, keep, T;
  int softmax, divide;      // scores are a softmax over all experts; weights are divided by their sum
  float scale, den_eps;
};

// A warp chooses the experts of one token: lane k < top ends with the k-th one and its weight.  buf: [2 (experts + groups)] floats.
template <int NE>
__device__ __forceinline__ void choose(const Router& a, int t, float* buf, int lane, int& id, float& weight) {
  const float* z = a.z + (size_t)t * a.ld + a.col;
  float* choice = buf;
  float* score = buf + a.experts;
  float* sums = buf + 2 * a.experts;
  float* kept = sums + a.groups;
  float c[NE], most = 0.0f, sum_exp = 1.0f;
  if (a.softmax) {
    most = -INFINITY;
    sum_exp = 0.0f;
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      c[i] = lane + 32 * i < a.experts ? z[lane + 32 * i] : -INFINITY;
      most = fmaxf(most, c[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) most = fmaxf(most, __shfl_xor_sync(0xffffffffu, most, o));
#pragma unroll
    for (int i = 0; i < NE; ++i) sum_exp += expf(c[i] - most);
    sum_exp = warp_sum(sum_exp);
  }
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    const int e = lane + 32 * i;
    c[i] = -INFINITY;
    if (e < a.experts) {
      const float s = a.softmax ? expf(z[e] - most) / sum_exp : sigmoid(z[e]);
      // without a correction or groups, logits choose as their softmax does, and never tie where it underflows
      c[i] = a.correction != nullptr ? s + a.correction[e] : (a.softmax && a.keep == a.groups ? z[e] : s);
      score[e] = s;
      choice[e] = c[i];
    }
  }
  __syncwarp();
  if (a.keep < a.groups) {
    const int size = a.experts / a.groups;
    int lanes = 32;                              // lanes that share a group
    while (lanes > 1 && lanes * a.groups > 32) lanes >>= 1;
    for (int g0 = 0; g0 < a.groups; g0 += 32 / lanes) {
      const int g = g0 + lane / lanes;
      float b1 = -INFINITY, b2 = -INFINITY;
      if (g < a.groups)
        for (int j = lane % lanes; j < size; j += lanes) {
          const float v = choice[g * size + j];
          b2 = fmaxf(b2, fminf(b1, v));
          b1 = fmaxf(b1, v);
        }
      for (int o = lanes >> 1; o > 0; o >>= 1) {
        const float c1 = __shfl_xor_sync(0xffffffffu, b1, o), c2 = __shfl_xor_sync(0xffffffffu, b2, o);
        b2 = fmaxf(fmaxf(b2, c2), fminf(b1, c1));
        b1 = fmaxf(b1, c1);
      }
      if (g < a.groups && lane % lanes == 0) sums[g] = size > 1 ? b1 + b2 : b1;
    }
    __syncwarp();
    for (int g = lane; g < a.groups; g += 32) {
      int better = 0;
      for (int j = 0; j < a.groups; ++j) better += sums[j] > sums[g] || (sums[j] == sums[g] && j < g);
      kept[g] = better < a.keep ? 1.0f : 0.0f;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int e = lane + 32 * i;
      if (e < a.experts && kept[e / size] == 0.0f) c[i] = -INFINITY;
    }
  }
  id = 0;
  weight = 0.0f;
  float sum = 0.0f;
  for (int k = 0; k < a.top; ++k) {
    float v = c[0];
    int e = lane;
#pragma unroll
    for (int i = 1; i < NE; ++i)
      if (c[i] > v) {
        v = c[i];
        e = lane + 32 * i;
      }
    const int bits = __float_as_int(v);          // as an unsigned number of the same order
    const unsigned key = bits < 0 ? ~(unsigned)bits : (unsigned)bits | 0x80000000u;
    e = (int)__reduce_min_sync(0xffffffffu, key == __reduce_max_sync(0xffffffffu, key) ? (unsigned)e : 0x7fffffffu);
    e = min(e, a.experts - 1);
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (e == lane + 32 * i) c[i] = -INFINITY;
    const float s = score[e];
    sum += s;
    if (lane == k) {
      id = e;
      weight = s;
    }
  }
  weight = (a.divide ? weight / (sum + a.den_eps) : weight) * a.scale;
  __syncwarp();
}

// Warp 0: offsets (experts + 1) from counts; `lists` receives them and the chosen experts when given.
__device__ __forceinline__ void prefix(const int* counts, int experts, int* offsets, int* lists, int lane) {
  int total = 0, chosen = 0;
  for (int e0 = 0; e0 < experts; e0 += 32) {
    const int e = e0 + lane, n = e < experts ? counts[e] : 0;
    int v = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += u;
    }
    if (e < experts) offsets[e] = total + v - n;
    const unsigned some = __ballot_sync(0xffffffffu, n > 0);
    if (lists != nullptr) {
      if (e < experts) lists[e] = total + v - n;
      if (n > 0) lists[experts + 2 + chosen + __popc(some & ((1u << lane) - 1u))] = e;
    }
    chosen += __popc(some);
    total += __shfl_sync(0xffffffffu, v, 31);
  }
  if (lane == 0) {
    offsets[experts] = total;
    if (lists != nullptr) {
      lists[experts] = total;
      lists[experts + 1] = chosen;
    }
  }
}

template <int NE>
__global__ void __launch_bounds__(1024) route_small_kernel(Router a, int warps) {
  extern __shared__ float buf[];                 // [warps][2 (experts + groups)]
  __shared__ int s_id[kSmallPairs], s_place[kSmallPairs], s_count[kMaxExperts], s_off[kMaxExperts + 1];
  __shared__ float s_weight[kSmallPairs];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int e = threadIdx.x; e < a.experts; e += 1024) s_count[e] = 0;
  pdl_wait();
  pdl_trigger();
  __syncthreads();
  for (int t = warp; t < a.T && warp < warps; t += warps) {
    int id;
    float w;
    choose<NE>(a, t, buf + warp * 2 * (a.experts + a.groups), lane, id, w);
    if (lane < a.top) {
      const int p = t * a.top + lane;
      s_id[p] = id;
      s_weight[p] = w;
      s_place[p] = atomicAdd(&s_count[id], 1);
    }
  }
  __syncthreads();
  if (warp == 0) prefix(s_count, a.experts, s_off, a.lists, lane);
  __syncthreads();
  for (int p = threadIdx.x; p < a.T * a.top; p += 1024) {
    const int row = s_off[s_id[p]] + s_place[p];
    a.at[p] = row;
    a.token[row] = p / a.top;
    a.weight[row] = s_weight[p];
  }
}

// 8 tokens per CTA
template <int NE>
__global__ void __launch_bounds__(256) route_kernel(Router a) {
  extern __shared__ float buf[];                 // [8 warps][2 (experts + groups)]
  __shared__ int s_count[kMaxExperts], s_base[kMaxExperts];
  __shared__ int s_id[8 * kMaxTop], s_place[8 * kMaxTop];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t0 = blockIdx.x * 8, n = min(8, a.T - t0);
  for (int e = threadIdx.x; e < a.experts; e += 256) s_count[e] = 0;
  pdl_wait();
  pdl_trigger();
  __syncthreads();
  if (warp < n) {
    int id;
    float w;
    choose<NE>(a, t0 + warp, buf + warp * 2 * (a.experts + a.groups), lane, id, w);
    if (lane < a.top) {
      s_id[warp * a.top + lane] = id;
      s_place[warp * a.top + lane] = atomicAdd(&s_count[id], 1);
      a.pair_weight[(size_t)(t0 + warp) * a.top + lane] = w;
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < a.experts; e += 256)
    if (s_count[e] > 0) s_base[e] = atomicAdd(&a.counts[e], s_count[e]);
  __syncthreads();
  for (int p = threadIdx.x; p < n * a.top; p += 256)
    reinterpret_cast<int2*>(a.pair)[(size_t)t0 * a.top + p] = make_int2(s_id[p], s_base[s_id[p]] + s_place[p]);
}

// 8 tokens per CTA; xs (may be null): the tokens' rows of h (chunks of 8 elements) in sorted order
__global__ void __launch_bounds__(256) arrange_kernel(Router a, const bf16* h, int ldh, int chunks, bf16* xs, int ldx) {
  __shared__ int s_off[kMaxExperts + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * 8 + warp;
  pdl_wait();
  pdl_trigger();
  if (warp == 0) prefix(a.counts, a.experts, s_off, blockIdx.x == 0 ? a.lists : nullptr, lane);
  __syncthreads();
  if (t >= a.T) return;
  int row = -1;
  if (lane < a.top) {
    const size_t p = (size_t)t * a.top + lane;
    const int2 v = reinterpret_cast<const int2*>(a.pair)[p];
    row = min(max(s_off[v.x] + v.y, 0), a.T * a.top - 1);        // in range whatever the counters held
    a.at[p] = row;
    a.token[row] = t;
    a.weight[row] = a.pair_weight[p];
  }
  if (xs == nullptr) return;
  const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)t * ldh);
  for (int i0 = 0; i0 < chunks; i0 += 128) {
    uint4 v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (i0 + 32 * j + lane < chunks) v[j] = src[i0 + 32 * j + lane];
    for (int k = 0; k < a.top; ++k) {
      uint4* dst = reinterpret_cast<uint4*>(xs + (size_t)__shfl_sync(0xffffffffu, row, k) * ldx);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (i0 + 32 * j + lane < chunks) dst[i0 + 32 * j + lane] = v[j];
    }
  }
}

// ---- projections ----------------------------------------------------------------------------------------------------------------
struct Grouped {
  const bf16* W;            // [experts][n][kp]
  const int* lists;         // as above
  const int* token;         // input row of a sorted row; null: the sorted row itself
  const float* weight;      // gated epilogue: factor of a sorted row's outputs
  int n, k, kp, experts, rows;   // rows: sorted rows in all
  int ldx, ldo, glu;        // glu: the gated epilogue over interleaved gate / up rows
  Glu unit;
};

constexpr int kFewWarps = 8;

// grid (16 weight rows, chosen experts): NT groups of 8 rows at a time
template <int NT>
__global__ void __launch_bounds__(kFewWarps * 32) few_kernel(Grouped a, const bf16* x, float* out, bf16* out16) {
  constexpr int LD = 8 * NT + 1;
  __shared__ float red[kFewWarps][16][LD];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  pdl_wait();
  pdl_trigger();
  if ((int)blockIdx.y >= a.lists[a.experts + 1]) return;
  const int e = a.lists[a.experts + 2 + blockIdx.y], first = a.lists[e], last = min(a.lists[e + 1], a.rows);
  const int row0 = blockIdx.x * 16, chunks = a.kp >> 7;
  const bf16* w0 = a.W + ((size_t)e * a.n + min(row0 + g, a.n - 1)) * a.kp + 8 * t4;
  const bf16* w1 = a.W + ((size_t)e * a.n + min(row0 + g + 8, a.n - 1)) * a.kp + 8 * t4;
  for (int s0 = first; s0 < last; s0 += 8 * NT) {
    const int cnt = min(8 * NT, last - s0);
    uint4 wa[4], wb[4];
    auto load_w = [&](int c) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        wa[i] = *reinterpret_cast<const uint4*>(w0 + c * 128 + i * 32);
        wb[i] = *reinterpret_cast<const uint4*>(w1 + c * 128 + i * 32);
      }
    };
    if (warp < chunks) load_w(warp);
    const bf16* xr[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int s = s0 + min(8 * j + g, cnt - 1);
      xr[j] = x + (size_t)(a.token == nullptr ? s : a.token[s]) * a.ldx + 8 * t4;
    }
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
    for (int c = warp; c < chunks; c += kFewWarps) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t lo[4] = {wa[i].x, wb[i].x, wa[i].y, wb[i].y}, hi[4] = {wa[i].z, wb[i].z, wa[i].w, wb[i].w};
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          if (8 * j >= cnt) continue;
          const uint4 v = *reinterpret_cast<const uint4*>(xr[j] + c * 128 + i * 32);
          mma_bf16(acc[j], lo, v.x, v.y);
          mma_bf16(acc[j], hi, v.z, v.w);
        }
      }
      if (c + kFewWarps < chunks) load_w(c + kFewWarps);
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      red[warp][g][8 * j + 2 * t4] = acc[j][0];
      red[warp][g][8 * j + 2 * t4 + 1] = acc[j][1];
      red[warp][g + 8][8 * j + 2 * t4] = acc[j][2];
      red[warp][g + 8][8 * j + 2 * t4 + 1] = acc[j][3];
    }
    __syncthreads();
    if (!a.glu) {
      for (int i = threadIdx.x; i < 16 * cnt; i += kFewWarps * 32) {
        const int r = i & 15, t = i >> 4;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kFewWarps; ++w) v += red[w][r][t];
        if (row0 + r < a.n) out[(size_t)(s0 + t) * a.ldo + row0 + r] = v;
      }
    } else {
      for (int i = threadIdx.x; i < 8 * cnt; i += kFewWarps * 32) {
        const int r = i & 7, t = i >> 3;
        float gv = 0.0f, uv = 0.0f;
#pragma unroll
        for (int w = 0; w < kFewWarps; ++w) {
          gv += red[w][2 * r][t];
          uv += red[w][2 * r + 1][t];
        }
        if (row0 + 2 * r + 1 < a.n) out16[(size_t)(s0 + t) * a.ldo + (row0 >> 1) + r] = __float2bfloat16_rn(glu(a.unit, gv, uv) * a.weight[s0 + t]);
      }
    }
    __syncthreads();     // the partial sums are read before the next rows overwrite them
  }
}

// grid (64 weight rows, 64 sorted rows of an expert, experts), 256 threads with 4 x 4 outputs each
__global__ void __launch_bounds__(256) expert_f32_kernel(Grouped a, const float* x, float* out) {
  __shared__ float sw[16][68], sx[16][68];
  pdl_wait();
  pdl_trigger();
  const int e = blockIdx.z, first = a.lists[e] + blockIdx.y * 64, last = min(a.lists[e + 1], a.rows), n0 = blockIdx.x * 64;
  if (first >= last) return;
  const bf16* W = a.W + (size_t)e * a.n * a.kp;
  const int tn = threadIdx.x & 15, tt = threadIdx.x >> 4;
  const float* xrow[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int s = min(first + ((threadIdx.x + i * 256) >> 4), last - 1);
    xrow[i] = x + (size_t)(a.token == nullptr ? s : a.token[s]) * a.ldx;
  }
  float acc[4][4] = {};   // [sorted row][weight row]
  for (int k0 = 0; k0 < a.k; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256, r = idx >> 4, c = idx & 15;
      const bool kin = k0 + c < a.k;
      sw[c][r] = kin && n0 + r < a.n ? __bfloat162float(W[(size_t)(n0 + r) * a.kp + k0 + c]) : 0.0f;
      sx[c][r] = kin && first + r < last ? xrow[i][k0 + c] : 0.0f;
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
    const int s = first + tt * 4 + i;
    if (s >= last) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = n0 + tn * 4 + j;
      if (!a.glu) {
        if (r < a.n) out[(size_t)s * a.ldo + r] = acc[i][j];
      } else if ((j & 1) == 0 && r + 1 < a.n) {
        out[(size_t)s * a.ldo + (r >> 1)] = glu(a.unit, acc[i][j], acc[i][j + 1]) * a.weight[s];
      }
    }
  }
}

static bool fill(Router& a, const void* const* ptrs, const int* ints, const float* floats, int T) {
  a.z = (const float*)ptrs[0]; a.correction = (const float*)ptrs[1]; a.counts = (int*)ptrs[2]; a.pair = (int*)ptrs[3]; a.pair_weight = (float*)ptrs[4];
  a.lists = (int*)ptrs[5]; a.token = (int*)ptrs[6]; a.weight = (float*)ptrs[7]; a.at = (int*)ptrs[8];
  a.ld = ints[0]; a.col = ints[1]; a.experts = ints[2]; a.top = ints[3]; a.groups = ints[4]; a.keep = ints[5]; a.T = T;
  a.softmax = ints[6]; a.divide = ints[7]; a.scale = floats[0]; a.den_eps = floats[1];
  return T >= 1 && a.experts >= 1 && a.experts <= kMaxExperts && a.top >= 1 && a.top <= kMaxTop && a.groups >= 1 && a.experts % a.groups == 0 && a.keep >= 1 &&
         a.keep <= a.groups && a.top <= a.keep * (a.experts / a.groups) && (long long)T * a.top < (1ll << 30);
}

#define BONSAI_BY_EXPERTS(CALL)                                                                       \
  (a.experts <= 32 ? CALL(1)                                                                          \
                   : (a.experts <= 64 ? CALL(2) : (a.experts <= 128 ? CALL(4) : (a.experts <= 256 ? CALL(8) : CALL(16)))))

}  // namespace lay
}  // namespace bonsai

extern "C" {

// tokens that one CTA routes and sorts by itself
int bonsai_lay_route_small(int top) { return top < 1 || top > bonsai::lay::kMaxTop ? 0 : min(bonsai::lay::kSmallTokens, bonsai::lay::kSmallPairs / top); }

// Chooses and sorts.  ptrs = {logits, correction, counts, pair, pair_weight, lists, token, weight, at}, ints = {ld, col, experts, top,
// groups, keep, softmax, divide}, floats = {scale, den_eps}.  h bf16 [T][ldh] -> xs [T * top][ldx] in sorted order, `chunks` blocks of 8 columns (xs
// null: no copy).  Steps above bonsai_lay_route_small tokens need counts at zero (bonsai_lay_side_by_side leaves them so).
int bonsai_lay_route(const void* const* ptrs, const int* ints, const float* floats, int T, const void* h, int ldh, int chunks, void* xs, int ldx,
                     cudaStream_t stream) {
  using namespace bonsai::lay;
  Router a;
  if (!fill(a, ptrs, ints, floats, T)) return BONSAI_CUDA_BAD_ARG;
  const size_t buf = 2 * (a.experts + a.groups) * sizeof(float);
  if (xs == nullptr && T <= bonsai_lay_route_small(a.top)) {
    const int warps = min(min(T, 32), (int)(160 * 1024 / buf));
#define BONSAI_SMALL(NE) launch(route_small_kernel<NE>, dim3(1), 1024, warps * buf, stream, 1, 0, a, warps)
    return BONSAI_BY_EXPERTS(BONSAI_SMALL);
#undef BONSAI_SMALL
  }
  if (xs != nullptr && (chunks < 1 || ldh % 8 != 0 || ldx % 8 != 0 || ldh < 8 * chunks || ldx < 8 * chunks)) return BONSAI_CUDA_BAD_ARG;
#define BONSAI_LARGE(NE) launch(route_kernel<NE>, dim3((T + 7) / 8), 256, 8 * buf, stream, 1, 0, a)
  const int st = BONSAI_BY_EXPERTS(BONSAI_LARGE);
#undef BONSAI_LARGE
  if (st != BONSAI_CUDA_OK) return st;
  return launch(arrange_kernel, dim3((T + 7) / 8), 256, 0, stream, 1, 0, a, (const bf16*)h, ldh, chunks, (bf16*)xs, ldx);
}

// Projection of the sorted rows by their experts' matrices W [experts][n][kp], few rows per expert.  x bf16 (row token[s], or s when
// token is null); glu: out bf16 [rows][n / 2] = gated unit * weight[s]; otherwise out f32 [rows][n].  slots: most experts chosen.
int bonsai_lay_experts_few(const void* W, int experts, int n, int kp, const void* x, int ldx, const int* lists, const int* token, const float* weight, int rows,
                           int slots, int per_expert, void* out, int ldo, int glu, float limit, float alpha, float offset, float cubic, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (experts < 1 || experts > kMaxExperts || n < 1 || kp < 128 || kp % 128 != 0 || ldx < kp || ldx % 8 != 0 || rows < 1 || slots < 1 || slots > experts ||
      ldo < (glu ? n / 2 : n) || (glu && (n % 2 != 0 || weight == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  const Grouped a{(const bf16*)W, lists, token, weight, n, kp, kp, experts, rows, ldx, ldo, glu, Glu{limit, alpha, offset, cubic}};
  const dim3 grid((n + 15) / 16, slots);
#define BONSAI_FEW(NT) launch(few_kernel<NT>, grid, kFewWarps * 32, 0, stream, 1, 0, a, (const bf16*)x, (float*)out, (bf16*)out)
  return per_expert <= 8 ? BONSAI_FEW(1) : (per_expert <= 16 ? BONSAI_FEW(2) : BONSAI_FEW(4));
#undef BONSAI_FEW
}

// The same in 32 bits: x and out f32, at most `tokens` rows per expert.
int bonsai_lay_experts_f32(const void* W, int experts, int n, int k, int kp, const float* x, int ldx, const int* lists, const int* token, const float* weight,
                           int rows, int tokens, float* out, int ldo, int glu, float limit, float alpha, float offset, float cubic, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (experts < 1 || experts > kMaxExperts || n < 1 || k < 1 || kp < k || ldx < k || rows < 1 || tokens < 1 || tokens > 64 * 65535 ||
      ldo < (glu ? n / 2 : n) || (glu && (n % 2 != 0 || weight == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  const Grouped a{(const bf16*)W, lists, token, weight, n, k, kp, experts, rows, ldx, ldo, glu, Glu{limit, alpha, offset, cubic}};
  return launch(expert_f32_kernel, dim3((n + 63) / 64, (tokens + 63) / 64, experts), 256, 0, stream, 1, 0, a, x, out);
}

}  // extern "C"
