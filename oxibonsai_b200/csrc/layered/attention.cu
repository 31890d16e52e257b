// Attention of the layer-list decoders over a paged cache.  Every part is a parameter that a design may leave out:
//
//   score(i, j) = cap(q'_i . k'_j) - slope_h (i - j)       j <= i and (i - j < window, or i and j in one chunk, or j < keep)
//   out         = softmax(score) V * sigmoid(gate) * out_scale       [denominator + e^(sink_h)], one gate per head or per element
//
// with q' = rot(norm(q) [* w_q]) * scale [* (1 + coef ln(floor((i + 1) / every) + 1))], k' = rot(norm(k) [* w_k]) and
// cap(s) = s or c tanh(s / c); norm divides by the root mean square, rot turns pairs of dimensions by angles of the position.
// Projections may come without their biases, which are then added where a value is read.
//
// MAPS = 2, differential attention: every head has two queries and two keys [map 1 | map 2] over the same values, and with the two
// maps' outputs a1 and a2
//   o = a1 - lambda a2,    out = o / rms(o) * diff_scale * sigmoid(gate) * out_scale
// A key row holds both maps' keys, each in its half.
//
// Two kinds of cache rows (template parameter SEP):
//  * one row per token that is both key and value (designs whose values are the un-normalised keys): the row holds the projected
//    key, a float beside it the reciprocal root mean square, which multiplies the scores of its column.  Half the cache traffic
//    of separate rows, and a tile is staged once for S = Q K^T and O = P K;
//  * SEP: a row of finished keys and a row of values, both padded to the same row length.  Scores are capped, heads rotated and rows
//    of another layer used (k_col < 0: nothing is appended) only here.  Norm weights are applied to each side; with shared rows their
//    product is folded into the query.
//
// Rows of a batch are tokens: a row has a position and a slot (its sequence's block-table row).  `append_kernel` writes the
// rows' keys; `prompt_kernel` handles portions of prompts (tiles of 64 query rows = tokens x heads of one kv group; with two maps
// four warps have the rows of one, four those of the other); `decode_kernel` single tokens, whose append it does itself (a map is a
// query row of its own, zero in the other map's half); `f32_kernel` is the 32-bit mode for both.
// Only the page tiles that a window or a chunk can see are visited: the kept first tokens and the range behind its first position.
#include <cooperative_groups.h>
#include <type_traits>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

struct Attn {
  const float* proj;        // [T][ld]: q heads at q_col, k heads at k_col, one gate per head at g_col
  const float* q_norm;      // [dim]; null: no norm weights
  const float* k_norm;      // [dim]
  const float* q_bias;      // [heads * MAPS * dim]; null: none (the other two likewise)
  const float* k_bias;
  const float* v_bias;
  const float* slopes;      // [heads]; null: no distance bias
  const float* sinks;       // [heads]; null: no sink
  const float2* rot;        // [positions][rot_dims / 2] cosines and sines; null: no rotation
  const int* pos;           // [T]
  const int* slots;         // [T]
  const int* block_table;   // [slots][max_pages]
  void* pool;               // [pages][kv_heads][page_size][HD], bf16 (f32 in the 32-bit mode), columns past dim zero
  float* krms;              // [pages][kv_heads][page_size]; SEP: unused
  void* vpool;              // SEP: value rows, laid out like the pool
  void* out;                // [T][ldo], head h at h * vdim
  int ld, q_col, k_col, v_col, g_col, ldo;       // g_col < 0: no gate; k_col < 0: another layer appends the rows
  int heads, kv_heads, dim, vdim, max_pages, pshift;   // page size 1 << pshift
  int window, chunk, keep;  // <= 0: no window, no chunks
  int normed;               // queries and keys are divided by their root mean square
  int rot_dims, rot_pairs;  // rotated dimensions; pairs (2i, 2i + 1) instead of (i, i + rot_dims / 2)
  float eps, scale, out_scale;
  float softcap;            // <= 0: scores are not capped
  float temp_coef, temp_every;   // query temperature; coef 0: none
  int maps, gate_wide;      // gate_wide: a gate per output element
  float lambda, diff_scale; // two maps
};

// Calls f with "biases" and "norm weights" as types: code whose loads depend on neither at run time (a branch around a load keeps it
// from being issued with the others).  Two maps have both, shared rows no biases.
template <bool SEP, int MAPS, typename F>
__device__ __forceinline__ void with_flags(bool bias, bool norm, F f) {
  using Y = std::true_type;
  using N = std::false_type;
  if constexpr (MAPS == 2) {
    f(Y(), Y());
  } else {
    if constexpr (SEP) {
      if (bias) {
        if (norm) f(Y(), Y());
        else f(Y(), N());
        return;
      }
    }
    if (norm) f(N(), Y());
    else f(N(), N());
  }
}
__device__ __forceinline__ float biased(const float* p, const float* b, int i) { return b == nullptr ? p[i] : p[i] + b[i]; }

__device__ __forceinline__ float temperature(const Attn& a, int pos) {
  return a.temp_coef == 0.0f ? 1.0f : 1.0f + a.temp_coef * logf(floorf((float)(pos + 1) / a.temp_every) + 1.0f);
}
// factor of a head's outputs, and that of one element where gates are per element
__device__ __forceinline__ float gate(const Attn& a, size_t t, int head) {
  return a.g_col < 0 || a.gate_wide ? a.out_scale : a.out_scale * sigmoid(a.proj[t * a.ld + a.g_col + head]);
}
__device__ __forceinline__ float wide_gate(const Attn& a, size_t t, int head, int d) {
  return a.gate_wide ? sigmoid(a.proj[t * a.ld + a.g_col + head * a.vdim + d]) : 1.0f;
}
__device__ __forceinline__ const float2* angles(const Attn& a, int pos) { return a.rot == nullptr ? nullptr : a.rot + (size_t)pos * (a.rot_dims >> 1); }
// Scores arrive as base-2 logarithms, or with a cap as x = 2 log2(e) score / cap: cap * tanh(score / cap) * log2(e) from one
// exponential, tanh(y) = 1 - 2 / (e^2y + 1).
__device__ __forceinline__ float cap_score(float x, float cap_log2e) { return cap_log2e - __fdividef(2.0f * cap_log2e, ex2(x) + 1.0f); }

// first visible position outside the kept ones for a query at `p`
__device__ __forceinline__ int window_lo(const Attn& a, int p) {
  return a.window > 0 ? max(0, p - a.window + 1) : (a.chunk > 0 ? p - p % a.chunk : 0);
}
// position i, whose first visible one is lo, sees j
__device__ __forceinline__ bool sees(const Attn& a, int i, int lo, int j) { return j <= i && (j >= lo || j < a.keep); }
__device__ __forceinline__ size_t cache_row(const Attn& a, const int* bt, int kvh, int t) {
  return ((((size_t)bt[t >> a.pshift] * a.kv_heads + kvh) << a.pshift)) + (t & ((1 << a.pshift) - 1));
}

// A warp writes one token's row of kv head kvh: the key and its reciprocal root mean square, or the normalised key and the value.
template <int HD, bool SEP, int MAPS, typename C>
__device__ __forceinline__ void append_row(const Attn& a, const float* proj, int kvh, int pos, size_t row, int lane) {
  constexpr int KD = HD / MAPS;
  C* dst = static_cast<C*>(a.pool) + row * HD;
  const float* k = proj + a.k_col + kvh * MAPS * a.dim;
  if constexpr (SEP) {
    with_flags<SEP, MAPS>(a.k_bias != nullptr, a.k_norm != nullptr, [&](auto bias, auto norm) {
      constexpr bool BIAS = decltype(bias)::value, NORM = decltype(norm)::value;
      const float* v = proj + a.v_col + kvh * a.vdim;
      const float* vb = a.v_bias + kvh * a.vdim;
      C* vdst = static_cast<C*>(a.vpool) + row * HD;
      const float2* rot = angles(a, pos);
      float x[HD / 32], y[HD / 32], ss[MAPS];
#pragma unroll
      for (int m = 0; m < MAPS; ++m) ss[m] = 0.0f;
#pragma unroll
      for (int i = 0; i < HD / 32; ++i) {            // every load ahead of the first store
        const int c = lane + 32 * i, m = c / KD, d = c % KD;
        const float* km = k + m * a.dim;
        const float* kb = a.k_bias + (kvh * MAPS + m) * a.dim;
        auto raw = [&](int j) { return BIAS ? km[j] + kb[j] : km[j]; };
        float r = 0.0f;
        x[i] = 0.0f;
        if (d < a.dim) {
          r = raw(d);
          x[i] = rotated([&](int j) { return NORM ? raw(j) * a.k_norm[j] : raw(j); }, d, rot, a.rot_dims, a.rot_pairs);
        }
        y[i] = c < a.vdim ? (BIAS ? v[c] + vb[c] : v[c]) : 0.0f;
#pragma unroll
        for (int j = 0; j < MAPS; ++j) ss[j] += MAPS == 1 || m == j ? r * r : 0.0f;
      }
      float inv[MAPS];
#pragma unroll
      for (int m = 0; m < MAPS; ++m) inv[m] = a.normed ? 1.0f / sqrtf(warp_sum(ss[m]) / (float)a.dim + a.eps) : 1.0f;
#pragma unroll
      for (int i = 0; i < HD / 32; ++i) {
        store_act(dst + lane + 32 * i, x[i] * (MAPS == 1 || lane + 32 * i < KD ? inv[0] : inv[MAPS - 1]));
        store_act(vdst + lane + 32 * i, y[i]);
      }
    });
    return;
  }
  float ss = 0.0f;
#pragma unroll
  for (int d = lane; d < HD; d += 32) {
    const float v = d < a.dim ? k[d] : 0.0f;
    store_act(dst + d, v);
    ss += v * v;
  }
  ss = warp_sum(ss);
  if (lane == 0) a.krms[row] = 1.0f / sqrtf(ss / (float)a.dim + a.eps);
}

// grid (row groups of 4 x kv head): one warp per (row of the list, kv head)
template <int HD, bool SEP, int MAPS, typename C>
__global__ void append_kernel(Attn a, int first, int count) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, i = blockIdx.x * 4 + (threadIdx.x >> 5), kvh = blockIdx.y;
  if (i >= count) return;
  const int t = first + i;
  if (a.pos[t] >= (a.max_pages << a.pshift)) return;
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  append_row<HD, SEP, MAPS, C>(a, a.proj + (size_t)t * a.ld, kvh, a.pos[t], cache_row(a, bt, kvh, a.pos[t]), lane);
}

// weight of a query dimension: its own, and with shared rows the key's too
template <bool SEP>
__device__ __forceinline__ float query_weight(const Attn& a, int d) {
  return SEP ? a.q_norm[d] : a.q_norm[d] * a.k_norm[d];
}

// A warp normalises queries of a kv head and leaves q' * log2(e) in rows of dst (columns past dim zero): scores are base-2 logarithms; with
// a cap, q' * 2 log2(e) / cap.  place(r) names row r's projections, head, map, position and destination; rows r0, r0 + step, ..
// below r1, UN of them at a time.
struct QueryRow {
  const float* proj;
  int head, map, pos;
  bf16* dst;
};
template <int KD, bool SEP, int MAPS, int UN, typename P>
__device__ __forceinline__ void load_queries(const Attn& a, int r0, int r1, int step, P place, int lane) {
  with_flags<SEP, MAPS>(a.q_bias != nullptr, a.q_norm != nullptr, [&](auto bias, auto norm) {
    constexpr bool BIAS = decltype(bias)::value, NORM = decltype(norm)::value;
    constexpr int N = (KD + 31) / 32;
    for (int r = r0; r < r1; r += UN * step) {
      float v[UN][N], ss[UN];
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        const QueryRow row = place(min(r + u * step, r1 - 1));
        const float2* rot = angles(a, row.pos);
        const float* q = row.proj + a.q_col + (row.head * MAPS + row.map) * a.dim;
        const float* qb = a.q_bias + (row.head * MAPS + row.map) * a.dim;
        auto raw = [&](int j) { return BIAS ? q[j] + qb[j] : q[j]; };
        ss[u] = 0.0f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
          const int d = lane + 32 * i;
          float x = 0.0f;
          v[u][i] = 0.0f;
          if (d < KD && d < a.dim) {
            x = raw(d);
            v[u][i] = rotated([&](int j) { return NORM ? raw(j) * query_weight<SEP>(a, j) : raw(j); }, d, rot, a.rot_dims, a.rot_pairs);
          }
          ss[u] += x * x;
        }
      }
#pragma unroll
      for (int u = 0; u < UN; ++u) {
        if (r + u * step >= r1) break;
        const QueryRow row = place(r + u * step);
        const float f = a.scale * temperature(a, row.pos) * (a.softcap > 0.0f ? 2.0f * kLog2e / a.softcap : kLog2e) /
                        (a.normed ? sqrtf(warp_sum(ss[u]) / (float)a.dim + a.eps) : 1.0f);
#pragma unroll
        for (int i = 0; i < N; ++i)
          if (KD % 32 == 0 || lane + 32 * i < KD) row.dst[lane + 32 * i] = __float2bfloat16_rn(v[u][i] * f);
      }
    }
  });
}

// Row r (0 or 1) of a thread's accumulators times f and the gates of its head: out[t] for columns nt * 8 + 2 (lane & 3) and the next.
template <int HD>
__device__ __forceinline__ void store_row(const Attn& a, const float (&o)[HD / 8][4], int r, float f, size_t t, int head, int lane) {
  bf16* dst = static_cast<bf16*>(a.out) + t * a.ldo + head * a.vdim + (lane & 3) * 2;
  const bool pairs = ((a.vdim | a.ldo | (int)(reinterpret_cast<uintptr_t>(a.out) >> 1)) & 1) == 0;
  const int left = a.vdim - (lane & 3) * 2;
  auto store = [&](int nt, float x, float y) {
    if (pairs) {
      if (nt * 8 < left) *reinterpret_cast<uint32_t*>(dst + nt * 8) = pack_bf16(x, y);
    } else {
      if (nt * 8 < left) dst[nt * 8] = __float2bfloat16_rn(x);
      if (nt * 8 + 1 < left) dst[nt * 8 + 1] = __float2bfloat16_rn(y);
    }
  };
  if (!a.gate_wide) {
#pragma unroll
    for (int nt = 0; nt < HD / 8; ++nt) store(nt, o[nt][2 * r] * f, o[nt][2 * r + 1] * f);
    return;
  }
  const float* g = a.proj + t * a.ld + a.g_col + head * a.vdim + (lane & 3) * 2;
#pragma unroll
  for (int n0 = 0; n0 < HD / 8; n0 += 4) {
    float gv[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      gv[i][0] = (n0 + i) * 8 < left ? g[(n0 + i) * 8] : 0.0f;
      gv[i][1] = (n0 + i) * 8 + 1 < left ? g[(n0 + i) * 8 + 1] : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) store(n0 + i, o[n0 + i][2 * r] * f * sigmoid(gv[i][0]), o[n0 + i][2 * r + 1] * f * sigmoid(gv[i][1]));
  }
}

// ---- portions of prompts ------------------------------------------------------------------------------------------------------
// entries[e] = {first row, tokens, slot, first position}; tiles[i] = {entry, first token of the tile}.  A tile holds
// 64 / G tokens x the G query heads of one kv head.
template <int HD, bool SEP, int MAPS>
__global__ void __launch_bounds__(128 * MAPS) prompt_kernel(Attn a, const int4* entries, const int2* tiles) {
  constexpr int LD = HD + 8, KD = HD / MAPS, NTH = 128 * MAPS;
  constexpr bool kQReg = KD <= 128;   // query fragments stay in registers (else they are re-read from shared memory)
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);
  bf16* sK = sQ + 64 * LD;            // two stages of [64][LD]
  bf16* sV = sK + 2 * 64 * LD;        // SEP: two stages of [64][LD]
  float* sR = reinterpret_cast<float*>(sK + 2 * 64 * LD);   // otherwise two stages of 64 key factors
  const int kvh = blockIdx.x, lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, map = MAPS == 1 ? 0 : threadIdx.x >> 7;
  const int G = a.heads / a.kv_heads, tpt = 64 / G;
  pdl_wait();
  pdl_trigger();
  const int2 tl = tiles[gridDim.y - 1 - blockIdx.y];
  const int4 en = entries[tl.x];
  const int q0 = tl.y, ntok = min(tpt, en.y - q0), rows = ntok * G;
  const int pfirst = en.w + q0, plast = pfirst + ntok - 1;
  const int lo = window_lo(a, pfirst), hi = plast + 1;
  const int* bt = a.block_table + (size_t)en.z * a.max_pages;
  const bf16* pool = static_cast<const bf16*>(a.pool);

  auto fetch = [&](int kb, int st) {
    bf16* dst = sK + st * 64 * LD;
#pragma unroll 4
    for (int i = threadIdx.x; i < 64 * (HD / 8); i += NTH) {
      const int r = i / (HD / 8), c = (i % (HD / 8)) * 8, t = kb + r;
      const bool ok = t < hi;
      const size_t at = ok ? cache_row(a, bt, kvh, t) * HD + c : 0;
      cp_async16(dst + r * LD + c, pool + at, ok);
      if (SEP) cp_async16(sV + st * 64 * LD + r * LD + c, static_cast<const bf16*>(a.vpool) + at, ok);
    }
    if (!SEP && threadIdx.x < 64) sR[st * 64 + threadIdx.x] = kb + threadIdx.x < hi ? a.krms[cache_row(a, bt, kvh, kb + threadIdx.x)] : 0.0f;
  };
  // key tiles: those that hold kept tokens, then those of the window's range
  auto next = [&](int kb) {
    kb += 64;
    if (kb >= a.keep && kb + 64 <= lo) kb = lo & ~63;
    return kb;
  };
  int kb = next(-64);
  fetch(kb, 0);
  cp_async_commit();
  const int r0 = warp * 16, r1 = min(rows, r0 + 16);     // a warp loads its own rows and map
  load_queries<KD, SEP, MAPS, 4>(a, r0, r1, 1, [&](int r) {
    return QueryRow{a.proj + (size_t)(en.x + q0 + r / G) * a.ld, kvh * G + r % G, map, pfirst + r / G, sQ + r * LD + map * KD};
  }, lane);
  for (int r = max(r0, r1); r < r0 + 16; ++r)
    for (int d = lane; d < KD; d += 32) sQ[r * LD + map * KD + d] = __float2bfloat16_rn(0.0f);
  __syncwarp();
  uint32_t qf[kQReg ? KD / 16 : 1][4];
  if (kQReg) {
#pragma unroll
    for (int ks = 0; ks < (kQReg ? KD / 16 : 1); ++ks) ldsm4(qf[ks], frag_a(sQ, LD, warp * 16, map * KD + ks * 16, lane));
  }
  float o[HD / 8][4];
#pragma unroll
  for (int i = 0; i < HD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  int row[2], qpos[2], qlo[2], head[2];
  float slope[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    row[e] = warp * 16 + (lane >> 2) + 8 * e;
    qpos[e] = row[e] < rows ? pfirst + row[e] / G : -1;      // rows past the tile see nothing
    qlo[e] = window_lo(a, max(0, qpos[e]));
    head[e] = kvh * G + row[e] % G;
    slope[e] = a.slopes == nullptr ? 0.0f : a.slopes[head[e]] * kLog2e;
  }
  const int wfirst = pfirst + warp * 16 / G, wlast = min(plast, pfirst + (warp * 16 + 15) / G);   // positions of this warp's rows
  const bool wlive = warp * 16 + 15 < rows;
  const int wlo = window_lo(a, wlast);
  const float cap = a.softcap * kLog2e;
  for (int it = 0; kb < hi; ++it) {
    const int nx = next(kb);
    if (nx < hi) fetch(nx, (it + 1) & 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const bf16* k = sK + (it & 1) * 64 * LD;
    const bf16* v = SEP ? sV + (it & 1) * 64 * LD : k;
    const float* kr = sR + (it & 1) * 64;
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < KD / 16; ++ks) {
      uint32_t qt[4];
      if (!kQReg) ldsm4(qt, frag_a(sQ, LD, warp * 16, map * KD + ks * 16, lane));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        ldsm4(b, frag_b_rows(k, LD, np * 16, map * KD + ks * 16, lane));
        mma_bf16(s[2 * np], kQReg ? qf[kQReg ? ks : 0] : qt, b[0], b[1]);
        mma_bf16(s[2 * np + 1], kQReg ? qf[kQReg ? ks : 0] : qt, b[2], b[3]);
      }
    }
    const bool whole = wlive && kb + 63 <= wfirst && (kb >= wlo || kb + 63 < a.keep);
    float nm[2] = {mx[0], mx[1]};
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      const int c = nt * 8 + (lane & 3) * 2;
      const float2 f = SEP ? make_float2(1.0f, 1.0f) : *reinterpret_cast<const float2*>(kr + c);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = e >> 1, j = kb + c + (e & 1);
        if (!SEP) s[nt][e] *= (e & 1) ? f.y : f.x;
        if (SEP && a.softcap > 0.0f) s[nt][e] = cap_score(s[nt][e], cap);
        s[nt][e] -= slope[r] * (float)(qpos[r] - j);
        if (!whole && !sees(a, qpos[r], qlo[r], j)) s[nt][e] = -INFINITY;
        nm[r] = fmaxf(nm[r], s[nt][e]);
      }
    }
    float base[2], resc[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 1));
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 2));
      base[r] = nm[r] == -INFINITY ? 0.0f : nm[r];           // nothing visible yet: every term is ex2(-inf) = 0
      resc[r] = ex2(mx[r] - base[r]);
      mx[r] = nm[r];
      l[r] *= resc[r];
    }
    uint32_t p[8][2];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = ex2(s[nt][e] - base[e >> 1]);
        l[e >> 1] += v[e];
      }
      p[nt][0] = pack_bf16(v[0], v[1]);
      p[nt][1] = pack_bf16(v[2], v[3]);
    }
#pragma unroll
    for (int i = 0; i < HD / 8; ++i) {
      o[i][0] *= resc[0]; o[i][1] *= resc[0];
      o[i][2] *= resc[1]; o[i][3] *= resc[1];
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      const uint32_t pa[4] = {p[2 * ks][0], p[2 * ks][1], p[2 * ks + 1][0], p[2 * ks + 1][1]};
#pragma unroll
      for (int np = 0; np < HD / 16; ++np) {
        uint32_t b[4];
        ldsm4_t(b, frag_b_cols(v, LD, ks * 16, np * 16, lane));
        mma_bf16(o[2 * np], pa, b[0], b[1]);
        mma_bf16(o[2 * np + 1], pa, b[2], b[3]);
      }
    }
    __syncthreads();   // every warp is done with this stage before it is refilled
    kb = nx;
  }
  cp_async_wait<0>();
  if constexpr (MAPS == 2) {           // the second map's outputs meet the first one's where the tiles were
    constexpr int OLD = HD + 8;
    float* so = reinterpret_cast<float*>(sK);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
      l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
      if (map == 0 || row[r] >= rows) continue;
      const float f = 1.0f / l[r];
#pragma unroll
      for (int nt = 0; nt < HD / 8; ++nt)
        *reinterpret_cast<float2*>(so + row[r] * OLD + nt * 8 + (lane & 3) * 2) = make_float2(o[nt][2 * r] * f, o[nt][2 * r + 1] * f);
    }
    __syncthreads();
    if (map != 0) return;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const bool live = row[r] < rows;
      const float f = live ? 1.0f / l[r] : 0.0f;
      float ss = 0.0f;
#pragma unroll
      for (int nt = 0; nt < HD / 8; ++nt) {        // columns past vdim are zero on both sides
        const float2 u = live ? *reinterpret_cast<const float2*>(so + row[r] * OLD + nt * 8 + (lane & 3) * 2) : make_float2(0.0f, 0.0f);
        o[nt][2 * r] = o[nt][2 * r] * f - a.lambda * u.x;
        o[nt][2 * r + 1] = o[nt][2 * r + 1] * f - a.lambda * u.y;
        ss += o[nt][2 * r] * o[nt][2 * r] + o[nt][2 * r + 1] * o[nt][2 * r + 1];
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (!live) continue;
      const size_t t = en.x + q0 + row[r] / G;
      store_row<HD>(a, o, r, a.diff_scale * gate(a, t, head[r]) / sqrtf(ss / (float)a.vdim + a.eps), t, head[r], lane);
    }
    return;
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (row[r] >= rows) continue;
    const size_t t = en.x + q0 + row[r] / G;
    float f = gate(a, t, head[r]);
    if (a.sinks == nullptr) {
      f /= l[r];   // the query's own position is always visible
    } else {
      const float sink = a.sinks[head[r]] * kLog2e, top = fmaxf(mx[r], sink), down = ex2(mx[r] - top);
      f *= down / (l[r] * down + ex2(sink - top));
    }
    store_row<HD>(a, o, r, f, t, head[r], lane);
  }
}

// ---- single tokens --------------------------------------------------------------------------------------------------------------
// grid (kv heads x groups of 16 query rows (heads x maps), splits, rows); the splits of one row form a cluster and meet in distributed
// shared memory.  A warp walks 16-token tiles of the visible range; the split that holds the row's own position appends its
// key before it reads it.
// tiles a warp keeps in flight, one of them in use; warps of a CTA
constexpr int decode_stages(int hd, bool sep) { return sep ? (hd <= 64 ? 4 : (hd <= 192 ? 3 : 2)) : (hd <= 128 ? 4 : 2); }
constexpr int decode_warps(int hd, bool sep) { return sep && hd > 128 ? 4 : 8; }

template <int HD, bool SEP, int MAPS>
__global__ void __launch_bounds__(32 * decode_warps(HD, SEP)) decode_kernel(Attn a) {
  constexpr int KD = HD / MAPS;
  constexpr int LD = HD + 8, NW = decode_warps(HD, SEP), NTH = 32 * NW, NST = decode_stages(HD, SEP);
  constexpr int kTile = 16 * LD;      // elements of a tile
  constexpr int kStage = SEP ? 2 * kTile : kTile;   // keys, then values
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);                    // [16][LD]
  float* res = reinterpret_cast<float*>(sQ + kTile);               // this CTA's merged rows [16][HD + 2]
  bf16* tiles = reinterpret_cast<bf16*>(res + 16 * (HD + 2));      // [warp][stage][tile], later the warps' partial rows
  float* part = reinterpret_cast<float*>(tiles);                   // [warp][16][HD + 2]
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int G = a.heads / a.kv_heads, mg = (MAPS * G + 15) / 16;
  const int kvh = blockIdx.x / mg, h0 = (blockIdx.x % mg) * 16, nh = min(16, MAPS * G - h0);
  auto head_of = [&](int r) { return kvh * G + (h0 + r) / MAPS; };
  const int split = blockIdx.y, nsplit = gridDim.y;
  // the row's place and the keys of earlier positions are older than the kernel before this one
  const int t = blockIdx.z;
  const int pos = a.pos[t];
  if (pos >= (a.max_pages << a.pshift)) {    // no page can hold it: the whole cluster leaves
    pdl_wait();
    pdl_trigger();
    return;
  }
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  const bf16* pool = static_cast<const bf16*>(a.pool);
  const int lo16 = window_lo(a, pos) >> 4, end16 = (pos >> 4) + 1;
  const int lo = window_lo(a, pos), nkeep = min((a.keep + 15) >> 4, lo16);   // tiles of kept tokens before the window's first tile
  const int ntiles = nkeep + end16 - lo16;
  const int per = (ntiles + nsplit - 1) / nsplit;
  const int b0 = split * per, b1 = min(ntiles, b0 + per);
  const bool owner = a.k_col >= 0 && b1 == ntiles && b0 < b1;            // holds the last tile, the row's own position, and appends it
  bf16* wt = tiles + warp * NST * kStage;
  float* wf = reinterpret_cast<float*>(tiles + NW * NST * kStage) + warp * NST * 16;   // key factors of the tiles
  auto first_token = [&](int j) { return (j < nkeep ? j : lo16 + j - nkeep) << 4; };
  auto issue = [&](int j, int st) {     // a tile lies in one page: its rows and factors are contiguous
    const int tb = first_token(j);
    const size_t row = cache_row(a, bt, kvh, tb);
#pragma unroll
    for (int i = 0; i < 16 * (HD / 8) / 32; ++i) {
      const int idx = lane + 32 * i, r = idx / (HD / 8), c = (idx % (HD / 8)) * 8;
      cp_async16(wt + st * kStage + r * LD + c, pool + (row + r) * HD + c, tb + r <= pos);
      if (SEP) cp_async16(wt + st * kStage + kTile + r * LD + c, static_cast<const bf16*>(a.vpool) + (row + r) * HD + c, tb + r <= pos);
    }
    if (!SEP && lane < 4) cp_async16(wf + st * 16 + lane * 4, a.krms + row + lane * 4, true);
  };
  const int j0 = b0 + warp;
  auto is_new = [&](int j) { return owner && j == b1 - 1; };              // the tile that receives the row's own key
#pragma unroll
  for (int st = 0; st < NST - 1; ++st)
    if (j0 + st * NW < b1 && !is_new(j0 + st * NW)) issue(j0 + st * NW, st);
  pdl_wait();
  pdl_trigger();
  const float* prow = a.proj + (size_t)t * a.ld;
  load_queries<KD, SEP, MAPS, 16 / NW>(a, warp, nh, NW, [&](int r) {
    const int m = (h0 + r) % MAPS;
    return QueryRow{prow, head_of(r), m, pos, sQ + r * LD + m * KD};
  }, lane);
  for (int r = warp; r < 16; r += NW)
    for (int d = lane; d < HD; d += 32)
      if (r >= nh || (MAPS == 2 && d / KD != (h0 + r) % MAPS)) sQ[r * LD + d] = __float2bfloat16_rn(0.0f);
  if (owner && warp == NW - 1) {
    append_row<HD, SEP, MAPS, bf16>(a, prow, kvh, pos, cache_row(a, bt, kvh, pos), lane);
    __threadfence();
  }
  __syncthreads();
  float o[HD / 8][4];
#pragma unroll
  for (int i = 0; i < HD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  const int g = lane >> 2;
  float slope[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) slope[r] = a.slopes == nullptr ? 0.0f : a.slopes[head_of(min(g + 8 * r, nh - 1))] * kLog2e;
  const float cap = a.softcap * kLog2e;
#pragma unroll
  for (int st = 0; st < NST - 1; ++st) {
    if (j0 + st * NW < b1 && is_new(j0 + st * NW)) issue(j0 + st * NW, st);
    cp_async_commit();
  }
  float ahead[MAPS == 2 ? HD / 32 : 1];       // two maps: the gates of this warp's head
  if (MAPS == 2) {
    const int hh = split * NW + warp;
#pragma unroll
    for (int i = 0; i < HD / 32; ++i)
      ahead[MAPS == 2 ? i : 0] = hh < nh / 2 && lane + 32 * i < a.vdim ? wide_gate(a, t, head_of(2 * hh), lane + 32 * i) : 1.0f;
  }
  constexpr bool kQReg = HD <= 128;
  uint32_t qf[kQReg ? HD / 16 : 1][4];
  if (kQReg) {
#pragma unroll
    for (int ks = 0; ks < (kQReg ? HD / 16 : 1); ++ks) ldsm4(qf[ks], frag_a(sQ, LD, 0, ks * 16, lane));
  }
  int it = 0;
  for (int j = j0; j < b1; j += NW, ++it) {
    cp_async_wait<NST - 2>();
    __syncwarp();
    if (j + (NST - 1) * NW < b1) issue(j + (NST - 1) * NW, (it + NST - 1) % NST);
    cp_async_commit();
    const bf16* k = wt + (it % NST) * kStage;
    const bf16* v = SEP ? k + kTile : k;
    const float* kf = wf + (it % NST) * 16;
    const int tb = first_token(j);
    float s[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < HD / 16; ++ks) {
      uint32_t q[4], b[4];
      if (!kQReg) ldsm4(q, frag_a(sQ, LD, 0, ks * 16, lane));
      ldsm4(b, frag_b_rows(k, LD, 0, ks * 16, lane));
      mma_bf16(s[0], kQReg ? qf[kQReg ? ks : 0] : q, b[0], b[1]);
      mma_bf16(s[1], kQReg ? qf[kQReg ? ks : 0] : q, b[2], b[3]);
    }
    float nm[2] = {mx[0], mx[1]}, base[2], resc[2];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = nt * 8 + (lane & 3) * 2 + (e & 1), j1 = tb + c;
        if (!SEP) s[nt][e] *= kf[c];
        if (SEP && a.softcap > 0.0f) s[nt][e] = cap_score(s[nt][e], cap);
        s[nt][e] -= slope[e >> 1] * (float)(pos - j1);
        if (!sees(a, pos, lo, j1)) s[nt][e] = -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], s[nt][e]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 1));
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 2));
      base[r] = nm[r] == -INFINITY ? 0.0f : nm[r];
      resc[r] = ex2(mx[r] - base[r]);
      mx[r] = nm[r];
      l[r] *= resc[r];
    }
    uint32_t pa[4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = ex2(s[nt][e] - base[e >> 1]);
        l[e >> 1] += v[e];
      }
      pa[2 * nt] = pack_bf16(v[0], v[1]);
      pa[2 * nt + 1] = pack_bf16(v[2], v[3]);
    }
#pragma unroll
    for (int i = 0; i < HD / 8; ++i) {
      o[i][0] *= resc[0]; o[i][1] *= resc[0];
      o[i][2] *= resc[1]; o[i][3] *= resc[1];
    }
#pragma unroll
    for (int np = 0; np < HD / 16; ++np) {
      uint32_t b[4];
      ldsm4_t(b, frag_b_cols(v, LD, 0, np * 16, lane));
      mma_bf16(o[2 * np], pa, b[0], b[1]);
      mma_bf16(o[2 * np + 1], pa, b[2], b[3]);
    }
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();     // the tiles are free: the warps' partial rows take their place
  constexpr int ST = HD + 2;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (g + 8 * r >= nh) continue;
    float* dst = part + (warp * 16 + g + 8 * r) * ST;
#pragma unroll
    for (int nt = 0; nt < HD / 8; ++nt) {
      dst[nt * 8 + (lane & 3) * 2] = o[nt][2 * r];
      dst[nt * 8 + (lane & 3) * 2 + 1] = o[nt][2 * r + 1];
    }
    if ((lane & 3) == 0) {
      dst[HD] = mx[r];
      dst[HD + 1] = l[r];
    }
  }
  __syncthreads();
  // the warps' factors, once per row
  float own = -INFINITY, most, sum = 0.0f;
  const int fr = threadIdx.x / NW, fw = threadIdx.x % NW;
  static_assert(16 * NW <= NTH && (NW & (NW - 1)) == 0 && NW <= 32, "a thread per row and warp");
  if (fr < nh) own = part[(fw * 16 + fr) * ST + HD];
  most = own;
#pragma unroll
  for (int o = NW / 2; o > 0; o >>= 1) most = fmaxf(most, __shfl_xor_sync(0xffffffffu, most, o));
  if (fr < nh) {
    const float f = own == -INFINITY ? 0.0f : ex2(own - most);
    float* src = part + (fw * 16 + fr) * ST;
    src[HD] = f;
    sum = f * src[HD + 1];
  }
#pragma unroll
  for (int o = NW / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  if (fr < nh && fw == 0) {
    res[fr * ST + HD] = most;
    res[fr * ST + HD + 1] = sum;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * HD; i += NTH) {
    const int r = i / HD, d = i % HD;
    float acc = 0.0f;
#pragma unroll
    for (int w = 0; w < NW; ++w) acc = fmaf(part[(w * 16 + r) * ST + HD], part[(w * 16 + r) * ST + d], acc);
    res[r * ST + d] = acc;
  }
  if (nsplit > 1) cluster.sync();
  else __syncthreads();
  if constexpr (MAPS == 2) {           // a warp takes a head: its two rows are neighbours
    for (int hh = split * NW + warp; hh < nh / 2; hh += nsplit * NW) {
      float f[2][8], L[2] = {0.0f, 0.0f};                       // factors of the splits
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        float M = -INFINITY;
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          f[m][s] = s < nsplit ? (nsplit > 1 ? cluster.map_shared_rank(res, s) : res)[(2 * hh + m) * ST + HD] : -INFINITY;
          M = fmaxf(M, f[m][s]);
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          f[m][s] = f[m][s] == -INFINITY ? 0.0f : ex2(f[m][s] - M);
          if (s < nsplit) L[m] += f[m][s] * (nsplit > 1 ? cluster.map_shared_rank(res, s) : res)[(2 * hh + m) * ST + HD + 1];
        }
      }
      const float i1 = 1.0f / L[0], i2 = a.lambda / L[1];
      float o2[HD / 32], ss = 0.0f;
#pragma unroll
      for (int i = 0; i < HD / 32; ++i) {
        float x1 = 0.0f, x2 = 0.0f;
#pragma unroll
        for (int s = 0; s < 8; ++s)
          if (s < nsplit) {
            const float* src = (nsplit > 1 ? cluster.map_shared_rank(res, s) : res) + 2 * hh * ST + lane + 32 * i;
            x1 += f[0][s] * src[0];
            x2 += f[1][s] * src[ST];
          }
        o2[i] = x1 * i1 - x2 * i2;                               // columns past vdim are zero
        ss += o2[i] * o2[i];
      }
      const int h = head_of(2 * hh);
      const float g2 = a.diff_scale * gate(a, t, h) / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
#pragma unroll
      for (int i = 0; i < HD / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < a.vdim) static_cast<bf16*>(a.out)[(size_t)t * a.ldo + h * a.vdim + d] = __float2bfloat16_rn(o2[i] * g2 * (hh == split * NW + warp ? ahead[MAPS == 2 ? i : 0] : wide_gate(a, t, h, d)));
      }
    }
    if (nsplit > 1) cluster.sync();
    return;
  }
  // every CTA of the cluster finishes its share of the outputs
  for (int i = split * NTH + threadIdx.x; i < nh * a.vdim; i += nsplit * NTH) {
    const int r = i / a.vdim, d = i % a.vdim;
    float M = -INFINITY, acc = 0.0f, L = 0.0f;
    for (int s = 0; s < nsplit; ++s) M = fmaxf(M, (nsplit > 1 ? cluster.map_shared_rank(res, s) : res)[r * ST + HD]);
    for (int s = 0; s < nsplit; ++s) {
      const float* src = (nsplit > 1 ? cluster.map_shared_rank(res, s) : res) + r * ST;
      const float f = src[HD] == -INFINITY ? 0.0f : ex2(src[HD] - M);
      acc += f * src[d];
      L += f * src[HD + 1];
    }
    const int h = head_of(r);
    if (a.sinks != nullptr) {
      const float sink = a.sinks[h] * kLog2e, top = fmaxf(M, sink), down = ex2(M - top);
      acc *= down;
      L = L * down + ex2(sink - top);
    }
    static_cast<bf16*>(a.out)[(size_t)t * a.ldo + h * a.vdim + d] = __float2bfloat16_rn(acc / L * gate(a, t, h) * wide_gate(a, t, h, d));
  }
  if (nsplit > 1) cluster.sync();   // nobody leaves while its rows are being read
}

// ---- 32-bit mode ------------------------------------------------------------------------------------------------------------------
// grid (heads, rows): four warps take the visible keys in turn, exact f32 products and exponentials
template <int HD, bool SEP, int MAPS>
__global__ void __launch_bounds__(128) f32_kernel(Attn a) {
  constexpr int KD = HD / MAPS, NK = (KD + 31) / 32;
  __shared__ float sm[MAPS][4][HD + 2], s32[32];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, t = blockIdx.y, kvh = h / (a.heads / a.kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int pos = a.pos[t];
  if (pos >= (a.max_pages << a.pshift)) return;
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  const float* pool = static_cast<const float*>(a.pool);
  const float2* rot = angles(a, pos);
  const float slope = a.slopes == nullptr ? 0.0f : a.slopes[h], scale = a.scale * temperature(a, pos);
  const int lo = window_lo(a, pos), nkeep = min(a.keep, lo);
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    const float* qr = a.proj + (size_t)t * a.ld + a.q_col + (h * MAPS + mp) * a.dim;
    const float* qb = a.q_bias == nullptr ? nullptr : a.q_bias + (h * MAPS + mp) * a.dim;
    float q[NK], o[HD / 32], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int d = lane + 32 * i;
      const bool in = d < KD && d < a.dim;
      const float raw = in ? biased(qr, qb, d) : 0.0f;
      q[i] = in ? rotated([&](int j) { return biased(qr, qb, j) * (a.q_norm == nullptr ? 1.0f : query_weight<SEP>(a, j)); }, d, rot, a.rot_dims, a.rot_pairs) : 0.0f;
      ss += raw * raw;
    }
#pragma unroll
    for (int i = 0; i < HD / 32; ++i) o[i] = 0.0f;
    const float rq = a.normed ? 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps) : 1.0f;
#pragma unroll
    for (int i = 0; i < NK; ++i) q[i] *= rq;
    float m = -INFINITY, l = 0.0f;
    for (int i = warp; i < nkeep + pos + 1 - lo; i += 4) {
      const int j = i < nkeep ? i : lo + i - nkeep;
      const size_t row = cache_row(a, bt, kvh, j);
      float k[NK], s = 0.0f;
#pragma unroll
      for (int c = 0; c < NK; ++c) {
        k[c] = KD % 32 == 0 || lane + 32 * c < KD ? pool[row * HD + mp * KD + lane + 32 * c] : 0.0f;
        s = fmaf(q[c], k[c], s);
      }
      s = warp_sum(s) * scale * (SEP ? 1.0f : a.krms[row]);
      if (SEP && a.softcap > 0.0f) s = a.softcap * tanhf(s / a.softcap);
      s -= slope * (float)(pos - j);
      const float nm = fmaxf(m, s), f = expf(m - nm), p = expf(s - nm);
      m = nm;
      l = l * f + p;
#pragma unroll
      for (int c = 0; c < HD / 32; ++c) o[c] = o[c] * f + p * (SEP ? static_cast<const float*>(a.vpool)[row * HD + lane + 32 * c] : k[c < NK ? c : 0]);
    }
#pragma unroll
    for (int c = 0; c < HD / 32; ++c) sm[mp][warp][lane + 32 * c] = o[c];
    if (lane == 0) {
      sm[mp][warp][HD] = m;
      sm[mp][warp][HD + 1] = l;
    }
  }
  __syncthreads();
  float M[MAPS], inv[MAPS];
#pragma unroll
  for (int mp = 0; mp < MAPS; ++mp) {
    float L = 0.0f;
    M[mp] = -INFINITY;
    for (int w = 0; w < 4; ++w) M[mp] = fmaxf(M[mp], sm[mp][w][HD]);
    if (a.sinks != nullptr) {
      M[mp] = fmaxf(M[mp], a.sinks[h]);
      L = expf(a.sinks[h] - M[mp]);
    }
    for (int w = 0; w < 4; ++w) L += expf(sm[mp][w][HD] - M[mp]) * sm[mp][w][HD + 1];
    inv[mp] = 1.0f / L;
  }
  auto value = [&](int mp, int d) {
    float acc = 0.0f;
    for (int w = 0; w < 4; ++w) acc += expf(sm[mp][w][HD] - M[mp]) * sm[mp][w][d];
    return acc * inv[mp];
  };
  auto head_value = [&](int d) { return MAPS == 1 ? value(0, d) : value(0, d) - a.lambda * value(MAPS - 1, d); };
  float f = gate(a, t, h);
  if (MAPS == 2) {
    float ss = 0.0f;
    for (int d = threadIdx.x; d < a.vdim; d += 128) ss += head_value(d) * head_value(d);
    f *= a.diff_scale / sqrtf(block_sum(ss, s32) / (float)a.vdim + a.eps);
  }
  for (int d = threadIdx.x; d < a.vdim; d += 128)
    static_cast<float*>(a.out)[(size_t)t * a.ldo + h * a.vdim + d] = head_value(d) * f * wide_gate(a, t, h, d);
}

template <int HD, bool SEP, int MAPS>
static int run_append(const Attn& a, int first, int count, int f32, cudaStream_t stream) {
  const dim3 grid((count + 3) / 4, a.kv_heads);
  return f32 ? launch(append_kernel<HD, SEP, MAPS, float>, grid, 128, 0, stream, 1, 0, a, first, count)
             : launch(append_kernel<HD, SEP, MAPS, bf16>, grid, 128, 0, stream, 1, 0, a, first, count);
}
template <int HD, bool SEP, int MAPS>
static int run_prompt(const Attn& a, const int* entries, const int* tiles, int ntiles, cudaStream_t stream) {
  const size_t smem = (size_t)(SEP ? 5 : 3) * 64 * (HD + 8) * sizeof(bf16) + (SEP ? 0 : 128 * sizeof(float));
  cudaFuncSetAttribute(prompt_kernel<HD, SEP, MAPS>, cudaFuncAttributePreferredSharedMemoryCarveout, (int)cudaSharedmemCarveoutMaxShared);
  return launch(prompt_kernel<HD, SEP, MAPS>, dim3(a.kv_heads, ntiles), 128 * MAPS, smem, stream, 1, 0, a, (const int4*)entries, (const int2*)tiles);
}
template <int HD, bool SEP, int MAPS>
static int run_decode(const Attn& a, int nrows, int nsplit, cudaStream_t stream) {
  const int mg = (MAPS * (a.heads / a.kv_heads) + 15) / 16;
  constexpr int NW = decode_warps(HD, SEP), NST = decode_stages(HD, SEP);
  constexpr size_t smem = (size_t)16 * (HD + 8) * sizeof(bf16) * (1 + NW * NST * (SEP ? 2 : 1)) + (size_t)16 * (HD + 2) * sizeof(float) +
                          (SEP ? 0 : (size_t)NW * NST * 16 * sizeof(float));
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  return launch(decode_kernel<HD, SEP, MAPS>, dim3(a.kv_heads * mg, nsplit, nrows), 32 * NW, smem, stream, nsplit, 1, a);
}
template <int HD, bool SEP, int MAPS>
static int run_f32(const Attn& a, int T, cudaStream_t stream) {
  return launch(f32_kernel<HD, SEP, MAPS>, dim3(a.heads, T), 128, 0, stream, 1, 0, a);
}

static int padded_dim(int dim) {
  const int sizes[] = {32, 64, 96, 128, 192, 256};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

// elements of a cache row
static int row_dim(const Attn& a) { return padded_dim(a.maps * a.dim > a.vdim ? a.maps * a.dim : a.vdim); }

static bool fill(Attn& a, const void* const* ptrs, const int* ints, const float* floats) {
  a.proj = (const float*)ptrs[0]; a.q_norm = (const float*)ptrs[1]; a.k_norm = (const float*)ptrs[2]; a.slopes = (const float*)ptrs[3];
  a.pos = (const int*)ptrs[4]; a.slots = (const int*)ptrs[5]; a.block_table = (const int*)ptrs[6]; a.pool = const_cast<void*>(ptrs[7]);
  a.krms = (float*)ptrs[8]; a.vpool = const_cast<void*>(ptrs[9]); a.out = const_cast<void*>(ptrs[10]); a.sinks = (const float*)ptrs[11];
  a.rot = (const float2*)ptrs[12]; a.q_bias = (const float*)ptrs[13]; a.k_bias = (const float*)ptrs[14]; a.v_bias = (const float*)ptrs[15];
  a.ld = ints[0]; a.q_col = ints[1]; a.k_col = ints[2]; a.v_col = ints[3]; a.g_col = ints[4]; a.ldo = ints[5]; a.heads = ints[6];
  a.kv_heads = ints[7]; a.dim = ints[8]; a.vdim = ints[9]; a.max_pages = ints[10];
  for (a.pshift = 0; (2 << a.pshift) <= ints[11]; ++a.pshift) {}
  a.window = ints[12]; a.keep = ints[13]; a.normed = ints[14]; a.rot_dims = a.rot == nullptr ? 0 : ints[15]; a.rot_pairs = ints[16];
  a.chunk = ints[17]; a.maps = ints[18]; a.gate_wide = ints[19];
  a.eps = floats[0]; a.scale = floats[1]; a.out_scale = floats[2]; a.softcap = floats[3]; a.temp_coef = floats[4]; a.temp_every = floats[5];
  a.lambda = floats[6]; a.diff_scale = floats[7];
  if (a.window <= 0 && a.chunk <= 0) a.keep = 0;       // everything is visible
  if (a.vpool == nullptr ? a.krms == nullptr || a.vdim != a.dim || a.softcap > 0.0f || a.rot != nullptr || !a.normed || a.k_col < 0 || a.maps != 1 ||
                              a.q_bias != nullptr || a.k_bias != nullptr || a.v_bias != nullptr
                        : a.vdim < 1) return false;
  if (a.rot != nullptr && (a.rot_dims < 2 || a.rot_dims % 2 != 0 || a.rot_dims > a.dim)) return false;
  if (a.maps != 1 && (a.maps != 2 || a.sinks != nullptr || a.q_norm == nullptr || a.q_bias == nullptr)) return false;
  if ((a.q_bias == nullptr) != (a.v_bias == nullptr) || (a.k_col >= 0 && (a.q_bias == nullptr) != (a.k_bias == nullptr))) return false;
  if (a.window > 0 && a.chunk > 0) return false;
  return a.heads >= 1 && a.kv_heads >= 1 && a.heads % a.kv_heads == 0 && a.heads / a.kv_heads <= 64 && a.dim >= 1 &&
         row_dim(a) > 0 && a.pshift >= 4 && (1 << a.pshift) == ints[11] && a.keep >= 0 &&
         (a.temp_coef == 0.0f || a.temp_every > 0.0f) && (a.q_norm == nullptr) == (a.k_norm == nullptr);
}

#define BONSAI_ONE_DIM(D, CALL)                                                                                              \
  case D: {                                                                                                                  \
    constexpr int HD = D;                                                                                                    \
    if (a.maps == 2) { constexpr bool SEP = true; constexpr int MAPS = 2; return CALL; }                                     \
    if (a.vpool != nullptr) { constexpr bool SEP = true; constexpr int MAPS = 1; return CALL; }                              \
    constexpr bool SEP = false;                                                                                              \
    constexpr int MAPS = 1;                                                                                                  \
    return CALL;                                                                                                             \
  }
#define BONSAI_BY_DIM(CALL)                                 \
  switch (row_dim(a)) {                                     \
    BONSAI_ONE_DIM(32, CALL)                                \
    BONSAI_ONE_DIM(64, CALL)                                \
    BONSAI_ONE_DIM(96, CALL)                                \
    BONSAI_ONE_DIM(128, CALL)                               \
    BONSAI_ONE_DIM(192, CALL)                               \
    BONSAI_ONE_DIM(256, CALL)                               \
    default: return BONSAI_CUDA_BAD_ARG;                    \
  }

}  // namespace lay
}  // namespace bonsai

extern "C" {

// elements of a cache row for a head size (with two maps: both keys together, or the value if that is longer); 0: not supported
int bonsai_lay_attn_row(int dim) { return dim < 1 ? 0 : bonsai::lay::padded_dim(dim); }

// Arguments of all launches: ptrs = {proj, q_norm, k_norm, slopes, pos, slots, block_table, pool, krms, vpool, out, sinks, rot, q_bias,
// k_bias, v_bias} (null where a design has none, the biases together; two maps have biases and norm weights; vpool null: rows are key and value; rot has a row for every position the pages
// hold), ints = {ld, q_col, k_col, v_col, g_col, ldo, heads, kv_heads, dim, vdim, max_pages, page_size, window, keep, normed, rot_dims,
// rot_pairs, chunk, maps, gate_wide}, floats = {eps, scale, out_scale, softcap, temp_coef, temp_every, lambda, diff_scale}.

// Writes the keys of rows first .. first + count - 1.
int bonsai_lay_attn_append(const void* const* ptrs, const int* ints, const float* floats, int first, int count, int f32, cudaStream_t stream) {
  using namespace bonsai::lay;
  Attn a;
  if (!fill(a, ptrs, ints, floats) || count < 1 || first < 0 || a.k_col < 0) return BONSAI_CUDA_BAD_ARG;
  BONSAI_BY_DIM((run_append<HD, SEP, MAPS>(a, first, count, f32, stream)))
}

// entries int4 [..] {first row, tokens, slot, first position}, tiles int2 [ntiles] {entry, first token}; a tile has
// 64 / (heads / kv_heads) tokens.  The rows' keys must have been appended.
int bonsai_lay_attn_prompt(const void* const* ptrs, const int* ints, const float* floats, const int* entries, const int* tiles, int ntiles,
                           cudaStream_t stream) {
  using namespace bonsai::lay;
  Attn a;
  if (!fill(a, ptrs, ints, floats) || ntiles < 1 || ntiles > 65535) return BONSAI_CUDA_BAD_ARG;
  BONSAI_BY_DIM((run_prompt<HD, SEP, MAPS>(a, entries, tiles, ntiles, stream)))
}

// One token in each of the rows 0 .. nrows - 1, its key appended here.
int bonsai_lay_attn_decode(const void* const* ptrs, const int* ints, const float* floats, int nrows, int nsplit, cudaStream_t stream) {
  using namespace bonsai::lay;
  Attn a;
  if (!fill(a, ptrs, ints, floats) || nrows < 1 || nrows > 65535 || (nsplit != 1 && nsplit != 2 && nsplit != 4 && nsplit != 8)) return BONSAI_CUDA_BAD_ARG;
  BONSAI_BY_DIM((run_decode<HD, SEP, MAPS>(a, nrows, nsplit, stream)))
}

// All T rows, 32-bit throughout; the rows' keys must have been appended.
int bonsai_lay_attn_f32(const void* const* ptrs, const int* ints, const float* floats, int T, cudaStream_t stream) {
  using namespace bonsai::lay;
  Attn a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 65535) return BONSAI_CUDA_BAD_ARG;
  BONSAI_BY_DIM((run_f32<HD, SEP, MAPS>(a, T, stream)))
}

}  // extern "C"
