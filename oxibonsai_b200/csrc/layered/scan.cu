// Element-wise recurrences: every channel has its own decay at every token.
//
// minGRU: z = sigmoid(z + z_b), u = u + u_b, c = u + 1/2 where u >= 0 and sigmoid(u) elsewhere,
//   S <- (1 - z) S + z c,   out = S * silu(g)
// Prompts are scanned in time as well: a warp has 32 channels (a lane each) of kGruTokens tokens in registers, eight warps and the CTAs
// of a cluster have the tokens that follow, and the composed maps S -> A S + B of warps and CTAs meet in shared memory.  The projections
// are read once.
//
// Selective scan (Mamba): per channel c and state n, with dt = softplus(dt_raw + dt_b), A < 0,
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,   y_c = sum_n S[c, n] C_n + D_c x_c,   out = y * silu(z)
// LN lanes share a channel, NS states each in registers.  Prompts stage tiles of kScanTokens tokens with asynchronous copies, two ahead of
// the arithmetic; softplus, skip, gate and stores run over a tile at once.  A portion may be cut into segments that run side by
// side: first the local states of all but the last (from zero; their decay is exp(A sum of dt)), then every segment from the state its
// predecessors leave.
//
// State: f32, [row][channels] and [row][channels][NP] with the states padded to LN * NS.  A sequence's first token (position 0) starts
// from zero whatever its state row holds.  The 32-bit mode runs the same kernels on f32 activations with full-precision exponentials.
#include <cooperative_groups.h>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float silu(float v) { return v * sigmoid(v); }

// ---- minGRU ---------------------------------------------------------------------------------------------------------------------
struct Gru {
  const float* proj;        // [T][ld], z, u, g at their columns
  const float* z_bias;      // [width]
  const float* u_bias;
  float* S;                 // [row][width]
  const int* pos;
  const int* slots;
  const int* state_rows;
  void* out;                // [T][ldo]
  int ld, z_col, u_col, g_col, ldo, width;
};

__device__ __forceinline__ float candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid(u); }

// grid (channels, rows): single tokens
template <typename X>
__global__ void __launch_bounds__(128) gru_step_kernel(Gru a) {
  const int c = blockIdx.x * 128 + threadIdx.x, t = blockIdx.y;
  const bool on = c < a.width;
  float* S = a.S + (size_t)a.state_rows[a.slots[t]] * a.width + c;
  const float s0 = on && a.pos[t] > 0 ? *S : 0.0f;         // older than the kernel before this one
  const float zb = on ? a.z_bias[c] : 0.0f, ub = on ? a.u_bias[c] : 0.0f;
  pdl_wait();
  pdl_trigger();
  if (!on) return;
  const float* p = a.proj + (size_t)t * a.ld + c;
  const float zr = p[a.z_col] + zb, u = p[a.u_col] + ub, g = p[a.g_col];
  const float s = sigmoid(-zr) * s0 + sigmoid(zr) * candidate(u);
  *S = s;
  store_act(static_cast<X*>(a.out) + (size_t)t * a.ldo + c, s * silu(g));
}

constexpr int kGruTokens = 16, kGruWarps = 8;

// grid (32 channels x cluster, portions)
template <typename X>
__global__ void __launch_bounds__(32 * kGruWarps) gru_scan_kernel(Gru a, const int4* entries) {
  __shared__ float2 part[2][kGruWarps][32], whole[2][32];
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int ctas = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x / ctas) * 32 + lane;
  const bool on = c < a.width;
  pdl_wait();
  pdl_trigger();
  const int4 en = entries[blockIdx.y];
  float* S = a.S + (size_t)a.state_rows[en.z] * a.width + c;
  float state = on && en.w > 0 ? *S : 0.0f;                // of the tokens before this round's
  const float zb = on ? a.z_bias[c] : 0.0f, ub = on ? a.u_bias[c] : 0.0f;
  const float* base = a.proj + (size_t)en.x * a.ld + c;
  const int per_round = ctas * kGruWarps * kGruTokens, mine = (rank * kGruWarps + warp) * kGruTokens;
  int par = 0;
  for (int r0 = 0; r0 < en.y; r0 += per_round, par ^= 1) {
    const int t0 = r0 + mine, n = on ? min(kGruTokens, en.y - t0) : 0;
    float keep[kGruTokens], add[kGruTokens], gate[kGruTokens];
#pragma unroll
    for (int i = 0; i < kGruTokens; ++i) {
      const float* p = base + (size_t)(t0 + i) * a.ld;
      keep[i] = i < n ? p[a.z_col] : 0.0f;
      add[i] = i < n ? p[a.u_col] : 0.0f;
      gate[i] = i < n ? p[a.g_col] : 0.0f;
    }
    float A = 1.0f, B = 0.0f;
#pragma unroll
    for (int i = 0; i < kGruTokens; ++i) {
      const float zr = keep[i] + zb;
      add[i] = i < n ? sigmoid(zr) * candidate(add[i] + ub) : 0.0f;
      keep[i] = i < n ? sigmoid(-zr) : 1.0f;
      B = fmaf(keep[i], B, add[i]);
      A *= keep[i];
    }
    part[par][warp][lane] = make_float2(A, B);
    __syncthreads();
    if (ctas > 1) {
      if (warp == 0) {
        A = 1.0f;
        B = 0.0f;
#pragma unroll
        for (int w = 0; w < kGruWarps; ++w) {
          const float2 m = part[par][w][lane];
          A *= m.x;
          B = fmaf(m.x, B, m.y);
        }
        whole[par][lane] = make_float2(A, B);
      }
      cluster.sync();        // the other buffer is free again: everyone is past the reads of the round before the last
    }
    float s = state;
    if (ctas > 1) {
      for (int i = 0; i < ctas; ++i) {
        if (i == rank) s = state;
        const float2 m = *cluster.map_shared_rank(&whole[par][lane], i);
        state = fmaf(m.x, state, m.y);
      }
    } else {
#pragma unroll
      for (int w = 0; w < kGruWarps; ++w) {
        const float2 m = part[par][w][lane];
        state = fmaf(m.x, state, m.y);
      }
    }
    for (int w = 0; w < warp; ++w) {
      const float2 m = part[par][w][lane];
      s = fmaf(m.x, s, m.y);
    }
    X* dst = static_cast<X*>(a.out) + (size_t)(en.x + t0) * a.ldo + c;
#pragma unroll
    for (int i = 0; i < kGruTokens; ++i) {
      s = fmaf(keep[i], s, add[i]);
      if (i < n) store_act(dst + (size_t)i * a.ldo, s * silu(gate[i]));
    }
  }
  if (rank == 0 && warp == 0 && on) *S = state;
  if (ctas > 1) cluster.sync();     // nobody leaves while its maps are being read
}

// ---- selective scan ---------------------------------------------------------------------------------------------------------------
struct Scan {
  const float* proj;        // [T][ld], z at z_col
  const float* bc;          // [T][ldbc], B at b_col, C at c_col
  const float* dt;          // [T][lddt], before bias and softplus
  const void* x;            // [T][ldx], convolved and activated
  const float* dt_bias;     // [channels]
  const float* A;           // [channels][np], negative; 0 in the padding
  const float* D;           // [channels]
  float* S;                 // [row][channels][np]
  const int* pos;
  const int* slots;
  const int* state_rows;
  void* out;                // [T][ldo]
  float* seg_S;             // [segment][channels][np]
  float* seg_dt;            // [segment][channels]: sum of dt
  int ld, z_col, ldbc, b_col, c_col, lddt, ldx, ldo, channels, states, np;
};

template <bool EXACT>
__device__ __forceinline__ float decay(float dt, float A) { return EXACT ? expf(dt * A) : ex2(dt * A); }

// grid (channels, rows): single tokens, 128 threads
template <int LN, int NS, typename X>
__global__ void __launch_bounds__(128) scan_step_kernel(Scan a) {
  constexpr bool EXACT = sizeof(X) == 4;
  constexpr int CH = 128 / LN;
  const int ln = threadIdx.x % LN, own = blockIdx.x * CH + threadIdx.x / LN, c = min(own, a.channels - 1), t = blockIdx.y;
  const bool on = own < a.channels;
  float4 s[NS / 4], A[NS / 4];
  float* S = a.S + ((size_t)a.state_rows[a.slots[t]] * a.channels + c) * a.np + ln * NS;
  const bool zero = a.pos[t] == 0;
#pragma unroll
  for (int i = 0; i < NS / 4; ++i) {             // older than the kernel before this one
    s[i] = !zero ? *reinterpret_cast<const float4*>(S + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    A[i] = *reinterpret_cast<const float4*>(a.A + (size_t)c * a.np + ln * NS + 4 * i);
  }
  const float bias = a.dt_bias[c], D = a.D[c];
  pdl_wait();
  pdl_trigger();
  const float dt = softplus(a.dt[(size_t)t * a.lddt + c] + bias), x = load_act(static_cast<const X*>(a.x) + (size_t)t * a.ldx + c), dx = dt * x;
  const float z = a.proj[(size_t)t * a.ld + a.z_col + c];
  const float* b = a.bc + (size_t)t * a.ldbc + a.b_col + ln * NS;
  const float* cc = a.bc + (size_t)t * a.ldbc + a.c_col + ln * NS;
  const float dl = EXACT ? dt : dt * kLog2e;
  float y = 0.0f;
#pragma unroll
  for (int i = 0; i < NS / 4; ++i) {
    const bool in = ln * NS + 4 * i < a.states;
    const float4 bv = in ? *reinterpret_cast<const float4*>(b + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 cv = in ? *reinterpret_cast<const float4*>(cc + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    s[i].x = fmaf(decay<EXACT>(dl, A[i].x), s[i].x, dx * bv.x);
    s[i].y = fmaf(decay<EXACT>(dl, A[i].y), s[i].y, dx * bv.y);
    s[i].z = fmaf(decay<EXACT>(dl, A[i].z), s[i].z, dx * bv.z);
    s[i].w = fmaf(decay<EXACT>(dl, A[i].w), s[i].w, dx * bv.w);
    y = fmaf(s[i].x, cv.x, y);
    y = fmaf(s[i].y, cv.y, y);
    y = fmaf(s[i].z, cv.z, y);
    y = fmaf(s[i].w, cv.w, y);
    if (on) *reinterpret_cast<float4*>(S + 4 * i) = s[i];
  }
#pragma unroll
  for (int o = LN / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (ln == 0 && on) store_act(static_cast<X*>(a.out) + (size_t)t * a.ldo + c, fmaf(D, x, y) * silu(z));
}

constexpr int kScanTokens = 16, kScanStages = 3;

template <int BYTES>
__device__ __forceinline__ void cp_async(void* dst, const void* src, bool ok) {
  if constexpr (BYTES == 16) {
    cp_async16(dst, src, ok);
  } else {
    static_assert(BYTES == 8, "copies of 8 or 16 bytes");
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(ok ? 8 : 0) : "memory");
  }
}

template <int LN, int NS, typename X>
struct ScanTile {
  static constexpr int CH = 128 / LN, NP = LN * NS;
  float dt[kScanTokens][CH];
  float z[kScanTokens][CH];
  float B[kScanTokens][NP];
  float C[kScanTokens][NP];
  X x[kScanTokens][CH];
};

// kWhole: grid (channels, portions), list = {first row, tokens, slot, first position}.  kLocal and kResume: grid (channels, segments), list =
// {first row, tokens, slot, last of its portion}, prompts = {slot, first position, first segment, segments}, prompt_count of them.
template <int LN, int NS, int MODE, typename X>
__global__ void __launch_bounds__(128) scan_kernel(Scan a, const int4* list, const int4* prompts, int prompt_count) {
  using Tile = ScanTile<LN, NS, X>;
  constexpr bool EXACT = sizeof(X) == 4;
  constexpr int CH = Tile::CH, NP = Tile::NP, TT = kScanTokens;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  Tile* tiles = reinterpret_cast<Tile*>(smem_raw);
  __shared__ float sdx[TT][CH], sy[TT][CH + 1];
  const int ln = threadIdx.x % LN, ch = threadIdx.x / LN, c0 = blockIdx.x * CH, c = c0 + ch;
  const bool on = c < a.channels;
  float A[NS], S[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    A[i] = on ? a.A[(size_t)c * a.np + ln * NS + i] * (EXACT ? 1.0f : kLog2e) : 0.0f;
    S[i] = 0.0f;
  }
  pdl_wait();
  pdl_trigger();
  const int4 en = list[blockIdx.y];
  if (MODE == kLocal && en.w != 0) return;       // the last segment's state is not asked for
  float* state = a.S + ((size_t)a.state_rows[en.z] * a.channels + (on ? c : 0)) * a.np + ln * NS;
  auto fetch = [&](int t0, Tile& tile) {
    for (int i = threadIdx.x; i < TT * (CH / 4); i += 128) {
      const int r = i / (CH / 4), q = (i % (CH / 4)) * 4;
      const bool ok = t0 + r < en.y && c0 + q < a.channels;
      const size_t row = ok ? en.x + t0 + r : en.x;
      cp_async16(&tile.dt[r][q], a.dt + row * a.lddt + (ok ? c0 + q : 0), ok);
      if (MODE != kLocal) cp_async16(&tile.z[r][q], a.proj + row * a.ld + a.z_col + (ok ? c0 + q : 0), ok);
    }
    constexpr int XV = CH < 16 / (int)sizeof(X) ? CH : 16 / (int)sizeof(X);
    for (int i = threadIdx.x; i < TT * (CH / XV); i += 128) {
      const int r = i / (CH / XV), q = (i % (CH / XV)) * XV;
      const bool ok = t0 + r < en.y && c0 + q < a.channels;
      cp_async<XV * (int)sizeof(X)>(&tile.x[r][q], static_cast<const X*>(a.x) + (size_t)(ok ? en.x + t0 + r : en.x) * a.ldx + (ok ? c0 + q : 0), ok);
    }
    for (int i = threadIdx.x; i < TT * (NP / 4); i += 128) {
      const int r = i / (NP / 4), q = (i % (NP / 4)) * 4;
      const bool ok = t0 + r < en.y && q < a.states;
      const float* p = a.bc + (size_t)(ok ? en.x + t0 + r : en.x) * a.ldbc + (ok ? q : 0);
      cp_async16(&tile.B[r][q], p + a.b_col, ok);
      if (MODE != kLocal) cp_async16(&tile.C[r][q], p + a.c_col, ok);
    }
  };
#pragma unroll
  for (int s = 0; s < kScanStages - 1; ++s) {
    if (s * TT < en.y) fetch(s * TT, tiles[s]);
    cp_async_commit();
  }
  // the state the first token starts from
  if (MODE == kWhole) {
    if (en.w > 0 && on)
#pragma unroll
      for (int i = 0; i < NS; ++i) S[i] = state[i];
  } else if (MODE == kResume) {
    int e = 0;
    while (e + 1 < prompt_count && prompts[e + 1].z <= (int)blockIdx.y) ++e;
    const int4 pr = prompts[e];
    if (on) {
      if (pr.y > 0)
#pragma unroll
        for (int i = 0; i < NS; ++i) S[i] = state[i];
      for (int g = pr.z; g < (int)blockIdx.y; ++g) {
        const float sum = a.seg_dt[(size_t)g * a.channels + c];
        const float* ls = a.seg_S + ((size_t)g * a.channels + c) * a.np + ln * NS;
#pragma unroll
        for (int i = 0; i < NS; ++i) S[i] = fmaf(decay<EXACT>(sum, A[i]), S[i], ls[i]);
      }
    }
  }
  float sum = 0.0f;
  int st = 0;
  for (int t0 = 0; t0 < en.y; t0 += TT) {
    const int nx = t0 + (kScanStages - 1) * TT;
    if (nx < en.y) fetch(nx, tiles[(st + kScanStages - 1) % kScanStages]);
    cp_async_commit();
    cp_async_wait<kScanStages - 1>();
    __syncthreads();
    Tile& tile = tiles[st];
    const int n = min(TT, en.y - t0);
    for (int i = threadIdx.x; i < TT * CH; i += 128) {
      const int r = i / CH, q = i % CH;
      const float dt = r < n && c0 + q < a.channels ? softplus(tile.dt[r][q] + a.dt_bias[c0 + q]) : 0.0f;    // 0: the state stays
      tile.dt[r][q] = dt;
      sdx[r][q] = dt > 0.0f ? dt * load_act(&tile.x[r][q]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int r0 = 0; r0 < TT; r0 += 4) {
      float y[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float dt = tile.dt[r0 + j][ch], dx = sdx[r0 + j][ch];
        const float4* b = reinterpret_cast<const float4*>(&tile.B[r0 + j][ln * NS]);
        const float4* cc = reinterpret_cast<const float4*>(&tile.C[r0 + j][ln * NS]);
        float v = 0.0f;
        sum += dt;
#pragma unroll
        for (int i = 0; i < NS / 4; ++i) {
          const float4 bv = b[i];
          S[4 * i] = fmaf(decay<EXACT>(dt, A[4 * i]), S[4 * i], dx * bv.x);
          S[4 * i + 1] = fmaf(decay<EXACT>(dt, A[4 * i + 1]), S[4 * i + 1], dx * bv.y);
          S[4 * i + 2] = fmaf(decay<EXACT>(dt, A[4 * i + 2]), S[4 * i + 2], dx * bv.z);
          S[4 * i + 3] = fmaf(decay<EXACT>(dt, A[4 * i + 3]), S[4 * i + 3], dx * bv.w);
          if (MODE != kLocal) {
            const float4 cv = cc[i];
            v = fmaf(S[4 * i], cv.x, v);
            v = fmaf(S[4 * i + 1], cv.y, v);
            v = fmaf(S[4 * i + 2], cv.z, v);
            v = fmaf(S[4 * i + 3], cv.w, v);
          }
        }
        y[j] = v;
      }
      if (MODE != kLocal) {
        // lane j of every four ends with the sum of token r0 + j over the channel's lanes
        const bool h1 = ln & 1, h2 = ln & 2;
        float k0 = h1 ? y[1] : y[0], k1 = h1 ? y[3] : y[2];
        k0 += __shfl_xor_sync(0xffffffffu, h1 ? y[0] : y[1], 1);
        k1 += __shfl_xor_sync(0xffffffffu, h1 ? y[2] : y[3], 1);
        float k = h2 ? k1 : k0;
        k += __shfl_xor_sync(0xffffffffu, h2 ? k0 : k1, 2);
#pragma unroll
        for (int o = 4; o < LN; o <<= 1) k += __shfl_xor_sync(0xffffffffu, k, o);
        if (ln < 4) sy[r0 + ln][ch] = k;
      }
    }
    if (MODE != kLocal) {
      __syncthreads();
      for (int i = threadIdx.x; i < n * CH; i += 128) {
        const int r = i / CH, q = i % CH;
        if (c0 + q < a.channels)
          store_act(static_cast<X*>(a.out) + (size_t)(en.x + t0 + r) * a.ldo + c0 + q,
                    fmaf(a.D[c0 + q], load_act(&tile.x[r][q]), sy[r][q]) * silu(tile.z[r][q]));
      }
    }
    __syncthreads();
    st = (st + 1) % kScanStages;
  }
  if (!on) return;
  if (MODE == kLocal) {
    float* ls = a.seg_S + ((size_t)blockIdx.y * a.channels + c) * a.np + ln * NS;
#pragma unroll
    for (int i = 0; i < NS; ++i) ls[i] = S[i];
    if (ln == 0) a.seg_dt[(size_t)blockIdx.y * a.channels + c] = sum;
  } else if (MODE == kWhole || en.w != 0) {
#pragma unroll
    for (int i = 0; i < NS; ++i) state[i] = S[i];
  }
}

// f32 columns col .. col + n - 1 of T rows as bf16
__global__ void __launch_bounds__(256) narrow_kernel(const float* in, int ld, int col, int n, int T, bf16* out, int ldo) {
  pdl_wait();
  pdl_trigger();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)T * n) return;
  const int t = (int)(i / n), c = (int)(i % n);
  out[(size_t)t * ldo + c] = __float2bfloat16_rn(in[(size_t)t * ld + col + c]);
}

static bool fill(Gru& a, const void* const* ptrs, const int* ints) {
  a.proj = (const float*)ptrs[0]; a.z_bias = (const float*)ptrs[1]; a.u_bias = (const float*)ptrs[2]; a.S = (float*)ptrs[3]; a.pos = (const int*)ptrs[4];
  a.slots = (const int*)ptrs[5]; a.state_rows = (const int*)ptrs[6]; a.out = const_cast<void*>(ptrs[7]);
  a.ld = ints[0]; a.z_col = ints[1]; a.u_col = ints[2]; a.g_col = ints[3]; a.ldo = ints[4]; a.width = ints[5];
  return a.width >= 1 && a.ldo >= a.width;
}

// lanes per channel and states per lane
struct ScanShape {
  int ln, ns;
};
static ScanShape scan_shape(int states) {
  if (states < 1 || states > 256) return {0, 0};
  if (states <= 16) return {4, 4};
  if (states <= 32) return {4, 8};
  return {states <= 64 ? 8 : (states <= 128 ? 16 : 32), 8};
}

static bool fill(Scan& a, const void* const* ptrs, const int* ints) {
  a.proj = (const float*)ptrs[0]; a.bc = (const float*)ptrs[1]; a.dt = (const float*)ptrs[2]; a.x = ptrs[3]; a.dt_bias = (const float*)ptrs[4];
  a.A = (const float*)ptrs[5]; a.D = (const float*)ptrs[6]; a.S = (float*)ptrs[7]; a.pos = (const int*)ptrs[8]; a.slots = (const int*)ptrs[9];
  a.state_rows = (const int*)ptrs[10]; a.out = const_cast<void*>(ptrs[11]); a.seg_S = (float*)ptrs[12]; a.seg_dt = (float*)ptrs[13];
  a.ld = ints[0]; a.z_col = ints[1]; a.ldbc = ints[2]; a.b_col = ints[3]; a.c_col = ints[4]; a.lddt = ints[5]; a.ldx = ints[6]; a.ldo = ints[7];
  a.channels = ints[8]; a.states = ints[9];
  const ScanShape s = scan_shape(a.states);
  a.np = s.ln * s.ns;
  const int up = (a.channels + 3) / 4 * 4;
  return s.ln > 0 && a.channels >= 1 && a.ldo >= a.channels && a.lddt >= up && a.ldx >= up && a.ld >= a.z_col + up &&
         (a.ld | a.z_col | a.ldbc | a.b_col | a.c_col | a.lddt | a.ldx) % 4 == 0 && a.ldbc >= a.c_col + (a.states + 3) / 4 * 4;
}

#define BONSAI_SCAN(LN, NS, CALL) { constexpr int kLN = LN, kNS = NS; return CALL; }
#define BONSAI_BY_STATES(CALL)                                                 \
  {                                                                            \
    const ScanShape s = scan_shape(a.states);                                  \
    if (s.ns == 4) BONSAI_SCAN(4, 4, CALL)                                     \
    if (s.ln == 4) BONSAI_SCAN(4, 8, CALL)                                     \
    if (s.ln == 8) BONSAI_SCAN(8, 8, CALL)                                     \
    if (s.ln == 16) BONSAI_SCAN(16, 8, CALL)                                   \
    BONSAI_SCAN(32, 8, CALL)                                                   \
  }

template <int LN, int NS, typename X>
static int run_step(const Scan& a, int rows, cudaStream_t stream) {
  constexpr int CH = 128 / LN;
  return launch(scan_step_kernel<LN, NS, X>, dim3((a.channels + CH - 1) / CH, rows), 128, 0, stream, 1, 0, a);
}

template <int LN, int NS, typename X>
static int run_scan(const Scan& a, const int* entries, int count, const int* segments, int nseg, const int* prompts, cudaStream_t stream) {
  constexpr int CH = 128 / LN;
  constexpr size_t smem = kScanStages * sizeof(ScanTile<LN, NS, X>);
  static_assert(smem <= 200 * 1024 && sizeof(ScanTile<LN, NS, X>) % 16 == 0, "shared memory of a CTA");
  const int blocks = (a.channels + CH - 1) / CH;
  if (nseg == 0) return launch(scan_kernel<LN, NS, kWhole, X>, dim3(blocks, count), 128, smem, stream, 1, 0, a, (const int4*)entries, (const int4*)nullptr, 0);
  if constexpr (sizeof(X) == 2) {
    const int st = launch(scan_kernel<LN, NS, kLocal, X>, dim3(blocks, nseg), 128, smem, stream, 1, 0, a, (const int4*)segments, (const int4*)prompts, count);
    if (st != BONSAI_CUDA_OK) return st;
    return launch(scan_kernel<LN, NS, kResume, X>, dim3(blocks, nseg), 128, smem, stream, 1, 0, a, (const int4*)segments, (const int4*)prompts, count);
  }
  return BONSAI_CUDA_BAD_ARG;
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// minGRU: ptrs = {proj, z_bias, u_bias, S, pos, slots, state_rows, out}, ints = {ld, z_col, u_col, g_col, ldo, width}; out f32 when exact,
// otherwise bf16.  One token in each of the rows 0 .. rows - 1:
int bonsai_lay_gru_step(const void* const* ptrs, const int* ints, const float*, int rows, int exact, cudaStream_t stream) {
  using namespace bonsai::lay;
  Gru a;
  if (!fill(a, ptrs, ints) || rows < 1 || rows > 65535) return BONSAI_CUDA_BAD_ARG;
  const dim3 grid((a.width + 127) / 128, rows);
  return exact ? launch(gru_step_kernel<float>, grid, 128, 0, stream, 1, 0, a) : launch(gru_step_kernel<bf16>, grid, 128, 0, stream, 1, 0, a);
}

// Portions entries[e] = {first row, tokens, slot, first position}; cluster: CTAs (1, 2, 4 or 8) that share a portion's tokens.
int bonsai_lay_gru_scan(const void* const* ptrs, const int* ints, const float*, const int* entries, int count, int cluster, int exact, cudaStream_t stream) {
  using namespace bonsai::lay;
  Gru a;
  if (!fill(a, ptrs, ints) || count < 1 || count > 65535 || (cluster != 1 && cluster != 2 && cluster != 4 && cluster != 8)) return BONSAI_CUDA_BAD_ARG;
  const dim3 grid((a.width + 31) / 32 * cluster, count);
  return exact ? launch(gru_scan_kernel<float>, grid, 32 * kGruWarps, 0, stream, cluster, 0, a, (const int4*)entries)
               : launch(gru_scan_kernel<bf16>, grid, 32 * kGruWarps, 0, stream, cluster, 0, a, (const int4*)entries);
}
int bonsai_lay_gru_tokens() { return bonsai::lay::kGruTokens * bonsai::lay::kGruWarps; }

// states of a channel as they are stored (0: more than the kernels take), and channels of a CTA
int bonsai_lay_scan_states(int states) {
  const bonsai::lay::ScanShape s = bonsai::lay::scan_shape(states);
  return s.ln * s.ns;
}
int bonsai_lay_scan_channels(int states) {
  const bonsai::lay::ScanShape s = bonsai::lay::scan_shape(states);
  return s.ln > 0 ? 128 / s.ln : 0;
}

// Selective scan: ptrs = {proj, bc, dt, x, dt_bias, A, D, S, pos, slots, state_rows, out, seg_S, seg_dt}, ints = {ld, z_col, ldbc, b_col, c_col,
// lddt, ldx, ldo, channels, states}; x and out f32 when exact, otherwise bf16.  One token in each of the rows 0 .. rows - 1:
int bonsai_lay_scan_step(const void* const* ptrs, const int* ints, const float*, int rows, int exact, cudaStream_t stream) {
  using namespace bonsai::lay;
  Scan a;
  if (!fill(a, ptrs, ints) || rows < 1 || rows > 65535) return BONSAI_CUDA_BAD_ARG;
  if (exact) BONSAI_BY_STATES((run_step<kLN, kNS, float>(a, rows, stream)))
  BONSAI_BY_STATES((run_step<kLN, kNS, bf16>(a, rows, stream)))
}

// Portions as above, or (nseg > 0, not exact) their segments {first row, tokens, slot, last of its portion} with prompts {slot, first
// position, first segment, segments}.
int bonsai_lay_scan(const void* const* ptrs, const int* ints, const float*, const int* entries, int count, const int* segments, int nseg, const int* prompts,
                    int exact, cudaStream_t stream) {
  using namespace bonsai::lay;
  Scan a;
  if (!fill(a, ptrs, ints) || count < 1 || count > 65535 || nseg < 0 || nseg > 65535 || (nseg > 0 && (segments == nullptr || prompts == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  if (exact) BONSAI_BY_STATES((run_scan<kLN, kNS, float>(a, entries, count, segments, nseg, prompts, stream)))
  if (a.ldx % 8 != 0) return BONSAI_CUDA_BAD_ARG;
  BONSAI_BY_STATES((run_scan<kLN, kNS, bf16>(a, entries, count, segments, nseg, prompts, stream)))
}

int bonsai_lay_narrow(const float* in, int ld, int col, int n, int T, void* out, int ldo, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (n < 1 || T < 1 || ld < col + n || ldo < n) return BONSAI_CUDA_BAD_ARG;
  return launch(narrow_kernel, dim3((unsigned)(((long long)T * n + 255) / 256)), 256, 0, stream, 1, 0, in, ld, col, n, T, (bf16*)out, ldo);
}

}  // extern "C"
