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
// LN lanes share a channel, NS states each in registers.  Prompts stage tiles of kScanTokens tokens with asynchronous copies.  Between
// two barriers the warps prepare the step sizes of the next tile, step through one and finish the outputs of the one before.  A portion may be cut into segments that run side by
// side: first the local states of all but the last (from zero; their decay is exp(A sum of dt)), then every segment from the state its
// predecessors leave.
//
// State: f32, [row][channels] and [row][channels][NP] with the states padded to LN * NS.  A sequence's first token (position 0) starts
// from zero whatever its state row holds.  The 32-bit mode runs the same kernels on f32 activations with full-precision exponentials.
#include <cooperative_groups.h>
#include <type_traits>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

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

// 1 - sigmoid(z) and sigmoid(z) * candidate(u)
template <bool EXACT>
__device__ __forceinline__ float2 gru_map(float z, float u) {
  const float e = EXACT ? expf(-fabsf(z)) : ex2(-fabsf(z) * kLog2e), big = EXACT ? 1.0f / (1.0f + e) : __fdividef(1.0f, 1.0f + e), small = e * big;
  const float c = u >= 0.0f ? u + 0.5f : sigmoid_as<EXACT>(u);
  return z >= 0.0f ? make_float2(small, big * c) : make_float2(big, small * c);
}

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
  constexpr bool EXACT = sizeof(X) == 4;
  const float z = p[a.z_col] + zb, u = p[a.u_col] + ub, g = p[a.g_col];
  const float2 m = gru_map<EXACT>(z, u);
  const float s = fmaf(m.x, s0, m.y);
  *S = s;
  store_act(static_cast<X*>(a.out) + (size_t)t * a.ldo + c, s * silu_as<EXACT>(g));
}

constexpr int kGruTokens = 8, kGruWarps = 8;

// grid (32 channels x cluster, portions)
template <typename X>
__global__ void __launch_bounds__(32 * kGruWarps, 4) gru_scan_kernel(Gru a, const int4* entries) {
  constexpr bool EXACT = sizeof(X) == 4;
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
  float state = on && en.w > 0 ? *S : 0.0f;                // of the tokens ahead of these
  const float zb = on ? a.z_bias[c] : 0.0f, ub = on ? a.u_bias[c] : 0.0f;
  const float* base = a.proj + (size_t)en.x * a.ld + c;
  const int per_turn = ctas * kGruWarps * kGruTokens, mine = (rank * kGruWarps + warp) * kGruTokens;
  int par = 0;
  for (int r0 = 0; r0 < en.y; r0 += per_turn, par ^= 1) {
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
      const float2 m = gru_map<EXACT>(keep[i] + zb, add[i] + ub);
      add[i] = i < n ? m.y : 0.0f;
      keep[i] = i < n ? m.x : 1.0f;
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
      cluster.sync();        // the other buffer is free again: everyone is past the reads of two turns ago
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
      if (i < n) store_act(dst + (size_t)i * a.ldo, s * silu_as<EXACT>(gate[i]));
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
  alignas(16) float s[NS], A[NS];
  float* S = a.S + ((size_t)a.state_rows[a.slots[t]] * a.channels + c) * a.np + ln * NS;
  const bool zero = a.pos[t] == 0;
  constexpr int VW = NS < 4 ? NS : 4;
  using Vec = typename std::conditional<VW == 4, float4, float2>::type;
  auto load = [&](const float* p, float* v) { *reinterpret_cast<Vec*>(v) = *reinterpret_cast<const Vec*>(p); };
#pragma unroll
  for (int i = 0; i < NS; i += VW) {             // older than the kernel before this one
    load(S + i, s + i);
    load(a.A + (size_t)c * a.np + ln * NS + i, A + i);
#pragma unroll
    for (int j = 0; j < VW; ++j) s[i + j] = zero ? 0.0f : s[i + j];
  }
  const float bias = a.dt_bias[c], D = a.D[c];
  pdl_wait();
  pdl_trigger();
  const float dt = softplus_as<EXACT>(a.dt[(size_t)t * a.lddt + c] + bias), x = load_act(static_cast<const X*>(a.x) + (size_t)t * a.ldx + c), dx = dt * x;
  const float z = a.proj[(size_t)t * a.ld + a.z_col + c];
  const float* b = a.bc + (size_t)t * a.ldbc + a.b_col + ln * NS;
  const float* cc = a.bc + (size_t)t * a.ldbc + a.c_col + ln * NS;
  const float dl = EXACT ? dt : dt * kLog2e;
  float y = 0.0f;
#pragma unroll
  for (int i = 0; i < NS; i += VW) {
    alignas(16) float bv[VW], cv[VW];
#pragma unroll
    for (int j = 0; j < VW; ++j) bv[j] = cv[j] = 0.0f;
    if (ln * NS + i < (a.states + 3) / 4 * 4) {     // the projections are padded to four columns
      load(b + i, bv);
      load(cc + i, cv);
    }
#pragma unroll
    for (int j = 0; j < VW; ++j) {
      s[i + j] = fmaf(decay<EXACT>(dl, A[i + j]), s[i + j], dx * bv[j]);
      y = fmaf(s[i + j], cv[j], y);
    }
    if (on) *reinterpret_cast<Vec*>(S + i) = *reinterpret_cast<const Vec*>(s + i);
  }
#pragma unroll
  for (int o = LN / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (ln == 0 && on) store_act(static_cast<X*>(a.out) + (size_t)t * a.ldo + c, fmaf(D, x, y) * silu_as<EXACT>(z));
}

constexpr int kScanTokens = 16, kScanStages = 5;   // tiles: finished, stepped through, prepared, and two on their way

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
  float dx[kScanTokens][CH];      // dt x, then y
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
  const int ln = threadIdx.x % LN, ch = threadIdx.x / LN, c0 = blockIdx.x * CH;
  const bool on = c0 + ch < a.channels;
  const int c = on ? c0 + ch : 0;
  float A[NS], S[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    A[i] = on ? a.A[(size_t)c * a.np + ln * NS + i] * (EXACT ? 1.0f : kLog2e) : 0.0f;
    S[i] = 0.0f;
  }
  // of the channel this thread prepares and finishes
  static_assert(128 % CH == 0, "every thread keeps to one channel of a tile");
  const int pq = threadIdx.x % CH, pr = threadIdx.x / CH;
  const bool pin = c0 + pq < a.channels;
  const float bias = pin ? a.dt_bias[c0 + pq] : 0.0f, D = pin ? a.D[c0 + pq] : 0.0f;
  pdl_wait();
  pdl_trigger();
  const int4 en = list[blockIdx.y];
  if (MODE == kLocal && en.w != 0) return;       // the last segment's state is not asked for
  float* state = a.S + ((size_t)a.state_rows[en.z] * a.channels + c) * a.np + ln * NS;
  // copies of a tile: thread i has chunks i, i + 128, .. of each array, and where they come from in the next tile
  constexpr int QF = CH / 4, XV = CH < 16 / (int)sizeof(X) ? CH : 16 / (int)sizeof(X), QX = CH / XV, QN = NP / 4;
  constexpr int NF = (TT * QF + 127) / 128, NX = (TT * QX + 127) / 128, NN = (TT * QN + 127) / 128;
  const float *from_dt[NF], *from_z[NF], *from_b[NN];
  const X* from_x[NX];
  const int c_off = a.c_col - a.b_col;
#pragma unroll
  for (int k = 0; k < NF; ++k) {
    const int i = threadIdx.x + 128 * k, r = i / QF, q = min(c0 + (i % QF) * 4, (a.channels - 1) & ~3);
    from_dt[k] = a.dt + (size_t)(en.x + r) * a.lddt + q;
    from_z[k] = a.proj + (size_t)(en.x + r) * a.ld + a.z_col + q;
  }
#pragma unroll
  for (int k = 0; k < NX; ++k) {
    const int i = threadIdx.x + 128 * k;
    from_x[k] = static_cast<const X*>(a.x) + (size_t)(en.x + i / QX) * a.ldx + min(c0 + (i % QX) * XV, (a.channels - 1) / XV * XV);
  }
#pragma unroll
  for (int k = 0; k < NN; ++k) {
    const int i = threadIdx.x + 128 * k;
    from_b[k] = a.bc + (size_t)(en.x + i / QN) * a.ldbc + a.b_col + min((i % QN) * 4, (a.states - 1) & ~3);
  }
  auto fetch = [&](int t0, Tile& tile) {
#pragma unroll
    for (int k = 0; k < NF; ++k) {
      const int i = threadIdx.x + 128 * k, r = i / QF, q = (i % QF) * 4;
      if (TT * QF % 128 == 0 || i < TT * QF) {
        const bool ok = t0 + r < en.y;
        cp_async16(&tile.dt[r][q], ok ? from_dt[k] : a.dt, ok);
        if (MODE != kLocal) cp_async16(&tile.z[r][q], ok ? from_z[k] : a.dt, ok);
      }
      from_dt[k] += (size_t)TT * a.lddt;
      from_z[k] += (size_t)TT * a.ld;
    }
#pragma unroll
    for (int k = 0; k < NX; ++k) {
      const int i = threadIdx.x + 128 * k, r = i / QX, q = (i % QX) * XV;
      if (TT * QX % 128 == 0 || i < TT * QX) {
        const bool ok = t0 + r < en.y;
        cp_async<XV * (int)sizeof(X)>(&tile.x[r][q], ok ? (const void*)from_x[k] : a.dt, ok);
      }
      from_x[k] += (size_t)TT * a.ldx;
    }
#pragma unroll
    for (int k = 0; k < NN; ++k) {
      const int i = threadIdx.x + 128 * k, r = i / QN, q = (i % QN) * 4;
      if (TT * QN % 128 == 0 || i < TT * QN) {
        const bool ok = t0 + r < en.y && q < a.states;          // zeros in the padding
        cp_async16(&tile.B[r][q], ok ? from_b[k] : a.dt, ok);
        if (MODE != kLocal) cp_async16(&tile.C[r][q], ok ? from_b[k] + c_off : a.dt, ok);
      }
      from_b[k] += (size_t)TT * a.ldbc;
    }
  };
  constexpr int kAhead = kScanStages - 2;
#pragma unroll
  for (int s = 0; s < kAhead; ++s) {
    if (s * TT < en.y) fetch(s * TT, tiles[s]);
    cp_async_commit();
  }
  // step sizes of a tile; 0 past the end, where the state stays
  auto prepare = [&](int t0, Tile& tile) {
#pragma unroll
    for (int r = pr; r < TT; r += 128 / CH) {
      const bool in = t0 + r < en.y && pin;
      const float dt = in ? softplus_as<EXACT>(tile.dt[r][pq] + bias) : 0.0f;
      tile.dt[r][pq] = dt;
      tile.dx[r][pq] = in ? dt * load_act(&tile.x[r][pq]) : 0.0f;
    }
  };
  auto finish = [&](int t0, const Tile& tile) {
    X* dst = static_cast<X*>(a.out) + (size_t)(en.x + t0) * a.ldo + c0 + pq;
#pragma unroll
    for (int r = pr; r < TT; r += 128 / CH)
      if (t0 + r < en.y && pin) store_act(dst + (size_t)r * a.ldo, fmaf(D, load_act(&tile.x[r][pq]), tile.dx[r][pq]) * silu_as<EXACT>(tile.z[r][pq]));
  };
  // the state the first token starts from
  if (MODE == kWhole) {
    if (en.w > 0 && on)
#pragma unroll
      for (int i = 0; i < NS; ++i) S[i] = state[i];
  } else if (MODE == kResume) {
    int e = 0;
    while (e + 1 < prompt_count && prompts[e + 1].z <= (int)blockIdx.y) ++e;
    const int4 prompt = prompts[e];
    if (on) {
      if (prompt.y > 0)
#pragma unroll
        for (int i = 0; i < NS; ++i) S[i] = state[i];
      for (int g = prompt.z; g < (int)blockIdx.y; ++g) {
        const float through = a.seg_dt[(size_t)g * a.channels + c];
        const float* ls = a.seg_S + ((size_t)g * a.channels + c) * a.np + ln * NS;
#pragma unroll
        for (int i = 0; i < NS; ++i) S[i] = fmaf(decay<EXACT>(through, A[i]), S[i], ls[i]);
      }
    }
  }
  float sum = 0.0f;
  // four tokens of a tile: what they need, and the steps
  constexpr int VW = NS < 4 ? NS : 4;
  using Vec = typename std::conditional<VW == 4, float4, float2>::type;
  struct Four {
    float dt[4], dx[4];
    alignas(16) float B[4][NS], C[4][NS];
  };
  auto load_four = [&](const Tile& tile, int r0, Four& f) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      f.dt[j] = tile.dt[r0 + j][ch];
      f.dx[j] = tile.dx[r0 + j][ch];
#pragma unroll
      for (int i = 0; i < NS / VW; ++i) {
        *reinterpret_cast<Vec*>(&f.B[j][VW * i]) = *reinterpret_cast<const Vec*>(&tile.B[r0 + j][ln * NS + VW * i]);
        if (MODE != kLocal) *reinterpret_cast<Vec*>(&f.C[j][VW * i]) = *reinterpret_cast<const Vec*>(&tile.C[r0 + j][ln * NS + VW * i]);
      }
    }
  };
  auto step_four = [&](Tile& tile, int r0, const Four& f) {
    float y[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float v = 0.0f;
      if (MODE == kLocal) sum += f.dt[j];
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        S[i] = fmaf(decay<EXACT>(f.dt[j], A[i]), S[i], f.dx[j] * f.B[j][i]);
        if (MODE != kLocal) v = fmaf(S[i], f.C[j][i], v);
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
      if (ln < 4) tile.dx[r0 + ln][ch] = k;          // every lane of the channel has read these tokens' dx
    }
  };
  cp_async_wait<kAhead - 1>();
  __syncthreads();
  prepare(0, tiles[0]);
  int slot = 0;
  auto after = [&](int n) { return slot + n < kScanStages ? slot + n : slot + n - kScanStages; };
  for (int t0 = 0; t0 < en.y; t0 += TT, slot = after(1)) {
    cp_async_wait<kAhead - 2>();                     // the next tile has landed
    __syncthreads();
    if (t0 + kAhead * TT < en.y) fetch(t0 + kAhead * TT, tiles[after(kAhead)]);
    cp_async_commit();
    if (t0 + TT < en.y) prepare(t0 + TT, tiles[after(1)]);
    Tile& tile = tiles[slot];
    if constexpr (NS <= 4) {                         // a group's loads ahead of the steps of the one before
      Four f[2];
      load_four(tile, 0, f[0]);
#pragma unroll
      for (int g = 0; g < TT / 4; ++g) {
        if (g + 1 < TT / 4) load_four(tile, 4 * g + 4, f[(g + 1) & 1]);
        step_four(tile, 4 * g, f[g & 1]);
      }
    } else {
#pragma unroll
      for (int g = 0; g < TT / 4; ++g) {
        Four f;
        load_four(tile, 4 * g, f);
        step_four(tile, 4 * g, f);
      }
    }
    if (MODE != kLocal && t0 > 0) finish(t0 - TT, tiles[after(kScanStages - 1)]);
  }
  if (MODE != kLocal) {
    __syncthreads();
    slot = after(kScanStages - 1);
    finish((en.y - 1) / TT * TT, tiles[slot]);
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

// lanes per channel and states per lane: single tokens stream the state and take few lanes, prompts are short of warps and take many;
// both keep the same number of states
struct ScanShape {
  int ln, ns;
};
static ScanShape step_shape(int states) {
  if (states < 1 || states > 256) return {0, 0};
  if (states <= 16) return {4, 4};
  return {states <= 32 ? 4 : (states <= 64 ? 8 : (states <= 128 ? 16 : 32)), 8};
}
static ScanShape scan_shape(int states) {
  if (states < 1 || states > 256) return {0, 0};
  if (states <= 16) return {8, 2};
  return {states <= 32 ? 8 : (states <= 64 ? 16 : 32), states <= 128 ? 4 : 8};
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

#define BONSAI_SHAPE(LN, NS, CALL)             \
  if (s.ln == LN && s.ns == NS) {              \
    constexpr int kLN = LN, kNS = NS;          \
    return CALL;                               \
  }
#define BONSAI_STEP_SHAPES(CALL)                                                                                                              \
  {                                                                                                                                           \
    const ScanShape s = step_shape(a.states);                                                                                                 \
    BONSAI_SHAPE(4, 4, CALL) BONSAI_SHAPE(4, 8, CALL) BONSAI_SHAPE(8, 8, CALL) BONSAI_SHAPE(16, 8, CALL) BONSAI_SHAPE(32, 8, CALL)              \
  }
#define BONSAI_SCAN_SHAPES(CALL)                                                                                                              \
  {                                                                                                                                           \
    const ScanShape s = scan_shape(a.states);                                                                                                 \
    BONSAI_SHAPE(8, 2, CALL) BONSAI_SHAPE(8, 4, CALL) BONSAI_SHAPE(16, 4, CALL) BONSAI_SHAPE(32, 4, CALL) BONSAI_SHAPE(32, 8, CALL)             \
  }

template <int LN, int NS, typename X>
static int run_step(const Scan& a, int rows, cudaStream_t stream) {
  constexpr int CH = 128 / LN;
  return launch(scan_step_kernel<LN, NS, X>, dim3((a.channels + CH - 1) / CH, rows), 128, 0, stream, 1, 0, a);
}

template <int LN, int NS, typename X>
static int run_scan(const Scan& a, const int* entries, int count, const int* segments, int nseg, const int* prompts, cudaStream_t stream) {
  constexpr int CH = ScanTile<LN, NS, X>::CH;
  constexpr size_t smem = kScanStages * sizeof(ScanTile<LN, NS, X>);
  static_assert(smem <= 227 * 1024 && sizeof(ScanTile<LN, NS, X>) % 16 == 0, "shared memory of a CTA");
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
  if (exact) BONSAI_STEP_SHAPES((run_step<kLN, kNS, float>(a, rows, stream)))
  BONSAI_STEP_SHAPES((run_step<kLN, kNS, bf16>(a, rows, stream)))
  return BONSAI_CUDA_BAD_ARG;
}

// Portions as above, or (nseg > 0, not exact) their segments {first row, tokens, slot, last of its portion} with prompts {slot, first
// position, first segment, segments}.
int bonsai_lay_scan(const void* const* ptrs, const int* ints, const float*, const int* entries, int count, const int* segments, int nseg, const int* prompts,
                    int exact, cudaStream_t stream) {
  using namespace bonsai::lay;
  Scan a;
  if (!fill(a, ptrs, ints) || count < 1 || count > 65535 || nseg < 0 || nseg > 65535 || (nseg > 0 && (segments == nullptr || prompts == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  if (exact) BONSAI_SCAN_SHAPES((run_scan<kLN, kNS, float>(a, entries, count, segments, nseg, prompts, stream)))
  if (a.ldx % 8 != 0) return BONSAI_CUDA_BAD_ARG;
  BONSAI_SCAN_SHAPES((run_scan<kLN, kNS, bf16>(a, entries, count, segments, nseg, prompts, stream)))
  return BONSAI_CUDA_BAD_ARG;
}

int bonsai_lay_narrow(const float* in, int ld, int col, int n, int T, void* out, int ldo, cudaStream_t stream) {
  using namespace bonsai::lay;
  if (n < 1 || T < 1 || ld < col + n || ldo < n) return BONSAI_CUDA_BAD_ARG;
  return launch(narrow_kernel, dim3((unsigned)(((long long)T * n + 255) / 256)), 256, 0, stream, 1, 0, in, ld, col, n, T, (bf16*)out, ldo);
}

}  // extern "C"
