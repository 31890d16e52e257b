// Matrix-memory recurrence (mLSTM): per head a matrix S [dim][vdim], a vector n [dim] and a running maximum m, all f32.
//
//   i = cap tanh((W_i h + b_i) / cap), f = logsigmoid(cap tanh((W_f h + b_f) / cap))
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' likewise with k;  o = S'^T q / (max(|n' . q|, e^-m') + 1e-6)
//
// `step_kernel` runs the recurrence as written, a column tile of 64 values of one head per CTA with the state in registers.
// For single tokens (decode) the column tiles of a head form a cluster, exchange the sum of squares of the head's output
// through distributed shared memory, and write the finished activations (head norm, norm weight, output gate); for several
// tokens (32-bit mode) it leaves o for the gated head norm.
//
// `chunk_kernel` handles portions of prompts on the tensor cores, 64 tokens at a time.  With F the running sum of f inside the
// chunk and m_t from the recurrence itself (an associative scan), token t sees token s <= t with weight
// e^(F_t - F_s + i_s - m_t) and the chunk's initial state with weight e^(F_t + m_0 - m_t), so every exponent is <= 0:
//   o_t ~ sum_s w_ts (q_t . k_s) v_s + g_t S_0^T q_t,   n_t . q_t = sum_s w_ts (q_t . k_s) + g_t n_0 . q_t
// Gates, weights, normaliser and state are f32; the state and the weighted values enter their products as a bf16 pair
// (value and remainder), i.e. with 16 significant bits.
//
// A long prompt in few sequences leaves most SMs idle, since its chunks follow one another.  It is then cut into segments:
// every segment but the last first runs from an empty state (state products only), `combine_kernel` turns these local states
// into the state each segment starts from - with (F, m, S, n) of a segment: m' = max(F + m_prev, m),
// S' = e^(F + m_prev - m') S_prev + e^(m - m') S - and a second pass computes the outputs of all segments at once.
//
// State layout: S [row][head][DIM][VP], n [row][head][VP / 64][DIM], m [row][head][VP / 64] - every column tile keeps its own
// copy of n and m - with DIM, VP the padded sizes; the padding stays zero.  A sequence's first token (position 0) starts from
// zero whatever its state row holds.
#include <cooperative_groups.h>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

struct Mlstm {
  const float* proj;       // [T][ld]: q heads at q_col, k heads at k_col, v heads at v_col, gate at g_col, i at i_col, f at f_col
  const float* i_bias;     // [heads]
  const float* f_bias;
  const float* norm;       // [heads * vdim]
  float* S;
  float* n;
  float* m;
  const int* pos;          // [T]
  const int* slots;        // [T]
  const int* state_rows;   // [slots]
  void* out;               // finished activations [T][ldo] or o f32 [T][ldo]
  int ld, q_col, k_col, v_col, g_col, i_col, f_col, ldo;
  int heads, dim, vdim, vp;
  int vec;                 // head rows start on 16-byte boundaries
  float cap, eps, den_eps, q_scale;
  // segmented prompts: one state per segment, laid out like the pool's rows, and per column tile the local state's F and m
  float* seg_S;
  float* seg_n;
  float* seg_m;
  float* seg_F;
};

__device__ __forceinline__ float log_input_gate(const Mlstm& a, float raw, int h) { return a.cap * tanhf((raw + a.i_bias[h]) / a.cap); }
__device__ __forceinline__ float log_forget_gate(const Mlstm& a, float raw, int h) {
  const float x = a.cap * tanhf((raw + a.f_bias[h]) / a.cap);
  return fminf(x, 0.0f) - log1pf(expf(-fabsf(x)));
}

// grid (vp / 64, heads, entries); threads = 16 column quads x DG groups of state rows, DPT state rows per thread
// (DIM = DG * DPT).  ONE: one token in each of the rows 0 .. gridDim.z - 1, otherwise entries[e] = {first row, tokens, slot,
// first position}.  FINISH: finished outputs, clusters along x; otherwise o is stored.
template <int DG, int DPT, bool ONE, bool FINISH, typename OUT>
__global__ void __launch_bounds__(16 * DG) step_kernel(Mlstm a, const int4* entries) {
  static_assert(ONE || !FINISH, "only single tokens are finished here");
  constexpr int DIM = DG * DPT, NTH = 16 * DG;
  __shared__ float sq[DIM], sk[DIM], red[DG][68], s32[32];
  __shared__ float s_ss;
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int h = blockIdx.y, tile = blockIdx.x, ntile = gridDim.x;
  const int cq = threadIdx.x & 15, dg = threadIdx.x >> 4, col = tile * 64 + cq * 4;
  int t0, count, slot, pos0;
  if (ONE) {
    t0 = blockIdx.z;
    count = 1;
    slot = a.slots[t0];
    pos0 = a.pos[t0];
  } else {
    pdl_wait();            // the entry list may be written by the kernel before
    pdl_trigger();
    const int4 en = entries[blockIdx.z];
    t0 = en.x; count = en.y; slot = en.z; pos0 = en.w;
  }
  const size_t sh = (size_t)a.state_rows[slot] * a.heads + h;
  float* S = a.S + sh * DIM * a.vp + col;
  float* gn = a.n + (sh * ntile + tile) * DIM;
  float* gm = a.m + sh * ntile + tile;
  // the state is older than the kernel before this one
  float4 s[DPT];
#pragma unroll
  for (int i = 0; i < DPT; ++i)
    s[i] = pos0 == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (size_t)(dg + i * DG) * a.vp);
  float nv = threadIdx.x < DIM && pos0 != 0 ? gn[threadIdx.x] : 0.0f;     // thread d < DIM owns n[d]
  float nv2 = threadIdx.x + NTH < DIM && pos0 != 0 ? gn[threadIdx.x + NTH] : 0.0f;
  static_assert(DIM <= 2 * NTH, "a thread owns at most two elements of n");
  float m = pos0 == 0 ? 0.0f : *gm;
  if (ONE) {
    pdl_wait();
    pdl_trigger();
  }
  for (int tt = 0; tt < count; ++tt) {
    const float* p = a.proj + (size_t)(t0 + tt) * a.ld;
    for (int d = threadIdx.x; d < DIM; d += NTH) {
      sq[d] = d < a.dim ? p[a.q_col + h * a.dim + d] * a.q_scale : 0.0f;
      sk[d] = d < a.dim ? p[a.k_col + h * a.dim + d] : 0.0f;
    }
    float v[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) v[c] = col + c < a.vdim ? p[a.v_col + h * a.vdim + col + c] : 0.0f;
    const float ig = log_input_gate(a, p[a.i_col + h], h), fg = log_forget_gate(a, p[a.f_col + h], h);
    const float mn = fmaxf(fg + m, ig), fa = expf(fg + m - mn), ib = expf(ig - mn);
    m = mn;
    __syncthreads();
    float nq = 0.0f;
    if (threadIdx.x < DIM) {
      nv = fa * nv + ib * sk[threadIdx.x];
      nq = nv * sq[threadIdx.x];
    }
    if (threadIdx.x + NTH < DIM) {
      nv2 = fa * nv2 + ib * sk[threadIdx.x + NTH];
      nq += nv2 * sq[threadIdx.x + NTH];
    }
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const float kb = ib * sk[dg + i * DG], q = sq[dg + i * DG];
      s[i].x = fa * s[i].x + kb * v[0];
      s[i].y = fa * s[i].y + kb * v[1];
      s[i].z = fa * s[i].z + kb * v[2];
      s[i].w = fa * s[i].w + kb * v[3];
      acc.x += s[i].x * q;
      acc.y += s[i].y * q;
      acc.z += s[i].z * q;
      acc.w += s[i].w * q;
    }
    *reinterpret_cast<float4*>(&red[dg][cq * 4]) = acc;
    nq = block_sum(nq, s32);           // its barriers also order the stores to red
    const float den = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + a.den_eps);
    float o = 0.0f;
    const int oc = tile * 64 + threadIdx.x;
    if (threadIdx.x < 64) {
#pragma unroll
      for (int g = 0; g < DG; ++g) o += red[g][threadIdx.x];
      o *= den;
    }
    if (!FINISH) {
      if (threadIdx.x < 64 && oc < a.vdim) static_cast<float*>(a.out)[(size_t)(t0 + tt) * a.ldo + h * a.vdim + oc] = o;
      __syncthreads();                 // sq, sk and red are free
    } else {
      const float ss = block_sum(threadIdx.x < 64 ? o * o : 0.0f, s32);
      if (threadIdx.x == 0) s_ss = ss;
      float total = ss;
      if (ntile > 1) {
        cluster.sync();
        total = 0.0f;
        for (int r = 0; r < ntile; ++r) total += *cluster.map_shared_rank(&s_ss, r);
      }
      if (threadIdx.x < 64 && oc < a.vdim) {
        const int c = h * a.vdim + oc;
        const float y = o / sqrtf(total / (float)a.vdim + a.eps) * a.norm[c] * sigmoid(p[a.g_col + c]);
        store_act(static_cast<OUT*>(a.out) + (size_t)t0 * a.ldo + c, y);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < DPT; ++i) *reinterpret_cast<float4*>(S + (size_t)(dg + i * DG) * a.vp) = s[i];
  if (threadIdx.x < DIM) gn[threadIdx.x] = nv;
  if (threadIdx.x + NTH < DIM) gn[threadIdx.x + NTH] = nv2;
  if (threadIdx.x == 0) *gm = m;
  if (FINISH && ntile > 1) cluster.sync();   // nobody leaves while its sum is being read
}

// ---- portions of prompts ------------------------------------------------------------------------------------------------------------
constexpr int chunk_warps(int dim) { return dim >= 256 ? 16 : 8; }

template <int DIM>
struct ChunkSmem {
  static constexpr int LD = DIM + 8, NCH = chunk_warps(DIM) / 4;
  bf16 q[kL * LD], k[kL * LD];
  bf16 v[kL * kVLD], vh[kL * kVLD], vl[kL * kVLD];   // values; weighted values: leading part and remainder
  bf16 sh[DIM * kVLD], sl[DIM * kVLD];               // state at the start of the chunk: leading part and remainder
  bf16 p[kL * kVLD];                                 // weighted scores
  float n[DIM];
  struct alignas(16) Gates {
    float c[kL];        // i_s - F_s
    float r[kL];        // F_t - m_t
    float g[kL];        // weight of the initial state
    float em[kL];       // e^-m_t
    float w[kL];        // weight of token s in the final state
    float tail[4];      // decay of the state over the chunk, m and F at its end
  } gates[2];           // this chunk's and the next one's
  float rows[NCH][kL];  // row sums of p over the warps' key columns
  float nq[kL];         // q_t . n_0
};

// grid (vp / 64, heads, entries).  Warp w: rows (w & 3) * 16 .. + 15 of the chunk and group w >> 2 of the columns (keys and
// values); of the state two 16-row tiles and WN 8-column tiles.
// kWhole: entries {first row, tokens, slot, first position}, state from and to the pool.  kLocal / kResume: entries are the
// segments {first row, tokens, slot, last of its prompt}; kLocal leaves a segment's local state in its scratch row, kResume
// starts from the scratch row and writes the last segment's state to the pool.
template <int DIM, int MODE>
__global__ void __launch_bounds__(32 * chunk_warps(DIM), DIM <= 128 ? 2 : 1) chunk_kernel(Mlstm a, const int4* entries) {
  constexpr int LD = DIM + 8;
  constexpr int NW = chunk_warps(DIM), NTH = 32 * NW;
  constexpr int CW = 256 / NW;                       // columns of a warp's group: 64 / (NW / 4)
  constexpr int MT = DIM / 16, MG = MT / 2;          // 16-row tiles of the state, pairs of them
  constexpr int WM = 2, WN = 8 * MG / NW;            // state tiles of a warp
  static_assert(WN >= 2 && WN % 2 == 0 && MG * 8 == NW * WN, "state tiles over the warps");
  extern __shared__ __align__(16) uint8_t smem_raw[];
  ChunkSmem<DIM>& sm = *reinterpret_cast<ChunkSmem<DIM>*>(smem_raw);
  const int tile = blockIdx.x, ntile = gridDim.x, h = blockIdx.y, col0 = tile * kVT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = warp & 3, ch = warp >> 2;
  const int g = lane >> 2, t4 = lane & 3;
  pdl_wait();
  pdl_trigger();
  const int4 en = entries[blockIdx.z];
  if (MODE == kLocal && en.w) return;                // nothing resumes from the last segment's local state
  const size_t pool = (size_t)a.state_rows[en.z] * a.heads + h, seg = (size_t)blockIdx.z * a.heads + h;
  const size_t src = MODE == kWhole ? pool : seg, dst = MODE == kLocal ? seg : pool;
  const float* inS = (MODE == kWhole ? a.S : a.seg_S) + src * DIM * a.vp + col0;
  const float* in_n = (MODE == kWhole ? a.n : a.seg_n) + (src * ntile + tile) * DIM;
  const bool fresh = MODE == kLocal || (MODE == kWhole && en.w == 0);
  auto state_row = [&](int i) { return ((warp % MG) * 2 + i) * 16; };
  const int sc0 = (warp / MG) * WN * 8;              // first column of this warp's state tiles
  float st[WM][WN][4];
#pragma unroll
  for (int i = 0; i < WM; ++i)
#pragma unroll
    for (int j = 0; j < WN; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float2 v = make_float2(0.f, 0.f);
        if (!fresh) v = *reinterpret_cast<const float2*>(inS + (size_t)(state_row(i) + g + 8 * e) * a.vp + sc0 + j * 8 + 2 * t4);
        st[i][j][2 * e] = v.x;
        st[i][j][2 * e + 1] = v.y;
      }
  float nv[WM][4];      // n of this warp's state rows: column 0 of an accumulator tile (lanes with t4 == 0), warps with sc0 == 0
#pragma unroll
  for (int i = 0; i < WM; ++i) {
    nv[i][0] = fresh ? 0.0f : in_n[state_row(i) + g];
    nv[i][2] = fresh ? 0.0f : in_n[state_row(i) + g + 8];
    nv[i][1] = nv[i][3] = 0.0f;
  }
  // a local state has no floor at 0: its maximum starts empty
  float m0 = MODE == kLocal ? -INFINITY : (fresh ? 0.0f : (MODE == kWhole ? a.m : a.seg_m)[src * ntile + tile]);
  float Fsum = 0.0f;

  // One warp turns the raw gates of a chunk into its weights; it does so a chunk ahead, from values loaded earlier still.
  constexpr int kGateWarp = 4 * (NW / 4 - 1);        // the warp with the least other work: first rows, last columns
  float raw[2][2];                                   // this lane's two tokens: log forget gate's and log input gate's raw value
  auto load_raw = [&](int at) {
    const float* gp = a.proj + (size_t)(en.x + at + 2 * lane) * a.ld + h;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = at + 2 * lane + e < en.y;
      raw[e][0] = ok ? gp[(size_t)e * a.ld + a.f_col] : 0.0f;
      raw[e][1] = ok ? gp[(size_t)e * a.ld + a.i_col] : 0.0f;
    }
  };
  auto make_gates = [&](int at, float m0, typename ChunkSmem<DIM>::Gates& G) {
    // scan of (F, M): F_t = f_1 + .. + f_t, M_t = max over s <= t of F_t - F_s + i_s; two tokens per lane
    float f[2], ig[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = at + 2 * lane + e < en.y;
      f[e] = ok ? log_forget_gate(a, raw[e][0], h) : 0.0f;
      ig[e] = ok ? log_input_gate(a, raw[e][1], h) : -INFINITY;
    }
    float F = f[0] + f[1], M = fmaxf(ig[0] + f[1], ig[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(pm + F, M);
        F += pf;
      }
    }
    float eF = __shfl_up_sync(0xffffffffu, F, 1), eM = __shfl_up_sync(0xffffffffu, M, 1);   // before this lane's tokens
    if (lane == 0) {
      eF = 0.0f;
      eM = -INFINITY;
    }
    float Ft[2], Mt[2];
    Ft[0] = eF + f[0];
    Mt[0] = fmaxf(fmaxf(eM + f[0], ig[0]), Ft[0] + m0);
    Ft[1] = F;
    Mt[1] = fmaxf(M, Ft[1] + m0);
    const float FL = __shfl_sync(0xffffffffu, Ft[1], 31), mL = __shfl_sync(0xffffffffu, Mt[1], 31);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int s = 2 * lane + e;
      G.c[s] = ig[e] - Ft[e];
      G.r[s] = Ft[e] - Mt[e];
      G.g[s] = expf(Ft[e] + m0 - Mt[e]);
      G.em[s] = expf(-Mt[e]);
      G.w[s] = expf(FL - mL + ig[e] - Ft[e]);
    }
    if (lane == 0) {
      G.tail[0] = expf(FL + m0 - mL);
      G.tail[1] = mL;
      G.tail[2] = FL;
    }
  };
  if (warp == kGateWarp) {
    load_raw(0);
    make_gates(0, m0, sm.gates[0]);
  }

  for (int t0 = 0, it = 0; t0 < en.y; t0 += kL, ++it) {
    const int nt = min(kL, en.y - t0);
    const bool more = t0 + kL < en.y;
    const typename ChunkSmem<DIM>::Gates& G = sm.gates[it & 1];
    const float* base = a.proj + (size_t)(en.x + t0) * a.ld;
    // ---- stage the chunk: projections as bf16, the state as a bf16 pair, the gates ------------------------------------------------
    const float* qb = base + a.q_col + h * a.dim;
    const float* kb = base + a.k_col + h * a.dim;
    const float* vb = base + a.v_col + h * a.vdim + col0;
    if (a.vec) {
      constexpr int C4 = DIM / 4, N = kL * C4 / NTH, NB = N < 4 ? N : 4;   // float4 per thread, of which NB are in flight
      constexpr int NVV = kL * (kVT / 4) / NTH;
      const int d4 = a.dim >> 2, v4 = (a.vdim - col0) >> 2;
      float4 vv[NVV];
#pragma unroll
      for (int j = 0; j < NVV; ++j) {
        const int i = tid + j * NTH, r = i >> 4, c = i & 15;
        vv[j] = r < nt && c < v4 ? reinterpret_cast<const float4*>(vb + (size_t)r * a.ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int i0 = 0; i0 < N; i0 += NB) {
        float4 qv[NB], kv[NB];
#pragma unroll
        for (int j = 0; j < NB; ++j) {
          const int i = tid + (i0 + j) * NTH, r = i / C4, c = i % C4;
          const bool ok = r < nt && c < d4;
          if (MODE != kLocal) qv[j] = ok ? reinterpret_cast<const float4*>(qb + (size_t)r * a.ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
          kv[j] = ok ? reinterpret_cast<const float4*>(kb + (size_t)r * a.ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int j = 0; j < NB; ++j) {
          const int i = tid + (i0 + j) * NTH, r = i / C4, c = i % C4;
          if (MODE != kLocal)
            *reinterpret_cast<uint2*>(sm.q + r * LD + 4 * c) =
                make_uint2(pack_bf16(qv[j].x * a.q_scale, qv[j].y * a.q_scale), pack_bf16(qv[j].z * a.q_scale, qv[j].w * a.q_scale));
          *reinterpret_cast<uint2*>(sm.k + r * LD + 4 * c) = make_uint2(pack_bf16(kv[j].x, kv[j].y), pack_bf16(kv[j].z, kv[j].w));
        }
      }
#pragma unroll
      for (int j = 0; j < NVV; ++j) {
        const int i = tid + j * NTH, r = i >> 4, c = i & 15;
        *reinterpret_cast<uint2*>(sm.v + r * kVLD + 4 * c) = make_uint2(pack_bf16(vv[j].x, vv[j].y), pack_bf16(vv[j].z, vv[j].w));
      }
    } else {
      for (int i = tid; i < kL * DIM; i += NTH) {
        const int r = i / DIM, d = i % DIM;
        const bool ok = r < nt && d < a.dim;
        sm.q[r * LD + d] = __float2bfloat16_rn(ok ? qb[(size_t)r * a.ld + d] * a.q_scale : 0.0f);
        sm.k[r * LD + d] = __float2bfloat16_rn(ok ? kb[(size_t)r * a.ld + d] : 0.0f);
      }
      for (int i = tid; i < kL * kVT; i += NTH) {
        const int r = i / kVT, c = i % kVT;
        sm.v[r * kVLD + c] = __float2bfloat16_rn(r < nt && col0 + c < a.vdim ? vb[(size_t)r * a.ld + c] : 0.0f);
      }
    }
    if (MODE != kLocal)
#pragma unroll
    for (int i = 0; i < WM; ++i)
#pragma unroll
      for (int j = 0; j < WN; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int o = (state_row(i) + g + 8 * e) * kVLD + sc0 + j * 8 + 2 * t4;
          const float x = st[i][j][2 * e], y = st[i][j][2 * e + 1];
          const __nv_bfloat162 hi = __floats2bfloat162_rn(x, y);
          *reinterpret_cast<__nv_bfloat162*>(sm.sh + o) = hi;
          *reinterpret_cast<uint32_t*>(sm.sl + o) = pack_bf16(x - __bfloat162float(hi.x), y - __bfloat162float(hi.y));
        }
    if (MODE != kLocal && sc0 == 0 && t4 == 0) {
#pragma unroll
      for (int i = 0; i < WM; ++i) {
        sm.n[state_row(i) + g] = nv[i][0];
        sm.n[state_row(i) + g + 8] = nv[i][2];
      }
    }
    __syncthreads();
    // ---- weighted scores, the initial state's share, its normaliser, weighted values ---------------------------------------------
    if (more) {
      // the next chunk's projections into L2, its raw gates into registers
      const float* nb = base + (size_t)kL * a.ld;
      const int left = min(kL, en.y - t0 - kL);
      for (int i = tid; i < kL * (DIM / 32); i += NTH) {
        const int r = i / (DIM / 32), d = i % (DIM / 32) * 32;
        if (r < left && d < a.dim) {
          const float* p = nb + (size_t)r * a.ld + h * a.dim + d;
          if (MODE != kLocal) asm volatile("prefetch.global.L2 [%0];" ::"l"(p + a.q_col));
          asm volatile("prefetch.global.L2 [%0];" ::"l"(p + a.k_col));
        }
      }
      if (tid < 2 * kL && (tid >> 1) < left && col0 + (tid & 1) * 32 < a.vdim)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(nb + (size_t)(tid >> 1) * a.ld + a.v_col + h * a.vdim + col0 + (tid & 1) * 32));
      if (warp == kGateWarp) load_raw(t0 + kL);
    }
    float oi[CW / 8][4] = {};
    if constexpr (MODE != kLocal) {
    float s[CW / 8][4] = {};
    const bool live = ch * CW <= rg * 16 + 15;       // else all of these keys come after the rows
#pragma unroll 4
    for (int ks = 0; ks < MT; ++ks) {
      uint32_t q[4], b[4];
      ldsm4(q, frag_a(sm.q, LD, rg * 16, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < CW / 16; ++np) {
        if (live) {
          ldsm4(b, frag_b_rows(sm.k, LD, ch * CW + np * 16, ks * 16, lane));
          mma_bf16(s[2 * np], q, b[0], b[1]);
          mma_bf16(s[2 * np + 1], q, b[2], b[3]);
        }
        ldsm4_t(b, frag_b_cols(sm.sh, kVLD, ks * 16, ch * CW + np * 16, lane));
        mma_bf16(oi[2 * np], q, b[0], b[1]);
        mma_bf16(oi[2 * np + 1], q, b[2], b[3]);
        ldsm4_t(b, frag_b_cols(sm.sl, kVLD, ks * 16, ch * CW + np * 16, lane));
        mma_bf16(oi[2 * np], q, b[0], b[1]);
        mma_bf16(oi[2 * np + 1], q, b[2], b[3]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = rg * 16 + g + 8 * e;
      const float r = G.r[t];
      float sum = 0.0f;
#pragma unroll
      for (int j = 0; j < CW / 8; ++j) {
        const int k0 = ch * CW + j * 8 + 2 * t4;
        const float x = k0 <= t ? s[j][2 * e] * expf(r + G.c[k0]) : 0.0f;
        const float y = k0 + 1 <= t ? s[j][2 * e + 1] * expf(r + G.c[k0 + 1]) : 0.0f;
        sum += x + y;
        *reinterpret_cast<uint32_t*>(sm.p + t * kVLD + k0) = pack_bf16(x, y);
      }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if (t4 == 0) sm.rows[ch][t] = sum;
    }
    {
      constexpr int TPR = NTH / kL;                  // threads per row
      const int t = tid / TPR, d0 = (tid % TPR) * 8;
      float x = 0.0f;
#pragma unroll 4
      for (int d = d0; d < DIM; d += 8 * TPR) {
        const uint4 q = *reinterpret_cast<const uint4*>(sm.q + t * LD + d);
        const float4 n0 = *reinterpret_cast<const float4*>(sm.n + d), n1 = *reinterpret_cast<const float4*>(sm.n + d + 4);
        const __nv_bfloat162* qq = reinterpret_cast<const __nv_bfloat162*>(&q);
        const float2 q0 = __bfloat1622float2(qq[0]), q1 = __bfloat1622float2(qq[1]), q2 = __bfloat1622float2(qq[2]), q3 = __bfloat1622float2(qq[3]);
        x += q0.x * n0.x + q0.y * n0.y + q1.x * n0.z + q1.y * n0.w + q2.x * n1.x + q2.y * n1.y + q3.x * n1.z + q3.y * n1.w;
      }
#pragma unroll
      for (int o = 1; o < TPR; o <<= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
      if (tid % TPR == 0) sm.nq[t] = x;
    }
    }
    for (int i = tid; i < kL * (kVT / 2); i += NTH) {
      const int r = i / (kVT / 2), c = (i % (kVT / 2)) * 2;
      const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(sm.v + r * kVLD + c);
      const float x = G.w[r] * __bfloat162float(v.x), y = G.w[r] * __bfloat162float(v.y);
      const __nv_bfloat162 hi = __floats2bfloat162_rn(x, y);
      *reinterpret_cast<__nv_bfloat162*>(sm.vh + r * kVLD + c) = hi;
      *reinterpret_cast<uint32_t*>(sm.vl + r * kVLD + c) = pack_bf16(x - __bfloat162float(hi.x), y - __bfloat162float(hi.y));
    }
    __syncthreads();
    if constexpr (MODE != kLocal) {
    // ---- outputs ---------------------------------------------------------------------------------------------------------------------
    {
      const float g0 = G.g[rg * 16 + g], g1 = G.g[rg * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < CW / 8; ++j) {
        oi[j][0] *= g0; oi[j][1] *= g0;
        oi[j][2] *= g1; oi[j][3] *= g1;
      }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks > rg) break;
      uint32_t p[4], b[4];
      ldsm4(p, frag_a(sm.p, kVLD, rg * 16, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < CW / 16; ++np) {
        ldsm4_t(b, frag_b_cols(sm.v, kVLD, ks * 16, ch * CW + np * 16, lane));
        mma_bf16(oi[2 * np], p, b[0], b[1]);
        mma_bf16(oi[2 * np + 1], p, b[2], b[3]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = rg * 16 + g + 8 * e;
      if (t >= nt) continue;
      float nq = G.g[t] * sm.nq[t];
#pragma unroll
      for (int c = 0; c < NW / 4; ++c) nq += sm.rows[c][t];
      const float den = 1.0f / (fmaxf(fabsf(nq), G.em[t]) + a.den_eps);
      float* dst = static_cast<float*>(a.out) + (size_t)(en.x + t0 + t) * a.ldo + h * a.vdim + col0;
#pragma unroll
      for (int j = 0; j < CW / 8; ++j) {
        const int c = ch * CW + j * 8 + 2 * t4;
        if (col0 + c < a.vdim) dst[c] = oi[j][2 * e] * den;
        if (col0 + c + 1 < a.vdim) dst[c + 1] = oi[j][2 * e + 1] * den;
      }
    }
    }
    // ---- the state at the end of the chunk ------------------------------------------------------------------------------------------
    if (more && warp == kGateWarp) make_gates(t0 + kL, G.tail[1], sm.gates[(it + 1) & 1]);
    const float decay = G.tail[0];
    m0 = G.tail[1];
    Fsum += G.tail[2];
#pragma unroll
    for (int i = 0; i < WM; ++i)
#pragma unroll
      for (int j = 0; j < WN; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[i][j][e] *= decay;
#pragma unroll
    for (int i = 0; i < WM; ++i) {
      nv[i][0] *= decay;
      nv[i][2] *= decay;
    }
#pragma unroll
    for (int ks = 0; ks < kL / 16; ++ks) {
      uint32_t kt[WM][4], b[4];
#pragma unroll
      for (int i = 0; i < WM; ++i) ldsm4_t(kt[i], frag_a_cols(sm.k, LD, state_row(i), ks * 16, lane));
      if (sc0 == 0) {        // n: the weights themselves as a column, a bf16 pair
        const float2 w0 = *reinterpret_cast<const float2*>(G.w + ks * 16 + 2 * t4), w1 = *reinterpret_cast<const float2*>(G.w + ks * 16 + 8 + 2 * t4);
        const __nv_bfloat162 h0 = __floats2bfloat162_rn(w0.x, w0.y), h1 = __floats2bfloat162_rn(w1.x, w1.y);
        const uint32_t hi0 = g == 0 ? *reinterpret_cast<const uint32_t*>(&h0) : 0u, hi1 = g == 0 ? *reinterpret_cast<const uint32_t*>(&h1) : 0u;
        const uint32_t lo0 = g == 0 ? pack_bf16(w0.x - __bfloat162float(h0.x), w0.y - __bfloat162float(h0.y)) : 0u;
        const uint32_t lo1 = g == 0 ? pack_bf16(w1.x - __bfloat162float(h1.x), w1.y - __bfloat162float(h1.y)) : 0u;
#pragma unroll
        for (int i = 0; i < WM; ++i) {
          mma_bf16(nv[i], kt[i], hi0, hi1);
          mma_bf16(nv[i], kt[i], lo0, lo1);
        }
      }
#pragma unroll
      for (int np = 0; np < WN / 2; ++np) {
        ldsm4_t(b, frag_b_cols(sm.vh, kVLD, ks * 16, sc0 + np * 16, lane));
#pragma unroll
        for (int i = 0; i < WM; ++i) {
          mma_bf16(st[i][2 * np], kt[i], b[0], b[1]);
          mma_bf16(st[i][2 * np + 1], kt[i], b[2], b[3]);
        }
        ldsm4_t(b, frag_b_cols(sm.vl, kVLD, ks * 16, sc0 + np * 16, lane));
#pragma unroll
        for (int i = 0; i < WM; ++i) {
          mma_bf16(st[i][2 * np], kt[i], b[0], b[1]);
          mma_bf16(st[i][2 * np + 1], kt[i], b[2], b[3]);
        }
      }
    }
    __syncthreads();    // the staged tiles are free
  }
  if (MODE == kResume && !en.w) return;
  float* outS = (MODE == kLocal ? a.seg_S : a.S) + dst * DIM * a.vp + col0;
#pragma unroll
  for (int i = 0; i < WM; ++i)
#pragma unroll
    for (int j = 0; j < WN; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        *reinterpret_cast<float2*>(outS + (size_t)(state_row(i) + g + 8 * e) * a.vp + sc0 + j * 8 + 2 * t4) =
            make_float2(st[i][j][2 * e], st[i][j][2 * e + 1]);
  float* out_n = (MODE == kLocal ? a.seg_n : a.n) + (dst * ntile + tile) * DIM;
  if (sc0 == 0 && t4 == 0) {
#pragma unroll
    for (int i = 0; i < WM; ++i) {
      out_n[state_row(i) + g] = nv[i][0];
      out_n[state_row(i) + g + 8] = nv[i][2];
    }
  }
  if (tid == 0) {
    if (MODE == kLocal) *reinterpret_cast<float2*>(a.seg_F + 2 * (dst * ntile + tile)) = make_float2(Fsum, m0);
    else a.m[dst * ntile + tile] = m0;
  }
}

// Local states of the segments -> the states they start from.  grid (vp / 64 * 4, heads, prompts), 256 threads: a quarter of
// a column tile's state rows.  prompts[e] = {slot, first position, first segment, segments}.
template <int DIM>
__global__ void __launch_bounds__(256) combine_kernel(Mlstm a, const int4* prompts) {
  pdl_wait();
  pdl_trigger();
  const int tile = blockIdx.x >> 2, quarter = blockIdx.x & 3, ntile = gridDim.x >> 2, h = blockIdx.y;
  const int4 pr = prompts[blockIdx.z];
  const bool fresh = pr.y == 0;
  const size_t pool = (size_t)a.state_rows[pr.x] * a.heads + h;
  constexpr int N = DIM / 4 * 16 / 256;              // float4 per thread
  const int c = (threadIdx.x & 15) * 4, r0 = quarter * (DIM / 4) + (threadIdx.x >> 4);
  const bool vector = quarter == 0 && threadIdx.x < DIM;
  auto at = [&](float* S, size_t row, int i) { return reinterpret_cast<float4*>(S + (row * DIM + r0 + 16 * i) * a.vp + tile * 64 + c); };
  float4 s[N];
#pragma unroll
  for (int i = 0; i < N; ++i) s[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *at(a.S, pool, i);
  float n = vector && !fresh ? a.n[(pool * ntile + tile) * DIM + threadIdx.x] : 0.0f;
  float m = fresh ? 0.0f : a.m[pool * ntile + tile];
  for (int j = 0; j < pr.w; ++j) {
    const size_t row = (size_t)(pr.z + j) * a.heads + h, idx = row * ntile + tile;
    const bool last = j == pr.w - 1;                 // its scratch row holds no local state
    float4 d[N];
    float dn = 0.0f, fa = 0.0f, fb = 0.0f, mn = m;
    if (!last) {
#pragma unroll
      for (int i = 0; i < N; ++i) d[i] = *at(a.seg_S, row, i);
      if (vector) dn = a.seg_n[idx * DIM + threadIdx.x];
      const float2 loc = *reinterpret_cast<const float2*>(a.seg_F + 2 * idx);   // F and m of the local state
      mn = fmaxf(loc.x + m, loc.y);
      fa = expf(loc.x + m - mn);
      fb = expf(loc.y - mn);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) *at(a.seg_S, row, i) = s[i];
    if (vector) a.seg_n[idx * DIM + threadIdx.x] = n;
    if (vector && threadIdx.x == 0) a.seg_m[idx] = m;
    if (last) break;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      s[i].x = fa * s[i].x + fb * d[i].x;
      s[i].y = fa * s[i].y + fb * d[i].y;
      s[i].z = fa * s[i].z + fb * d[i].z;
      s[i].w = fa * s[i].w + fb * d[i].w;
    }
    n = fa * n + fb * dn;
    m = mn;
  }
}

static int padded_state_dim(int dim) {
  const int sizes[] = {64, 128, 256, 512};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

template <int DG, int DPT>
static int run_step(const Mlstm& a, const int* entries, int count, int mode, cudaStream_t stream) {
  const int nt = a.vp / kVT;
  const dim3 grid(nt, a.heads, count);
  const int4* en = (const int4*)entries;
  switch (mode) {
    case 0: return launch(step_kernel<DG, DPT, false, false, float>, grid, 16 * DG, 0, stream, 1, 0, a, en);
    case 1: return launch(step_kernel<DG, DPT, true, true, bf16>, grid, 16 * DG, 0, stream, nt, 0, a, en);
    case 2: return launch(step_kernel<DG, DPT, true, true, float>, grid, 16 * DG, 0, stream, nt, 0, a, en);
    default: return launch(step_kernel<DG, DPT, true, false, float>, grid, 16 * DG, 0, stream, 1, 0, a, en);
  }
}

template <int DIM>
static int run_chunk(const Mlstm& a, const int* entries, int count, const int* segs, int nsegs, const int* prompts, cudaStream_t stream) {
  const int nt = a.vp / kVT;
  constexpr size_t smem = sizeof(ChunkSmem<DIM>);
  if (nsegs == 0) return launch(chunk_kernel<DIM, kWhole>, dim3(nt, a.heads, count), 32 * chunk_warps(DIM), smem, stream, 1, 0, a, (const int4*)entries);
  int rc = launch(chunk_kernel<DIM, kLocal>, dim3(nt, a.heads, nsegs), 32 * chunk_warps(DIM), smem, stream, 1, 0, a, (const int4*)segs);
  if (rc == BONSAI_CUDA_OK) rc = launch(combine_kernel<DIM>, dim3(nt * 4, a.heads, count), 256, 0, stream, 1, 0, a, (const int4*)prompts);
  if (rc == BONSAI_CUDA_OK) rc = launch(chunk_kernel<DIM, kResume>, dim3(nt, a.heads, nsegs), 32 * chunk_warps(DIM), smem, stream, 1, 0, a, (const int4*)segs);
  return rc;
}

static bool fill(Mlstm& a, const void* const* ptrs, const int* ints, const float* floats) {
  a.proj = (const float*)ptrs[0]; a.i_bias = (const float*)ptrs[1]; a.f_bias = (const float*)ptrs[2]; a.norm = (const float*)ptrs[3];
  a.S = (float*)ptrs[4]; a.n = (float*)ptrs[5]; a.m = (float*)ptrs[6]; a.pos = (const int*)ptrs[7]; a.slots = (const int*)ptrs[8];
  a.state_rows = (const int*)ptrs[9]; a.out = const_cast<void*>(ptrs[10]);
  a.seg_S = (float*)ptrs[11]; a.seg_n = (float*)ptrs[12]; a.seg_m = (float*)ptrs[13]; a.seg_F = (float*)ptrs[14];
  a.ld = ints[0]; a.q_col = ints[1]; a.k_col = ints[2]; a.v_col = ints[3]; a.g_col = ints[4]; a.i_col = ints[5]; a.f_col = ints[6];
  a.ldo = ints[7]; a.heads = ints[8]; a.dim = ints[9]; a.vdim = ints[10]; a.vp = (a.vdim + kVT - 1) / kVT * kVT;
  a.vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && (a.ld | a.q_col | a.k_col | a.v_col) % 4 == 0 && (uintptr_t)a.proj % 16 == 0;
  a.cap = floats[0]; a.eps = floats[1]; a.den_eps = floats[2]; a.q_scale = floats[3];
  return a.heads >= 1 && a.heads <= 65535 && a.dim >= 1 && a.vdim >= 1 && padded_state_dim(a.dim) > 0;
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// padded state sizes: rows (0: not supported) and columns
int bonsai_lay_mlstm_dim(int dim) { return dim < 1 ? 0 : bonsai::lay::padded_state_dim(dim); }
int bonsai_lay_mlstm_vdim(int vdim) { return (vdim + bonsai::lay::kVT - 1) / bonsai::lay::kVT * bonsai::lay::kVT; }
// largest dim of the chunked kernel
int bonsai_lay_mlstm_chunk_dim() { return 256; }
// largest vdim whose single-token step finishes its outputs itself (one cluster per head)
int bonsai_lay_mlstm_fused_vdim() { return 8 * bonsai::lay::kVT; }

// tokens per chunk
int bonsai_lay_mlstm_chunk_tokens() { return bonsai::lay::kL; }

// ptrs = {proj, i_bias, f_bias, norm, S, n, m, pos, slots, state_rows, out, seg_S, seg_n, seg_m, seg_F}, ints = {ld, q_col, k_col, v_col, g_col, i_col,
// f_col, ldo, heads, dim, vdim}, floats = {cap, eps, den_eps, q_scale}.

// mode 0: entries (int4 {first row, tokens, slot, first position}), o f32; single tokens in rows 0 .. count - 1: mode 1 / 2
// finished bf16 / f32 activations, mode 3 o f32.
int bonsai_lay_mlstm_step(const void* const* ptrs, const int* ints, const float* floats, const int* entries, int count, int mode,
                          cudaStream_t stream) {
  using namespace bonsai::lay;
  Mlstm a;
  if (!fill(a, ptrs, ints, floats) || count < 1 || count > 65535 || mode < 0 || mode > 3 || (mode == 0 && entries == nullptr)) return BONSAI_CUDA_BAD_ARG;
  if ((mode == 1 || mode == 2) && a.vp / kVT > 8) return BONSAI_CUDA_BAD_ARG;
  switch (padded_state_dim(a.dim)) {
    case 64: return run_step<16, 4>(a, entries, count, mode, stream);
    case 128: return run_step<16, 8>(a, entries, count, mode, stream);
    case 256: return run_step<16, 16>(a, entries, count, mode, stream);
    default: return run_step<32, 16>(a, entries, count, mode, stream);
  }
}

// Portions of prompts, o f32.  nsegs > 0: cut into the segments segs int4 [nsegs] {first row, tokens (a multiple of the chunk
// except at a portion's end), slot, 1 for the last of its portion}, with prompts int4 [count] {slot, first position, first
// segment, segments} and scratch for nsegs states.
int bonsai_lay_mlstm_chunk(const void* const* ptrs, const int* ints, const float* floats, const int* entries, int count, const int* segs, int nsegs,
                           const int* prompts, cudaStream_t stream) {
  using namespace bonsai::lay;
  Mlstm a;
  if (!fill(a, ptrs, ints, floats) || count < 1 || count > 65535 || entries == nullptr || nsegs < 0 || nsegs > 65535) return BONSAI_CUDA_BAD_ARG;
  if (nsegs > 0 && (segs == nullptr || prompts == nullptr || a.seg_S == nullptr)) return BONSAI_CUDA_BAD_ARG;
  switch (padded_state_dim(a.dim)) {
    case 64: return run_chunk<64>(a, entries, count, segs, nsegs, prompts, stream);
    case 128: return run_chunk<128>(a, entries, count, segs, nsegs, prompts, stream);
    case 256: return run_chunk<256>(a, entries, count, segs, nsegs, prompts, stream);
    default: return BONSAI_CUDA_BAD_ARG;
  }
}

}  // extern "C"
