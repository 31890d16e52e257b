// Linear recurrences with one decay per head and token: S <- a_t S + b_t k_t v_t^T, o_t = S^T q_t [+ D v_t], S [dim][vdim] in f32.
//
// What a design chooses:
//  * decay: a fixed one per head (a_t = decay_h, b_t = 1), or from the input, dt = softplus(raw + bias_h), a_t = exp(-rate_h dt),
//    b_t = dt (state-space duality);
//  * features: q, k, v straight from the projections, through silu, through a causal convolution per channel and silu, or rotated
//    (first rot_dims dimensions, i paired with i + rot_dims / 2); k times key_scale; `groups` heads' worth of q and k, head h
//    using group h / (heads / groups);
//  * a skip D per head.
//
// `step_kernel` runs the recurrence as written, a column tile of 64 values of one head per CTA, the state in registers.  For
// single tokens it makes the features itself and, where the norm is per head, finishes the outputs (the column tiles of a head
// form a cluster and exchange their sums of squares).  For several tokens (32-bit mode, long keys) it reads prepared features.
// `features_kernel` prepares the features of prompt rows; `rec_chunk_kernel` runs portions of prompts on the tensor cores, 64 tokens
// at a time.  With F the running sum of log2 a inside the chunk, token t sees token s <= t with weight b_s 2^(F_t - F_s) and the
// chunk's initial state with weight 2^F_t, so no exponent is positive for decays up to 1:
//   o_t = sum_s b_s 2^(F_t - F_s) (q_t . k_s) v_s + 2^F_t S_0^T q_t,    S' = 2^F_L S_0 + sum_s b_s 2^(F_L - F_s) k_s v_s^T
// Decays, weights and state are f32; the state and the weighted values enter their products as a bf16 pair (value and
// remainder), i.e. with 16 significant bits.  Prompts long enough are cut into segments as in mlstm.cu: local states, their
// combination, outputs.
//
// State layout: S [row][head][DIM][VP] with padded sizes (the padding stays zero); the convolution's last inputs in a ring
// [row][taps][channels], the input of position p at p % taps, so that a token never writes where it reads.  A sequence's first
// token (position 0) starts from zero whatever its state row holds.
#include <cooperative_groups.h>

#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

struct LinRec {
  const float* proj;        // [T][ld]
  const float* decay;       // [heads]; null: decays from the input
  const float* rate;        // [heads]
  const float* dt_bias;     // [heads]
  const float* skip;        // [heads] or null
  const float* norm;        // [heads * vdim] or null: weight of the per-head norm
  const float* conv_w;      // [taps][channels], tap j: the input j tokens back
  const float* conv_b;      // [channels]
  float* ring;
  const double* freq;       // [rot_dims / 2]
  float* S;
  const int* pos;           // [T]
  const int* slots;         // [T]
  const int* state_rows;    // [slots]
  void* out;                // finished activations [T][ldo] or o f32 [T][ldo]
  void* feat;               // [T][ldf]: groups x dp of q, groups x dp of k, heads x ep of v (dp, ep: dim, vdim rounded up to 8)
  float* seg_S;             // one state per segment
  float* seg_F;             // [segment][head]: log2 of the local state's decay
  int ld, q_col, k_col, v_col, g_col, dt_col, conv_col, ldo, ldf;
  int heads, groups, dim, vdim, vp, dp, ep, act, taps, conv_n, rot_dims, gate_silu;
  float eps, key_scale, out_scale;
};

constexpr float kFloor = -80.0f;   // log2 of the smallest decay: keeps the sums of a chunk short of losing their last digits

__device__ __forceinline__ float silu(float v) { return v * sigmoid(v); }
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// cos and sin of position * frequency, the angle reduced in double precision
__device__ __forceinline__ float2 rotation(int pos, double freq) {
  constexpr double kTwoPi = 6.283185307179586476925;
  double x = (double)pos * freq;
  x -= kTwoPi * rint(x / kTwoPi);
  float s, c;
  sincosf((float)x, &s, &c);
  return make_float2(c, s);
}

// Column `col` of a single token's row p, convolved with the ring's inputs where the design has a convolution, and activated.
// here: pos % taps.
__device__ __forceinline__ float single_feature(const LinRec& a, const float* p, const float* ring, int pos, int here, int col) {
  float v = p[col];
  if (a.taps > 0) {
    const int c = col - a.conv_col;
    float x[3], w[3];                                // the first three inputs back, loaded at once
#pragma unroll
    for (int j = 1; j <= 3; ++j) {
      const bool ok = j < a.taps && j <= pos;
      x[j - 1] = ok ? ring[(here >= j ? here - j : here - j + a.taps) * a.conv_n + c] : 0.0f;
      w[j - 1] = ok ? a.conv_w[j * a.conv_n + c] : 0.0f;
    }
    v = fmaf(v, a.conv_w[c], a.conv_b[c]);
#pragma unroll
    for (int j = 0; j < 3; ++j) v = fmaf(w[j], x[j], v);
    for (int j = 4; j < a.taps && j <= pos; ++j) v = fmaf(a.conv_w[j * a.conv_n + c], ring[(here >= j ? here - j : here - j + a.taps) * a.conv_n + c], v);
  }
  return a.act ? silu(v) : v;
}

__device__ __forceinline__ float load_feature(const float* p) { return *p; }
__device__ __forceinline__ float load_feature(const bf16* p) { return __bfloat162float(*p); }

enum StepMode { kTokens, kSingle, kSingleDone };

// grid (vp / 64, heads, entries); threads = 16 column quads x DG groups of state rows, DPT state rows per thread
// (DIM = DG * DPT).  kTokens: entries[e] = {first row, tokens, slot, first position}, features of type X, o f32.  kSingle: one
// token in each of the rows 0 .. gridDim.z - 1, o f32; kSingleDone: finished outputs of type X, clusters along x.  early: what
// the kernel before this one writes is not read here, so the wait for it comes at the end.
template <int DG, int DPT, int MODE, typename X>
__global__ void __launch_bounds__(16 * DG) step_kernel(LinRec a, const int4* entries, int early) {
  constexpr int DIM = DG * DPT, NTH = 16 * DG;
  constexpr bool ONE = MODE != kTokens;
  __shared__ float sq[DIM], sk[DIM], sv[kVT], red[DG][68], s32[32];
  __shared__ float s_ss;
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int h = blockIdx.y, tile = blockIdx.x, ntile = gridDim.x, per = a.heads / a.groups, grp = h / per;
  const int tid = threadIdx.x, cq = tid & 15, dg = tid >> 4, col = tile * kVT + cq * 4;
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
  const int row = a.state_rows[slot];
  float* S = a.S + ((size_t)row * a.heads + h) * DIM * a.vp + col;
  float* ring = a.ring + (size_t)row * a.taps * a.conv_n;
  // the state is older than the kernel before this one
  float4 s[DPT];
#pragma unroll
  for (int i = 0; i < DPT; ++i)
    s[i] = pos0 == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + (size_t)(dg + i * DG) * a.vp);
  if (ONE && !early) {
    pdl_wait();
    pdl_trigger();
  }
  const float skip = a.skip == nullptr ? 0.0f : a.skip[h];
  const int here = ONE && a.taps > 0 ? pos0 % a.taps : 0;
  for (int tt = 0; tt < count; ++tt) {
    const float* p = a.proj + (size_t)(t0 + tt) * a.ld;
    if (ONE) {
      const int qc = a.q_col + grp * a.dim, kc = a.k_col + grp * a.dim, half = a.rot_dims >> 1;
      for (int i = tid; i < half; i += NTH) {
        const float2 cs = rotation(pos0, a.freq[i]);
        const float qu = single_feature(a, p, ring, pos0, here, qc + i), qv = single_feature(a, p, ring, pos0, here, qc + half + i);
        const float ku = single_feature(a, p, ring, pos0, here, kc + i), kv = single_feature(a, p, ring, pos0, here, kc + half + i);
        sq[i] = qu * cs.x - qv * cs.y;
        sq[half + i] = qv * cs.x + qu * cs.y;
        sk[i] = (ku * cs.x - kv * cs.y) * a.key_scale;
        sk[half + i] = (kv * cs.x + ku * cs.y) * a.key_scale;
      }
      for (int d = a.rot_dims + tid; d < DIM; d += NTH) {
        sq[d] = d < a.dim ? single_feature(a, p, ring, pos0, here, qc + d) : 0.0f;
        sk[d] = d < a.dim ? single_feature(a, p, ring, pos0, here, kc + d) * a.key_scale : 0.0f;
      }
      const int vt = NTH - 1 - tid;                  // the last threads: the first ones have a rotation to do
      if (vt < kVT) {
        const int c = tile * kVT + vt;
        sv[vt] = c < a.vdim ? single_feature(a, p, ring, pos0, here, a.v_col + h * a.vdim + c) : 0.0f;
      }
      if (a.taps > 0) {                              // this token's inputs join the ring, every channel from one CTA
        float* dst = ring + here * a.conv_n;
        for (int i = tid; i < min(kVT, a.vdim - tile * kVT); i += NTH) {
          const int cc = a.v_col + h * a.vdim + tile * kVT + i;
          dst[cc - a.conv_col] = p[cc];
        }
        if (tile == 0 && h % per == 0)
          for (int d = tid; d < a.dim; d += NTH) {
            dst[qc + d - a.conv_col] = p[qc + d];
            dst[kc + d - a.conv_col] = p[kc + d];
          }
      }
    } else {
      const X* f = static_cast<const X*>(a.feat) + (size_t)(t0 + tt) * a.ldf;
      for (int d = tid; d < DIM; d += NTH) {
        sq[d] = d < a.dim ? load_feature(f + grp * a.dp + d) : 0.0f;
        sk[d] = d < a.dim ? load_feature(f + (a.groups + grp) * a.dp + d) : 0.0f;
      }
      for (int i = tid; i < kVT; i += NTH) sv[i] = tile * kVT + i < a.vdim ? load_feature(f + 2 * a.groups * a.dp + h * a.ep + tile * kVT + i) : 0.0f;
    }
    float da, db = 1.0f;
    if (a.decay != nullptr) {
      da = a.decay[h];
    } else {
      db = softplus(p[a.dt_col + h] + a.dt_bias[h]);
      da = expf(-a.rate[h] * db);
    }
    __syncthreads();
    const float4 v = *reinterpret_cast<const float4*>(&sv[cq * 4]);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const float kb = db * sk[dg + i * DG], q = sq[dg + i * DG];
      s[i].x = da * s[i].x + kb * v.x;
      s[i].y = da * s[i].y + kb * v.y;
      s[i].z = da * s[i].z + kb * v.z;
      s[i].w = da * s[i].w + kb * v.w;
      acc.x += s[i].x * q;
      acc.y += s[i].y * q;
      acc.z += s[i].z * q;
      acc.w += s[i].w * q;
    }
    *reinterpret_cast<float4*>(&red[dg][cq * 4]) = acc;
    __syncthreads();
    float o = 0.0f;
    const int oc = tile * kVT + tid;
    if (tid < kVT) {
#pragma unroll
      for (int g = 0; g < DG; ++g) o += red[g][tid];
      o += skip * sv[tid];
    }
    if (MODE != kSingleDone) {
      if (tid < kVT && oc < a.vdim) static_cast<float*>(a.out)[(size_t)(t0 + tt) * a.ldo + h * a.vdim + oc] = o;
      if (!ONE) __syncthreads();         // sq, sk, sv and red are free
    } else {
      const float ss = block_sum(tid < kVT ? o * o : 0.0f, s32);
      if (tid == 0) s_ss = ss;
      float total = ss;
      if (ntile > 1) {
        cluster.sync();
        total = 0.0f;
        for (int r = 0; r < ntile; ++r) total += *cluster.map_shared_rank(&s_ss, r);
      }
      if (tid < kVT && oc < a.vdim) {
        const int c = h * a.vdim + oc;
        const float g = p[a.g_col + c], w = a.norm == nullptr ? 1.0f : a.norm[c];
        store_act(static_cast<X*>(a.out) + (size_t)t0 * a.ldo + c, o * (a.out_scale / sqrtf(total / (float)a.vdim + a.eps)) * w * (a.gate_silu ? silu(g) : sigmoid(g)));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < DPT; ++i) *reinterpret_cast<float4*>(S + (size_t)(dg + i * DG) * a.vp) = s[i];
  if (MODE == kSingleDone && ntile > 1) cluster.sync();   // nobody leaves while its sum is being read
  if (ONE && early) {
    pdl_wait();
    pdl_trigger();
  }
}

// ---- features of prompt rows ------------------------------------------------------------------------------------------------------
// Rows first .. first + count - 1, kFR per CTA; a thread has VEC feature columns.  Rows of one portion are neighbours; an input
// from before the portion comes from the ring.
constexpr int kFR = 8;
enum FeatureKind { kPlain, kRotary, kConv4, kConv };     // kConv4: up to four taps, the inputs back in registers

template <int VEC, int KIND, typename X>
__global__ void __launch_bounds__(128) features_kernel(LinRec a, int first, int count) {
  extern __shared__ float2 cs[];                     // [kFR][rot_dims / 2]
  pdl_wait();
  pdl_trigger();
  const int r0 = first + blockIdx.y * kFR, rows = min(kFR, first + count - r0), half = a.rot_dims >> 1;
  const int qk = a.groups * a.dp, f0 = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (KIND == kRotary) {
    if (blockIdx.x * 128 * VEC < 2 * qk)
      for (int i = threadIdx.x; i < rows * half; i += 128) cs[i] = rotation(a.pos[r0 + i / half], a.freq[i % half]);
    __syncthreads();
  }
  if (f0 >= 2 * qk + a.heads * a.ep) return;
  int d, size, col;
  const int what = f0 < qk ? 0 : (f0 < 2 * qk ? 1 : 2);
  if (what < 2) {
    const int f = f0 - what * qk, g = f / a.dp;
    d = f % a.dp;
    size = a.dim;
    col = (what == 0 ? a.q_col : a.k_col) + g * a.dim + d;
  } else {
    const int f = f0 - 2 * qk, h = f / a.ep;
    d = f % a.ep;
    size = a.vdim;
    col = a.v_col + h * a.vdim + d;
  }
  const bool in = d < size, rot = KIND == kRotary && what < 2 && d < a.rot_dims;
  auto load = [&](const float* p, float* v, bool ok) {
    if constexpr (VEC == 4) {
      const float4 q = ok ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
      v[0] = ok ? *p : 0.0f;
    }
  };
  float v[kFR][VEC], u[KIND == kRotary ? kFR : 1][VEC];
  const float* src = a.proj + (size_t)r0 * a.ld + col;
  const int partner = d < half ? half : -half;
#pragma unroll
  for (int r = 0; r < kFR; ++r) {
    load(src + (size_t)r * a.ld, v[r], in && r < rows);
    if (KIND == kRotary) load(src + (size_t)r * a.ld + partner, u[KIND == kRotary ? r : 0], rot && r < rows);
  }
  const int c = col - a.conv_col;
  bool same = false;                                 // all of these rows and the three before them belong to one portion
  float w[KIND == kConv4 ? 4 : 1][VEC], back[KIND == kConv4 ? 3 : 1][VEC], bias[VEC];   // back[j]: the input j + 1 rows back
  if (KIND == kConv4) {
#pragma unroll
    for (int j = 0; j < 4; ++j) load(a.conv_w + (size_t)j * a.conv_n + c, w[KIND == kConv4 ? j : 0], in && j < a.taps);
    if (r0 - 3 >= first) {
#pragma unroll
      for (int j = 1; j <= 3; ++j) load(src - (size_t)j * a.ld, back[KIND == kConv4 ? j - 1 : 0], in);
      same = a.slots[r0 - 3] == a.slots[r0 + rows - 1];
    }
  }
  if (KIND >= kConv4) load(a.conv_b + c, bias, in);
  // the input j rows before row t, a zero before the sequence's start
  auto earlier = [&](int t, int slot, int pos, int j, float* x) {
    bool here = t - j >= first;                      // the rows back to t - j belong to the same portion
    for (int i = 1; i <= j && here; ++i) here = a.slots[t - i] == slot;
    const float* ring = a.ring + ((size_t)a.state_rows[slot] * a.taps + (pos - j + a.taps * j) % a.taps) * a.conv_n + c;
    load(here ? a.proj + (size_t)(t - j) * a.ld + col : ring, x, in && j < a.taps && j <= pos);
  };
  int last = -1;                                     // slot of the row before
#pragma unroll
  for (int r = 0; r < kFR; ++r) {
    if (r >= rows) break;
    const int t = r0 + r;
    float y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = v[r][e];
    if constexpr (KIND == kConv4) {
      if (!same) {
        const int slot = a.slots[t];
        if (slot != last) {
          const int pos = a.pos[t];
#pragma unroll
          for (int j = 1; j <= 3; ++j) earlier(t, slot, pos, j, back[j - 1]);
          last = slot;
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        y[e] = fmaf(v[r][e], w[0][e], bias[e]);
        y[e] = fmaf(back[0][e], w[1][e], y[e]);
        y[e] = fmaf(back[1][e], w[2][e], y[e]);
        y[e] = fmaf(back[2][e], w[3][e], y[e]);
        back[2][e] = back[1][e];
        back[1][e] = back[0][e];
        back[0][e] = v[r][e];
      }
    }
    if constexpr (KIND == kConv) {
      const int slot = a.slots[t], pos = a.pos[t];
      float x[VEC], k[VEC];
      load(a.conv_w + c, k, in);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(v[r][e], k[e], bias[e]);
      for (int j = 1; j < a.taps && j <= pos; ++j) {
        earlier(t, slot, pos, j, x);
        load(a.conv_w + (size_t)j * a.conv_n + c, k, in);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(x[e], k[e], y[e]);
      }
    }
    if (a.act) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = silu(y[e]);
    }
    if constexpr (KIND == kRotary) {
      if (rot) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const float z = a.act ? silu(u[r][e]) : u[r][e];
          const float2 k = cs[r * half + (d < half ? d : d - half) + e];
          y[e] = d < half ? y[e] * k.x - z * k.y : y[e] * k.x + z * k.y;
        }
      }
    }
    if (what == 1) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] *= a.key_scale;
    }
    X* dst = static_cast<X*>(a.feat) + (size_t)t * a.ldf + f0;
    if constexpr (VEC == 4 && sizeof(X) == 2) {
      *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16(y[0], y[1]), pack_bf16(y[2], y[3]));
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) store_act(dst + e, in ? y[e] : 0.0f);
    }
  }
}

// The last inputs of every portion join the ring (after the features have read it).  grid (channels / 256, entries).
__global__ void __launch_bounds__(256) ring_kernel(LinRec a, const int4* entries) {
  pdl_wait();
  pdl_trigger();
  const int4 en = entries[blockIdx.y];
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.conv_n) return;
  float* ring = a.ring + (size_t)a.state_rows[en.z] * a.taps * a.conv_n + c;
  for (int i = max(0, en.y - a.taps + 1); i < en.y; ++i) ring[(size_t)((en.w + i) % a.taps) * a.conv_n] = a.proj[(size_t)(en.x + i) * a.ld + a.conv_col + c];
}

// ---- portions of prompts ------------------------------------------------------------------------------------------------------------
template <int DIM>
struct RecSmem {
  static constexpr int LD = DIM + 8;
  bf16 q[kL * LD], k[kL * LD];
  bf16 v[kL * kVLD], vh[kL * kVLD], vl[kL * kVLD];   // values; weighted values: leading part and remainder
  bf16 sh[DIM * kVLD], sl[DIM * kVLD];               // state at the start of the chunk: leading part and remainder
  bf16 p[kL * kVLD];                                 // weighted scores
  struct alignas(16) Gates {
    float F[kL];        // log2 of the decays up to and with token t
    float b[kL];
    float g[kL];        // 2^F_t
    float w[kL];        // weight of token s in the final state
    float tail[4];      // decay of the state over the chunk and its log2
  } gates[2];           // this chunk's and the next one's
};

constexpr int rec_warps(int dim) { return dim >= 256 ? 16 : 8; }

// grid (vp / 64, heads, entries).  Warp w: rows (w & 3) * 16 .. + 15 of the chunk and group w >> 2 of the columns (keys and
// values); of the state two 16-row tiles and WN 8-column tiles.
// kWhole: entries {first row, tokens, slot, first position}, state from and to the pool.  kLocal / kResume: entries are the
// segments {first row, tokens, slot, last of its prompt}; kLocal leaves a segment's local state in its scratch row, kResume
// starts from the scratch row and writes the last segment's state to the pool.
template <int DIM, int MODE>
__global__ void __launch_bounds__(32 * rec_warps(DIM), DIM <= 128 ? 2 : 1) rec_chunk_kernel(LinRec a, const int4* entries) {
  constexpr int LD = DIM + 8;
  constexpr int NW = rec_warps(DIM), NTH = 32 * NW;
  constexpr int CW = 256 / NW;                       // columns of a warp's group: 64 / (NW / 4)
  constexpr int MT = DIM / 16, MG = MT / 2;          // 16-row tiles of the state, pairs of them
  constexpr int WM = 2, WN = 8 * MG / NW;            // state tiles of a warp
  static_assert(WN >= 2 && WN % 2 == 0 && MG * 8 == NW * WN, "state tiles over the warps");
  extern __shared__ __align__(16) uint8_t smem_raw[];
  RecSmem<DIM>& sm = *reinterpret_cast<RecSmem<DIM>*>(smem_raw);
  const int tile = blockIdx.x, h = blockIdx.y, col0 = tile * kVT, grp = h / (a.heads / a.groups);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rg = warp & 3, ch = warp >> 2;
  const int g = lane >> 2, t4 = lane & 3;
  pdl_wait();
  pdl_trigger();
  const int4 en = entries[blockIdx.z];
  if (MODE == kLocal && en.w) return;                // nothing resumes from the last segment's local state
  const size_t pool = (size_t)a.state_rows[en.z] * a.heads + h, seg = (size_t)blockIdx.z * a.heads + h;
  const size_t src = MODE == kWhole ? pool : seg, dst = MODE == kLocal ? seg : pool;
  const bf16* feat = static_cast<const bf16*>(a.feat) + (size_t)en.x * a.ldf;
  const bf16* fq = feat + grp * a.dp;
  const bf16* fk = feat + (a.groups + grp) * a.dp;
  const bf16* fv = feat + 2 * a.groups * a.dp + h * a.ep + col0;
  auto stage_keys = [&](bf16* to, const bf16* from, int at) {
#pragma unroll
    for (int i = tid; i < kL * (DIM / 8); i += NTH) {
      const int r = i / (DIM / 8), c = (i % (DIM / 8)) * 8;
      const bool ok = at + r < en.y && c < a.dp;
      cp_async16(to + r * LD + c, from + (ok ? (size_t)(at + r) * a.ldf + c : 0), ok);
    }
  };
  auto stage_values = [&](int at) {
#pragma unroll
    for (int i = tid; i < kL * (kVT / 8); i += NTH) {
      const int r = i / (kVT / 8), c = (i % (kVT / 8)) * 8;
      const bool ok = at + r < en.y && col0 + c < a.ep;
      cp_async16(sm.v + r * kVLD + c, ok ? fv + (size_t)(at + r) * a.ldf + c : feat, ok);
    }
  };
  if (MODE != kLocal) stage_keys(sm.q, fq, 0);
  stage_keys(sm.k, fk, 0);
  stage_values(0);
  cp_async_commit();
  const float* inS = (MODE == kWhole ? a.S : a.seg_S) + src * DIM * a.vp + col0;
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
  const float skip = a.skip == nullptr ? 0.0f : a.skip[h];
  float Fsum = 0.0f;

  // One warp makes a chunk's decays and weights; it does so a chunk ahead, from values loaded earlier still.
  constexpr int kGateWarp = 4 * (NW / 4 - 1);        // the warp with the least other work: first rows, last columns
  float raw[2] = {0.0f, 0.0f};                       // this lane's two tokens
  const float fixed = a.decay != nullptr ? fmaxf(log2f(a.decay[h]), kFloor) : 0.0f;
  auto load_raw = [&](int at) {
    if (a.decay != nullptr) return;
#pragma unroll
    for (int e = 0; e < 2; ++e)
      raw[e] = at + 2 * lane + e < en.y ? a.proj[(size_t)(en.x + at + 2 * lane + e) * a.ld + a.dt_col + h] : 0.0f;
  };
  auto make_gates = [&](int at, typename RecSmem<DIM>::Gates& G) {
    float f[2], b[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = at + 2 * lane + e < en.y;
      if (a.decay != nullptr) {
        f[e] = ok ? fixed : 0.0f;
        b[e] = ok ? 1.0f : 0.0f;
      } else {
        const float dt = softplus(raw[e] + a.dt_bias[h]);
        f[e] = ok ? fmaxf(-a.rate[h] * dt * kLog2e, kFloor) : 0.0f;
        b[e] = ok ? dt : 0.0f;
      }
    }
    float F = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) F += pf;
    }
    const float Ft[2] = {F - f[1], F}, FL = __shfl_sync(0xffffffffu, F, 31);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int s = 2 * lane + e;
      G.F[s] = Ft[e];
      G.b[s] = b[e];
      G.g[s] = ex2(Ft[e]);
      G.w[s] = ex2(FL - Ft[e]) * b[e];
    }
    if (lane == 0) {
      G.tail[0] = ex2(FL);
      G.tail[1] = FL;
    }
  };
  if (warp == kGateWarp) {
    load_raw(0);
    make_gates(0, sm.gates[0]);
  }

  for (int t0 = 0, it = 0; t0 < en.y; t0 += kL, ++it) {
    const int nt = min(kL, en.y - t0);
    const bool more = t0 + kL < en.y;
    const typename RecSmem<DIM>::Gates& G = sm.gates[it & 1];
    // ---- the state as a bf16 pair, while the chunk's features arrive ----------------------------------------------------------------
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
    cp_async_wait<0>();
    __syncthreads();
    // ---- weighted scores, the initial state's share, weighted values -----------------------------------------------------------------
    if (more && warp == kGateWarp) load_raw(t0 + kL);
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
        const float Ft = G.F[t];
#pragma unroll
        for (int j = 0; j < CW / 8; ++j) {
          const int k0 = ch * CW + j * 8 + 2 * t4;
          const float2 Fs = *reinterpret_cast<const float2*>(&G.F[k0]), b = *reinterpret_cast<const float2*>(&G.b[k0]);
          const float x = k0 <= t ? s[j][2 * e] * ex2(Ft - Fs.x) * b.x : 0.0f;
          const float y = k0 + 1 <= t ? s[j][2 * e + 1] * ex2(Ft - Fs.y) * b.y : 0.0f;
          *reinterpret_cast<uint32_t*>(sm.p + t * kVLD + k0) = pack_bf16(x, y);
        }
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
    if (MODE != kLocal && more) {                    // the queries have been read
      stage_keys(sm.q, fq, t0 + kL);
      cp_async_commit();
    }
    // ---- outputs ---------------------------------------------------------------------------------------------------------------------
    if constexpr (MODE != kLocal) {
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
      const bool pairs = ((a.vdim | a.ldo) & 1) == 0;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = rg * 16 + g + 8 * e;
        if (t >= nt) continue;
        float* dst = static_cast<float*>(a.out) + (size_t)(en.x + t0 + t) * a.ldo + h * a.vdim + col0;
#pragma unroll
        for (int j = 0; j < CW / 8; ++j) {
          const int c = ch * CW + j * 8 + 2 * t4;
          float2 y = make_float2(oi[j][2 * e], oi[j][2 * e + 1]);
          if (skip != 0.0f) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sm.v + t * kVLD + c));
            y.x += skip * v.x;
            y.y += skip * v.y;
          }
          if (pairs) {
            if (col0 + c < a.vdim) *reinterpret_cast<float2*>(dst + c) = y;
          } else {
            if (col0 + c < a.vdim) dst[c] = y.x;
            if (col0 + c + 1 < a.vdim) dst[c + 1] = y.y;
          }
        }
      }
    }
    // ---- the state at the end of the chunk ------------------------------------------------------------------------------------------
    if (more && warp == kGateWarp) make_gates(t0 + kL, sm.gates[(it + 1) & 1]);
    const float decay = G.tail[0];
    Fsum += G.tail[1];
#pragma unroll
    for (int i = 0; i < WM; ++i)
#pragma unroll
      for (int j = 0; j < WN; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[i][j][e] *= decay;
#pragma unroll
    for (int ks = 0; ks < kL / 16; ++ks) {
      uint32_t kt[WM][4], b[4];
#pragma unroll
      for (int i = 0; i < WM; ++i) ldsm4_t(kt[i], frag_a_cols(sm.k, LD, state_row(i), ks * 16, lane));
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
    if (more) {
      stage_keys(sm.k, fk, t0 + kL);
      stage_values(t0 + kL);
      cp_async_commit();
    }
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
  if (MODE == kLocal && tile == 0 && tid == 0) a.seg_F[dst] = Fsum;
}

// Local states of the segments -> the states they start from.  grid (vp / 64 * 4, heads, prompts), 256 threads: a quarter of
// a column tile's state rows.  prompts[e] = {slot, first position, first segment, segments}.
template <int DIM>
__global__ void __launch_bounds__(256) rec_combine_kernel(LinRec a, const int4* prompts) {
  pdl_wait();
  pdl_trigger();
  const int tile = blockIdx.x >> 2, quarter = blockIdx.x & 3, h = blockIdx.y;
  const int4 pr = prompts[blockIdx.z];
  const bool fresh = pr.y == 0;
  const size_t pool = (size_t)a.state_rows[pr.x] * a.heads + h;
  constexpr int N = DIM / 4 * 16 / 256;              // float4 per thread
  const int c = (threadIdx.x & 15) * 4, r0 = quarter * (DIM / 4) + (threadIdx.x >> 4);
  auto at = [&](float* S, size_t row, int i) { return reinterpret_cast<float4*>(S + (row * DIM + r0 + 16 * i) * a.vp + tile * kVT + c); };
  float4 s[N];
#pragma unroll
  for (int i = 0; i < N; ++i) s[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *at(a.S, pool, i);
  for (int j = 0; j < pr.w; ++j) {
    const size_t row = (size_t)(pr.z + j) * a.heads + h;
    const bool last = j == pr.w - 1;                 // its scratch row holds no local state
    float4 d[N];
    float f = 0.0f;
    if (!last) {
#pragma unroll
      for (int i = 0; i < N; ++i) d[i] = *at(a.seg_S, row, i);
      f = ex2(a.seg_F[row]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) *at(a.seg_S, row, i) = s[i];
    if (last) break;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      s[i].x = f * s[i].x + d[i].x;
      s[i].y = f * s[i].y + d[i].y;
      s[i].z = f * s[i].z + d[i].z;
      s[i].w = f * s[i].w + d[i].w;
    }
  }
}

static int padded_rec_dim(int dim) {
  const int sizes[] = {64, 128, 256, 512};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

template <int DG, int DPT>
static int run_rec_step(const LinRec& a, const int* entries, int count, int mode, int f32, int early, cudaStream_t stream) {
  const int nt = a.vp / kVT, th = 16 * DG;
  const dim3 grid(nt, a.heads, count);
  const int4* en = (const int4*)entries;
  if (mode == kTokens)
    return f32 ? launch(step_kernel<DG, DPT, kTokens, float>, grid, th, 0, stream, 1, 0, a, en, 0)
               : launch(step_kernel<DG, DPT, kTokens, bf16>, grid, th, 0, stream, 1, 0, a, en, 0);
  if (mode == kSingle) return launch(step_kernel<DG, DPT, kSingle, float>, grid, th, 0, stream, 1, 0, a, en, early);
  return f32 ? launch(step_kernel<DG, DPT, kSingleDone, float>, grid, th, 0, stream, nt, 0, a, en, early)
             : launch(step_kernel<DG, DPT, kSingleDone, bf16>, grid, th, 0, stream, nt, 0, a, en, early);
}

template <int DIM>
static int run_rec_chunk(const LinRec& a, const int* entries, int count, const int* segs, int nsegs, const int* prompts, cudaStream_t stream) {
  const int nt = a.vp / kVT, th = 32 * rec_warps(DIM);
  constexpr size_t smem = sizeof(RecSmem<DIM>);
  if (nsegs == 0) return launch(rec_chunk_kernel<DIM, kWhole>, dim3(nt, a.heads, count), th, smem, stream, 1, 0, a, (const int4*)entries);
  int rc = launch(rec_chunk_kernel<DIM, kLocal>, dim3(nt, a.heads, nsegs), th, smem, stream, 1, 0, a, (const int4*)segs);
  if (rc == BONSAI_CUDA_OK) rc = launch(rec_combine_kernel<DIM>, dim3(nt * 4, a.heads, count), 256, 0, stream, 1, 0, a, (const int4*)prompts);
  if (rc == BONSAI_CUDA_OK) rc = launch(rec_chunk_kernel<DIM, kResume>, dim3(nt, a.heads, nsegs), th, smem, stream, 1, 0, a, (const int4*)segs);
  return rc;
}

static bool fill(LinRec& a, const void* const* ptrs, const int* ints, const float* floats) {
  a.proj = (const float*)ptrs[0]; a.decay = (const float*)ptrs[1]; a.rate = (const float*)ptrs[2]; a.dt_bias = (const float*)ptrs[3];
  a.skip = (const float*)ptrs[4]; a.norm = (const float*)ptrs[5]; a.conv_w = (const float*)ptrs[6]; a.conv_b = (const float*)ptrs[7];
  a.ring = (float*)ptrs[8]; a.freq = (const double*)ptrs[9]; a.S = (float*)ptrs[10]; a.pos = (const int*)ptrs[11]; a.slots = (const int*)ptrs[12];
  a.state_rows = (const int*)ptrs[13]; a.out = const_cast<void*>(ptrs[14]); a.feat = const_cast<void*>(ptrs[15]); a.seg_S = (float*)ptrs[16];
  a.seg_F = (float*)ptrs[17];
  a.ld = ints[0]; a.q_col = ints[1]; a.k_col = ints[2]; a.v_col = ints[3]; a.g_col = ints[4]; a.dt_col = ints[5]; a.conv_col = ints[6];
  a.ldo = ints[7]; a.ldf = ints[8]; a.heads = ints[9]; a.groups = ints[10]; a.dim = ints[11]; a.vdim = ints[12]; a.act = ints[13];
  a.taps = ints[14]; a.conv_n = ints[15]; a.rot_dims = ints[16]; a.gate_silu = ints[17];
  a.eps = floats[0]; a.key_scale = floats[1]; a.out_scale = floats[2];
  if (a.heads < 1 || a.heads > 65535 || a.groups < 1 || a.heads % a.groups != 0 || a.dim < 1 || a.vdim < 1 || padded_rec_dim(a.dim) == 0) return false;
  a.vp = (a.vdim + kVT - 1) / kVT * kVT;
  a.dp = (a.dim + 7) / 8 * 8;
  a.ep = (a.vdim + 7) / 8 * 8;
  if (a.decay == nullptr && (a.rate == nullptr || a.dt_bias == nullptr)) return false;
  if (a.taps < 0 || (a.taps > 0 && (a.conv_w == nullptr || a.conv_b == nullptr || a.ring == nullptr || a.conv_n < 1))) return false;
  if (a.rot_dims < 0 || a.rot_dims > a.dim || a.rot_dims % 2 != 0 || (a.rot_dims > 0 && (a.freq == nullptr || a.taps > 0))) return false;
  return a.S != nullptr && a.ldf >= 2 * a.groups * a.dp + a.heads * a.ep && a.ldf % 8 == 0;
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// padded state sizes: rows (0: not supported) and columns
int bonsai_lay_rec_dim(int dim) { return dim < 1 ? 0 : bonsai::lay::padded_rec_dim(dim); }
int bonsai_lay_rec_vdim(int vdim) { return (vdim + bonsai::lay::kVT - 1) / bonsai::lay::kVT * bonsai::lay::kVT; }
// columns of the prepared features
int bonsai_lay_rec_features_width(int heads, int groups, int dim, int vdim) { return 2 * groups * ((dim + 7) / 8 * 8) + heads * ((vdim + 7) / 8 * 8); }
// largest dim of the chunked kernel; largest vdim whose single-token step finishes its outputs itself (one cluster per head)
int bonsai_lay_rec_chunk_dim() { return 256; }
int bonsai_lay_rec_fused_vdim() { return 8 * bonsai::lay::kVT; }

// Arguments of all launches: ptrs = {proj, decay, rate, dt_bias, skip, norm, conv_w, conv_b, ring, freq, S, pos, slots, state_rows,
// out, feat, seg_S, seg_F} (null where a design has none), ints = {ld, q_col, k_col, v_col, g_col, dt_col, conv_col, ldo, ldf, heads,
// groups, dim, vdim, act, taps, conv_n, rot_dims, gate_silu}, floats = {eps, key_scale, out_scale}.

// Features of the rows first .. first + count - 1, bf16 or f32.
int bonsai_lay_rec_features(const void* const* ptrs, const int* ints, const float* floats, int first, int count, int f32, cudaStream_t stream) {
  using namespace bonsai::lay;
  LinRec a;
  if (!fill(a, ptrs, ints, floats) || first < 0 || count < 1 || count > 65535 * kFR || a.feat == nullptr) return BONSAI_CUDA_BAD_ARG;
  const uintptr_t at = (uintptr_t)a.proj | (uintptr_t)a.conv_w | (uintptr_t)a.conv_b | (uintptr_t)a.ring;
  const bool vec = ((a.dim | a.vdim | a.ld | a.q_col | a.k_col | a.v_col | a.conv_col | a.conv_n | (a.rot_dims / 2)) & 3) == 0 && at % 16 == 0;
  const int quads = (2 * a.groups * a.dp + a.heads * a.ep) / (vec ? 4 : 1);
  const dim3 grid((quads + 127) / 128, (count + kFR - 1) / kFR);
  const size_t smem = (size_t)kFR * (a.rot_dims / 2) * sizeof(float2);
#define BONSAI_FEATURES(KIND)                                                                                     \
  (f32 ? (vec ? launch(features_kernel<4, KIND, float>, grid, 128, smem, stream, 1, 0, a, first, count)           \
              : launch(features_kernel<1, KIND, float>, grid, 128, smem, stream, 1, 0, a, first, count))          \
       : (vec ? launch(features_kernel<4, KIND, bf16>, grid, 128, smem, stream, 1, 0, a, first, count)            \
              : launch(features_kernel<1, KIND, bf16>, grid, 128, smem, stream, 1, 0, a, first, count)))
  if (a.taps > 0) return a.taps <= 4 ? BONSAI_FEATURES(kConv4) : BONSAI_FEATURES(kConv);
  return a.rot_dims > 0 ? BONSAI_FEATURES(kRotary) : BONSAI_FEATURES(kPlain);
#undef BONSAI_FEATURES
}

// The portions' last inputs join the convolution's ring; after the features.
int bonsai_lay_rec_ring(const void* const* ptrs, const int* ints, const float* floats, const int* entries, int count, cudaStream_t stream) {
  using namespace bonsai::lay;
  LinRec a;
  if (!fill(a, ptrs, ints, floats) || a.taps < 1 || count < 1 || count > 65535 || entries == nullptr) return BONSAI_CUDA_BAD_ARG;
  return launch(ring_kernel, dim3((a.conv_n + 255) / 256, count), 256, 0, stream, 1, 0, a, (const int4*)entries);
}

// mode 0: entries (int4 {first row, tokens, slot, first position}) from prepared features (f32: their type), o f32; single tokens
// in rows 0 .. count - 1: mode 1 o f32, mode 2 finished activations (f32 or bf16).  early: the launch before this one writes
// nothing that is read here.
int bonsai_lay_rec_step(const void* const* ptrs, const int* ints, const float* floats, const int* entries, int count, int mode, int f32, int early,
                        cudaStream_t stream) {
  using namespace bonsai::lay;
  LinRec a;
  if (!fill(a, ptrs, ints, floats) || count < 1 || count > 65535 || mode < 0 || mode > 2 || (mode == 0 && (entries == nullptr || a.feat == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  if (mode == 2 && a.vp / kVT > 8) return BONSAI_CUDA_BAD_ARG;
  switch (padded_rec_dim(a.dim)) {
    case 64: return run_rec_step<16, 4>(a, entries, count, mode, f32, early, stream);
    case 128: return run_rec_step<16, 8>(a, entries, count, mode, f32, early, stream);
    case 256: return run_rec_step<16, 16>(a, entries, count, mode, f32, early, stream);
    default: return run_rec_step<32, 16>(a, entries, count, mode, f32, early, stream);
  }
}

// Portions of prompts from bf16 features, o f32.  nsegs > 0: cut into the segments segs int4 [nsegs] {first row, tokens (a multiple
// of the chunk except at a portion's end), slot, 1 for the last of its portion}, with prompts int4 [count] {slot, first position,
// first segment, segments} and scratch for nsegs states.
int bonsai_lay_rec_chunk(const void* const* ptrs, const int* ints, const float* floats, const int* entries, int count, const int* segs, int nsegs,
                         const int* prompts, cudaStream_t stream) {
  using namespace bonsai::lay;
  LinRec a;
  if (!fill(a, ptrs, ints, floats) || count < 1 || count > 65535 || entries == nullptr || nsegs < 0 || nsegs > 65535 || a.feat == nullptr)
    return BONSAI_CUDA_BAD_ARG;
  if (nsegs > 0 && (segs == nullptr || prompts == nullptr || a.seg_S == nullptr || a.seg_F == nullptr)) return BONSAI_CUDA_BAD_ARG;
  switch (padded_rec_dim(a.dim)) {
    case 64: return run_rec_chunk<64>(a, entries, count, segs, nsegs, prompts, stream);
    case 128: return run_rec_chunk<128>(a, entries, count, segs, nsegs, prompts, stream);
    case 256: return run_rec_chunk<256>(a, entries, count, segs, nsegs, prompts, stream);
    default: return BONSAI_CUDA_BAD_ARG;
  }
}

}  // extern "C"
