// Attention over a compressed cache: per token one normalised latent c and one rotated key part that all heads share,
//
//   c = norm(W_c h) * w,  k_h = [W_uk,h c, rot(W_r h)],  v_h = W_uv,h c,  q_h = [u_h, rot(r_h)]
//   out_h = (softmax(scale q_h . k_h) V_h) * sigmoid(gate) * out_scale                  one gate per element
//
// The paged cache holds rows [c | rotated part], each part padded with zeros to 16 elements, the row to 32.  Two ways to the same sum:
//
//  * absorbed, for single tokens and short portions: (W_uk,h^T u_h) . c instead of u_h . (W_uk,h c), and the weighted sum of the
//    latents goes through W_uv,h afterwards, so all heads read the same cache row once.  `query_kernel` appends the rows' latents
//    and makes the queries, `decode_kernel` leaves one partial sum per split of the keys, `value_kernel` joins the splits,
//    expands and gates.  A row is a token with a position and a slot, so tokens of one portion need not know of each other;
//  * expanded, for longer portions: `gather_kernel` brings the sequence's rows together, one product makes every head's keys and
//    values of them, and `prompt_kernel` is ordinary attention with one key/value head per query head.
//
// `f32_kernel` is the 32-bit mode, absorbed.
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

struct Latent {
  const float* proj;        // [T][ld]: queries at q_col ([dim | rot_dim] per head), latent at c_col, shared key part at r_col, gates at g_col
  const float* c_norm;      // [rank]
  const float2* rot;        // [positions][rot_dim / 2] cosines and sines
  const int* pos;           // [T]
  const int* slots;         // [T]
  const int* block_table;   // [slots][max_pages]
  void* pool;               // [pages][page_size][row], bf16 (f32 in the 32-bit mode)
  const bf16* wk;           // [heads][rp][dk]: key expansion, transposed, zero in the padding
  const bf16* wv;           // [heads][vdim][rk]: value expansion, zero in the padding
  bf16* q;                  // [rows][heads][row]: absorbed queries times scale * log2(e)
  float* part;              // [rows][splits][heads][rp]: sums of ex2(score - max) c
  float2* ml;               // [rows][splits][heads]: maximum and sum of ex2(score - max)
  void* out;                // [T][ldo], head h at h * vdim
  int ld, q_col, c_col, r_col, g_col, ldo;
  int heads, dim, rot_dim, vdim, rank, max_pages, pshift;   // page size 1 << pshift
  int rp, row, dk, rk;      // rank to 16, the row, dim to 32, rank to 32
  float eps, scale, out_scale;
};

__device__ __forceinline__ size_t latent_row(const Latent& a, const int* bt, int t) {
  return ((size_t)bt[t >> a.pshift] << a.pshift) + (t & ((1 << a.pshift) - 1));
}
__device__ __forceinline__ const float2* latent_angles(const Latent& a, int pos) { return a.rot + (size_t)pos * (a.rot_dim >> 1); }

// A warp writes the cache row of batch row t.
template <typename C>
__device__ __forceinline__ void append_latent(const Latent& a, int t, int lane) {
  const int pos = a.pos[t];
  if (pos >= (a.max_pages << a.pshift)) return;
  C* dst = static_cast<C*>(a.pool) + latent_row(a, a.block_table + (size_t)a.slots[t] * a.max_pages, pos) * a.row;
  const float* c = a.proj + (size_t)t * a.ld + a.c_col;
  const float* r = a.proj + (size_t)t * a.ld + a.r_col;
  float ss = 0.0f;
  for (int d = lane; d < a.rank; d += 32) ss += c[d] * c[d];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
  for (int d = lane; d < a.rp; d += 32) store_act(dst + d, d < a.rank ? c[d] * inv * a.c_norm[d] : 0.0f);
  const float2* rot = latent_angles(a, pos);
  for (int d = lane; d < a.row - a.rp; d += 32) store_act(dst + a.rp + d, d < a.rot_dim ? rotated(r, d, rot, a.rot_dim, 1) : 0.0f);
}

template <typename C>
__global__ void __launch_bounds__(128) latent_append_kernel(Latent a, int first, int count) {
  pdl_wait();
  pdl_trigger();
  const int i = blockIdx.x * 4 + (threadIdx.x >> 5);
  if (i < count) append_latent<C>(a, first + i, threadIdx.x & 31);
}

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// acc (16 rows of W at `w` x 8 tokens) over kp inputs: a lane loads 16 contiguous bytes of a row as A registers, the tokens in `sx`
// (rows of ldx elements) go through the same permutation of every 32 inputs.
__device__ __forceinline__ void rows_by_tokens(float* acc, const bf16* w0, const bf16* w1, const bf16* sx, int ldx, int kp, int lane) {
  const int g = lane >> 2, t4 = lane & 3;
  acc[0] = acc[1] = acc[2] = acc[3] = 0.0f;
#pragma unroll 4
  for (int k = 0; k < kp; k += 32) {
    const uint4 a = *reinterpret_cast<const uint4*>(w0 + k + 8 * t4), b = *reinterpret_cast<const uint4*>(w1 + k + 8 * t4);
    const uint4 v = *reinterpret_cast<const uint4*>(sx + g * ldx + k + 8 * t4);
    const uint32_t lo[4] = {a.x, b.x, a.y, b.y}, hi[4] = {a.z, b.z, a.w, b.w};
    mma_bf16(acc, lo, v.x, v.y);
    mma_bf16(acc, hi, v.z, v.w);
  }
}

// ---- absorbed -----------------------------------------------------------------------------------------------------------------
// grid (heads + 1, groups of 8 rows): queries of one head, or (the last column) the rows' cache entries
__global__ void __launch_bounds__(256) query_kernel(Latent a, int T) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* sq = reinterpret_cast<bf16*>(smem_raw);       // [8][dk + 8]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.x, t = blockIdx.y * 8 + warp, ldq = a.dk + 8;
  const bf16* w = a.wk + (size_t)head * a.rp * a.dk;
  if (head < a.heads)
    for (int i = threadIdx.x * 64; i < a.rp * a.dk; i += 256 * 64) prefetch_l2(w + i);
  pdl_wait();
  pdl_trigger();
  if (head == a.heads) {
    if (t < T) append_latent<bf16>(a, t, lane);
    return;
  }
  const float f = a.scale * kLog2e;
  const float* q = a.proj + (size_t)min(t, T - 1) * a.ld + a.q_col + head * (a.dim + a.rot_dim);
  for (int d = lane; d < a.dk; d += 32) sq[warp * ldq + d] = __float2bfloat16_rn(d < a.dim ? q[d] : 0.0f);
  if (t < T) {
    bf16* dst = a.q + ((size_t)t * a.heads + head) * a.row + a.rp;
    const int pos = a.pos[t];
    const bool ok = pos < (a.max_pages << a.pshift);
    const float2* rot = latent_angles(a, ok ? pos : 0);
    for (int d = lane; d < a.row - a.rp; d += 32) dst[d] = __float2bfloat16_rn(d < a.rot_dim ? rotated(q + a.dim, d, rot, a.rot_dim, 1) * f : 0.0f);
  }
  __syncthreads();
  const int g = lane >> 2, t4 = lane & 3, t0 = blockIdx.y * 8;
  for (int r0 = warp * 16; r0 < a.rp; r0 += 128) {
    float acc[4];
    rows_by_tokens(acc, w + (size_t)(r0 + g) * a.dk, w + (size_t)(r0 + g + 8) * a.dk, sq, ldq, a.dk, lane);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int tok = t0 + 2 * t4 + (e & 1), r = r0 + g + 8 * (e >> 1);
      if (tok < T) a.q[((size_t)tok * a.heads + head) * a.row + r] = __float2bfloat16_rn(acc[e] * f);
    }
  }
}

// grid (groups of 16 MT heads, splits, rows).  A CTA walks tiles of 64 keys of its split: the warps share the scores by head group
// and keys, the softmax by heads, and the weighted sum by latent columns (CB blocks of 16 a warp).
template <int CB, int MT>
__global__ void __launch_bounds__(256) latent_decode_kernel(Latent a) {
  constexpr int H = 16 * MT, LDS = 68, LDP = 72;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int ld = a.row + 8;
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);           // [H][ld]
  bf16* sK = sQ + H * ld;                                 // two stages of [64][ld]
  float* sS = reinterpret_cast<float*>(sK + 2 * 64 * ld); // [H][LDS] scores
  bf16* sP = reinterpret_cast<bf16*>(sS + H * LDS);       // [H][LDP] weights
  float* sF = reinterpret_cast<float*>(sP + H * LDP);     // [H] factors of the sums so far
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int h0 = blockIdx.x * H, nh = min(H, a.heads - h0), split = blockIdx.y, nsplit = gridDim.y, t = blockIdx.z;
  const int pos = a.pos[t];
  const bool held = pos < (a.max_pages << a.pshift);      // otherwise no page can hold the row: its output is not defined
  const int ntiles = held ? (pos >> 6) + 1 : 0, per = (ntiles + nsplit - 1) / nsplit;
  const int b0 = split * per, b1 = min(ntiles, b0 + per);
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  const bf16* pool = static_cast<const bf16*>(a.pool);
  const int chunks = a.row >> 3;
  auto fetch = [&](int tile, int st) {
    bf16* dst = sK + st * 64 * ld;
    for (int i = threadIdx.x; i < 64 * chunks; i += 256) {
      const int r = i / chunks, c = (i - r * chunks) * 8, k = tile * 64 + r;
      cp_async16(dst + r * ld + c, pool + (k <= pos ? latent_row(a, bt, k) * a.row + c : 0), k <= pos);
    }
  };
  // rows of this batch are appended by the kernel before this one; a tile that ends 64 tokens before this one holds none of them
  const bool early = b0 < b1 && b0 * 64 + 64 <= pos - 63;
  if (early) fetch(b0, 0);
  pdl_wait();
  pdl_trigger();
  float2* ml = a.ml + ((size_t)t * nsplit + split) * a.heads + h0;
  if (b0 >= b1) {
    for (int i = threadIdx.x; i < nh; i += 256) ml[i] = make_float2(-INFINITY, 0.0f);
    return;
  }
  if (!early) fetch(b0, 0);
  cp_async_commit();
  const bf16* q = a.q + ((size_t)t * a.heads + h0) * a.row;
  for (int i = threadIdx.x; i < H * chunks; i += 256) {
    const int r = i / chunks, c = (i - r * chunks) * 8;
    *reinterpret_cast<uint4*>(sQ + r * ld + c) = r < nh ? *reinterpret_cast<const uint4*>(q + (size_t)r * a.row + c) : make_uint4(0u, 0u, 0u, 0u);
  }
  float o[MT][2 * CB][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2 * CB; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.0f;
  float mx[2 * MT], l[2 * MT];                            // heads warp * 2 MT + i
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) mx[i] = -INFINITY, l[i] = 0.0f;
  const int mt = warp % MT, key0 = (warp / MT) * 8 * MT;  // this warp's scores: 16 heads x 8 MT keys
  for (int tile = b0; tile < b1; ++tile) {
    const bf16* k = sK + ((tile - b0) & 1) * 64 * ld;
    cp_async_wait<0>();
    __syncthreads();     // the tile has landed, and everyone is done with the other stage
    if (tile + 1 < b1) fetch(tile + 1, (tile + 1 - b0) & 1);
    cp_async_commit();
    float s[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
    if constexpr (MT == 1) {
      const bf16* kb = k + (key0 + (lane & 7)) * ld + (lane >> 3) * 8;
      for (int c = 0; c < a.row; c += 32) {
        uint32_t qa[4], qb[4], b[4];
        ldsm4(qa, frag_a(sQ, ld, 0, c, lane));
        ldsm4(qb, frag_a(sQ, ld, 0, c + 16, lane));
        ldsm4(b, kb + c);
        mma_bf16(s[0], qa, b[0], b[1]);
        mma_bf16(s[0], qb, b[2], b[3]);
      }
    } else {
#pragma unroll 2
      for (int c = 0; c < a.row; c += 16) {
        uint32_t qa[4];
        ldsm4(qa, frag_a(sQ, ld, mt * 16, c, lane));
#pragma unroll
        for (int i = 0; i < MT / 2; ++i) {
          uint32_t b[4];
          ldsm4(b, frag_b_rows(k, ld, key0 + 16 * i, c, lane));
          mma_bf16(s[2 * i], qa, b[0], b[1]);
          mma_bf16(s[2 * i + 1], qa, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = key0 + 8 * i + 2 * t4 + (e & 1);
        sS[(mt * 16 + g + 8 * (e >> 1)) * LDS + c] = tile * 64 + c <= pos ? s[i][e] : -INFINITY;
      }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      const int r = warp * 2 * MT + i;
      const float s0 = sS[r * LDS + lane], s1 = sS[r * LDS + 32 + lane];
      const float nm = fmaxf(mx[i], warp_max(fmaxf(s0, s1)));      // the first key of a tile is always visible
      const float p0 = ex2(s0 - nm), p1 = ex2(s1 - nm), f = ex2(mx[i] - nm);
      mx[i] = nm;
      l[i] = l[i] * f + p0 + p1;                          // this lane's keys
      sP[r * LDP + lane] = __float2bfloat16_rn(p0);
      sP[r * LDP + 32 + lane] = __float2bfloat16_rn(p1);
      if (lane == 0) sF[r] = f;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = sF[m * 16 + g], f1 = sF[m * 16 + g + 8];
#pragma unroll
      for (int i = 0; i < 2 * CB; ++i) {
        o[m][i][0] *= f0; o[m][i][1] *= f0;
        o[m][i][2] *= f1; o[m][i][3] *= f1;
      }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t p[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4(p[m], frag_a(sP, LDP, m * 16, ks * 16, lane));
#pragma unroll
      for (int j = 0; j < CB; ++j) {
        const int c = (warp * CB + j) * 16;
        if (c >= a.rp) continue;
        uint32_t b[4];
        ldsm4_t(b, frag_b_cols(k, ld, ks * 16, c, lane));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(o[m][2 * j], p[m], b[0], b[1]);
          mma_bf16(o[m][2 * j + 1], p[m], b[2], b[3]);
        }
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) {
    const int r = warp * 2 * MT + i;
    const float sum = warp_sum(l[i]);
    if (lane == 0 && r < nh) ml[r] = make_float2(mx[i], sum);
  }
  float* part = a.part + (((size_t)t * nsplit + split) * a.heads + h0) * a.rp;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2 * CB; ++i) {
      const int c = (warp * CB + i / 2) * 16 + (i & 1) * 8 + 2 * t4;
      if (c >= a.rp) continue;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = m * 16 + g + 8 * e;
        if (r < nh) *reinterpret_cast<float2*>(part + (size_t)r * a.rp + c) = make_float2(o[m][i][2 * e], o[m][i][2 * e + 1]);
      }
    }
}

constexpr int kMaxSplits = 64;

// grid (heads, groups of 8 rows): the splits' sums become one latent per row, which is expanded and gated
__global__ void __launch_bounds__(256) value_kernel(Latent a, int T, int nsplit) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* so = reinterpret_cast<bf16*>(smem_raw);           // [8][rk + 8]
  __shared__ float sw[8][kMaxSplits];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.x, t0 = blockIdx.y * 8, ldo = a.rk + 8;
  const bf16* w = a.wv + (size_t)head * a.vdim * a.rk;
  for (int i = threadIdx.x * 64; i < a.vdim * a.rk; i += 256 * 64) prefetch_l2(w + i);
  pdl_wait();
  pdl_trigger();
  {
    const int t = min(t0 + warp, T - 1);
    const float2* ml = a.ml + (size_t)t * nsplit * a.heads + head;
    float2 v[2];
    float M = -INFINITY, L = 0.0f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      v[i] = s < nsplit ? ml[(size_t)s * a.heads] : make_float2(-INFINITY, 0.0f);
      M = fmaxf(M, v[i].x);
    }
    M = warp_max(M);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      v[i].x = v[i].y > 0.0f ? ex2(v[i].x - M) : 0.0f;
      L += v[i].x * v[i].y;
    }
    L = warp_sum(L);
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (lane + 32 * i < nsplit) sw[warp][lane + 32 * i] = v[i].x > 0.0f ? v[i].x / L : 0.0f;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 8 * (a.rk >> 2); i += 256) {
    const int r = i / (a.rk >> 2), c = (i - r * (a.rk >> 2)) * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t0 + r < T && c < a.rp) {
      const float* p = a.part + ((size_t)(t0 + r) * nsplit * a.heads + head) * a.rp + c;
#pragma unroll 4
      for (int s = 0; s < nsplit; ++s) {
        const float f = sw[r][s];
        if (f == 0.0f) continue;                          // nothing was written there
        const float4 v = *reinterpret_cast<const float4*>(p + (size_t)s * a.heads * a.rp);
        acc.x += f * v.x; acc.y += f * v.y; acc.z += f * v.z; acc.w += f * v.w;
      }
    }
    *reinterpret_cast<uint2*>(so + r * ldo + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
  __syncthreads();
  const int g = lane >> 2, t4 = lane & 3;
  for (int r0 = warp * 16; r0 < a.vdim; r0 += 128) {
    float acc[4];
    rows_by_tokens(acc, w + (size_t)min(r0 + g, a.vdim - 1) * a.rk, w + (size_t)min(r0 + g + 8, a.vdim - 1) * a.rk, so, ldo, a.rk, lane);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = t0 + 2 * t4 + (e & 1), d = head * a.vdim + r0 + g + 8 * (e >> 1);
      if (t < T && r0 + g + 8 * (e >> 1) < a.vdim)
        static_cast<bf16*>(a.out)[(size_t)t * a.ldo + d] = __float2bfloat16_rn(acc[e] * a.out_scale * sigmoid(a.proj[(size_t)t * a.ld + a.g_col + d]));
    }
  }
}

// ---- expanded -----------------------------------------------------------------------------------------------------------------
// contexts[e] = {first scratch row, cached tokens, slot, 0}: the sequence's cache rows, one after another
__global__ void __launch_bounds__(256) gather_kernel(Latent a, const int4* contexts, bf16* lat, int ldl) {
  pdl_wait();
  pdl_trigger();
  const int4 c = contexts[blockIdx.y];
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= c.y) return;
  const bf16* src = static_cast<const bf16*>(a.pool) + latent_row(a, a.block_table + (size_t)c.z * a.max_pages, t) * a.row;
  bf16* dst = lat + (size_t)(c.x + t) * ldl;
  for (int i = lane; i < a.row >> 3; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
}

struct Expanded {
  const bf16* kv;           // [scratch rows][ldkv]: per head dim8 keys, then vdim8 values (dim and vdim to 8)
  const bf16* lat;          // [scratch rows][ldl]: the gathered cache rows
  int ldkv, ldl, dim8, vdim8;
};

// entries[e] = {first row, tokens, slot, first position}, contexts as above, tiles[i] = {entry, first token of 128}; grid (heads, tiles)
template <int KD, int VD>
__global__ void __launch_bounds__(256) latent_prompt_kernel(Latent a, Expanded x, const int4* entries, const int4* contexts, const int2* tiles) {
  constexpr int LK = KD + 8, LV = VD + 8;
  constexpr bool kQReg = KD <= 128 || (KD <= 192 && VD <= 128);      // query fragments stay in registers
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* sQ = reinterpret_cast<bf16*>(smem_raw);           // [128][LK]
  bf16* sK = sQ + 128 * LK;                               // two stages of [64][LK]
  bf16* sV = sK + 2 * 64 * LK;                            // two stages of [64][LV]
  const int head = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  pdl_trigger();
  const int2 tl = tiles[gridDim.y - 1 - blockIdx.y];
  const int4 en = entries[tl.x], ctx = contexts[tl.x];
  const int q0 = tl.y, ntok = min(128, en.y - q0), pfirst = en.w + q0, hi = pfirst + ntok;
  const bf16* kv = x.kv + (size_t)ctx.x * x.ldkv + head * (x.dim8 + x.vdim8);
  const bf16* lat = x.lat + (size_t)ctx.x * x.ldl + a.rp;
  const int kcols = x.dim8 + ((a.rot_dim + 7) & ~7);
  auto fetch = [&](int kb, int st) {
    bf16* dk = sK + st * 64 * LK;
    bf16* dv = sV + st * 64 * LV;
#pragma unroll 2
    for (int i = threadIdx.x; i < 64 * (KD / 8); i += 256) {
      const int r = i / (KD / 8), c = (i % (KD / 8)) * 8, t = kb + r;
      const bf16* src = c < x.dim8 ? kv + (size_t)t * x.ldkv + c : lat + (size_t)t * x.ldl + c - x.dim8;
      const bool ok = t < hi && c < kcols;
      cp_async16(dk + r * LK + c, ok ? src : kv, ok);
    }
#pragma unroll 2
    for (int i = threadIdx.x; i < 64 * (VD / 8); i += 256) {
      const int r = i / (VD / 8), c = (i % (VD / 8)) * 8, t = kb + r;
      const bool ok = t < hi && c < x.vdim8;
      cp_async16(dv + r * LV + c, ok ? kv + (size_t)t * x.ldkv + x.dim8 + c : kv, ok);
    }
  };
  fetch(0, 0);
  cp_async_commit();
  const float f = a.scale * kLog2e;
  for (int r = warp * 16; r < warp * 16 + 16; ++r) {
    const float* q = a.proj + (size_t)(en.x + q0 + min(r, ntok - 1)) * a.ld + a.q_col + head * (a.dim + a.rot_dim);
    const float2* rot = latent_angles(a, pfirst + min(r, ntok - 1));
    for (int d = lane; d < KD; d += 32) {
      const int e = d - x.dim8;
      const float v = d < a.dim ? q[d] : (e >= 0 && e < a.rot_dim ? rotated(q + a.dim, e, rot, a.rot_dim, 1) : 0.0f);
      sQ[r * LK + d] = __float2bfloat16_rn(v * f);
    }
  }
  __syncwarp();
  uint32_t qf[kQReg ? KD / 16 : 1][4];
  if (kQReg) {
#pragma unroll
    for (int ks = 0; ks < (kQReg ? KD / 16 : 1); ++ks) ldsm4(qf[ks], frag_a(sQ, LK, warp * 16, ks * 16, lane));
  }
  float o[VD / 8][4];
#pragma unroll
  for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  const int row0 = warp * 16 + (lane >> 2), wfirst = pfirst + warp * 16;     // this thread's rows: row0 and row0 + 8
  const bool live = warp * 16 < ntok;                                        // a warp without rows only helps with the copies
  for (int it = 0, kb = 0; kb < hi; ++it, kb += 64) {
    cp_async_wait<0>();
    __syncthreads();     // the tile has landed, and everyone is done with the other stage
    if (kb + 64 < hi) fetch(kb + 64, (it + 1) & 1);
    cp_async_commit();
    if (!live || kb > wfirst + 15) continue;              // all of the tile's keys lie behind this warp's rows
    const bf16* k = sK + (it & 1) * 64 * LK;
    const bf16* v = sV + (it & 1) * 64 * LV;
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < KD / 16; ++ks) {
      uint32_t qt[4];
      if (!kQReg) ldsm4(qt, frag_a(sQ, LK, warp * 16, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        ldsm4(b, frag_b_rows(k, LK, np * 16, ks * 16, lane));
        mma_bf16(s[2 * np], kQReg ? qf[kQReg ? ks : 0] : qt, b[0], b[1]);
        mma_bf16(s[2 * np + 1], kQReg ? qf[kQReg ? ks : 0] : qt, b[2], b[3]);
      }
    }
    float nm[2] = {mx[0], mx[1]};
    const bool whole = kb + 63 <= wfirst;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = kb + nt * 8 + (lane & 3) * 2 + (e & 1);
        if (!whole && j > pfirst + row0 + 8 * (e >> 1)) s[nt][e] = -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], s[nt][e]);
      }
    float base[2], resc[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 1));
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 2));
      base[r] = nm[r] == -INFINITY ? 0.0f : nm[r];
      resc[r] = ex2(mx[r] - base[r]);
      mx[r] = nm[r];
      l[r] *= resc[r];
    }
    uint32_t p[8][2];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) {
      float e[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        e[i] = ex2(s[nt][i] - base[i >> 1]);
        l[i >> 1] += e[i];
      }
      p[nt][0] = pack_bf16(e[0], e[1]);
      p[nt][1] = pack_bf16(e[2], e[3]);
    }
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
      o[i][0] *= resc[0]; o[i][1] *= resc[0];
      o[i][2] *= resc[1]; o[i][3] *= resc[1];
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      const uint32_t pa[4] = {p[2 * ks][0], p[2 * ks][1], p[2 * ks + 1][0], p[2 * ks + 1][1]};
#pragma unroll
      for (int np = 0; np < VD / 16; ++np) {
        uint32_t b[4];
        ldsm4_t(b, frag_b_cols(v, LV, ks * 16, np * 16, lane));
        mma_bf16(o[2 * np], pa, b[0], b[1]);
        mma_bf16(o[2 * np + 1], pa, b[2], b[3]);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = row0 + 8 * r;
    if (row >= ntok) continue;
    const size_t t = en.x + q0 + row;
    const float inv = a.out_scale / l[r];
    const float* gate = a.proj + t * a.ld + a.g_col + head * a.vdim;
    bf16* dst = static_cast<bf16*>(a.out) + t * a.ldo + head * a.vdim;
#pragma unroll
    for (int nt = 0; nt < VD / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = nt * 8 + (lane & 3) * 2 + e;
        if (d < a.vdim) dst[d] = __float2bfloat16_rn(o[nt][2 * r + e] * inv * sigmoid(gate[d]));
      }
  }
}

// ---- 32-bit mode ----------------------------------------------------------------------------------------------------------------
// grid (heads, rows): exact f32 products and exponentials; four warps take the keys in turn
constexpr int kMaxRank = 512, kMaxRot = 256;

__global__ void __launch_bounds__(128) latent_f32_kernel(Latent a) {
  constexpr int NC = kMaxRank / 32, NR = kMaxRot / 32;
  __shared__ float sq[kMaxRank + kMaxRot], sm[4][kMaxRank + 2];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, pos = a.pos[t];
  if (pos >= (a.max_pages << a.pshift)) return;
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  const float* pool = static_cast<const float*>(a.pool);
  const float* q = a.proj + (size_t)t * a.ld + a.q_col + h * (a.dim + a.rot_dim);
  const float2* rot = latent_angles(a, pos);
  for (int r = threadIdx.x; r < a.rank; r += 128) {
    const bf16* w = a.wk + ((size_t)h * a.rp + r) * a.dk;
    float s = 0.0f;
    for (int d = 0; d < a.dim; ++d) s = fmaf(q[d], __bfloat162float(w[d]), s);
    sq[r] = s;
  }
  for (int d = threadIdx.x; d < a.rot_dim; d += 128) sq[a.rank + d] = rotated(q + a.dim, d, rot, a.rot_dim, 1);
  __syncthreads();
  float o[NC], m = -INFINITY, l = 0.0f;
#pragma unroll
  for (int c = 0; c < NC; ++c) o[c] = 0.0f;
  for (int j = warp; j <= pos; j += 4) {
    const float* row = pool + latent_row(a, bt, j) * a.row;
    float k[NC], s = 0.0f;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int d = lane + 32 * c;
      k[c] = d < a.rank ? row[d] : 0.0f;
      if (d < a.rank) s = fmaf(sq[d], k[c], s);
    }
#pragma unroll
    for (int c = 0; c < NR; ++c) {
      const int d = lane + 32 * c;
      if (d < a.rot_dim) s = fmaf(sq[a.rank + d], row[a.rp + d], s);
    }
    s = warp_sum(s) * a.scale;
    const float nm = fmaxf(m, s), f = expf(m - nm), p = expf(s - nm);
    m = nm;
    l = l * f + p;
#pragma unroll
    for (int c = 0; c < NC; ++c) o[c] = o[c] * f + p * k[c];
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) sm[warp][lane + 32 * c] = o[c];
  if (lane == 0) {
    sm[warp][kMaxRank] = m;
    sm[warp][kMaxRank + 1] = l;
  }
  __syncthreads();
  float M = -INFINITY, L = 0.0f;
  for (int w = 0; w < 4; ++w) M = fmaxf(M, sm[w][kMaxRank]);
  for (int w = 0; w < 4; ++w) L += expf(sm[w][kMaxRank] - M) * sm[w][kMaxRank + 1];
  for (int r = threadIdx.x; r < a.rank; r += 128) {
    float acc = 0.0f;
    for (int w = 0; w < 4; ++w) acc += expf(sm[w][kMaxRank] - M) * sm[w][r];
    sq[r] = acc / L;
  }
  __syncthreads();
  for (int d = warp; d < a.vdim; d += 4) {
    const bf16* w = a.wv + ((size_t)h * a.vdim + d) * a.rk;
    float s = 0.0f;
    for (int r = lane; r < a.rank; r += 32) s = fmaf(sq[r], __bfloat162float(w[r]), s);
    s = warp_sum(s);
    if (lane == 0)
      static_cast<float*>(a.out)[(size_t)t * a.ldo + h * a.vdim + d] = s * a.out_scale * sigmoid(a.proj[(size_t)t * a.ld + a.g_col + h * a.vdim + d]);
  }
}

// ---- launches ---------------------------------------------------------------------------------------------------------------------
static int up(int n, int m) { return (n + m - 1) / m * m; }
static int latent_row_size(int rank, int rot) { return up(up(rank, 16) + up(rot, 16), 32); }

static bool fill(Latent& a, const void* const* ptrs, const int* ints, const float* floats) {
  a.proj = (const float*)ptrs[0]; a.c_norm = (const float*)ptrs[1]; a.rot = (const float2*)ptrs[2]; a.pos = (const int*)ptrs[3];
  a.slots = (const int*)ptrs[4]; a.block_table = (const int*)ptrs[5]; a.pool = const_cast<void*>(ptrs[6]); a.wk = (const bf16*)ptrs[7];
  a.wv = (const bf16*)ptrs[8]; a.q = (bf16*)const_cast<void*>(ptrs[9]); a.part = (float*)const_cast<void*>(ptrs[10]);
  a.ml = (float2*)const_cast<void*>(ptrs[11]); a.out = const_cast<void*>(ptrs[12]);
  a.ld = ints[0]; a.q_col = ints[1]; a.c_col = ints[2]; a.r_col = ints[3]; a.g_col = ints[4]; a.ldo = ints[5]; a.heads = ints[6]; a.dim = ints[7];
  a.rot_dim = ints[8]; a.vdim = ints[9]; a.rank = ints[10]; a.max_pages = ints[11];
  for (a.pshift = 0; (2 << a.pshift) <= ints[12]; ++a.pshift) {}
  a.eps = floats[0]; a.scale = floats[1]; a.out_scale = floats[2];
  a.rp = up(a.rank, 16); a.row = latent_row_size(a.rank, a.rot_dim); a.dk = up(a.dim, 32); a.rk = up(a.rank, 32);
  return a.heads >= 1 && a.dim >= 1 && a.rot_dim >= 2 && a.rot_dim % 2 == 0 && a.rot_dim <= kMaxRot && a.vdim >= 1 && a.rank >= 1 && a.rank <= kMaxRank &&
         a.max_pages >= 1 && (1 << a.pshift) == ints[12];
}

template <int CB, int MT>
static int run_latent_decode(const Latent& a, int T, int nsplit, cudaStream_t stream) {
  constexpr int H = 16 * MT;
  const size_t smem = (size_t)(H + 128) * (a.row + 8) * sizeof(bf16) + H * (68 * sizeof(float) + 72 * sizeof(bf16) + sizeof(float));
  if (smem > 227 * 1024) return BONSAI_CUDA_BAD_ARG;
  return launch(latent_decode_kernel<CB, MT>, dim3((a.heads + H - 1) / H, nsplit, T), 256, smem, stream, 1, 0, a);
}

template <int KD, int VD>
static int run_latent_prompt(const Latent& a, const Expanded& x, const int* entries, const int* contexts, const int* tiles, int ntiles, cudaStream_t stream) {
  const size_t smem = (size_t)(256 * (KD + 8) + 128 * (VD + 8)) * sizeof(bf16);
  static_assert((size_t)(256 * (KD + 8) + 128 * (VD + 8)) * sizeof(bf16) <= 227 * 1024, "shared memory of a CTA");
  return launch(latent_prompt_kernel<KD, VD>, dim3(a.heads, ntiles), 256, smem, stream, 1, 0, a, x, (const int4*)entries, (const int4*)contexts,
                (const int2*)tiles);
}

}  // namespace lay
}  // namespace bonsai

extern "C" {

// elements of a cache row
int bonsai_lay_latent_row(int rank, int rot_dim) { return rank < 1 || rot_dim < 2 ? 0 : bonsai::lay::latent_row_size(rank, rot_dim); }
int bonsai_lay_latent_max_splits() { return bonsai::lay::kMaxSplits; }
// heads that one CTA of the decode kernel serves
int bonsai_lay_latent_group(int heads) { return heads <= 16 ? 16 : 32; }

// Arguments of all launches: ptrs = {proj, c_norm, rot, pos, slots, block_table, pool, wk, wv, q, part, ml, out}, ints = {ld, q_col,
// c_col, r_col, g_col, ldo, heads, dim, rot_dim, vdim, rank, max_pages, page_size}, floats = {eps, scale, out_scale}.  rot has a row for
// every position the pages hold.

// Writes the cache rows of batch rows first .. first + count - 1.
int bonsai_lay_latent_append(const void* const* ptrs, const int* ints, const float* floats, int first, int count, int f32, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || first < 0 || count < 1) return BONSAI_CUDA_BAD_ARG;
  return f32 ? launch(latent_append_kernel<float>, dim3((count + 3) / 4), 128, 0, stream, 1, 0, a, first, count)
             : launch(latent_append_kernel<bf16>, dim3((count + 3) / 4), 128, 0, stream, 1, 0, a, first, count);
}

// Rows 0 .. T - 1: cache rows and absorbed queries.
int bonsai_lay_latent_query(const void* const* ptrs, const int* ints, const float* floats, int T, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 8 * 65535) return BONSAI_CUDA_BAD_ARG;
  return launch(query_kernel, dim3(a.heads + 1, (T + 7) / 8), 256, 8 * (a.dk + 8) * sizeof(bf16), stream, 1, 0, a, T);
}

// Rows 0 .. T - 1, their cache rows and queries made: partial sums of `nsplit` splits of the keys.
int bonsai_lay_latent_decode(const void* const* ptrs, const int* ints, const float* floats, int T, int nsplit, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 65535 || nsplit < 1 || nsplit > kMaxSplits) return BONSAI_CUDA_BAD_ARG;
  const int cb = (a.rp + 127) / 128;
#define BONSAI_LATENT(CB) (a.heads <= 16 ? run_latent_decode<CB, 1>(a, T, nsplit, stream) : run_latent_decode<CB, 2>(a, T, nsplit, stream))
  return cb == 1 ? BONSAI_LATENT(1) : (cb == 2 ? BONSAI_LATENT(2) : (cb == 3 ? BONSAI_LATENT(3) : BONSAI_LATENT(4)));
#undef BONSAI_LATENT
}

// Rows 0 .. T - 1: joins the splits, expands and gates.
int bonsai_lay_latent_value(const void* const* ptrs, const int* ints, const float* floats, int T, int nsplit, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 8 * 65535 || nsplit < 1 || nsplit > kMaxSplits) return BONSAI_CUDA_BAD_ARG;
  return launch(value_kernel, dim3(a.heads, (T + 7) / 8), 256, 8 * (a.rk + 8) * sizeof(bf16), stream, 1, 0, a, T, nsplit);
}

// contexts int4 [n] {first scratch row, cached tokens (at most `longest`), slot, 0}: their cache rows into lat (rows of ldl elements)
int bonsai_lay_latent_gather(const void* const* ptrs, const int* ints, const float* floats, const int* contexts, int n, int longest, void* lat, int ldl,
                             cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || n < 1 || n > 65535 || longest < 1 || ldl < a.row || ldl % 8 != 0) return BONSAI_CUDA_BAD_ARG;
  return launch(gather_kernel, dim3((longest + 7) / 8, n), 256, 0, stream, 1, 0, a, (const int4*)contexts, (bf16*)lat, ldl);
}

// entries int4 [..] {first row, tokens, slot, first position} with contexts of the same index, tiles int2 [ntiles] {entry, first token
// of 128}; kv: the expanded keys and values of the gathered rows, per head dim and vdim columns, each padded to 8
int bonsai_lay_latent_prompt(const void* const* ptrs, const int* ints, const float* floats, const int* entries, const int* contexts, const int* tiles,
                             int ntiles, const void* kv, int ldkv, const void* lat, int ldl, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || ntiles < 1 || ntiles > 65535 || ldkv % 8 != 0 || ldl % 8 != 0) return BONSAI_CUDA_BAD_ARG;
  const Expanded x{(const bf16*)kv, (const bf16*)lat, ldkv, ldl, up(a.dim, 8), up(a.vdim, 8)};
  const int kd = x.dim8 + up(a.rot_dim, 8), vd = a.vdim;
#define BONSAI_LATENT_PROMPT(KD, VD) run_latent_prompt<KD, VD>(a, x, entries, contexts, tiles, ntiles, stream)
#define BONSAI_LATENT_VD(KD) (vd <= 64 ? BONSAI_LATENT_PROMPT(KD, 64) : (vd <= 128 ? BONSAI_LATENT_PROMPT(KD, 128) : BONSAI_LATENT_PROMPT(KD, 256)))
  if (kd > 256 || vd > 256) return BONSAI_CUDA_BAD_ARG;
  return kd <= 64 ? BONSAI_LATENT_VD(64) : (kd <= 128 ? BONSAI_LATENT_VD(128) : (kd <= 192 ? BONSAI_LATENT_VD(192) : BONSAI_LATENT_VD(256)));
#undef BONSAI_LATENT_VD
#undef BONSAI_LATENT_PROMPT
}

// All T rows, 32-bit throughout; their cache rows must have been appended.
int bonsai_lay_latent_f32(const void* const* ptrs, const int* ints, const float* floats, int T, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 65535) return BONSAI_CUDA_BAD_ARG;
  return launch(latent_f32_kernel, dim3(a.heads, T), 128, 0, stream, 1, 0, a);
}

}  // extern "C"
