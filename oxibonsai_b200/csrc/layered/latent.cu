// Attention over a compressed cache: per token one normalised latent c and one rotated key part that all heads share,
//
//   c = norm(W_c h) * w,  k_h = [W_uk,h c, rot(W_r h)],  v_h = W_uv,h c,  q_h = [u_h, rot(r_h)]
//   out_h = (softmax(scale q_h . k_h) V_h) * sigmoid(gate) * out_scale                  one gate per element
//
// The paged cache holds rows [c | rotated part], each part padded with zeros to 16 elements, the row to 32.  Two ways to the same sum:
//
//  * absorbed, for single tokens and short portions: (W_uk,h^T u_h) . c instead of u_h . (W_uk,h c), and the weighted sum of the
//    latents goes through W_uv,h afterwards, so all heads read the same cache row once.  `query_kernel` appends the rows' latents
//    and makes the queries, `latent_decode_kernel` leaves one partial sum per cluster of CTAs that share the keys, `value_kernel`
//    joins those, expands and gates.  A row is a token with a position and a slot, so tokens of one portion need not know of each other;
//  * expanded, for longer portions: `gather_kernel` brings the sequence's rows together, one product makes every head's keys and
//    values of them, and `prompt_kernel` is ordinary attention with one key/value head per query head.
//
// `f32_kernel` is the 32-bit mode, absorbed.
#include <cooperative_groups.h>
#include <cuda.h>

#include "cuda/tcgen05.cuh"
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

constexpr int kMaxRank = 512, kMaxRot = 256, kMaxSplits = 128, kMaxCluster = 8, kMaxParts = 16;

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
  bf16* q;                  // [rows][heads][row]: absorbed queries times scale * log2(e), columns in the order of `query_at`
  float* part;              // [rows][parts][heads][rp]: sums of ex2(score - max) c
  float2* ml;               // [rows][parts][heads]: maximum and sum of ex2(score - max)
  int* status;              // set to 1 when a copy does not arrive
  void* out;                // [T][ldo], head h at h * vdim
  int ld, q_col, c_col, r_col, g_col, ldo;
  int heads, dim, rot_dim, vdim, rank, max_pages, pshift;   // page size 1 << pshift
  int rp, row, dk, rk;      // rank to 16, the row, dim to 32, rank to 32
  int q_rows, parts;        // rows of q, and of part and ml over all rows and parts
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
  if ((a.rank & 3) == 0 && ((a.ld | a.c_col) & 3) == 0) {
    float4 v[kMaxRank / 128];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kMaxRank / 128; ++i) {
      const int d = 4 * lane + 128 * i;
      v[i] = d < a.rank ? *reinterpret_cast<const float4*>(c + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
#pragma unroll
    for (int i = 0; i < kMaxRank / 128; ++i) {
      const int d = 4 * lane + 128 * i;
      if (d >= a.rp) continue;
      const float4 w = d < a.rank ? *reinterpret_cast<const float4*>(a.c_norm + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      store_act4(dst + d, make_float4(v[i].x * inv * w.x, v[i].y * inv * w.y, v[i].z * inv * w.z, v[i].w * inv * w.w));
    }
  } else {
    float ss = 0.0f;
    for (int d = lane; d < a.rank; d += 32) ss += c[d] * c[d];
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
    for (int d = lane; d < a.rp; d += 32) store_act(dst + d, d < a.rank ? c[d] * inv * a.c_norm[d] : 0.0f);
  }
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

// 16 rows of a weight matrix over NK steps of 32 inputs `stride` steps apart, as A registers: a lane loads 16 contiguous bytes of a row,
// so the inputs inside every 32 are permuted; `rows_by_tokens` reads the tokens (rows of ldx elements in shared memory) through the
// same permutation.
template <int NK>
struct WeightRows {
  uint4 a[NK], b[NK];
  __device__ __forceinline__ void load(const bf16* w0, const bf16* w1, int first, int stride, int steps, int lane) {
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int k = first + i * stride;
      if (k >= steps) continue;
      a[i] = *reinterpret_cast<const uint4*>(w0 + 32 * k + 8 * (lane & 3));
      b[i] = *reinterpret_cast<const uint4*>(w1 + 32 * k + 8 * (lane & 3));
    }
  }
  template <int NT>
  __device__ __forceinline__ void rows_by_tokens(float (&acc)[NT][4], const bf16* sx, int ldx, int first, int stride, int steps, int lane) const {
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int k = first + i * stride;
      if (k >= steps) continue;
      const uint32_t lo[4] = {a[i].x, b[i].x, a[i].y, b[i].y}, hi[4] = {a[i].z, b[i].z, a[i].w, b[i].w};
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const uint4 v = *reinterpret_cast<const uint4*>(sx + (8 * j + (lane >> 2)) * ldx + 32 * k + 8 * (lane & 3));
        mma_bf16(acc[j], lo, v.x, v.y);
        mma_bf16(acc[j], hi, v.z, v.w);
      }
    }
  }
};

// ---- absorbed -----------------------------------------------------------------------------------------------------------------
// Place of column c of an absorbed query: in every 32 columns the eight that a lane holds as A registers of two steps are neighbours.
__device__ __forceinline__ int query_at(int c) { return (c & ~31) | ((c & 6) << 2) | ((c & 16) >> 2) | ((c & 8) >> 2) | (c & 1); }

// One grid of three kinds of CTAs: cache entries (8 rows), the rotated parts of the queries (32 pairs of row and head), and the absorbed
// parts (128 latent columns of one head for 8 NT rows).
template <int NT, int NK>
__global__ void __launch_bounds__(256) query_kernel(Latent a, int T, int blocks) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* sq = reinterpret_cast<bf16*>(smem_raw);       // [8 NT][dk + 8]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, appends = (T + 7) / 8, turns = (T * a.heads + 31) / 32;
  int job = blockIdx.x;
  if (job < appends + turns) {
    pdl_wait();
    pdl_trigger();
    if (job < appends) {
      if (job * 8 + warp < T) append_latent<bf16>(a, job * 8 + warp, lane);
      return;
    }
    const float f = a.scale * kLog2e;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int pair = (job - appends) * 32 + warp * 4 + i, t = pair / a.heads, head = pair - t * a.heads;
      if (t >= T) return;
      const float* q = a.proj + (size_t)t * a.ld + a.q_col + head * (a.dim + a.rot_dim) + a.dim;
      bf16* dst = a.q + (size_t)pair * a.row;
      const int pos = a.pos[t];
      const float2* rot = latent_angles(a, pos < (a.max_pages << a.pshift) ? pos : 0);
      for (int d = lane; d < a.row - a.rp; d += 32)
        dst[query_at(a.rp + d)] = __float2bfloat16_rn(d < a.rot_dim ? rotated(q, d, rot, a.rot_dim, 1) * f : 0.0f);
    }
    return;
  }
  job -= appends + turns;
  const int head = job / blocks % a.heads, r0 = (job % blocks) * 128 + warp * 16, t0 = job / (blocks * a.heads) * 8 * NT;
  const int ldq = a.dk + 8, g = lane >> 2, t4 = lane & 3, steps = a.dk >> 5;
  const bf16* w = a.wk + ((size_t)head * a.rp + min(r0, a.rp - 16) + g) * a.dk;
  WeightRows<NK> wr;
  wr.load(w, w + 8 * a.dk, 0, 1, steps, lane);        // weights depend on no earlier kernel
  pdl_wait();
  pdl_trigger();
  const float* q = a.proj + a.q_col + head * (a.dim + a.rot_dim);
#pragma unroll 8
  for (int i = threadIdx.x; i < 8 * NT * a.dk; i += 256) {
    const int r = i / a.dk, d = i - r * a.dk;
    sq[r * ldq + d] = __float2bfloat16_rn(d < a.dim ? q[(size_t)min(t0 + r, T - 1) * a.ld + d] : 0.0f);
  }
  __syncthreads();
  if (r0 >= a.rp) return;
  float acc[NT][4];
  wr.rows_by_tokens<NT>(acc, sq, ldq, 0, 1, steps, lane);
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int tok = t0 + 8 * j + 2 * t4 + (e & 1), r = r0 + g + 8 * (e >> 1);
      if (tok < T) a.q[((size_t)tok * a.heads + head) * a.row + query_at(r)] = __float2bfloat16_rn(acc[j][e] * a.scale * kLog2e);
    }
}

__device__ __forceinline__ void tma_rows(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_addr(dst)), "l"(map),
               "r"(x), "r"(y), "r"(smem_addr(bar))
               : "memory");
}

// grid (groups of 16 MT heads, splits, rows), the splits in clusters.  A CTA walks tiles of 64 keys of its split, which TMA copies
// bring in as blocks of 64 columns (128-byte swizzle): sixteen warps share the scores by head group, keys and quarters of the
// row (the queries' share stays in registers), the softmax by heads, and the weighted sum by latent columns (CB blocks of 16 a warp).  The CTAs of a cluster meet in distributed shared memory and leave
// one sum.  rows_map: the cache rows [pages * page_size][row] in boxes of 64 columns x min(64, page size) rows.
constexpr int kBlockBytes = 64 * 128;

// element (r, c) of a staged tile, c at the start of 8 columns
__device__ __forceinline__ const bf16* tile_at(const uint8_t* k, int r, int c) {
  return reinterpret_cast<const bf16*>(k + (c >> 6) * kBlockBytes + r * 128 + ((((c >> 3) & 7) ^ (r & 7)) << 4));
}

template <int CB, int MT>
__global__ void __launch_bounds__(512) latent_decode_kernel(const __grid_constant__ CUtensorMap rows_map, Latent a, int cl) {
  constexpr int H = 16 * MT, LDS = 72, LDP = 72, NK = 5, NTH = 512;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ uint64_t full[2];
  __shared__ float2 s_ml[H];
  __shared__ float s_f[kMaxCluster][H];
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int blocks = (a.row + 63) >> 6, stage = blocks * kBlockBytes;
  uint8_t* sK = reinterpret_cast<uint8_t*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);   // two stages, later this CTA's sums
  float* sS = reinterpret_cast<float*>(sK + 2 * stage);   // [4][H][LDS] scores from the quarters of the row
  bf16* sP = reinterpret_cast<bf16*>(sS + 4 * H * LDS);   // [H][LDP] weights
  float* sF = reinterpret_cast<float*>(sP + H * LDP);     // [H] factors of the sums so far
  float* sO = reinterpret_cast<float*>(sK);               // [H][rp + 8]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int h0 = blockIdx.x * H, nh = min(H, a.heads - h0), split = blockIdx.y, nsplit = gridDim.y, t = blockIdx.z;
  const int pos = a.pos[t];
  const bool held = pos < (a.max_pages << a.pshift);      // otherwise no page can hold the row: its output is not defined
  const int ntiles = held ? (pos >> 6) + 1 : 0, per = (ntiles + nsplit - 1) / nsplit;
  const int b0 = split * per, b1 = min(ntiles, b0 + per);
  const int* bt = a.block_table + (size_t)a.slots[t] * a.max_pages;
  if (threadIdx.x == 0) {
    tc::mbar_init(&full[0], blocks);
    tc::mbar_init(&full[1], blocks);
    tc::mbar_fence_init();
  }
  __syncthreads();
  const int box = min(64, 1 << a.pshift);                 // rows of a copy: they lie in one page
  auto first_row = [&](int tile) { return tile < ntiles ? (int)latent_row(a, bt, tile * 64) : 0; };
  auto fetch = [&](int tile, int st, int row) {           // one thread of `blocks` warps each; pages past the last position are not touched
    const int n = (min(64, pos + 1 - tile * 64) + box - 1) / box;
    tc::mbar_arrive_expect_tx(&full[st], (uint32_t)(n * box * 128));
    for (int i = 0; i < n; ++i)
      tma_rows(sK + st * stage + warp * kBlockBytes + i * box * 128, &rows_map, warp * 64, i == 0 ? row : (int)latent_row(a, bt, tile * 64 + i * box), &full[st]);
  };
  const bool copies = lane == 0 && warp < blocks;
  int next_row = copies ? first_row(b0) : 0;
  // rows of this batch are appended by the kernel before this one; a tile that ends 64 tokens before this one holds none of them
  const bool early = b0 < b1 && b0 * 64 + 64 <= pos - 63;
  if (early && copies) fetch(b0, 0, next_row);
  pdl_wait();
  pdl_trigger();
  float mx[MT], l[MT];                                    // heads warp * MT + i
#pragma unroll
  for (int i = 0; i < MT; ++i) mx[i] = -INFINITY, l[i] = 0.0f;
  if (b0 < b1) {
    if (!early && copies) fetch(b0, 0, next_row);
    if (copies) next_row = first_row(b0 + 1);
    // this warp's scores: 16 heads x 16 MT keys over blocks kq, kq + 4, .. of 32 columns
    const int mt = warp % MT, kq = (warp / MT) & 3, key0 = (warp / (4 * MT)) * 16 * MT, nk = ((a.row >> 5) - kq + 3) >> 2;
    uint4 q0[NK], q1[NK];                                 // the queries' share: A registers of two steps each
    {
      const int r0 = mt * 16 + g;
      const bf16* p0 = a.q + ((size_t)t * a.heads + h0 + min(r0, nh - 1)) * a.row + 32 * kq + 8 * t4;
      const bf16* p1 = a.q + ((size_t)t * a.heads + h0 + min(r0 + 8, nh - 1)) * a.row + 32 * kq + 8 * t4;
#pragma unroll
      for (int i = 0; i < NK; ++i)
        if (i < nk) {
          q0[i] = *reinterpret_cast<const uint4*>(p0 + 128 * i);
          q1[i] = *reinterpret_cast<const uint4*>(p1 + 128 * i);
        }
    }
    float o[MT][2 * CB][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < 2 * CB; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.0f;
    for (int tile = b0; tile < b1; ++tile) {
      const int st = (tile - b0) & 1;
      uint8_t* k = sK + st * stage;
      __syncthreads();     // everyone is done with the other stage
      if (tile + 1 < b1 && copies) {
        fetch(tile + 1, st ^ 1, next_row);
        next_row = first_row(tile + 2);                   // used a tile later
      }
      if (!tc::mbar_wait(&full[st], ((tile - b0) >> 1) & 1) && lane == 0) atomicExch(a.status, 1);
      if (tile == ntiles - 1) {     // rows behind the last position may hold anything: their weights are zero, so they must be finite
        for (int i = threadIdx.x + (pos + 1 - tile * 64) * 8; i < 64 * 8; i += NTH)
          for (int b = 0; b < blocks; ++b) *reinterpret_cast<uint4*>(k + b * kBlockBytes + i * 16) = make_uint4(0u, 0u, 0u, 0u);
        __syncthreads();
      }
      float s[2 * MT][4];     // 16 heads x 16 MT keys
#pragma unroll
      for (int i = 0; i < 2 * MT; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
      for (int ks = 0; ks < NK; ++ks) {
        if (ks >= nk) continue;
        const uint32_t qa[2][4] = {{q0[ks].x, q1[ks].x, q0[ks].y, q1[ks].y}, {q0[ks].z, q1[ks].z, q0[ks].w, q1[ks].w}};
        uint32_t b[2][MT][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < MT; ++i)
            ldsm4(b[u][i], tile_at(k, key0 + 16 * i + (lane & 7) + ((lane >> 4) << 3), (kq + 4 * ks) * 32 + 16 * u + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma_bf16(s[2 * i], qa[u], b[u][i][0], b[u][i][1]);
            mma_bf16(s[2 * i + 1], qa[u], b[u][i][2], b[u][i][3]);
          }
      }
#pragma unroll
      for (int i = 0; i < 2 * MT; ++i)
#pragma unroll
        for (int e = 0; e < 4; e += 2)
          *reinterpret_cast<float2*>(sS + (kq * H + mt * 16 + g + 4 * e) * LDS + key0 + 8 * i + 2 * t4) = make_float2(s[i][e], s[i][e + 1]);
      __syncthreads();
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const int r = warp * MT + i;
        float2 u[4], v;
#pragma unroll
        for (int p = 0; p < 4; ++p) u[p] = *reinterpret_cast<const float2*>(sS + (p * H + r) * LDS + 2 * lane);
        v.x = tile * 64 + 2 * lane <= pos ? (u[0].x + u[1].x) + (u[2].x + u[3].x) : -INFINITY;
        v.y = tile * 64 + 2 * lane + 1 <= pos ? (u[0].y + u[1].y) + (u[2].y + u[3].y) : -INFINITY;
        const float nm = fmaxf(mx[i], warp_max(fmaxf(v.x, v.y)));      // the first key of a tile is always visible
        const float p0 = ex2(v.x - nm), p1 = ex2(v.y - nm), f = ex2(mx[i] - nm);
        mx[i] = nm;
        l[i] = l[i] * f + p0 + p1;                          // this lane's keys
        *reinterpret_cast<uint32_t*>(sP + r * LDP + 2 * lane) = pack_bf16(p0, p1);
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
          ldsm4_t(b, tile_at(k, ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, c + (lane >> 4) * 8));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][2 * j], p[m], b[0], b[1]);
            mma_bf16(o[m][2 * j + 1], p[m], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();     // the tiles are free: the sums take their place
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < 2 * CB; ++i) {
        const int c = (warp * CB + i / 2) * 16 + (i & 1) * 8 + 2 * t4;
        if (c >= a.rp) continue;
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(sO + (m * 16 + g + 8 * e) * (a.rp + 8) + c) = make_float2(o[m][i][2 * e], o[m][i][2 * e + 1]);
      }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const float sum = warp_sum(l[i]);
    if (lane == 0) s_ml[warp * MT + i] = make_float2(mx[i], sum);
  }
  if (cl > 1) cluster.sync();
  else __syncthreads();
  // every CTA of the cluster finishes its share of the heads and columns
  const int rank = split % cl, nparts = nsplit / cl;
  const size_t base = ((size_t)t * nparts + split / cl) * a.heads + h0;
  const int quads = a.rp >> 2;
  if (threadIdx.x < H) {
    float2 ml[kMaxCluster];
    float M = -INFINITY, L = 0.0f;
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s) {
      if (s >= cl) break;
      ml[s] = (cl > 1 ? cluster.map_shared_rank(s_ml, s) : s_ml)[threadIdx.x];
      M = fmaxf(M, ml[s].x);
    }
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s) {
      if (s >= cl) break;
      const float f = ml[s].y > 0.0f ? ex2(ml[s].x - M) : 0.0f;     // a split without keys left nothing
      L += f * ml[s].y;
      s_f[s][threadIdx.x] = f;
    }
    if (rank == 0 && threadIdx.x < nh) a.ml[base + threadIdx.x] = make_float2(M, L);
  }
  __syncthreads();
  for (int i = rank * NTH + threadIdx.x; i < nh * quads; i += cl * NTH) {
    const int r = i / quads, c = (i - r * quads) * 4;
    float4 v[kMaxCluster], acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s)
      if (s < cl) v[s] = *reinterpret_cast<const float4*>((cl > 1 ? cluster.map_shared_rank(sO, s) : sO) + r * (a.rp + 8) + c);
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s) {
      const float f = s < cl ? s_f[s][r] : 0.0f;
      if (f > 0.0f) {
        acc.x += f * v[s].x; acc.y += f * v[s].y; acc.z += f * v[s].z; acc.w += f * v[s].w;
      }
    }
    *reinterpret_cast<float4*>(a.part + (base + r) * a.rp + c) = acc;
  }
  if (cl > 1) {     // nobody leaves while its sums are being read; the reads are over when their values are stored
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
  }
}

// grid (heads x blocks of 16 RT value columns, groups of 8 NT rows): the partial sums become one latent per row, which is expanded
// (the warps share the columns and the latent) and gated
template <int NT, int RT>
__global__ void __launch_bounds__(256) value_kernel(Latent a, int T, int nparts, int blocks) {
  constexpr int SH = 8 / RT, NC = 16 * RT, NI = NT * kMaxRank / 128;     // shares of the latent, columns, blocks of 4 latents a thread joins
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* so = reinterpret_cast<bf16*>(smem_raw);           // [8 NT][rk + 8]
  __shared__ float sw[8 * NT][kMaxParts], sv[SH][8 * NT][NC + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.x / blocks, d0 = (blockIdx.x % blocks) * NC, t0 = blockIdx.y * 8 * NT;
  const int ldo = a.rk + 8, g = lane >> 2, t4 = lane & 3, steps = a.rk >> 5, r0 = d0 + (warp % RT) * 16, share = warp / RT;
  const bf16* w = a.wv + (size_t)head * a.vdim * a.rk;
  WeightRows<kMaxRank / 32 / SH> wr;
  wr.load(w + (size_t)min(r0 + g, a.vdim - 1) * a.rk, w + (size_t)min(r0 + g + 8, a.vdim - 1) * a.rk, share, SH, steps, lane);
  pdl_wait();
  pdl_trigger();
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int i = warp + 8 * j;
    const float2* ml = a.ml + (size_t)min(t0 + i, T - 1) * nparts * a.heads + head;
    const float2 v = lane < nparts ? ml[(size_t)lane * a.heads] : make_float2(-INFINITY, 0.0f);
    const float M = warp_max(v.x), f = v.y > 0.0f ? ex2(v.x - M) : 0.0f, L = warp_sum(f * v.y);
    if (lane < nparts) sw[i][lane] = f > 0.0f ? f / L : 0.0f;
  }
  __syncthreads();
  const int quads = a.rk >> 2;
  float4 acc4[NI];
#pragma unroll
  for (int j = 0; j < NI; ++j) acc4[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll (NT == 1 ? 4 : 1)
  for (int s = 0; s < nparts; ++s) {                      // a part without keys is zero
    float4 v[NI];
#pragma unroll
    for (int j = 0; j < NI; ++j) {
      const int i = threadIdx.x + 256 * j, r = i / quads, c = (i - r * quads) * 4;
      v[j] = r < 8 * NT && t0 + r < T && c < a.rp
                 ? *reinterpret_cast<const float4*>(a.part + (((size_t)(t0 + r) * nparts + s) * a.heads + head) * a.rp + c)
                 : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < NI; ++j) {
      const float f = sw[min((threadIdx.x + 256 * j) / quads, 8 * NT - 1)][s];
      acc4[j].x += f * v[j].x; acc4[j].y += f * v[j].y; acc4[j].z += f * v[j].z; acc4[j].w += f * v[j].w;
    }
  }
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    const int i = threadIdx.x + 256 * j, r = i / quads, c = (i - r * quads) * 4;
    if (r < 8 * NT) *reinterpret_cast<uint2*>(so + r * ldo + c) = make_uint2(pack_bf16(acc4[j].x, acc4[j].y), pack_bf16(acc4[j].z, acc4[j].w));
  }
  float gate[NT][NC / 32];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int b = 0; b < NC / 32; ++b) {
      const int t = t0 + warp + 8 * j, d = d0 + lane + 32 * b;
      gate[j][b] = t < T && d < a.vdim ? a.proj[(size_t)t * a.ld + a.g_col + head * a.vdim + d] : 0.0f;
    }
  __syncthreads();
  float acc[NT][4];
  wr.template rows_by_tokens<NT>(acc, so, ldo, share, SH, steps, lane);
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) sv[share][8 * j + 2 * t4 + (e & 1)][(warp % RT) * 16 + g + 8 * (e >> 1)] = acc[j][e];
  __syncthreads();
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int b = 0; b < NC / 32; ++b) {
      const int i = warp + 8 * j, c = lane + 32 * b;
      if (t0 + i >= T || d0 + c >= a.vdim) continue;
      float v = 0.0f;
#pragma unroll
      for (int p = 0; p < SH; ++p) v += sv[p][i][c];
      static_cast<bf16*>(a.out)[(size_t)(t0 + i) * a.ldo + head * a.vdim + d0 + c] = __float2bfloat16_rn(v * a.out_scale * sigmoid(gate[j][b]));
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
  a.ml = (float2*)const_cast<void*>(ptrs[11]); a.status = (int*)const_cast<void*>(ptrs[12]); a.out = const_cast<void*>(ptrs[13]);
  a.ld = ints[0]; a.q_col = ints[1]; a.c_col = ints[2]; a.r_col = ints[3]; a.g_col = ints[4]; a.ldo = ints[5]; a.heads = ints[6]; a.dim = ints[7];
  a.rot_dim = ints[8]; a.vdim = ints[9]; a.rank = ints[10]; a.max_pages = ints[11];
  for (a.pshift = 0; (2 << a.pshift) <= ints[12]; ++a.pshift) {}
  a.q_rows = ints[13]; a.parts = ints[14];
  a.eps = floats[0]; a.scale = floats[1]; a.out_scale = floats[2];
  a.rp = up(a.rank, 16); a.row = latent_row_size(a.rank, a.rot_dim); a.dk = up(a.dim, 32); a.rk = up(a.rank, 32);
  return a.heads >= 1 && a.dim >= 1 && a.rot_dim >= 2 && a.rot_dim % 2 == 0 && a.rot_dim <= kMaxRot && a.vdim >= 1 && a.dim <= 256 && a.rank >= 1 && a.rank <= kMaxRank &&
         a.max_pages >= 1 && a.pshift >= 4 && (1 << a.pshift) == ints[12];
}

template <int CB, int MT>
static int run_latent_decode(const CUtensorMap& map, const Latent& a, int T, int nsplit, int cl, cudaStream_t stream) {
  constexpr int H = 16 * MT;
  const size_t tiles = (size_t)2 * ((a.row + 63) / 64) * kBlockBytes;
  const size_t smem = 1024 + tiles + H * (4 * 72 * sizeof(float) + 72 * sizeof(bf16) + sizeof(float));
  if (smem > 225 * 1024 || a.row > 640 || (size_t)H * (a.rp + 8) * sizeof(float) > tiles) return BONSAI_CUDA_BAD_ARG;   // the sums take the tiles' place
  return launch(latent_decode_kernel<CB, MT>, dim3((a.heads + H - 1) / H, nsplit, T), 512, smem, stream, cl, 1, map, a, cl);
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
// most splits of the keys, and most of them that share a sum
int bonsai_lay_latent_max_splits() { return bonsai::lay::kMaxSplits; }
int bonsai_lay_latent_max_cluster() { return bonsai::lay::kMaxCluster; }
// heads that one CTA of the decode kernel serves
int bonsai_lay_latent_group(int heads) { return heads <= 16 ? 16 : 32; }

// Arguments of all launches: ptrs = {proj, c_norm, rot, pos, slots, block_table, pool, wk, wv, q, part, ml, status, out}, ints = {ld, q_col,
// c_col, r_col, g_col, ldo, heads, dim, rot_dim, vdim, rank, max_pages, page_size, q_rows, parts, pool_pages}, floats = {eps, scale,
// out_scale}.  rot has a row for every position the pages hold; q, part and ml have rows for q_rows rows and `parts` parts in all.

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
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > a.q_rows || T > 65535) return BONSAI_CUDA_BAD_ARG;
  const int blocks = (a.rp + 127) / 128;
#define BONSAI_QUERY_NK(NT, NK) \
  launch(query_kernel<NT, NK>, dim3((T + 7) / 8 + (T * a.heads + 31) / 32 + a.heads * blocks * ((T + 8 * NT - 1) / (8 * NT))), 256, \
         8 * NT * (a.dk + 8) * sizeof(bf16), stream, 1, 0, a, T, blocks)
#define BONSAI_QUERY(NT) (a.dk <= 128 ? BONSAI_QUERY_NK(NT, 4) : BONSAI_QUERY_NK(NT, 8))
  return T <= 8 ? BONSAI_QUERY(1) : (T <= 16 ? BONSAI_QUERY(2) : BONSAI_QUERY(4));
#undef BONSAI_QUERY
#undef BONSAI_QUERY_NK
}

// Rows 0 .. T - 1, their cache rows and queries made: the keys in `nsplit` splits, one partial sum for `cl` (1, 2, 4 or 8) of them.
int bonsai_lay_latent_decode(const void* const* ptrs, const int* ints, const float* floats, int T, int nsplit, int cl, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 65535 || nsplit < 1 || nsplit > kMaxSplits || (cl != 1 && cl != 2 && cl != 4 && cl != 8) ||
      nsplit % cl != 0 || nsplit / cl > kMaxParts || a.status == nullptr || T > a.q_rows || (long long)T * (nsplit / cl) > a.parts)
    return BONSAI_CUDA_BAD_ARG;
  CUtensorMap map;
  const cuuint64_t dims[2] = {(cuuint64_t)a.row, (cuuint64_t)ints[15] << a.pshift}, strides[1] = {(cuuint64_t)a.row * sizeof(bf16)};
  const cuuint32_t box[2] = {64, (cuuint32_t)(a.pshift < 6 ? 1 << a.pshift : 64)}, step[2] = {1, 1};
  if (ints[15] < 1 || cuTensorMapEncodeTiled(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.pool, dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return BONSAI_CUDA_BAD_ARG;
  const int cb = (a.rp + 255) / 256;
#define BONSAI_LATENT(CB) (a.heads <= 16 ? run_latent_decode<CB, 1>(map, a, T, nsplit, cl, stream) : run_latent_decode<CB, 2>(map, a, T, nsplit, cl, stream))
  return cb == 1 ? BONSAI_LATENT(1) : BONSAI_LATENT(2);
#undef BONSAI_LATENT
}

// Rows 0 .. T - 1: joins `nparts` partial sums, expands and gates.
int bonsai_lay_latent_value(const void* const* ptrs, const int* ints, const float* floats, int T, int nparts, cudaStream_t stream) {
  using namespace bonsai::lay;
  Latent a;
  if (!fill(a, ptrs, ints, floats) || T < 1 || T > 65535 || nparts < 1 || nparts > kMaxParts || (long long)T * nparts > a.parts) return BONSAI_CUDA_BAD_ARG;
  const int blocks = T <= 8 ? (a.vdim + 31) / 32 : (a.vdim + 63) / 64;
#define BONSAI_VALUE(NT, RT)                                                                                                                  \
  launch(value_kernel<NT, RT>, dim3(a.heads * blocks, (T + 8 * NT - 1) / (8 * NT)), 256, 8 * NT * (a.rk + 8) * sizeof(bf16), stream, 1, 0, a, T, \
         nparts, blocks)
  return T <= 8 ? BONSAI_VALUE(1, 2) : BONSAI_VALUE(2, 4);
#undef BONSAI_VALUE
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
