// The steps between sublayers with every part optional, and the causal convolution over tokens that several designs put in front of a
// projection.
//
// `row_step_kernel`, one CTA per row:
//   u = sigmoid(gate) (y + bias) + the chosen experts' rows        what a sublayer computed
//   x <- x + mult * norm(u) * w                                    or the start of the stream, where nothing came before
//   x <- x + scale * table[token] + step                           what a loop adds ahead of a pass; also the embedding itself
//   n = norm(x) * next                                             the next input, or the input of the head
//   h = n + conv(n)                                                conv: a causal convolution per channel
// Norms divide each of `groups` equal parts by its own root mean square.  A group belongs to a power of two of threads, each with KEEP
// chunks of VEC columns in registers, so a group's sum is a shuffle and, above a warp, one exchange.
//
// The convolution's inputs of earlier tokens are f32 in a ring [row][taps][channels], the input of position p at p % taps: a token
// never writes where it reads.  Steps of single tokens convolve in the row kernel.  Otherwise the row kernel leaves n as f32 and
// `conv_kernel` follows: a thread has a few channels of up to kConvRows tokens of one portion; the portion's first tile alone reads the ring
// and, afterwards, stores the portion's last inputs there.
#include "layered/layered.cuh"

namespace bonsai {
namespace lay {

constexpr int kConvRows = 16, kMaxTaps = kConvRows;

struct RowStep {
  float* x;                 // [T][width]
  const float* y;           // [T][ldy]; null: none
  const float* y_bias;      // [width] or null
  const float* y_gate;      // [T][ldg], one per row; null: 1
  const void* e;            // expert rows [..][lde], bf16 or f32; row at[t * top + k] is token t's k-th
  const int* at;
  int* counts;              // [experts], left zero; may be null
  const float* w;           // [width]; null: u as it is
  const bf16* table;        // [vocab][ld_table] or null
  const int* tokens;
  const float* step;        // [width] or null
  const float* next;        // [width]; null: n = x
  float* n32;               // [T][ldn] f32: receives n where the convolution follows
  void* h;                  // [T][ldh], bf16 or f32; null: x only
  const float* conv;        // [taps][width], tap j: the input j tokens back; null: h = n
  float* ring;
  const int* pos;
  const int* slots;
  const int* state_rows;
  const int* rows;          // x is read at rows[i] and nothing is written there; null: row i
  int ldy, ldg, lde, e_f32, top, experts, width, groups, ld_table, ldn, ldh, h_f32, taps, fresh, inline_conv;
  float eps, mult, scale;
};

// KEEP chunks of VEC columns per thread, tg = 2^tshift threads per group
template <int VEC, int KEEP, bool CONV>
__global__ void __launch_bounds__(KEEP * VEC > 8 ? 1024 : 512, KEEP * VEC > 8 || CONV ? 1 : 3) row_step_kernel(RowStep a, int tshift) {
  __shared__ float sums[2][32];
  const int tg = 1 << tshift, grp = threadIdx.x >> tshift, l = threadIdx.x & (tg - 1), gw = a.width / a.groups;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x, row = a.rows == nullptr ? t : a.rows[t];
  int col[KEEP];
  bool on[KEEP];
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (l + i * tg) * VEC;
    on[i] = grp < a.groups && c < gw;
    col[i] = on[i] ? grp * gw + c : 0;
  }
  auto load = [&](const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
      v[0] = *p;
    }
  };
  auto load16 = [&](const bf16* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      const uint2 q = *reinterpret_cast<const uint2*>(p);
      const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
      v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
    } else {
      v[0] = __bfloat162float(*p);
    }
  };
  auto store = [&](float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
  };
  // 1 / sqrt(mean + eps) of this thread's group
  auto inverse = [&](float ss, float* s) {
    for (int o = min(tg, 32) >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (tg > 32) {
      if (lane == 0) s[warp] = ss;
      __syncthreads();
      const int nw = tg >> 5, w0 = warp & ~(nw - 1);
      ss = 0.0f;
      for (int i = 0; i < nw; ++i) ss += s[w0 + i];
    }
    return 1.0f / sqrtf(ss / (float)gw + a.eps);
  };
  constexpr bool kEarly = KEEP * VEC <= 8;         // registers for weights ahead of the sums they follow
  // inputs of earlier tokens, older than the kernel before this one unless this is a step's first
  constexpr int kBack = CONV && KEEP * VEC <= 8 ? 3 : 0;
  float back[KEEP][kBack > 0 ? kBack : 1][VEC];
  int pos = 0;
  float* ring = nullptr;
  if (CONV) {
    if (a.fresh) pdl_wait();
    pos = a.pos[t];
    ring = a.ring + (size_t)a.state_rows[a.slots[t]] * a.taps * a.width;
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
#pragma unroll
      for (int j = 0; j < kBack; ++j) {
#pragma unroll
        for (int v = 0; v < VEC; ++v) back[i][j][v] = 0.0f;
        if (on[i] && j + 1 < a.taps && j + 1 <= pos) load(ring + (size_t)((pos - j - 1) % a.taps) * a.width + col[i], back[i][j]);
      }
    if (!a.fresh) pdl_wait();
  } else {
    pdl_wait();
  }
  pdl_trigger();
  if (t == 0 && a.counts != nullptr)
    for (int i = threadIdx.x; i < a.experts; i += blockDim.x) a.counts[i] = 0;
  // columns that are off read column 0 and count as zero: no branch stands between the loads
  auto off = [&](int i, float (&v)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = on[i] ? v[e] : 0.0f;
  };
  float x[KEEP][VEC];
  float* xr = a.x + (size_t)row * a.width;
  if (!a.fresh) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) load(xr + col[i], x[i]);
  } else {
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
#pragma unroll
      for (int v = 0; v < VEC; ++v) x[i][v] = 0.0f;
  }
  if (a.y != nullptr || a.top > 0) {
    float u[KEEP][VEC], w[kEarly ? KEEP : 1][VEC], ss = 0.0f;
    if (a.y != nullptr) {
      const float* yr = a.y + (size_t)t * a.ldy;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) load(yr + col[i], u[i]);
      if (a.y_bias != nullptr) {
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
          float b[VEC];
          load(a.y_bias + col[i], b);
#pragma unroll
          for (int v = 0; v < VEC; ++v) u[i][v] += b[v];
        }
      }
      if (a.y_gate != nullptr) {
        const float g = sigmoid(a.y_gate[(size_t)t * a.ldg]);
#pragma unroll
        for (int i = 0; i < KEEP; ++i)
#pragma unroll
          for (int v = 0; v < VEC; ++v) u[i][v] *= g;
      }
    } else {
#pragma unroll
      for (int i = 0; i < KEEP; ++i)
#pragma unroll
        for (int v = 0; v < VEC; ++v) u[i][v] = 0.0f;
    }
    auto add_expert = [&](int k, auto load_row) {
      const size_t er = (size_t)a.at[t * a.top + k] * a.lde;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        float b[VEC];
        load_row(er + col[i], b);
#pragma unroll
        for (int v = 0; v < VEC; ++v) u[i][v] += b[v];
      }
    };
    if (a.e_f32) {
#pragma unroll(kEarly ? 2 : 1)
      for (int k = 0; k < a.top; ++k) add_expert(k, [&](size_t at, float (&b)[VEC]) { load(static_cast<const float*>(a.e) + at, b); });
    } else {
#pragma unroll(kEarly ? 4 : 1)
      for (int k = 0; k < a.top; ++k) add_expert(k, [&](size_t at, float (&b)[VEC]) { load16(static_cast<const bf16*>(a.e) + at, b); });
    }
    float f = a.mult;
    if (a.w != nullptr) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        if (kEarly) load(a.w + col[i], w[kEarly ? i : 0]);
        off(i, u[i]);
#pragma unroll
        for (int v = 0; v < VEC; ++v) ss += u[i][v] * u[i][v];
      }
      f *= inverse(ss, sums[0]);
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        if (!kEarly) load(a.w + col[i], w[0]);
#pragma unroll
        for (int v = 0; v < VEC; ++v) x[i][v] = fmaf(u[i][v] * f, w[kEarly ? i : 0][v], x[i][v]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < KEEP; ++i)
#pragma unroll
        for (int v = 0; v < VEC; ++v) x[i][v] = fmaf(u[i][v], f, x[i][v]);
    }
  }
  if (a.table != nullptr || a.step != nullptr) {
    const bf16* tr = a.table == nullptr ? nullptr : a.table + (size_t)a.tokens[t] * a.ld_table;
    if (tr != nullptr) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        float b[VEC];
        load16(tr + col[i], b);
#pragma unroll
        for (int v = 0; v < VEC; ++v) x[i][v] = fmaf(b[v], a.scale, x[i][v]);
      }
    }
    if (a.step != nullptr) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        float b[VEC];
        load(a.step + col[i], b);
#pragma unroll
        for (int v = 0; v < VEC; ++v) x[i][v] += b[v];
      }
    }
  }
  if (a.rows == nullptr) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (on[i]) store(xr + col[i], x[i]);
  }
  if (a.h == nullptr) return;
  if (a.next != nullptr) {
    float ss = 0.0f, w[kEarly ? KEEP : 1][VEC];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      if (kEarly) load(a.next + col[i], w[kEarly ? i : 0]);
      off(i, x[i]);
#pragma unroll
      for (int v = 0; v < VEC; ++v) ss += x[i][v] * x[i][v];
    }
    const float f = inverse(ss, sums[1]);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      if (!kEarly) load(a.next + col[i], w[0]);
#pragma unroll
      for (int v = 0; v < VEC; ++v) x[i][v] *= f * w[kEarly ? i : 0][v];
    }
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    if (!on[i]) continue;
    if (CONV) {
      float w[VEC], y[VEC];
      load(a.conv + col[i], w);
      store(ring + (size_t)(pos % a.taps) * a.width + col[i], x[i]);
#pragma unroll
      for (int v = 0; v < VEC; ++v) y[v] = x[i][v] * w[v];
#pragma unroll
      for (int j = 0; j < kBack; ++j) {
        if (j + 1 >= a.taps) break;
        load(a.conv + (size_t)(j + 1) * a.width + col[i], w);
#pragma unroll
        for (int v = 0; v < VEC; ++v) y[v] = fmaf(back[i][j][v], w[v], y[v]);
      }
      for (int j = kBack + 1; j < a.taps && j <= pos; ++j) {
        float b[VEC];
        load(ring + (size_t)((pos - j) % a.taps) * a.width + col[i], b);
        load(a.conv + (size_t)j * a.width + col[i], w);
#pragma unroll
        for (int v = 0; v < VEC; ++v) y[v] = fmaf(b[v], w[v], y[v]);
      }
#pragma unroll
      for (int v = 0; v < VEC; ++v) x[i][v] += y[v];
    } else if (a.n32 != nullptr) {
      store(a.n32 + (size_t)t * a.ldn + col[i], x[i]);
      continue;
    }
    if (a.h_f32) {
      store(static_cast<float*>(a.h) + (size_t)t * a.ldh + col[i], x[i]);
    } else {
      bf16* dst = static_cast<bf16*>(a.h) + (size_t)t * a.ldh + col[i];
      if constexpr (VEC == 4) store_act4(dst, make_float4(x[i][0], x[i][1], x[i][2], x[i][3]));
      else store_act(dst, x[i][0]);
    }
  }
}

// ---- convolution --------------------------------------------------------------------------------------------------------------
struct Conv {
  const float* in;          // [T][ld], channels at col
  const float* w;           // [taps][channels], tap j: the input j tokens back
  const float* bias;        // [channels] or null
  float* ring;              // [row][taps][channels]
  const int* pos;
  const int* slots;
  const int* state_rows;
  void* out;                // [T][ldo]
  int ld, col, channels, taps, ldo, out_f32;
  int add, silu;            // the input itself is added; silu
};

// grid (channels, single rows and then tiles); tiles[i] = {portion, first token of the tile}, entries[e] = {first row, tokens, slot,
// first position}.  KT: taps, 0 = any number.
template <int VEC, int KT>
__global__ void __launch_bounds__(128) conv_kernel(Conv a, int singles, const int4* entries, const int2* tiles) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  pdl_wait();
  pdl_trigger();
  if (c >= a.channels) return;
  const int taps = KT > 0 ? KT : a.taps;
  int first, q0 = 0, n = 1, total = 1, slot, pos0;
  if ((int)blockIdx.y < singles) {
    first = blockIdx.y;
    slot = a.slots[first];
    pos0 = a.pos[first];
  } else {
    const int2 tl = tiles[blockIdx.y - singles];
    const int4 en = entries[tl.x];
    first = en.x; total = en.y; slot = en.z; pos0 = en.w;
    q0 = tl.y;
    n = min(kConvRows, total - q0);
  }
  float* ring = a.ring + (size_t)a.state_rows[slot] * taps * a.channels + c;
  const float* in = a.in + (size_t)first * a.ld + a.col + c;
  auto load = [&](const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
      v[0] = *p;
    }
  };
  auto input = [&](int i, float (&v)[VEC]) {         // of the portion's token i, which may lie before the portion
    if (i >= 0) load(in + (size_t)i * a.ld, v);
    else if (pos0 + i >= 0) load(ring + (size_t)((pos0 + i) % taps) * a.channels, v);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = 0.0f;
    }
  };
  auto finish = [&](int i, const float (&x)[VEC], float (&y)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (a.add) y[e] += x[e];
      if (a.silu) y[e] = a.out_f32 ? silu_as<true>(y[e]) : silu_as<false>(y[e]);
    }
    const size_t at = (size_t)(first + q0 + i) * a.ldo + c;
    if constexpr (VEC == 4) {
      const float4 q = make_float4(y[0], y[1], y[2], y[3]);
      if (a.out_f32) store_act4(static_cast<float*>(a.out) + at, q);
      else store_act4(static_cast<bf16*>(a.out) + at, q);
    } else if (a.out_f32) {
      store_act(static_cast<float*>(a.out) + at, y[0]);
    } else {
      store_act(static_cast<bf16*>(a.out) + at, y[0]);
    }
  };
  float bias[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) bias[e] = 0.0f;
  if (a.bias != nullptr) load(a.bias + c, bias);
  if constexpr (KT > 0) {
    float w[KT][VEC], back[KT][VEC];                  // back[j]: the input j tokens back
#pragma unroll
    for (int j = 0; j < KT; ++j) load(a.w + (size_t)j * a.channels + c, w[j]);
#pragma unroll
    for (int j = 1; j < KT; ++j) input(q0 - j, back[j]);
    for (int i0 = 0; i0 < n; i0 += 8) {
      float x[8][VEC];
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i0 + i < n) load(in + (size_t)(q0 + i0 + i) * a.ld, x[i]);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (i0 + i >= n) break;
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          y[e] = fmaf(x[i][e], w[0][e], bias[e]);
#pragma unroll
          for (int j = 1; j < KT; ++j) y[e] = fmaf(back[j][e], w[j][e], y[e]);
        }
#pragma unroll
        for (int j = KT - 1; j > 1; --j)
#pragma unroll
          for (int e = 0; e < VEC; ++e) back[j][e] = back[j - 1][e];
        if (KT > 1) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) back[KT > 1 ? 1 : 0][e] = x[i][e];
        }
        finish(i0 + i, x[i], y);
      }
    }
  } else {
    for (int i = 0; i < n; ++i) {
      float x[VEC], y[VEC];
      load(in + (size_t)(q0 + i) * a.ld, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = bias[e];
      for (int j = 0; j < taps; ++j) {
        float b[VEC], w[VEC];
        input(q0 + i - j, b);
        load(a.w + (size_t)j * a.channels + c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(b[e], w[e], y[e]);
      }
      finish(i, x, y);
    }
  }
  if (q0 == 0) {                                     // this thread alone has read these channels of the ring
    for (int i = max(0, total - taps); i < total; ++i) {
      float v[VEC];
      load(in + (size_t)i * a.ld, v);
      float* dst = ring + (size_t)((pos0 + i) % taps) * a.channels;
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
      else *dst = v[0];
    }
  }
}

template <typename... P>
static bool aligned16(const P*... p) { return ((reinterpret_cast<uintptr_t>(p) | ...) & 15) == 0; }

}  // namespace lay
}  // namespace bonsai

extern "C" {

int bonsai_lay_conv_rows() { return bonsai::lay::kConvRows; }
int bonsai_lay_conv_taps() { return bonsai::lay::kMaxTaps; }

// ptrs = {x, y, y_bias, y_gate, w, table, tokens, step, next, n32, h, conv, ring, pos, slots, state_rows}, ints = {ldy, ldg, width, groups,
// ld_table, ldn, ldh, h_f32, taps, fresh}, floats = {eps, mult, scale} (null: left out; see RowStep).  T rows; e, lde, e_f32, at, top, counts,
// experts: expert rows (top 0: none); rows: only the norm of the rows of a list; conv_here: the convolution is done here (single
// tokens in every row), otherwise n goes to n32.
int bonsai_lay_row_step(const void* const* ptrs, const int* ints, const float* floats, int T, const void* e, int lde, int e_f32, const int* at, int top,
                        int* counts, int experts, const int* rows, int conv_here, cudaStream_t stream) {
  using namespace bonsai::lay;
  RowStep a;
  a.x = (float*)ptrs[0]; a.y = (const float*)ptrs[1]; a.y_bias = (const float*)ptrs[2]; a.y_gate = (const float*)ptrs[3]; a.w = (const float*)ptrs[4];
  a.table = (const bf16*)ptrs[5]; a.tokens = (const int*)ptrs[6]; a.step = (const float*)ptrs[7]; a.next = (const float*)ptrs[8];
  a.n32 = (float*)ptrs[9]; a.h = const_cast<void*>(ptrs[10]); a.conv = (const float*)ptrs[11]; a.ring = (float*)ptrs[12]; a.pos = (const int*)ptrs[13];
  a.slots = (const int*)ptrs[14]; a.state_rows = (const int*)ptrs[15];
  a.ldy = ints[0]; a.ldg = ints[1]; a.width = ints[2]; a.groups = ints[3]; a.ld_table = ints[4]; a.ldn = ints[5]; a.ldh = ints[6]; a.h_f32 = ints[7];
  a.taps = ints[8]; a.fresh = ints[9];
  a.eps = floats[0]; a.mult = floats[1]; a.scale = floats[2];
  a.e = e; a.lde = lde; a.e_f32 = e_f32; a.at = at; a.top = top; a.counts = counts; a.experts = experts; a.rows = rows;
  const bool conv = a.conv != nullptr && conv_here;
  a.inline_conv = conv;
  if (a.conv == nullptr || conv) a.n32 = nullptr;
  if (T < 1 || a.x == nullptr || a.width < 1 || a.groups < 1 || a.width % a.groups != 0 || top < 0 || (top > 0 && (e == nullptr || at == nullptr || lde < a.width)) ||
      (a.y != nullptr && a.ldy < a.width) || (a.table != nullptr && (a.tokens == nullptr || a.ld_table < a.width)) || (a.h != nullptr && a.ldh < a.width) ||
      (a.conv != nullptr && (a.taps < 1 || a.taps > kMaxTaps || a.h == nullptr || (conv ? a.ring == nullptr : a.n32 == nullptr || a.ldn < a.width))) ||
      (rows != nullptr && (a.y != nullptr || top > 0 || a.table != nullptr || a.step != nullptr || a.conv != nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  const int gw = a.width / a.groups;
  const bool vec = gw % 4 == 0 && a.ldy % 4 == 0 && a.ld_table % 4 == 0 && a.ldn % 4 == 0 && a.ldh % 4 == 0 && (top == 0 || lde % 4 == 0) &&
                   aligned16(a.x, a.y, a.y_bias, a.w, (const char*)a.table, a.step, a.next, a.n32, (const char*)a.h, a.conv, a.ring, (const char*)e);
  // threads per group: the fewest with which the chunks of a group fit, at most 512 (1024 with many chunks) in all
  auto shift = [&](int per) {
    int s = 0;
    while ((per << s) < gw) ++s;
    return s;
  };
  auto fits = [&](int per, int most) { return ((long long)a.groups << shift(per)) <= most; };
#define BONSAI_STEP(VEC, KEEP)                                                                                                     \
  {                                                                                                                                \
    const int s = shift((VEC) * (KEEP)), th = ((a.groups << s) + 31) / 32 * 32;                                                    \
    return conv ? launch(row_step_kernel<VEC, KEEP, true>, dim3(T), th, 0, stream, 1, 0, a, s)                                      \
                : launch(row_step_kernel<VEC, KEEP, false>, dim3(T), th, 0, stream, 1, 0, a, s);                                    \
  }
  if (vec && fits(4, 128)) BONSAI_STEP(4, 1)
  if (vec && fits(8, 512)) BONSAI_STEP(4, 2)
  if (vec && fits(16, 1024)) BONSAI_STEP(4, 4)
  if (fits(4, 512)) BONSAI_STEP(1, 4)
  if (fits(16, 1024)) BONSAI_STEP(1, 16)
#undef BONSAI_STEP
  return BONSAI_CUDA_BAD_ARG;
}

// ptrs = {in, w, bias, ring, pos, slots, state_rows, out}, ints = {ld, col, channels, taps, ldo, out_f32, add, silu}: the rows 0 .. singles - 1 are
// single tokens, then tiles of bonsai_lay_conv_rows() tokens.
int bonsai_lay_conv(const void* const* ptrs, const int* ints, const float*, int singles, const int* entries, const int* tiles, int ntiles, cudaStream_t stream) {
  using namespace bonsai::lay;
  Conv a;
  a.in = (const float*)ptrs[0]; a.w = (const float*)ptrs[1]; a.bias = (const float*)ptrs[2]; a.ring = (float*)ptrs[3]; a.pos = (const int*)ptrs[4];
  a.slots = (const int*)ptrs[5]; a.state_rows = (const int*)ptrs[6]; a.out = const_cast<void*>(ptrs[7]);
  a.ld = ints[0]; a.col = ints[1]; a.channels = ints[2]; a.taps = ints[3]; a.ldo = ints[4]; a.out_f32 = ints[5]; a.add = ints[6]; a.silu = ints[7];
  if (singles < 0 || ntiles < 0 || singles + ntiles < 1 || singles + ntiles > 65535 || a.taps < 1 || a.taps > kMaxTaps || a.channels < 1 ||
      a.ld < a.col + a.channels || a.ldo < a.channels || (ntiles > 0 && (entries == nullptr || tiles == nullptr)))
    return BONSAI_CUDA_BAD_ARG;
  const bool vec = a.channels % 4 == 0 && a.ld % 4 == 0 && a.col % 4 == 0 && a.ldo % 4 == 0 && aligned16(a.in, a.w, a.bias, a.ring, (const char*)a.out);
#define BONSAI_CONV(VEC, KT)                                                                                                       \
  launch(conv_kernel<VEC, KT>, dim3((a.channels + 128 * VEC - 1) / (128 * VEC), singles + ntiles), 128, 0, stream, 1, 0, a, singles, \
         (const int4*)entries, (const int2*)tiles)
  if (!vec) return BONSAI_CONV(1, 0);
  switch (a.taps) {
    case 2: return BONSAI_CONV(4, 2);
    case 3: return BONSAI_CONV(4, 3);
    case 4: return BONSAI_CONV(4, 4);
    default: return BONSAI_CONV(4, 0);
  }
#undef BONSAI_CONV
}

}  // extern "C"
