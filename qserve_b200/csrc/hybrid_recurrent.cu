// qserve_b200 -- recurrent layers of the hybrid decoders that read short causal convolutions.
//
//   state space (Mamba-2):  S <- a S + dt B x^T,  y = S^T C + D x    per head a [N, Dv] fp32 state; x, B, C pass a convolution and silu, a and dt are
//                           one number per (token, head); y * silu(z) is brought to unit RMS in equal parts.  The scan itself is a mode of the
//                           linear-scan kernel (hybrid_linear.cu); its first and last step are here.
//   gated linear unit (RG-LRU):  S <- a S + sqrt(1 - a^2) i u        per channel one fp32 number; u is the convolved branch, a and i come from
//                           block-diagonal projections of u (a batched product between the two kernels here); the output is S * gelu_tanh(y).
//                           Runs of at least a tile of tokens are scanned tile by tile: every tile's own (product of a, end state from
//                           zero) first, then the tiles' start states, then the tiles again from there.
//
// Batch tables: see hybrid.cu.  Convolution states (fp32): [slots][taps - 1][channels], oldest input first.
#include <cuda_bf16.h>
#include <math.h>

#include <algorithm>

#include "../../include/qserve_b200.h"
#include "common.cuh"
#include "hybrid_common.cuh"
#include "launch.h"

namespace qs {
namespace {

using namespace hyb;

constexpr int kMaxTaps = 17;

// The convolution's inputs of one token, channels c .. c + V - 1: `back` tokens before row t.  Inputs ahead of the portion come from the
// convolution state, inputs ahead of the sequence are zero; `in_bias` (may be null) belongs to the inputs.
template <typename ST, int V>
__device__ __forceinline__ void conv_input(float (&x)[V], const ST* __restrict__ in, long long stride, const float* __restrict__ in_bias,
                                           const float* st, int t, int local, int pos, int back, int taps, int C, int c) {
#pragma unroll
  for (int v = 0; v < V; ++v) x[v] = 0.f;
  if (pos - back < 0) return;
  if (local - back >= 0) {
    const ST* p = in + (size_t)(t - back) * stride + c;
    if constexpr (V == 4) {
      const float4 q = ld4(p);
      x[0] = q.x; x[1] = q.y; x[2] = q.z; x[3] = q.w;
    } else {
      x[0] = ldf(p);
    }
    if (in_bias != nullptr) {
#pragma unroll
      for (int v = 0; v < V; ++v) x[v] += in_bias[c + v];
    }
  } else {
    const float* p = st + (size_t)(taps - 1 + local - back) * C + c;
#pragma unroll
    for (int v = 0; v < V; ++v) x[v] = p[v];
  }
}

// Convolution of row t at channels c .. c + V - 1 (bias included).  In a step of single tokens the thread is the only reader of its channels'
// state and shifts the token's input in (`shift`); other steps do that in conv_state_kernel afterwards.
template <typename ST, int V>
__device__ __forceinline__ void conv_row(float (&y)[V], const ST* __restrict__ in, long long stride, const float* __restrict__ in_bias, float* st,
                                         const float* __restrict__ w, const float* __restrict__ b, int t, int local, int pos, int taps, int C, int c,
                                         bool shift) {
#pragma unroll
  for (int v = 0; v < V; ++v) y[v] = b != nullptr ? b[c + v] : 0.f;
  for (int j = 0; j < taps; ++j) {
    float x[V];
    conv_input<ST, V>(x, in, stride, in_bias, st, t, local, pos, taps - 1 - j, taps, C, c);
#pragma unroll
    for (int v = 0; v < V; ++v) y[v] += w[(size_t)(c + v) * taps + j] * x[v];
    if (shift && j > 0) {  // input j is slot j - 1 of the next token's state; slot j is read before slot j is written
#pragma unroll
      for (int v = 0; v < V; ++v) st[(size_t)(j - 1) * C + c + v] = x[v];
    }
  }
}

// The same for a walk over neighbouring rows, `TAPS` known: the channels' weights and the window of inputs stay in registers.
template <typename ST, int V, int TAPS>
struct ConvWalk {
  float w[V][TAPS], b[V], xb[V], x[TAPS][V];
  int entry = -1;

  __device__ __forceinline__ ConvWalk(const float* __restrict__ cw, const float* __restrict__ cb, const float* __restrict__ in_bias, int c) {
#pragma unroll
    for (int v = 0; v < V; ++v) {
      b[v] = cb != nullptr ? cb[c + v] : 0.f;
      xb[v] = in_bias != nullptr ? in_bias[c + v] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[v][j] = cw[(size_t)(c + v) * TAPS + j];
    }
  }
  __device__ __forceinline__ void row(float (&y)[V], const ST* __restrict__ in, long long stride, const float* __restrict__ in_bias, float* st, int t, int e,
                                      int local, int pos, int C, int c, bool shift) {
    if (e != entry) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) conv_input<ST, V>(x[j], in, stride, in_bias, st, t, local, pos, TAPS - 1 - j, TAPS, C, c);
      entry = e;
    } else {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) x[j][v] = x[j + 1][v];
    }
    const ST* p = in + (size_t)t * stride + c;
    if constexpr (V == 4) {
      const float4 q = ld4(p);
      x[TAPS - 1][0] = q.x; x[TAPS - 1][1] = q.y; x[TAPS - 1][2] = q.z; x[TAPS - 1][3] = q.w;
    } else {
      x[TAPS - 1][0] = ldf(p);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) {
      x[TAPS - 1][v] += xb[v];
      y[v] = b[v];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) y[v] += w[v][j] * x[j][v];
    }
    if (shift) {
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) st[(size_t)(j - 1) * C + c + v] = x[j][v];
    }
  }
};
// any number of taps
template <typename ST, int V>
struct ConvWalk<ST, V, 0> {
  const float *cw, *cb;
  int taps;
  __device__ __forceinline__ ConvWalk(const float* w, const float* b, int n) : cw(w), cb(b), taps(n) {}
  __device__ __forceinline__ void row(float (&y)[V], const ST* __restrict__ in, long long stride, const float* __restrict__ in_bias, float* st, int t, int,
                                      int local, int pos, int C, int c, bool shift) {
    conv_row<ST, V>(y, in, stride, in_bias, st, cw, cb, t, local, pos, taps, C, c, shift);
  }
};
template <typename ST, int V, int TAPS>
__device__ __forceinline__ ConvWalk<ST, V, TAPS> conv_walk(const float* w, const float* b, const float* in_bias, int taps, int c) {
  if constexpr (TAPS == 0) return ConvWalk<ST, V, 0>(w, b, taps);
  else return ConvWalk<ST, V, TAPS>(w, b, in_bias, c);
}

// silu as the storage type needs it: the special-function unit's exponential and division for bfloat16 results, the exact ones for fp32
template <typename ST> __device__ __forceinline__ float silu_as(float z) { return sizeof(ST) == 2 ? z * fast_sigmoid(z) : silu_f(z); }

// the sequence's convolution state after a portion: its last taps - 1 inputs (older ones shift out)
template <typename ST>
__global__ void conv_state_kernel(float* __restrict__ conv_state, const ST* __restrict__ in, long long stride, const float* __restrict__ in_bias,
                                  const int* __restrict__ entry_start, const int* __restrict__ entry_len, const int* __restrict__ entry_slot,
                                  const int* __restrict__ entry_pos0, int C, int taps) {
  const int e = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int n = entry_len[e], s0 = entry_start[e], keep = taps - 1;
  float* st = conv_state + (size_t)entry_slot[e] * keep * C + c;
  const bool fresh = entry_pos0[e] == 0;
  const float bias = in_bias != nullptr ? in_bias[c] : 0.f;
  for (int i = 0; i < keep; ++i) {  // slot i takes an input that lies further on in the old state: no slot is read after it was written
    const int src = n - keep + i;   // index in the portion, negative: older than the portion
    float v;
    if (src >= 0) v = ldf(in + (size_t)(s0 + src) * stride + c) + bias;
    else v = fresh ? 0.f : st[(size_t)(keep + src) * C];
    st[(size_t)i * C] = v;
  }
}

// ---------------------------------------------------------------------------------------------------------------------------------
// state space, step 1.  projection row: [inner z | inner x | G*N B | G*N C | H dt], inner = H * Dv
//   prepared row (ssd_row_floats): [inner x | G*N B | G*N C | H dt | H a]:  x, B, C convolved and through silu, dt <- softplus(dt + dt_bias),
//   a = exp(-exp(A_log) dt)
// grid (runs of `run` tokens, blocks of 128 V channels)
// ---------------------------------------------------------------------------------------------------------------------------------
template <typename ST, int V, int TAPS>
__global__ void __launch_bounds__(128) ssd_prepare_kernel(float* __restrict__ prep, const ST* __restrict__ proj, long long stride,
                                                          const float* __restrict__ conv_w, const float* __restrict__ conv_b, float* conv_state,
                                                          const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                          const int* __restrict__ tok_entry, const int* __restrict__ tok_pos,
                                                          const int* __restrict__ entry_start, const int* __restrict__ entry_slot, int T, int H, int G,
                                                          int N, int Dv, int taps, int run, int shift) {
  const int inner = H * Dv, C = inner + 2 * G * N, P = ssd_row_floats(H, G, N, Dv);
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  const int t0 = blockIdx.x * run, t1 = min(T, t0 + run);
  auto walk = conv_walk<ST, V, TAPS>(conv_w, conv_b, nullptr, taps, min(c, C - V));
  for (int t = t0; t < t1; ++t) {
    const int e = tok_entry[t];
    float* o = prep + (size_t)t * P;
    if (c < C) {
      float y[V];
      walk.row(y, proj + inner, stride, nullptr, conv_state + (size_t)entry_slot[e] * (taps - 1) * C, t, e, t - entry_start[e], tok_pos[t], C, c, shift != 0);
#pragma unroll
      for (int v = 0; v < V; ++v) y[v] = silu_as<ST>(y[v]);
      if constexpr (V == 4) st4(o + c, make_float4(y[0], y[1], y[2], y[3]));
      else o[c] = y[0];
    }
    if (blockIdx.y == 0)
      for (int h = threadIdx.x; h < H; h += 128) {
        const float z = ldf(proj + (size_t)t * stride + inner + C + h) + dt_bias[h];
        const float dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
        o[C + h] = dt;
        o[C + H + h] = expf(-expf(a_log[h]) * dt);
      }
  }
}

// state space, step 3: y <- y * silu(z), unit RMS in equal parts of the row, times norm_w and a constant.  One block per (token, part); the part
// waits in shared memory between its two passes.
template <typename ST>
__global__ void __launch_bounds__(256) ssd_out_kernel(ST* __restrict__ out, long long out_stride, const float* __restrict__ y, const ST* __restrict__ z,
                                                      long long z_stride, const float* __restrict__ norm_w, float out_scale, float eps, int inner,
                                                      int part, int vec) {
  extern __shared__ __align__(16) float ys[];  // [part]
  __shared__ float red[33];
  const int t = blockIdx.x, c0 = blockIdx.y * part;
  const float* yr = y + (size_t)t * inner + c0;
  const ST* zr = z + (size_t)t * z_stride + c0;
  ST* o = out + (size_t)t * out_stride + c0;
  float ss = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < part; i += blockDim.x * 4) {
      float4 a = ld4(yr + i);
      const float4 g = ld4(zr + i);
      a.x *= silu_as<ST>(g.x); a.y *= silu_as<ST>(g.y); a.z *= silu_as<ST>(g.z); a.w *= silu_as<ST>(g.w);
      ss += (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w);
      st4(ys + i, a);
    }
  } else {
    for (int i = threadIdx.x; i < part; i += blockDim.x) {
      const float a = yr[i] * silu_as<ST>(ldf(zr + i));
      ss += a * a;
      ys[i] = a;
    }
  }
  const float r = out_scale / sqrtf(block_sum(ss, red) / (float)part + eps);
  if (vec) {  // every thread reads back what it wrote itself
    for (int i = threadIdx.x * 4; i < part; i += blockDim.x * 4) {
      const float4 a = ld4(ys + i), w = ld4(norm_w + c0 + i);
      st4(o + i, make_float4(a.x * r * w.x, a.y * r * w.y, a.z * r * w.z, a.w * r * w.w));
    }
  } else {
    for (int i = threadIdx.x; i < part; i += blockDim.x) stf(o + i, ys[i] * r * norm_w[c0 + i]);
  }
}

// ---------------------------------------------------------------------------------------------------------------------------------
// gated linear unit.  projection row: [W y | W x] (biases not yet added)
// step 1: u = convolution of x + x_bias, in the storage type [T][W]
// ---------------------------------------------------------------------------------------------------------------------------------
template <typename ST, int V, int TAPS>
__global__ void __launch_bounds__(128) lru_conv_kernel(ST* __restrict__ u, const ST* __restrict__ proj, long long stride, const float* __restrict__ x_bias,
                                                       const float* __restrict__ conv_w, const float* __restrict__ conv_b, float* conv_state,
                                                       const int* __restrict__ tok_entry, const int* __restrict__ tok_pos,
                                                       const int* __restrict__ entry_start, const int* __restrict__ entry_slot, int T, int W, int taps,
                                                       int run, int shift) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  if (c >= W) return;
  const int t0 = blockIdx.x * run, t1 = min(T, t0 + run);
  auto walk = conv_walk<ST, V, TAPS>(conv_w, conv_b, x_bias, taps, c);
  for (int t = t0; t < t1; ++t) {
    const int e = tok_entry[t];
    float y[V];
    walk.row(y, proj + W, stride, x_bias, conv_state + (size_t)entry_slot[e] * (taps - 1) * W, t, e, t - entry_start[e], tok_pos[t], W, c, shift != 0);
    if constexpr (V == 4) st4(u + (size_t)t * W + c, make_float4(y[0], y[1], y[2], y[3]));
    else stf(u + (size_t)t * W + c, y[0]);
  }
}

// step 2 (between the kernels): gate logits z fp32 [blocks][T][2 W / blocks]: a block's r logits, then its i logits.
// step 3: the recurrence.  One token of one channel: r = sigmoid(z_r + r_bias), i = sigmoid(z_i + i_bias), log a = rate * r (rate < 0 per
// channel), S <- a S + sqrt(1 - a^2) i u with 1 - a^2 = -expm1(2 log a).
// A thread owns V neighbouring channels of one block (V = 2: the channels of a block are even in number and aligned).
template <int V>
struct LruChannels {
  const float* zr;    // r logits of row 0; rows are zs floats apart
  size_t zs, zi;      // zi: distance of the i logits
  float rb[V], ib[V], rate[V];

  __device__ __forceinline__ LruChannels(const float* z, const float* r_bias, const float* i_bias, const float* rates, int T, int W, int blocks, int c) {
    const int wb = W / blocks, b = c / wb, j = c - b * wb;
    zr = z + (size_t)b * T * 2 * wb + j;
    zs = 2 * (size_t)wb;
    zi = wb;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      rb[v] = r_bias[c + v];
      ib[v] = i_bias[c + v];
      rate[v] = rates[c + v];
    }
  }
};
template <int V> __device__ __forceinline__ void load_row(float (&x)[V], const float* p) {
  if constexpr (V == 2) {
    const float2 q = *reinterpret_cast<const float2*>(p);
    x[0] = q.x; x[1] = q.y;
  } else {
    x[0] = *p;
  }
}
template <int V> __device__ __forceinline__ void load_row(float (&x)[V], const __nv_bfloat16* p) {
  if constexpr (V == 2) {
    const uint32_t q = *reinterpret_cast<const uint32_t*>(p);
    x[0] = __uint_as_float(q << 16); x[1] = __uint_as_float(q & 0xffff0000u);
  } else {
    x[0] = ldf(p);
  }
}
template <int V> __device__ __forceinline__ void store_row(float* p, const float (&x)[V]) {
#pragma unroll
  for (int v = 0; v < V; ++v) p[v] = x[v];
}
template <int V> __device__ __forceinline__ void store_row(__nv_bfloat16* p, const float (&x)[V]) {
  if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16(x[0], x[1]);
  else stf(p, x[0]);
}

// FAST (bfloat16 storage): fp32 throughout, with the special-function unit's exponentials, divisions and square root (relative error about 2^-21) and
// 1 - a^2 = -expm1(x), x = 2 log a, from the exponential series where a^2 is close to 1
template <bool FAST>
__device__ __forceinline__ void lru_gates(float& a, float& b, float zr, float zi, float u, float rate) {
  if (FAST) {
    const float la = rate * fast_sigmoid(zr), x = 2.f * la;
    a = fast_exp2(la * 1.4426950408889634f);
    const float series = -x * (1.f + x * (1.f / 2.f) * (1.f + x * (1.f / 3.f) * (1.f + x * (1.f / 4.f) * (1.f + x * (1.f / 5.f) * (1.f + x * (1.f / 6.f))))));
    const float m = x > -0.25f ? series : 1.f - a * a;
    float root;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(m));
    b = root * fast_sigmoid(zi) * u;
    return;
  }
  const float la = rate * sigmoid_f(zr);
  a = expf(la);
  b = sqrtf(-expm1f(2.f * la)) * sigmoid_f(zi) * u;
}

constexpr int kLruBatch = 4;  // tokens whose inputs are on their way at once

// what a tile of rows does to a state: S <- A S + B.  sums [n_tiles][2][W]
template <typename ST, int V>
__global__ void __launch_bounds__(128) lru_tile_sums_kernel(float* __restrict__ sums, const ST* __restrict__ u, const float* __restrict__ z,
                                                            const float* __restrict__ r_bias, const float* __restrict__ i_bias,
                                                            const float* __restrict__ rate, const int* __restrict__ tile_entry,
                                                            const int* __restrict__ tile_row0, const int* __restrict__ entry_start,
                                                            const int* __restrict__ entry_len, int T, int W, int blocks, int tile_rows) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V, tile = blockIdx.x;
  if (c >= W) return;
  const int e = tile_entry[tile], r0 = tile_row0[tile], n = min(tile_rows, entry_len[e] - r0), s0 = entry_start[e] + r0;
  const LruChannels<V> k(z, r_bias, i_bias, rate, T, W, blocks, c);
  float A[V], S[V];
#pragma unroll
  for (int v = 0; v < V; ++v) { A[v] = 1.f; S[v] = 0.f; }
  for (int j = 0; j < n; j += kLruBatch) {
    float zr[kLruBatch][V], zi[kLruBatch][V], uu[kLruBatch][V];
#pragma unroll
    for (int q = 0; q < kLruBatch; ++q) {
      const size_t t = s0 + min(j + q, n - 1);
      load_row<V>(zr[q], k.zr + t * k.zs);
      load_row<V>(zi[q], k.zr + t * k.zs + k.zi);
      load_row<V>(uu[q], u + t * W + c);
    }
#pragma unroll
    for (int q = 0; q < kLruBatch; ++q) {
      if (j + q >= n) break;
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float a, b;
        lru_gates<sizeof(ST) == 2>(a, b, zr[q][v] + k.rb[v], zi[q][v] + k.ib[v], uu[q][v], k.rate[v]);
        A[v] *= a;
        S[v] = a * S[v] + b;
      }
    }
  }
  store_row<V>(sums + (size_t)tile * 2 * W + c, A);
  store_row<V>(sums + ((size_t)tile * 2 + 1) * W + c, S);
}

// start state of every tile, over the tile's A.  An entry's tiles are neighbours; the block of its first tile walks them, eight at a time.
__global__ void __launch_bounds__(128) lru_tile_starts_kernel(float* __restrict__ sums, const float* __restrict__ state, const int* __restrict__ tile_entry,
                                                              const int* __restrict__ tile_row0, const int* __restrict__ entry_len,
                                                              const int* __restrict__ entry_slot, const int* __restrict__ entry_pos0, int W, int tile_rows) {
  constexpr int U = 8;
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (tile_row0[blockIdx.x] != 0 || c >= W) return;
  const int e = tile_entry[blockIdx.x], n = (entry_len[e] + tile_rows - 1) / tile_rows;
  float S = entry_pos0[e] == 0 ? 0.f : state[(size_t)entry_slot[e] * W + c];
  float* p = sums + (size_t)blockIdx.x * 2 * W + c;
  for (int i = 0; i < n; i += U) {
    float A[U], B[U];
#pragma unroll
    for (int q = 0; q < U; ++q) {
      const size_t at = (size_t)min(i + q, n - 1) * 2 * W;
      A[q] = p[at];
      B[q] = p[at + W];
    }
#pragma unroll
    for (int q = 0; q < U; ++q) {
      if (i + q >= n) break;
      p[(size_t)(i + q) * 2 * W] = S;
      S = A[q] * S + B[q];
    }
  }
}

// The recurrence over a tile (tiles != 0: start state from sums) or over a whole entry of fewer than long_min tokens (tiles == 0: start state
// from the slot; longer entries are left to the tiles), read out through the gelu branch.  The slot takes the state after the entry's last row.
template <typename ST, int V>
__global__ void __launch_bounds__(128) lru_scan_kernel(ST* __restrict__ out, long long out_stride, float* state, const float* __restrict__ sums,
                                                       const ST* __restrict__ u, const float* __restrict__ z, const ST* __restrict__ y, long long y_stride,
                                                       const float* __restrict__ y_bias, const float* __restrict__ r_bias,
                                                       const float* __restrict__ i_bias, const float* __restrict__ rate,
                                                       const int* __restrict__ tile_entry, const int* __restrict__ tile_row0,
                                                       const int* __restrict__ entry_start, const int* __restrict__ entry_len,
                                                       const int* __restrict__ entry_slot, const int* __restrict__ entry_pos0, int tiles, int long_min, int T,
                                                       int W, int blocks, int tile_rows) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  const int e = tiles ? tile_entry[blockIdx.x] : blockIdx.x;
  const int len = entry_len[e], r0 = tiles ? tile_row0[blockIdx.x] : 0, n = tiles ? min(tile_rows, len - r0) : len;
  if (c >= W || (!tiles && len >= long_min)) return;
  const int s0 = entry_start[e] + r0;
  float* slot = state + (size_t)entry_slot[e] * W + c;
  const LruChannels<V> k(z, r_bias, i_bias, rate, T, W, blocks, c);
  float yb[V], S[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    yb[v] = y_bias[c + v];
    S[v] = tiles ? sums[(size_t)blockIdx.x * 2 * W + c + v] : (entry_pos0[e] == 0 ? 0.f : slot[v]);
  }
  for (int j = 0; j < n; j += kLruBatch) {
    float zr[kLruBatch][V], zi[kLruBatch][V], uu[kLruBatch][V], yy[kLruBatch][V];
#pragma unroll
    for (int q = 0; q < kLruBatch; ++q) {
      const size_t t = s0 + min(j + q, n - 1);
      load_row<V>(zr[q], k.zr + t * k.zs);
      load_row<V>(zi[q], k.zr + t * k.zs + k.zi);
      load_row<V>(uu[q], u + t * W + c);
      load_row<V>(yy[q], y + t * y_stride + c);
    }
#pragma unroll
    for (int q = 0; q < kLruBatch; ++q) {
      if (j + q >= n) break;
      float o[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float a, b;
        lru_gates<sizeof(ST) == 2>(a, b, zr[q][v] + k.rb[v], zi[q][v] + k.ib[v], uu[q][v], k.rate[v]);
        S[v] = a * S[v] + b;
        const float g = yy[q][v] + yb[v], w = 2.f * 0.7978845608028654f * (g + 0.044715f * g * g * g);
        o[v] = S[v] * g * (sizeof(ST) == 2 ? fast_sigmoid(w) : sigmoid_f(w));   // gelu_tanh(g) = g 0.5 (1 + tanh(w / 2)) = g sigmoid(w)
      }
      store_row<V>(out + (size_t)(s0 + j + q) * out_stride + c, o);
    }
  }
  if (r0 + n == len) store_row<V>(slot, S);
}

template <typename ST>
int launch_conv_state(float* conv_state, const ST* in, long long stride, const float* in_bias, const int* entry_start, const int* entry_len,
                      const int* entry_slot, const int* entry_pos0, int E, int C, int taps, cudaStream_t s) {
  if (taps > 1)
    conv_state_kernel<ST><<<dim3((C + 127) / 128, E), 128, 0, s>>>(conv_state, in, stride, in_bias, entry_start, entry_len, entry_slot, entry_pos0, C, taps);
  return check_cuda(cudaGetLastError(), "hyb convolution state");
}

bool aligned(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

// tokens a block of a convolution kernel walks: neighbours find each other's rows in the cache once there are blocks enough
int conv_run(int T) { return T >= 2048 ? 16 : T >= 512 ? 4 : 1; }

template <typename ST>
int launch_state_space(void* out, long long out_stride, float* prep, float* o_raw, const void* proj_, long long stride, const float* conv_w,
                       const float* conv_b, float* conv_state, float* state, const float* a_log, const float* dt_bias, const float* skip,
                       const float* norm_w, int norm_groups, float out_scale, const int* tok_entry, const int* tok_pos, const int* entry_start,
                       const int* entry_len, const int* entry_slot, const int* entry_pos0, int T, int E, int H, int G, int N, int Dv, int taps, float eps,
                       cudaStream_t s) {
  const ST* proj = static_cast<const ST*>(proj_);
  const int inner = H * Dv, C = inner + 2 * G * N, run = conv_run(T), shift = T == E && taps > 1;
  const bool v4 = C % 4 == 0 && inner % 4 == 0 && stride % 4 == 0 && aligned(proj, 4 * sizeof(ST)) && aligned(prep, 16);
  dim3 grid((T + run - 1) / run, (C + (v4 ? 512 : 128) - 1) / (v4 ? 512 : 128));
  auto prepare = !v4 ? ssd_prepare_kernel<ST, 1, 0> : taps == 4 ? ssd_prepare_kernel<ST, 4, 4> : taps == 3 ? ssd_prepare_kernel<ST, 4, 3>
                 : taps == 2 ? ssd_prepare_kernel<ST, 4, 2> : ssd_prepare_kernel<ST, 4, 0>;
  prepare<<<grid, 128, 0, s>>>(prep, proj, stride, conv_w, conv_b, conv_state, a_log, dt_bias, tok_entry, tok_pos, entry_start, entry_slot, T, H, G, N, Dv,
                               taps, run, shift);
  if (!shift)
    if (int rc = launch_conv_state<ST>(conv_state, proj + inner, stride, nullptr, entry_start, entry_len, entry_slot, entry_pos0, E, C, taps, s)) return rc;
  if (int rc = ssd_scan(o_raw, prep, state, skip, entry_start, entry_len, entry_slot, entry_pos0, T, E, H, G, N, Dv, s)) return rc;
  const int part = inner / norm_groups, threads = part >= 1024 ? 256 : 128;
  const size_t smb = (size_t)part * sizeof(float);
  const int vec = part % 4 == 0 && stride % 4 == 0 && out_stride % 4 == 0 && aligned(proj, 4 * sizeof(ST)) && aligned(out, 4 * sizeof(ST)) &&
                  aligned(o_raw, 16) && aligned(norm_w, 16);
  if (smb > 48 * 1024) cudaFuncSetAttribute(ssd_out_kernel<ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smb);
  ssd_out_kernel<ST><<<dim3(T, norm_groups), threads, smb, s>>>((ST*)out, out_stride, o_raw, proj, stride, norm_w, out_scale, eps, inner, part, vec);
  return check_cuda(cudaGetLastError(), "hyb_state_space");
}

template <typename ST>
int launch_lru_conv(void* u, const void* proj_, long long stride, const float* x_bias, const float* conv_w, const float* conv_b, float* conv_state,
                    const int* tok_entry, const int* tok_pos, const int* entry_start, const int* entry_len, const int* entry_slot, const int* entry_pos0,
                    int T, int E, int W, int taps, cudaStream_t s) {
  const ST* proj = static_cast<const ST*>(proj_);
  const int run = conv_run(T), shift = T == E && taps > 1;
  const bool v4 = W % 4 == 0 && stride % 4 == 0 && aligned(proj, 4 * sizeof(ST)) && aligned(u, 4 * sizeof(ST));
  dim3 grid((T + run - 1) / run, (W + (v4 ? 512 : 128) - 1) / (v4 ? 512 : 128));
  auto conv = !v4 ? lru_conv_kernel<ST, 1, 0> : taps == 4 ? lru_conv_kernel<ST, 4, 4> : taps == 3 ? lru_conv_kernel<ST, 4, 3>
              : taps == 2 ? lru_conv_kernel<ST, 4, 2> : lru_conv_kernel<ST, 4, 0>;
  conv<<<grid, 128, 0, s>>>((ST*)u, proj, stride, x_bias, conv_w, conv_b, conv_state, tok_entry, tok_pos, entry_start, entry_slot, T, W, taps, run, shift);
  if (!shift) return launch_conv_state<ST>(conv_state, proj + W, stride, x_bias, entry_start, entry_len, entry_slot, entry_pos0, E, W, taps, s);
  return check_cuda(cudaGetLastError(), "hyb_lru_conv");
}

template <typename ST, int V>
int launch_lru_scan_cols(void* out, long long out_stride, float* state, float* sums, const void* u, const float* z, const void* proj, long long stride,
                         const float* y_bias, const float* r_bias, const float* i_bias, const float* rate, const int* tile_entry, const int* tile_row0,
                         int n_tiles, int n_short, const int* entry_start, const int* entry_len, const int* entry_slot, const int* entry_pos0, int T, int E,
                         int W, int blocks, int tile_rows, int long_min, cudaStream_t s) {
  const int cols = (W + 128 * V - 1) / (128 * V);
  if (n_tiles > 0) {
    dim3 grid(n_tiles, cols);
    lru_tile_sums_kernel<ST, V><<<grid, 128, 0, s>>>(sums, (const ST*)u, z, r_bias, i_bias, rate, tile_entry, tile_row0, entry_start, entry_len, T, W, blocks,
                                                     tile_rows);
    lru_tile_starts_kernel<<<dim3(n_tiles, (W + 127) / 128), 128, 0, s>>>(sums, state, tile_entry, tile_row0, entry_len, entry_slot, entry_pos0, W, tile_rows);
    lru_scan_kernel<ST, V><<<grid, 128, 0, s>>>((ST*)out, out_stride, state, sums, (const ST*)u, z, (const ST*)proj, stride, y_bias, r_bias, i_bias, rate,
                                                tile_entry, tile_row0, entry_start, entry_len, entry_slot, entry_pos0, 1, long_min, T, W, blocks, tile_rows);
  }
  if (n_short > 0)
    lru_scan_kernel<ST, V><<<dim3(E, cols), 128, 0, s>>>((ST*)out, out_stride, state, nullptr, (const ST*)u, z, (const ST*)proj, stride, y_bias, r_bias, i_bias,
                                                         rate, nullptr, nullptr, entry_start, entry_len, entry_slot, entry_pos0, 0, long_min, T, W, blocks,
                                                         tile_rows);
  return check_cuda(cudaGetLastError(), "hyb_lru_scan");
}

template <typename ST>
int launch_lru_scan(void* out, long long out_stride, float* state, float* sums, const void* u, const float* z, const void* proj, long long stride,
                    const float* y_bias, const float* r_bias, const float* i_bias, const float* rate, const int* tile_entry, const int* tile_row0,
                    int n_tiles, int n_short, const int* entry_start, const int* entry_len, const int* entry_slot, const int* entry_pos0, int T, int E,
                    int W, int blocks, int tile_rows, int long_min, cudaStream_t s) {
  // two channels per thread for prompts; a step of few rows needs the threads
  const bool two = n_tiles > 0 && (W / blocks) % 2 == 0 && stride % 2 == 0 && out_stride % 2 == 0 && aligned(u, 8) && aligned(z, 8) && aligned(proj, 8) && aligned(out, 8);
  auto run = two ? launch_lru_scan_cols<ST, 2> : launch_lru_scan_cols<ST, 1>;
  return run(out, out_stride, state, sums, u, z, proj, stride, y_bias, r_bias, i_bias, rate, tile_entry, tile_row0, n_tiles, n_short, entry_start, entry_len,
             entry_slot, entry_pos0, T, E, W, blocks, tile_rows, long_min, s);
}

}  // namespace
}  // namespace qs

using namespace qs;

#define QS_DT(dtype, CALL_BF16, CALL_F32)                                               \
  do {                                                                                  \
    if ((dtype) == QS_DTYPE_BF16) { CALL_BF16; }                                        \
    else if ((dtype) == QS_DTYPE_F32) { CALL_F32; }                                     \
    else return set_error(qs::QS_ERR_INVALID, "dtype must be QS_DTYPE_BF16 or QS_DTYPE_F32"); \
  } while (0)

extern "C" {

int qs_hyb_state_space_prep_floats(int heads, int groups, int state_n, int vdim) { return hyb::ssd_row_floats(heads, groups, state_n, vdim); }

int qs_hyb_state_space(void* out, int64_t out_stride, float* prep, float* o_raw, const void* proj, int64_t stride, const float* conv_w,
                       const float* conv_b, float* conv_state, float* state, const float* a_log, const float* dt_bias, const float* skip,
                       const float* norm_w, int norm_groups, float out_scale, const int32_t* tok_entry, const int32_t* tok_pos,
                       const int32_t* entry_start, const int32_t* entry_len, const int32_t* entry_slot, const int32_t* entry_pos0, int tokens_n,
                       int entries, int heads, int groups, int state_n, int vdim, int taps, float eps, int dtype, void* stream) {
  QS_REQUIRE(out && prep && o_raw && proj && conv_w && state && a_log && dt_bias && skip && norm_w, "hyb_state_space: null tensor");
  QS_REQUIRE(tok_entry && tok_pos && entry_start && entry_len && entry_slot && entry_pos0, "hyb_state_space: null batch table");
  QS_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && vdim > 0 && state_n > 0 && state_n <= 512, "hyb_state_space: groups divide heads, 0 < state <= 512");
  QS_REQUIRE(taps >= 1 && taps <= kMaxTaps && (taps == 1 || conv_state != nullptr), "hyb_state_space: 1..17 convolution taps");
  QS_REQUIRE(norm_groups > 0 && (heads * vdim) % norm_groups == 0 && (heads * vdim) / norm_groups <= 51200, "hyb_state_space: norm groups divide the row");
  if (tokens_n == 0) return qs::QS_OK;
  cudaStream_t s = (cudaStream_t)stream;
  QS_DT(dtype,
        return launch_state_space<__nv_bfloat16>(out, out_stride, prep, o_raw, proj, stride, conv_w, conv_b, conv_state, state, a_log, dt_bias, skip, norm_w,
                                                 norm_groups, out_scale, tok_entry, tok_pos, entry_start, entry_len, entry_slot, entry_pos0, tokens_n,
                                                 entries, heads, groups, state_n, vdim, taps, eps, s),
        return launch_state_space<float>(out, out_stride, prep, o_raw, proj, stride, conv_w, conv_b, conv_state, state, a_log, dt_bias, skip, norm_w,
                                         norm_groups, out_scale, tok_entry, tok_pos, entry_start, entry_len, entry_slot, entry_pos0, tokens_n, entries,
                                         heads, groups, state_n, vdim, taps, eps, s));
}

int qs_hyb_lru_conv(void* u, const void* proj, int64_t stride, const float* x_bias, const float* conv_w, const float* conv_b, float* conv_state,
                    const int32_t* tok_entry, const int32_t* tok_pos, const int32_t* entry_start, const int32_t* entry_len, const int32_t* entry_slot,
                    const int32_t* entry_pos0, int tokens_n, int entries, int width, int taps, int dtype, void* stream) {
  QS_REQUIRE(u && proj && conv_w, "hyb_lru_conv: null tensor");
  QS_REQUIRE(tok_entry && tok_pos && entry_start && entry_len && entry_slot && entry_pos0, "hyb_lru_conv: null batch table");
  QS_REQUIRE(width > 0 && taps >= 1 && taps <= kMaxTaps && (taps == 1 || conv_state != nullptr), "hyb_lru_conv: 1..17 convolution taps");
  if (tokens_n == 0) return qs::QS_OK;
  cudaStream_t s = (cudaStream_t)stream;
  QS_DT(dtype,
        return launch_lru_conv<__nv_bfloat16>(u, proj, stride, x_bias, conv_w, conv_b, conv_state, tok_entry, tok_pos, entry_start, entry_len, entry_slot,
                                              entry_pos0, tokens_n, entries, width, taps, s),
        return launch_lru_conv<float>(u, proj, stride, x_bias, conv_w, conv_b, conv_state, tok_entry, tok_pos, entry_start, entry_len, entry_slot,
                                      entry_pos0, tokens_n, entries, width, taps, s));
}

int qs_hyb_lru_scan(void* out, int64_t out_stride, float* state, float* sums, const void* u, const float* z, const void* proj, int64_t stride,
                    const float* y_bias, const float* r_bias, const float* i_bias, const float* rate, const int32_t* tile_entry, const int32_t* tile_row0,
                    int n_tiles, int n_short, const int32_t* entry_start, const int32_t* entry_len, const int32_t* entry_slot, const int32_t* entry_pos0,
                    int tokens_n, int entries, int width, int blocks, int tile_rows, int long_min, int dtype, void* stream) {
  QS_REQUIRE(out && state && u && z && proj && y_bias && r_bias && i_bias && rate, "hyb_lru_scan: null tensor");
  QS_REQUIRE(entry_start && entry_len && entry_slot && entry_pos0, "hyb_lru_scan: null batch table");
  QS_REQUIRE(n_tiles == 0 || (tile_entry && tile_row0 && sums && tile_rows > 0), "hyb_lru_scan: null tile table");
  QS_REQUIRE(width > 0 && blocks > 0 && width % blocks == 0 && long_min > 0, "hyb_lru_scan: blocks divide the width");
  if (tokens_n == 0) return qs::QS_OK;
  cudaStream_t s = (cudaStream_t)stream;
  QS_DT(dtype,
        return launch_lru_scan<__nv_bfloat16>(out, out_stride, state, sums, u, z, proj, stride, y_bias, r_bias, i_bias, rate, tile_entry, tile_row0, n_tiles,
                                              n_short, entry_start, entry_len, entry_slot, entry_pos0, tokens_n, entries, width, blocks, tile_rows,
                                              long_min, s),
        return launch_lru_scan<float>(out, out_stride, state, sums, u, z, proj, stride, y_bias, r_bias, i_bias, rate, tile_entry, tile_row0, n_tiles, n_short,
                                      entry_start, entry_len, entry_slot, entry_pos0, tokens_n, entries, width, blocks, tile_rows, long_min, s));
}

}  // extern "C"
