// A short causal convolution over time on every channel of a projection, continued across steps from a state slot that
// holds the request's last taps - 1 input rows.  Each output is a sum over the taps in ascending order in fp32, from
// this step's rows or the slot's, so the result does not depend on where a prompt was cut.
#include <algorithm>

#include "common.cuh"
#include "elt_access.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

constexpr int SC_MAX_TAPS = 16;

// a block per token and slice of the channels (few tokens: one channel per thread; many: a thread walks its channels);
// a channel's taps are summed in ascending order
template <typename E>
__global__ void __launch_bounds__(256) short_conv_kernel(ShortConvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int b = a.token_req[t], r0 = a.qsl[b], pos = a.positions[t], taps = a.taps;
  const float* sp = a.state + (int64_t)a.slots[b] * a.slot_stride;      // [taps - 1, C]: row s holds the input of position p0 - (taps - 1) + s
  const E* x = (const E*)a.x;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < a.C; c += gridDim.y * blockDim.x) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;                  // the input of position pos - back
      if (pos - back < 0) continue;
      const int row = t - back;
      const float u = row >= r0 ? ldf(x + (int64_t)row * a.ldx + c) : sp[(int64_t)(taps - 1 - (r0 - row)) * a.C + c];
      acc = fmaf(ldf((const E*)a.w + (int64_t)c * taps + j), u, acc);
    }
    stf((E*)a.y + (int64_t)t * a.ldy + c, acc);
  }
}

// the same, four neighbouring channels per thread (8-byte loads of 16-bit rows, 16-byte ones of fp32 rows and of the slot)
template <typename E>
__global__ void __launch_bounds__(256) short_conv_vec_kernel(ShortConvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int b = a.token_req[t], r0 = a.qsl[b], pos = a.positions[t], taps = a.taps;
  const float* sp = a.state + (int64_t)a.slots[b] * a.slot_stride;
  const E* x = (const E*)a.x;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < a.C; c += gridDim.y * blockDim.x * 4) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;
      if (pos - back < 0) continue;
      const int row = t - back;
      float u[4];
      if (row >= r0) ld4(x + (int64_t)row * a.ldx + c, u); else ld4(sp + (int64_t)(taps - 1 - (r0 - row)) * a.C + c, u);
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[k] = fmaf(ldf((const E*)a.w + (int64_t)(c + k) * taps + j), u[k], acc[k]);
    }
    st4((E*)a.y + (int64_t)t * a.ldy + c, acc);
  }
}

// one block per request: the slot's rows move up by the step's row count and the step's last rows follow
template <typename E>
__global__ void __launch_bounds__(256) short_conv_save_kernel(ShortConvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x, r0 = a.qsl[b], n = a.qsl[b + 1] - r0, keep = a.taps - 1;
  if (n <= 0 || keep <= 0 || c >= a.C) return;
  const bool fresh = a.positions[r0] == 0;
  float* sp = a.state + (int64_t)a.slots[b] * a.slot_stride;
  const E* x = (const E*)a.x;
  float v[SC_MAX_TAPS];
#pragma unroll
  for (int s = 0; s < SC_MAX_TAPS - 1; ++s) {         // every row is read before any is written
    const int src = s + n;                            // in the old numbering of the slot's rows
    v[s] = 0.f;
    if (s < keep) {
      if (src >= keep) v[s] = ldf(x + (int64_t)(r0 + src - keep) * a.ldx + c);
      else if (!fresh) v[s] = sp[(int64_t)src * a.C + c];
    }
  }
#pragma unroll
  for (int s = 0; s < SC_MAX_TAPS - 1; ++s) if (s < keep) sp[(int64_t)s * a.C + c] = v[s];
}

// One warp per (token, head of head_dim channels) for the unit heads and per (token, 128 channels) for the rest: the
// convolution's sums, the silu and a head's sum of squares stay in the warp's registers.  VEC: four neighbouring channels
// per lane and pass.
template <typename E, typename O, bool VEC>
__global__ void __launch_bounds__(256) short_conv_silu_heads_kernel(ConvHeadsArgs a, int items) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int W = VEC ? 4 : 1, MAXP = 256 / (32 * W);
  const int lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (int64_t)a.T * items) return;
  const int t = (int)(item / items), u = (int)(item % items);
  const bool unit = u < a.unit_heads;
  const int c0 = unit ? u * a.head_dim : a.unit_heads * a.head_dim + (u - a.unit_heads) * 128;
  const int n = unit ? a.head_dim : min(128, a.C - c0);
  const int b = a.token_req[t], r0 = a.qsl[b], pos = a.positions[t], taps = a.taps;
  float* sp = a.state + (int64_t)a.slots[b] * a.slot_stride;      // [taps - 1, C], oldest first
  const E* x = (const E*)a.x;
  float acc[MAXP][W];
  float ss = 0.f;
#pragma unroll
  for (int p = 0; p < MAXP; ++p) {
    const int k = (p * 32 + lane) * W;
#pragma unroll
    for (int q = 0; q < W; ++q) acc[p][q] = 0.f;
    if (k < n) {
      const int c = c0 + k;
      if (a.bias) {
#pragma unroll
        for (int q = 0; q < W; ++q) acc[p][q] = ldf((const E*)a.bias + c + q);
      }
      for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;                  // the input of position pos - back
        if (pos - back < 0) continue;
        const int row = t - back;
        float in[4], w[4];
        if (VEC) {
          if (row >= r0) ld4(x + (int64_t)row * a.ldx + c, in); else ld4(sp + (int64_t)(taps - 1 - (r0 - row)) * a.C + c, in);
          ld4((const E*)a.w + (int64_t)j * a.C + c, w);
        } else {
          in[0] = row >= r0 ? ldf(x + (int64_t)row * a.ldx + c) : sp[(int64_t)(taps - 1 - (r0 - row)) * a.C + c];
          w[0] = ldf((const E*)a.w + (int64_t)j * a.C + c);
        }
#pragma unroll
        for (int q = 0; q < W; ++q) acc[p][q] = fmaf(w[q], in[q], acc[p][q]);
      }
      if (a.inline_save) {                              // one row per request: this lane alone touches these channels of the slot
        for (int s = 0; s + 1 < taps; ++s) {
#pragma unroll
          for (int q = 0; q < W; ++q) sp[(int64_t)s * a.C + c + q] = s + 2 < taps ? sp[(int64_t)(s + 1) * a.C + c + q] : ldf(x + (int64_t)t * a.ldx + c + q);
        }
      }
#pragma unroll
      for (int q = 0; q < W; ++q) {
        const float v = acc[p][q];
        acc[p][q] = v / (1.f + expf(-v));
        ss = fmaf(acc[p][q], acc[p][q], ss);
      }
    }
  }
  float f = 1.f;
  if (unit) {
    f = 1.f / sqrtf(warp_sum(ss) + a.unit_eps);
    if (u < a.scaled_heads) f *= a.head_scale;
  }
  O* y = (O*)a.y + (int64_t)t * a.ldy + c0;
#pragma unroll
  for (int p = 0; p < MAXP; ++p) {
    const int k = (p * 32 + lane) * W;
    if (k < n) {
#pragma unroll
      for (int q = 0; q < W; ++q) acc[p][q] *= f;
      if constexpr (VEC) st4(y + k, acc[p]); else stf(y + k, acc[p][0]);
    }
  }
}

// The same for two to four taps and 16-byte rows: a warp keeps its channels' weights and the last taps - 1 inputs in registers
// over a strip of TS tokens, so every input row is read once, and requests all rows of the strip before it uses the first.
// MAXP: passes of 128 channels (heads of up to 128 * MAXP channels).
template <typename E, typename O, int TAPS, int TS, int MAXP>
__global__ void __launch_bounds__(256) short_conv_silu_heads_strip_kernel(ConvHeadsArgs a, int items) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int u = (int)(item % items);
  const int64_t strip = item / items;
  if (strip * TS >= a.T) return;
  const int t0 = (int)strip * TS, nt = min(TS, a.T - t0);
  const bool unit = u < a.unit_heads;
  const int c0 = unit ? u * a.head_dim : a.unit_heads * a.head_dim + (u - a.unit_heads) * 128;
  const int n = unit ? a.head_dim : min(128, a.C - c0);
  const int ml = min(t0 + lane % TS, a.T - 1);                      // lane i knows token t0 + i's request, first row and position
  const int mb = a.token_req[ml], mr = a.qsl[mb], mp = a.positions[ml];
  const E* x = (const E*)a.x;
  float cur[MAXP][TS][4], win[MAXP][TAPS - 1][4], w[MAXP][TAPS][4], bias[MAXP][4] = {};
#pragma unroll
  for (int p = 0; p < MAXP; ++p) {
    const int k = (p * 32 + lane) * 4;
    if (k < n) {
#pragma unroll
      for (int i = 0; i < TS; ++i) if (i < nt) ld4(x + (int64_t)(t0 + i) * a.ldx + c0 + k, cur[p][i]);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) ld4((const E*)a.w + (int64_t)j * a.C + c0 + k, w[p][j]);
      if (a.bias) ld4((const E*)a.bias + c0 + k, bias[p]);
    }
  }
#pragma unroll
  for (int i = 0; i < TS; ++i) {
    if (i >= nt) break;
    const int t = t0 + i, r0 = __shfl_sync(0xffffffffu, mr, i), pos = __shfl_sync(0xffffffffu, mp, i), b = __shfl_sync(0xffffffffu, mb, i);
    const bool fill = i == 0 || t == r0;                             // the inputs before this row: rows of the step, the slot's, or zeros
    float* sp = a.state + (int64_t)a.slots[b] * a.slot_stride;
    float ss = 0.f, y[MAXP][4];
#pragma unroll
    for (int p = 0; p < MAXP; ++p) {
      const int k = (p * 32 + lane) * 4, c = c0 + k;
#pragma unroll
      for (int q = 0; q < 4; ++q) y[p][q] = 0.f;
      if (k < n) {
        if (fill) {
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) {
            const int back = TAPS - 1 - j, row = t - back;
            if (pos - back < 0) { win[p][j][0] = win[p][j][1] = win[p][j][2] = win[p][j][3] = 0.f; }
            else if (row >= r0) ld4(x + (int64_t)row * a.ldx + c, win[p][j]);
            else ld4(sp + (int64_t)(TAPS - 1 - (r0 - row)) * a.C + c, win[p][j]);
          }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float acc = bias[p][q];
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[p][j][q], win[p][j][q], acc);
          acc = fmaf(w[p][TAPS - 1][q], cur[p][i][q], acc);
#pragma unroll
          for (int j = 0; j + 1 < TAPS - 1; ++j) win[p][j][q] = win[p][j + 1][q];
          win[p][TAPS - 2][q] = cur[p][i][q];
          y[p][q] = acc / (1.f + expf(-acc));
          ss = fmaf(y[p][q], y[p][q], ss);
        }
        if (a.inline_save) {                                         // one row per request: this lane alone touches these channels of the slot
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) st4(sp + (int64_t)j * a.C + c, win[p][j]);
        }
      }
    }
    float f = 1.f;
    if (unit) {
      f = 1.f / sqrtf(warp_sum(ss) + a.unit_eps);
      if (u < a.scaled_heads) f *= a.head_scale;
    }
#pragma unroll
    for (int p = 0; p < MAXP; ++p) {
      const int k = (p * 32 + lane) * 4;
      if (k < n) {
#pragma unroll
        for (int q = 0; q < 4; ++q) y[p][q] *= f;
        st4((O*)a.y + (int64_t)t * a.ldy + c0 + k, y[p]);
      }
    }
  }
}

template <typename E, typename O, int TAPS, int TS>
cudaError_t launch_strip(const ConvHeadsArgs& a, int items, cudaStream_t st) {
  const dim3 grid((unsigned)(((int64_t)((a.T + TS - 1) / TS) * items + 7) / 8));
  return a.head_dim <= 128 ? launch_pdl(short_conv_silu_heads_strip_kernel<E, O, TAPS, TS, 1>, grid, dim3(256), 0, st, a, items)
                           : launch_pdl(short_conv_silu_heads_strip_kernel<E, O, TAPS, TS, 2>, grid, dim3(256), 0, st, a, items);
}
template <typename E, typename O>
cudaError_t launch_silu_heads(const ConvHeadsArgs& a, int items, cudaStream_t st) {
  if (a.vec && a.taps >= 2 && a.taps <= 4) {
    const bool many = a.T >= 32 && a.T > a.B;                       // prompt pieces: strips of eight rows; single tokens: a warp per (row, head)
    if (a.taps == 2) return many ? launch_strip<E, O, 2, 8>(a, items, st) : launch_strip<E, O, 2, 1>(a, items, st);
    if (a.taps == 3) return many ? launch_strip<E, O, 3, 8>(a, items, st) : launch_strip<E, O, 3, 1>(a, items, st);
    return many ? launch_strip<E, O, 4, 8>(a, items, st) : launch_strip<E, O, 4, 1>(a, items, st);
  }
  const dim3 grid((unsigned)(((int64_t)a.T * items + 7) / 8));
  return a.vec ? launch_pdl(short_conv_silu_heads_kernel<E, O, true>, grid, dim3(256), 0, st, a, items) : launch_pdl(short_conv_silu_heads_kernel<E, O, false>, grid, dim3(256), 0, st, a, items);
}

}  // namespace

int short_conv_silu_heads(const ConvHeadsArgs& a0, cudaStream_t st) {
  if (a0.T <= 0) return 0;
  ConvHeadsArgs a = a0;
  KGE_REQUIRE(a.taps >= 1 && a.taps <= SC_MAX_TAPS && a.C > 0 && a.head_dim > 0 && a.head_dim <= 256 && a.unit_heads * a.head_dim <= a.C,
              "short_conv_silu_heads: %d taps, %d heads of %d of %d channels", a.taps, a.unit_heads, a.head_dim, a.C);
  const int items = a.unit_heads + (a.C - a.unit_heads * a.head_dim + 127) / 128;
  a.vec = a.C % 4 == 0 && (a.unit_heads == 0 || a.head_dim % 4 == 0) && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.slot_stride % 4 == 0 &&
          ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.bias) |
            reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
  cudaError_t ce;
  if (a.elt == KGE_ELT_F32) ce = launch_silu_heads<float, float>(a, items, st);
  else ce = a.out_elt ? launch_silu_heads<__nv_bfloat16, __nv_bfloat16>(a, items, st) : launch_silu_heads<__nv_bfloat16, float>(a, items, st);
  KGE_CUDA_OK(ce);
  if (a.inline_save || a.taps < 2) return 0;
  ShortConvArgs s;      // the slots' rows move up after every row of the step has been read
  s.x = a.x; s.ldx = a.ldx; s.C = a.C; s.taps = a.taps; s.state = a.state; s.slot_stride = a.slot_stride; s.slots = a.slots; s.qsl = a.qsl; s.positions = a.positions; s.B = a.B; s.T = a.T;
  const dim3 sg(a.B, (a.C + 255) / 256);
  KGE_CUDA_OK(a.elt == KGE_ELT_F32 ? launch_pdl(short_conv_save_kernel<float>, sg, dim3(256), 0, st, s) : launch_pdl(short_conv_save_kernel<__nv_bfloat16>, sg, dim3(256), 0, st, s));
  return 0;
}

int short_conv_state(const ShortConvArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.taps >= 1 && a.taps <= SC_MAX_TAPS && a.C > 0 && a.x != a.y, "short_conv_state: %d taps on %d channels", a.taps, a.C);
  const int cb = (a.C + 255) / 256;
  KGE_REQUIRE(cb <= 65535, "short_conv_state: %d channels", a.C);
  const int cy = std::max(1, std::min(cb, 2048 / std::max(a.T, 1)));     // about 2048 blocks at least, else a block per token
  const bool vec = a.C % 4 == 0 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.slot_stride % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
  if (vec) {
    const int cv = std::max(1, std::min((a.C / 4 + 255) / 256, 2048 / std::max(a.T, 1)));
    if (a.elt == KGE_ELT_F32) KGE_CUDA_OK(launch_pdl(short_conv_vec_kernel<float>, dim3(a.T, cv), dim3(256), 0, st, a));
    else KGE_CUDA_OK(launch_pdl(short_conv_vec_kernel<__nv_bfloat16>, dim3(a.T, cv), dim3(256), 0, st, a));
    if (a.elt == KGE_ELT_F32) KGE_CUDA_OK(launch_pdl(short_conv_save_kernel<float>, dim3(a.B, cb), dim3(256), 0, st, a));
    else KGE_CUDA_OK(launch_pdl(short_conv_save_kernel<__nv_bfloat16>, dim3(a.B, cb), dim3(256), 0, st, a));
    return 0;
  }
  if (a.elt == KGE_ELT_F32) {
    KGE_CUDA_OK(launch_pdl(short_conv_kernel<float>, dim3(a.T, cy), dim3(256), 0, st, a));
    KGE_CUDA_OK(launch_pdl(short_conv_save_kernel<float>, dim3(a.B, cb), dim3(256), 0, st, a));
  } else {
    KGE_CUDA_OK(launch_pdl(short_conv_kernel<__nv_bfloat16>, dim3(a.T, cy), dim3(256), 0, st, a));
    KGE_CUDA_OK(launch_pdl(short_conv_save_kernel<__nv_bfloat16>, dim3(a.B, cb), dim3(256), 0, st, a));
  }
  return 0;
}

}  // namespace kge
